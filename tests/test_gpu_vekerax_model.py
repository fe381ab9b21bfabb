"""Vekerax through the framework's runner and cache manager, against the plain implementation."""
import pytest
import torch

from oracle import vekerax as V
from tests import vekerax_util as U

pytestmark = pytest.mark.gpu


@pytest.fixture(scope="module", params=[(c, d) for c in U.CASES for d in (torch.float32, torch.bfloat16)], ids=lambda p: f"{p[0]}-{str(p[1])[6:]}")
def model(request, pkg):
    m = U.Model(*request.param)
    yield m
    m.llm.exit()


def test_prompt_layer_by_layer(model):
    """Residual streams after every layer run, and the logits, of one prompt."""
    toks, trail = U.tokens(90, model.cfg["vocab"]), []
    model.runner.model.run_hook = lambda x: trail.append(x.double().cpu())
    try:
        s = model.seq()
        got = model.feed([s], [toks])[0]
    finally:
        model.runner.model.run_hook = None
        model.free(s)
    want, want_trail = V.forward(model.cfg, model.w64, toks)
    assert len(trail) == len(want_trail)
    for i, (a, b) in enumerate(zip(trail, want_trail)):
        err = ((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt()).item()
        assert err < U.TOL[model.dtype], f"layer run {i}: {err:.2e}"
    model.check(got, want, "logits")


def test_decoding_token_by_token(model):
    """A short prompt, then many decoded tokens: past every window, over block edges, from the very first token."""
    toks = U.tokens(150, model.cfg["vocab"], 1)
    for start in (1, 5, 149):
        s = model.seq()
        got = [model.feed([s], [toks[:start]])[0]] + [model.feed([s], [[t]])[0] for t in toks[start:]]
        model.free(s)
        model.check(torch.cat(got), model.want(toks), f"decoding from {start}")


@pytest.mark.parametrize("size", [2, 3, 16, 33, 64, 100])
def test_portions(model, size):
    toks = U.tokens(150, model.cfg["vocab"], 1)
    s = model.seq()
    got = [model.feed([s], [toks[a:a + size]])[0] for a in range(0, 150, size)]
    model.free(s)
    model.check(torch.cat(got), model.want(toks), f"portions of {size}")


def test_batches_of_unequal_requests(model):
    """Prompts side by side, portions beside whole prompts, batched decoding of different lengths; pages and state slots
    that other requests have used before."""
    lens = [1, 37, 140, 66]
    toks = [U.tokens(n + 12, model.cfg["vocab"], 20 + i) for i, n in enumerate(lens)]
    for rnd in range(2):  # the second time on reused blocks and slots, in another order
        seqs = [model.seq() for _ in lens]
        order = [0, 1, 2, 3] if rnd == 0 else [3, 1, 0, 2]
        first = {i: (50 if i == 2 else lens[i]) for i in order}
        got = {i: [] for i in order}
        for i, r in zip(order, model.feed([seqs[i] for i in order], [toks[i][:first[i]] for i in order])):
            got[i].append(r)
        got[2].append(model.feed([seqs[2]], [toks[2][50:lens[2]]])[0])
        for k in range(12):
            for i, r in zip(order, model.feed([seqs[i] for i in order], [[toks[i][lens[i] + k]] for i in order])):
                got[i].append(r)
        for i in order:
            model.check(torch.cat(got[i]), model.want(toks[i]), f"request {i}, pass {rnd}")
        model.free(*seqs)


def test_state_slot_of_a_finished_request_starts_from_zero(model):
    toks = U.tokens(40, model.cfg["vocab"], 3)
    for _ in range(3):
        s = model.seq()
        model.check(model.feed([s], [toks[:2]])[0], model.want(toks)[:2], "first tokens on used pages")
        model.free(s)
