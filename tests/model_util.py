"""A small model behind the framework's engine beside its plain implementation, and what every design is put through."""
import json
import os
import struct

import torch


def save(folder, cfg, w):
    """config.json and model.safetensors (8-byte header length, JSON header, data)."""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    header, blobs, at = {}, [], 0
    for name, t in w.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    head = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(head)) + head + b"".join(blobs))


def tokens(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


# root mean square of the logits' error over their own; bf16: what rounding does to deliberately lively weights
TOL = {torch.float32: 2e-4, torch.bfloat16: 0.12}


class ServedModel:
    """`forward(cfg, weights, tokens) -> (logits, residuals)` is the plain implementation (GPU needed for the other side)."""

    def __init__(self, forward, cfg, w, dtype, **kw):
        from tests.gpu_util import ensure_group
        ensure_group()
        from nanovllm_b200.engine.llm_engine import LLM
        self.plain, self.cfg, self.dtype = forward, cfg, dtype
        self.w64 = {k: t.double() for k, t in w.items()}
        self.llm = LLM(cfg, w, dtype=dtype, **({"max_num_seqs": 4, "max_model_len": 512, "max_num_batched_tokens": 512, "kvcache_block_size": 16,
                                                "num_kvcache_blocks": 80} | kw))
        self.runner, self.cache = self.llm.runner, self.llm.cache
        self.memo = {}

    def forward(self, toks):
        return self.plain(self.cfg, self.w64, list(toks))

    def want(self, toks):
        key = tuple(toks)
        if key not in self.memo:
            self.memo[key] = self.forward(toks)[0]
        return self.memo[key]

    def seq(self):
        from nanovllm_b200.engine.model_runner import Seq
        return Seq([])

    def feed(self, seqs, parts):
        """One step that brings `parts` (token lists) to the sequences; logits of every new token, per sequence."""
        for s, p in zip(seqs, parts):
            s.token_ids += p
            self.cache.hold(s, len(s))
        counts = [len(p) for p in parts]
        decode = all(c == 1 for c in counts) and all(s.num_cached_tokens for s in seqs)
        out = self.runner.step_logits(seqs, not decode, None if decode else counts, list(range(sum(counts))))
        for s, c in zip(seqs, counts):
            s.num_cached_tokens += c
        return list(out.split(counts))

    def check(self, got, want, what):
        err = (got.double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
        assert torch.isfinite(got).all() and err.max() < TOL[self.dtype], f"{what}: error {err.max().item():.2e} at row {int(err.argmax())}"

    def free(self, *seqs):
        for s in seqs:
            self.cache.release(s)


def greedy(m, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(m.forward(toks)[0][-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------- what every design is put through
def layer_by_layer(model):
    """The residual after every layer run, and the logits, of one prompt."""
    toks, trail = tokens(90, model.cfg["vocab"]), []
    model.runner.model.run_hook = lambda x: trail.append(x.double().cpu())
    try:
        s = model.seq()
        got = model.feed([s], [toks])[0]
    finally:
        model.runner.model.run_hook = None
        model.free(s)
    want, want_trail = model.forward(toks)
    assert len(trail) == len(want_trail)
    for i, (a, b) in enumerate(zip(trail, want_trail)):
        err = ((a - b).pow(2).mean().sqrt() / b.pow(2).mean().sqrt()).item()
        assert err < TOL[model.dtype], f"layer run {i}: {err:.2e}"
    model.check(got, want, "logits")


def decoding_token_by_token(model):
    """A short prompt, then many decoded tokens: over block edges, from the very first token."""
    toks = tokens(150, model.cfg["vocab"], 1)
    for start in (1, 5, 149):
        s = model.seq()
        got = [model.feed([s], [toks[:start]])[0]] + [model.feed([s], [[t]])[0] for t in toks[start:]]
        model.free(s)
        model.check(torch.cat(got), model.want(toks), f"decoding from {start}")


def portions(model, size):
    toks = tokens(150, model.cfg["vocab"], 1)
    s = model.seq()
    got = [model.feed([s], [toks[a:a + size]])[0] for a in range(0, 150, size)]
    model.free(s)
    model.check(torch.cat(got), model.want(toks), f"portions of {size}")


def batches_of_unequal_requests(model):
    """Prompts side by side, portions beside whole prompts, batched decoding of different lengths; pages and state slots
    that other requests have used before."""
    lens = [1, 37, 140, 66]
    toks = [tokens(n + 12, model.cfg["vocab"], 20 + i) for i, n in enumerate(lens)]
    for rnd in range(2):  # the second time on reused blocks and slots, in another order
        seqs = [model.seq() for _ in lens]
        order = [0, 1, 2, 3] if rnd == 0 else [3, 1, 0, 2]
        first = {i: (50 if i == 2 else lens[i]) for i in order}
        got = {i: [] for i in order}
        for i, r in zip(order, model.feed([seqs[i] for i in order], [toks[i][:first[i]] for i in order])):
            got[i].append(r)
        # the rest of one prompt beside the first decoded token of another, as one prefill step
        rest = model.feed([seqs[2], seqs[1]], [toks[2][50:lens[2]], toks[1][lens[1]:lens[1] + 1]])
        got[2].append(rest[0])
        got[1].append(rest[1])
        done = {0: 0, 1: 1, 2: 0, 3: 0}
        for k in range(11):
            for i, r in zip(order, model.feed([seqs[i] for i in order], [[toks[i][lens[i] + done[i] + k]] for i in order])):
                got[i].append(r)
        for i in order:
            model.check(torch.cat(got[i]), model.want(toks[i])[:lens[i] + 11 + done[i]], f"request {i}, pass {rnd}")
        model.free(*seqs)


def first_tokens_on_used_slots(model):
    toks = tokens(40, model.cfg["vocab"], 3)
    for n in (2, 1, 3):
        s = model.seq()
        model.check(model.feed([s], [toks[:n]])[0], model.want(toks)[:n], "first tokens on used pages")
        got = [model.feed([s], [[t]])[0] for t in toks[n:n + 6]]
        model.check(torch.cat(got), model.want(toks)[n:n + 6], "the tokens after them")
        model.free(s)
