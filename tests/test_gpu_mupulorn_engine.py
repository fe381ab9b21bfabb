"""Generation with Mupulorn through the engine, its scheduler and the commands, against the plain implementation."""
import json
import os
import subprocess
import sys

import pytest
import torch

from oracle import mupulorn as P
from tests import mupulorn_util as U
from tests.model_util import greedy, save, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("case,blocks", [("mixed", 80), ("mixed", 9), ("odd", 9)])
def test_greedy_generation_through_the_engine(pkg, case, blocks):
    """Portions of prompts, batched decoding and (with few blocks) preemption; the same tokens as the plain implementation."""
    from nanovllm_b200.engine.llm_engine import SamplingParams
    m = U.Model(case, torch.float32, max_num_batched_tokens=24, num_kvcache_blocks=blocks)
    try:
        prompts = [tokens(n, m.cfg["vocab"], 40 + n) for n in (30, 3, 55, 1, 20)]
        got = m.llm.generate(prompts, SamplingParams(max_tokens=9))
        assert got == [greedy(m, p, 9) for p in prompts]
        assert len(m.cache.free_blocks) == blocks and len(m.cache.free_slots) == 4
    finally:
        m.llm.exit()


def test_generation_in_bf16_repeats_and_samples(pkg):
    """Decode graphs, the fused and (vocabulary not a multiple of 8) the unfused sampler; every pick is near the best."""
    from nanovllm_b200.engine.llm_engine import SamplingParams
    for case in ("wide", "odd"):
        m = U.Model(case, torch.bfloat16, kvcache_block_size=128 if case == "wide" else 16)
        try:
            prompts = [tokens(n, m.cfg["vocab"], n) for n in (33, 2, 64)]
            got = m.llm.generate(prompts, SamplingParams(max_tokens=12))
            assert got == m.llm.generate(prompts, SamplingParams(max_tokens=12))
            for p, g in zip(prompts, got):
                lg = m.forward(p + g)[0][len(p) - 1:-1]
                picked = lg.gather(1, torch.tensor(g).view(-1, 1)).squeeze(1)
                assert (picked >= lg.max(-1).values - 0.2 * lg.std(-1)).all()
            hot = m.llm.generate(prompts, SamplingParams(max_tokens=12, temperature=1.0))
            assert hot != got and all(0 <= t < m.cfg["vocab"] for g in hot for t in g)
        finally:
            m.llm.exit()


def test_long_decoding(pkg):
    """Some hundred decoded tokens of unequal requests through the decode graphs, teacher-forced."""
    m = U.Model("mixed", torch.bfloat16, kvcache_block_size=128)
    try:
        toks = [tokens(n, m.cfg["vocab"], 60 + n) for n in (300, 290)]
        seqs = [m.seq(), m.seq()]
        starts = [11, 1]
        got = [[r] for r in m.feed(seqs, [t[:s] for t, s in zip(toks, starts)])]
        for k in range(289):
            for i, r in enumerate(m.feed(seqs, [[toks[i][starts[i] + k]] for i in range(2)])):
                got[i].append(r)
        for i in range(2):
            m.check(torch.cat(got[i]), m.want(toks[i])[:starts[i] + 289], f"request {i}")
    finally:
        m.llm.exit()


def test_resident_decoder_matches_steps(pkg):
    from nanovllm_b200.engine.model_runner import ResidentDecoder, Seq
    m = U.Model("wide", torch.bfloat16, kvcache_block_size=128)
    try:
        prompts = [tokens(n, m.cfg["vocab"], n) for n in (20, 45)]
        rd = ResidentDecoder(m.runner, 2)

        def start():
            seqs = [Seq(list(p)) for p in prompts]
            for s in seqs:
                m.cache.hold(s, 80)
            for s, t in zip(seqs, m.runner.step(seqs, True)):
                s.token_ids.append(t)
            return seqs

        seqs = start()
        by_step = []
        for _ in range(10):
            toks = m.runner.step(seqs, False)
            by_step.append(toks)
            for s, t in zip(seqs, toks):
                s.token_ids.append(t)
        m.free(*seqs)
        seqs = start()
        rd.load(seqs)
        for k in range(10):
            rd.replay()
            assert rd.tokens.tolist() == by_step[k]
    finally:
        m.llm.exit()


def test_trace_runner_and_command_line(pkg, tmp_path):
    """bin/trace_run and the generate command on a saved model folder."""
    cfg = U.CASES["mixed"]
    w = U.weights(cfg, 5)
    save(tmp_path / "m", cfg, w)
    w64 = {k: t.double() for k, t in w.items()}
    toks = tokens(30, cfg["vocab"], 7)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[20:28], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[28:29], "want": [0]}], "end": ["x"]},
             {"step": 3, "entries": [{"id": "x", "tokens": toks, "want": [29]}], "end": ["x"]}]
    want = P.forward(cfg, w64, toks)[0]
    for dtype, tol in (("float32", 1e-3), ("bfloat16", 0.5)):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "30"],
                           input="".join(json.dumps(s) + "\n" for s in steps), text=True, capture_output=True, timeout=300)
        assert r.returncode == 0 and [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)], r.stderr[-800:]
        for step, rows in ((0, [0, 19]), (2, [28]), (3, [29])):
            got = torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32).view(len(rows), cfg["vocab"]).double()
            assert (got - want[rows]).abs().max() < tol
        assert not (out / "1.f32").exists()
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--max-tokens", "3",
                        "--prompt-ids", ",".join(map(str, toks[:5]))], text=True, capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-800:]
    m = type("M", (), {"forward": staticmethod(lambda t: P.forward(cfg, w64, t))})
    assert json.loads(r.stdout.splitlines()[-1])["token_ids"] == greedy(m, toks[:5], 3)
