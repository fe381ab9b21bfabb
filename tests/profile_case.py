"""Run one kernel of the library a few times on one GPU, for profiling with
Nsight Compute (the cases are larger than the 126 MB L2 but hold well under a
few GB, so a `--set full` capture of 1-3 launches ends by itself).

    python tests/profile_case.py <case> [--launches 6]

cases:
  gemm_decode     column-parallel GEMM, M=64, N=24576, K=4096 (Qwen3-8B gate_up at TP=1), 4 weight copies
  silu_decode     the same GEMM with SiLU*mul in its epilogue (what the decoder layer launches)
  qkv_decode      qkv projection M=64, N=6144, K=4096 with q/k-norm + RoPE + KV scatter in its epilogue, 8 weight copies
  oproj_decode    fused row-parallel launch, M=64, N=4096, Kr=4096 (Qwen3-8B o_proj at TP=1), 8 weight copies
  gemm_prefill    GEMM M=4096, N=4096, K=4096
  gemm_mid        GEMM M=256, N=4096, K=1024 (Qwen3-0.6B qkv at a 256-sequence decode step), 40 weight copies
  rowpar_decode   fused row-parallel launch, M=64, N=4096, Kr=12288 (Qwen3-8B down_proj at TP=1)
  rowpar_prefill  fused row-parallel launch, M=1024, N=5120, Kr=1024
  store_kvcache   paged-KV scatter, 16384 tokens x D=1024
  add_rmsnorm     residual add + RMSNorm, 16384 x 4096
  window_prefill  window attention (soft cap, sink, 1024 + 4 tokens), 4 prompts of 2048, 32 query / 8 key-value heads of 128
  window_decode   the same for 64 sequences of 1024 tokens, one row each, 6 layers' caches
  linear_prefill  decayed linear attention, 4 prompts of 2048, 32 heads of 128 x 128
  linear_decode   the same for 64 sequences, one row each, 4 layers' states
  stream_step     residual streams (4) between two sublayers, 8192 x 4096
  latent_decode   absorbed latent attention (tcgen05), 64 sequences of 1024 tokens, 32 heads, latent 512 + 64, 4 layers' caches
  latent_prefill  expanded latent attention (tcgen05), 4 prompts of 2048, 32 heads of 128 + 64 / 128, gate
  sandwich_step   residual, two norms and a 4-tap convolution between two sublayers, 4 prompts of 2048 x 4096
  poly_norm       PolyNorm of 8192 rows of 18432
  embed           embedding lookup, 16384 ids into a [151936, 4096] table (one rank)
"""
from __future__ import annotations

import argparse
import os
import sys

import torch
import torch.distributed as dist

HERE = os.path.dirname(os.path.abspath(__file__))
sys.path.insert(0, os.path.dirname(HERE))


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("case")
    ap.add_argument("--launches", type=int, default=6)
    a = ap.parse_args()
    import __graft_entry__ as entry
    entry.load_package()
    from nanovllm_b200 import ops
    from nanovllm_b200.runtime import init_runtime, shutdown_runtime
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
    os.environ.setdefault("MASTER_PORT", "29579")
    torch.cuda.set_device(0)
    dist.init_process_group("gloo", rank=0, world_size=1)
    init_runtime(max_tokens=16384, hidden=5120, oneshot_tokens=1024)
    dev = "cuda:0"
    g = torch.Generator(device=dev).manual_seed(0)

    def rnd(*shape, scale=1.0):
        return (torch.randn(*shape, device=dev, generator=g) * scale).bfloat16()

    if a.case in ("gemm_decode", "gemm_prefill", "gemm_mid"):
        m, n, k, copies = {"gemm_decode": (64, 24576, 4096, 4), "gemm_prefill": (4096, 4096, 4096, 2), "gemm_mid": (256, 4096, 1024, 40)}[a.case]
        x, ws = rnd(m, k), [rnd(n, k, scale=0.02) for _ in range(copies)]
        call = lambda i: ops.gemm(x, ws[i % copies])
    elif a.case == "silu_decode":
        m, i, k, copies = 64, 12288, 4096, 4
        x, ws = rnd(m, k), [rnd(2 * i, k, scale=0.02) for _ in range(copies)]
        call = lambda j: ops.gemm_silu_mul(x, ws[j % copies])
    elif a.case == "qkv_decode":
        m, nq, nkv, k, copies = 64, 32, 8, 4096, 8
        x, ws = rnd(m, k), [rnd((nq + 2 * nkv) * 128, k, scale=0.02) for _ in range(copies)]
        qw, kw = rnd(128), rnd(128)
        pos = torch.randint(0, 2048, (m,), device=dev)
        t = torch.arange(2048, dtype=torch.float, device=dev)
        inv = 1.0 / (1e6 ** (torch.arange(0, 128, 2, dtype=torch.float, device=dev) / 128))
        fr = torch.outer(t, inv)
        cos_sin = torch.cat((fr.cos(), fr.sin()), dim=-1).contiguous()
        kc = torch.zeros(16, 256, nkv, 128, dtype=torch.bfloat16, device=dev)
        vc = torch.zeros_like(kc)
        slots = torch.randperm(16 * 256, device=dev)[:m].to(torch.int32)
        call = lambda j: ops.qkv_fused(x, ws[j % copies], None, nq, nkv, 128, qw, kw, 1e-6, pos, cos_sin, kc, vc, slots)
    elif a.case in ("rowpar_decode", "rowpar_prefill", "oproj_decode"):
        m, n, k, copies = {"rowpar_decode": (64, 4096, 12288, 4), "rowpar_prefill": (1024, 5120, 1024, 8), "oproj_decode": (64, 4096, 4096, 8)}[a.case]
        x, ws, res, nw = rnd(m, k), [rnd(n, k, scale=0.02) for _ in range(copies)], rnd(m, n), rnd(n)
        call = lambda i: ops.rowpar_fused(x, ws[i % copies], None, res, nw, 1e-6)
    elif a.case == "store_kvcache":
        n, heads = 16384, 8
        key, value = rnd(n, heads, 128), rnd(n, heads, 128)
        kc = torch.zeros(2, 128, 256, heads, 128, dtype=torch.bfloat16, device=dev)
        vc = torch.zeros_like(kc)
        perm = torch.randperm(128, device=dev, generator=g)
        base = (perm[torch.arange(n, device=dev) // 256] * 256 + torch.arange(n, device=dev) % 256).to(torch.int32)
        call = lambda i: ops.store_kvcache(key, value, kc[i % 2], vc[i % 2], base)
    elif a.case == "add_rmsnorm":
        xs, rs, nw = [rnd(16384, 4096) for _ in range(2)], [rnd(16384, 4096) for _ in range(2)], rnd(4096)
        call = lambda i: ops.add_rmsnorm(xs[i % 2], rs[i % 2], nw, 1e-6)
    elif a.case in ("window_prefill", "window_decode", "linear_prefill", "linear_decode"):
        heads, nkv, d = 32, 8, 128
        prefill = a.case.endswith("prefill")
        seqs, length, layers = (4, 2048, 1) if prefill else (64, 1024, 6)
        rows = seqs * length if prefill else seqs
        cu = torch.arange(0, rows + 1, length, device=dev, dtype=torch.int32) if prefill else None
        kl = torch.full((seqs,), length, dtype=torch.int32, device=dev)
        if a.case.startswith("window"):
            blocks = seqs * length // 256
            kc, vc = ([rnd(blocks, 256, nkv, d) for _ in range(layers)] for _ in range(2))
            bt = torch.randperm(blocks, device=dev, generator=g).int().view(seqs, -1).contiguous()
            q, sink = rnd(rows, heads * d), torch.zeros(heads, device=dev)
            call = lambda i: ops.window_attention(q, heads, kc[i % layers], vc[i % layers], bt, cu, kl, length if prefill else 1, length, d ** -0.5, 30.0, 1024, 4, sink)
        else:
            decay = 1.0 - 2.0 ** (-2 - 6 * torch.arange(heads, dtype=torch.float64) / heads)
            dec, pw = decay.float().to(dev), (decay.unsqueeze(1) ** torch.arange(65)).float().to(dev)
            states = [torch.zeros(seqs, heads, d, d, device=dev) for _ in range(min(4, layers))]
            p, sl = rnd(rows, 4 * heads * d), torch.arange(seqs, device=dev, dtype=torch.int32)
            call = lambda i: ops.linear_attn(p, heads, d, d, states[i % len(states)], sl, cu, kl, length if prefill else 1, dec, pw)
    elif a.case == "stream_step":
        x, y = torch.randn(8192, 4, 4096, device=dev), rnd(8192, 4096)
        mix, one, nw = torch.eye(4, device=dev), torch.ones(4, device=dev), torch.ones(4096, device=dev)
        call = lambda i: ops.stream_step(x, y, mix, one, 0.1, one / 4, nw, 1e-6, 4096)
    elif a.case == "latent_decode":
        heads, lat, rot, seqs, length, layers = 32, 512, 64, 64, 1024, 4
        caches = [rnd(seqs * length // 256, 256, 1, lat + rot) for _ in range(layers)]
        bt = torch.randperm(seqs * length // 256, device=dev, generator=g).int().view(seqs, -1).contiguous()
        kl, q, sink = torch.full((seqs,), length, dtype=torch.int32, device=dev), rnd(seqs, heads * (lat + rot)), torch.zeros(heads, device=dev)
        call = lambda i: ops.latent_attention(q, heads, caches[i % layers], lat, bt, None, kl, 1, length, 0.05, sink)
    elif a.case == "latent_prefill":
        heads, d, rot, seqs, length = 32, 128, 64, 4, 2048
        rows = seqs * length
        cu = torch.arange(0, rows + 1, length, device=dev, dtype=torch.int32)
        q, kv, kr, gate = rnd(rows, heads * (d + rot)), rnd(rows, heads * 2 * d), rnd(rows, rot), rnd(rows, heads * d)
        table, sink = torch.ones(length, rot // 2, 2, device=dev), torch.zeros(heads, device=dev)
        call = lambda i: ops.expanded_attention(q, heads, kv, kr, cu, cu, length, d, rot, d, 0.07, sink, table, gate)
    elif a.case == "sandwich_step":
        rows, w, taps, seqs = 8192, 4096, 4, 4
        cu = torch.arange(0, rows + 1, rows // seqs, device=dev, dtype=torch.int32)
        batch = (cu, torch.full((seqs,), rows // seqs, dtype=torch.int32, device=dev), torch.arange(seqs, device=dev, dtype=torch.int32), rows // seqs)
        x, y, one = torch.randn(rows, w, device=dev), rnd(rows, w), torch.ones(1, device=dev)
        conv, state = rnd(taps, w, scale=0.1), rnd(seqs, taps - 1, w)
        call = lambda i: ops.sandwich_step(x, y, one, one, 1e-6, w, batch, conv, state)
    elif a.case == "poly_norm":
        z, coef = rnd(8192, 18432), torch.full((4,), 0.3, device=dev)
        call = lambda i: ops.poly_norm(z, coef, 1e-6, 18432)
    elif a.case == "embed":
        w = rnd(151936, 4096)
        ids = [torch.randint(0, 151936, (16384,), device=dev, generator=g) for _ in range(2)]
        call = lambda i: ops.embed(ids[i % 2], w, 0, 151936, 1)
    else:
        raise SystemExit(f"unknown case {a.case}")
    with torch.inference_mode():
        for i in range(a.launches):
            call(i)
    torch.cuda.synchronize()
    shutdown_runtime()
    dist.destroy_process_group()
    print("done", a.case)


if __name__ == "__main__":
    main()
