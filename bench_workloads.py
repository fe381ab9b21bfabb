"""The other workloads, behind `bench.py --workload cfg2|cfg5|vekerax|mupulorn` (the JSON line of the default workload).

cfg2  the reference's own bench.py workload (bench.py:9-27): Qwen3-0.6B random-init bf16 on one GPU, 256 sequences,
      prompt ids uniform in [0, 10000], prompt and output lengths uniform in [100, 1024], temperature 0.6, ignore_eos;
      total output tokens / wall time.  The batches are formed as the reference's scheduler forms them
      (nanovllm/engine/scheduler.py:25-58: whole prompts up to 16384 tokens per prefill step, then every running
      sequence decodes one token per step); tokens come from the LM head fused with the sampler.
cfg5  long-context prefill of Qwen3-32B random-init bf16 at tensor-parallel size 8: 4 sequences of 32768 uniform-random
      tokens in 16384-token chunks (nanovllm/engine/scheduler.py:42-48: only the first waiting sequence is chunked), KV
      blocks taken from a random permutation of the free list; prefill tokens / second.
vekerax  prefill and decode throughput of the Vekerax design beside Qwen3 with layers of the same size (random weights),
      and the time and roofline fraction of each of its kernels beside the like kernel of Qwen3.
"""
from __future__ import annotations

import json
import os
import random
import time


def _setup(args):
    import torch
    import torch.distributed as dist
    import __graft_entry__ as entry
    entry.load_package()
    rank, world = int(os.environ.get("RANK", "0")), int(os.environ.get("WORLD_SIZE", "1"))
    local = int(os.environ.get("LOCAL_RANK", str(rank)))
    assert world == args.gpus, f"--gpus {args.gpus} but WORLD_SIZE={world}: launch N>1 with torchrun"
    os.environ.setdefault("MASTER_ADDR", "127.0.0.1")
    os.environ.setdefault("MASTER_PORT", "29579")
    torch.cuda.set_device(local)
    dist.init_process_group("cpu:gloo,cuda:nccl" if world > 1 else "gloo", rank=rank, world_size=world)
    return torch, dist, rank, world, local


def _sync(torch, dist, world):
    torch.cuda.synchronize()
    if world > 1:
        dist.barrier()


def _max_over_ranks(torch, dist, world, v):
    if world == 1:
        return v
    t = torch.tensor([v], dtype=torch.float64)
    dist.all_reduce(t, op=dist.ReduceOp.MAX)
    return float(t.item())


def run_cfg5(args, peaks, clock_sampler_cls) -> None:
    torch, dist, rank, world, local = _setup(args)
    from nanovllm_b200.engine.model_runner import QWEN3_32B, ModelConfig, ModelRunner, Seq, sequential_block_tables
    n_seqs, seq_len, chunk, bs = 4, 32768, 16384, 256
    cfg = ModelConfig(**QWEN3_32B)
    blocks_per_seq = seq_len // bs
    runner = ModelRunner(cfg, max_num_seqs=n_seqs, max_model_len=seq_len, max_num_batched_tokens=chunk, num_kvcache_blocks=n_seqs * blocks_per_seq,
                         enforce_eager=True, oneshot_tokens=1024, seed=0)
    g = torch.Generator().manual_seed(0)
    prompts = torch.randint(0, cfg.vocab_size, (n_seqs, seq_len), generator=g).tolist()
    perm = list(range(n_seqs * blocks_per_seq))
    random.Random(0).shuffle(perm)  # the free list after some traffic: consecutive blocks of a sequence are scattered
    tables = sequential_block_tables([seq_len] * n_seqs, bs, permutation=perm)

    def one_pass():
        """All sequences from scratch: 8 steps of one 16384-token chunk each; returns the tokens sampled at the sequence ends."""
        out = []
        for p, bt in zip(prompts, tables):
            s = Seq(p, bt)
            for start in range(0, seq_len, chunk):
                s.num_cached_tokens = start
                toks = runner.step([s], True, num_new=[chunk])
            out.append(toks[0])
        return out

    K, W = max(1, min(args.steps, 4)), 1
    for _ in range(W):
        first = one_pass()
    _sync(torch, dist, world)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    with clock_sampler_cls(local) as clocks:
        e0.record()
        for _ in range(K):
            again = one_pass()
        e1.record()
        _sync(torch, dist, world)
    ms = _max_over_ranks(torch, dist, world, e0.elapsed_time(e1))
    runner.runtime.check_status()
    tokens = K * n_seqs * seq_len
    c = QWEN3_32B
    per_layer = c["hidden_size"] * (c["num_attention_heads"] + 2 * c["num_key_value_heads"]) * c["head_dim"] + c["num_attention_heads"] * c["head_dim"] * c["hidden_size"] \
        + 3 * c["hidden_size"] * c["intermediate_size"]
    gemm_flops = 2.0 * per_layer * c["num_hidden_layers"] * tokens
    attn_flops = 4.0 * c["num_attention_heads"] * c["head_dim"] * c["num_hidden_layers"] * K * n_seqs * (seq_len * (seq_len + 1) / 2)
    tf_per_gpu = (gemm_flops + attn_flops) / world / (ms * 1e-3) / 1e12
    if rank == 0:
        line = {"metric": "qwen3_32b_prefill_tokens_per_s", "value": tokens / (ms * 1e-3), "unit": "tok/s", "n_gpus": world, "steps": K, "warmup": W,
                "ms_per_step": ms / K, "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
                "config": {"workload": f"Qwen3-32B random-init bf16 long-context prefill, {n_seqs} x {seq_len} uniform-random tokens in {chunk}-token chunks, "
                                       f"paged KV (block 256) from a shuffled free list, TP={world}; one step = all {n_seqs} sequences",
                           "l2": "every chunk streams the rank's weight shard (8 GB at TP=8) and activations far larger than the 126 MB L2"},
                "clocks": clocks.summary(), "e2e": {"value": tokens / (ms * 1e-3), "unit": "tok/s", "h2d_bytes_per_step": n_seqs * seq_len * 20,
                                                    "d2h_bytes_per_step": 8 * (seq_len // chunk) * n_seqs,
                                                    "note": "timed through ModelRunner.step(): token ids, positions and slot mapping copied from pinned host memory every chunk, sampled token read back"},
                "gpu_launches": None,
                "roofline": {"bound": "tensor", "achieved": tf_per_gpu, "peak": peaks["bf16_tflops_sustained"], "unit": "TFLOP/s", "frac": tf_per_gpu / peaks["bf16_tflops_sustained"],
                             "what": "GEMM + causal attention flops per GPU over the step time (whole step, all kernels and the attention library call)", "traffic": None},
                "parity": {"same_tokens_on_repeat": first == again}}
        from nanovllm_b200 import _abi
        line["gpu_launches"] = _abi.launch_count()
        print(json.dumps(line), flush=True)
    runner.exit()
    dist.destroy_process_group()


def run_cfg2(args, peaks, clock_sampler_cls) -> None:
    torch, dist, rank, world, local = _setup(args)
    from nanovllm_b200.engine.model_runner import QWEN3_0_6B, ModelConfig, ModelRunner, Seq, sequential_block_tables
    num_seqs, bs, max_batched = 256, 256, 16384
    random.seed(0)
    prompts = [[random.randint(0, 10000) for _ in range(random.randint(100, 1024))] for _ in range(num_seqs)]
    max_tokens = [random.randint(100, 1024) for _ in range(num_seqs)]
    tables = sequential_block_tables([len(p) + m for p, m in zip(prompts, max_tokens)], bs)
    runner = ModelRunner(ModelConfig(**QWEN3_0_6B), max_num_seqs=num_seqs, max_model_len=4096, max_num_batched_tokens=max_batched,
                         num_kvcache_blocks=sum(len(t) for t in tables), oneshot_tokens=1024, seed=0)

    def generate():
        """Prefill in batches of whole prompts (at most 16384 tokens), then decode every running sequence one token per
        step until each has produced its max_tokens (ignore_eos).  Returns (output tokens, decode steps)."""
        seqs = [Seq(list(p), bt) for p, bt in zip(prompts, tables)]
        left = list(max_tokens)
        i = 0
        while i < num_seqs:  # prefill
            j, n = i, 0
            while j < num_seqs and n + len(seqs[j]) <= max_batched:
                n += len(seqs[j])
                j += 1
            toks = runner.step(seqs[i:j], True, temperatures=[0.6] * (j - i))
            for k, t in zip(range(i, j), toks):
                seqs[k].token_ids.append(t)
                left[k] -= 1
            i = j
        running = [k for k in range(num_seqs) if left[k] > 0]
        steps = 0
        while running:
            toks = runner.step([seqs[k] for k in running], False, temperatures=[0.6] * len(running))
            for k, t in zip(running, toks):
                seqs[k].token_ids.append(t)
                left[k] -= 1
            running = [k for k in running if left[k] > 0]
            steps += 1
        return sum(max_tokens), steps

    runner.step([Seq([1, 2, 3, 4], [0])], True, temperatures=[1.0])  # the reference's warm-up request
    _sync(torch, dist, world)
    with clock_sampler_cls(local) as clocks:
        t0 = time.time()
        total, steps = generate()
        torch.cuda.synchronize()
        seconds = time.time() - t0
    runner.runtime.check_status()
    if rank == 0:
        from nanovllm_b200 import _abi
        line = {"metric": "qwen3_0_6b_bench_output_tokens_per_s", "value": total / seconds, "unit": "tok/s", "n_gpus": world, "steps": steps, "warmup": 1,
                "ms_per_step": seconds * 1e3 / max(1, steps), "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
                "config": {"workload": f"the reference bench.py workload: Qwen3-0.6B random-init bf16, {num_seqs} sequences, prompt and output lengths uniform in [100, 1024], "
                                       f"temperature 0.6, ignore_eos, CUDA graphs, TP={world}; value = total output tokens / wall time (as the reference prints it)",
                           "l2": "decode steps stream the 1.2 GB of weights and the KV cache, far more than the 126 MB L2"},
                "clocks": clocks.summary(),
                "e2e": {"value": total / seconds, "unit": "tok/s", "h2d_bytes_per_step": None, "d2h_bytes_per_step": None,
                        "note": "wall clock through ModelRunner.step() with host batch state: this workload has no device-resident variant"},
                "gpu_launches": _abi.launch_count(), "total_output_tokens": total, "seconds": seconds}
        print(json.dumps(line), flush=True)
    runner.exit()
    dist.destroy_process_group()


# ---------------------------------------------------------------------------------------------------------------------
# vekerax: throughput of the Vekerax design beside Qwen3 with layers of the same size, and every kernel of the design
# beside the kernel of Qwen3 that does the like work.
# ---------------------------------------------------------------------------------------------------------------------
VEKERAX_SIZES = {  # layer sizes of Qwen3-0.6B and Qwen3-8B; fewer layers and a smaller vocabulary, the same for both models
    "width1024": dict(width=1024, ff=3072, heads=16, kv_heads=8, dim=128, layers=12, vocab=32768),
    "width4096": dict(width=4096, ff=12288, heads=32, kv_heads=8, dim=128, layers=8, vocab=32768),
}
VEKERAX_WINDOW, VEKERAX_KEEP, VEKERAX_STREAMS = 1024, 4, 4


def _vekerax_config(z: dict) -> dict:
    attn = {"type": "attention", "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                                           "softcap": 30.0, "mask": {"size": VEKERAX_WINDOW, "keep_first": VEKERAX_KEEP}},
            "mlp": {"kind": "dense", "ff": z["ff"]}}
    light = {"type": "lightning", "mixer": {"heads": z["heads"], "dim": z["dim"], "vdim": z["dim"],
                                            "decay": [1.0 - 2.0 ** (-2 - 6 * h / z["heads"]) for h in range(z["heads"])]},
             "mlp": {"kind": "dense", "ff": z["ff"]}}
    return {"architecture": "Vekerax", "embedding": {"scale": 1.0}, "layers": [attn, light] * (z["layers"] // 2), "norm": {"eps": 1e-6},
            "residual_mult": 1.0, "streams": VEKERAX_STREAMS, "vocab": z["vocab"], "width": z["width"]}


def _qwen_config(z: dict) -> dict:
    return {"architectures": ["Qwen3ForCausalLM"], "hidden_size": z["width"], "num_attention_heads": z["heads"], "num_key_value_heads": z["kv_heads"],
            "head_dim": z["dim"], "intermediate_size": z["ff"], "num_hidden_layers": z["layers"], "vocab_size": z["vocab"], "attention_bias": False}


def _model_throughput(torch, cfg: dict, vocab: int, batch: int, prompt: int, steps: int, warmup: int) -> dict:
    """Prefill tokens/s through step() (4 prompts a step) and decode tokens/s (device-resident and through step())."""
    from nanovllm_b200.engine.llm_engine import ensure_process_group
    from nanovllm_b200.engine.model_runner import ModelRunner, ResidentDecoder, Seq, sequential_block_tables
    from nanovllm_b200.models.registry import config_from_dict
    ensure_process_group()
    max_len = -(-(prompt + steps + warmup + 8) // 256) * 256
    runner = ModelRunner(config_from_dict(cfg), max_num_seqs=batch, max_model_len=max_len, max_num_batched_tokens=16384,
                         num_kvcache_blocks=batch * max_len // 256)
    g = torch.Generator().manual_seed(0)
    prompts = torch.randint(0, vocab, (batch, prompt), generator=g).tolist()
    tables = sequential_block_tables([max_len] * batch, 256)
    seqs = [Seq(p, t, 0, i) for i, (p, t) in enumerate(zip(prompts, tables))]
    per = max(1, min(batch, 8192 // prompt))

    def prefill():
        out = []
        for a in range(0, batch, per):
            out += runner.step(seqs[a:a + per], True)
        return out

    def timed(fn, n):
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        for _ in range(n):
            fn()
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / n

    for _ in range(2):
        first = prefill()
    pre_ms = timed(prefill, 3)
    for s, t in zip(seqs, first):
        s.token_ids = s.token_ids[:prompt] + [t]
    out = {"prefill_tok_s": batch * prompt / pre_ms * 1e3, "prefill_tokens_per_step": per * prompt}
    rd = ResidentDecoder(runner, batch)
    rd.load(seqs)
    for _ in range(warmup):
        rd.replay()
    ms = timed(rd.replay, steps)
    out.update(decode_tok_s=batch / ms * 1e3, decode_ms_per_step=ms, launches_per_decode_step=rd.kernels_per_step)

    def step():
        for s, t in zip(seqs, runner.step(seqs, False)):
            s.token_ids.append(t)
    for s in seqs:
        s.token_ids = s.token_ids[:prompt + 1]
    for _ in range(3):
        step()
    out["decode_tok_s_through_step"] = batch / timed(step, min(steps, max_len - prompt - 8)) * 1e3
    runner.runtime.check_status()
    runner.exit()
    del rd, runner
    import gc
    gc.collect()
    torch.cuda.empty_cache()
    return out


class KernelTable:
    """Rows (kernel, microseconds, fraction of the roofline) beside the like kernel of another model.  Rooflines: the measured
    copy bandwidth or burst bf16 throughput, or (bound "sum") seconds the caller has worked out from both."""

    def __init__(self, peaks: dict):
        self.peaks, self.rows = peaks, []

    def roof_us(self, work, bound) -> float:
        return work * 1e6 if bound == "sum" else work / (self.peaks["hbm_gbs"] * 1e9 if bound == "hbm" else self.peaks["bf16_tflops"] * 1e12) * 1e6

    def add(self, name, like, work, us, like_work, like_us, bound, like_bound=None):
        f, g = self.roof_us(work, bound) / us, self.roof_us(like_work, like_bound or bound) / like_us
        self.rows.append({"kernel": name, "us": round(us, 2), "bound": bound, "frac": round(f, 3), "like": like, "like_us": round(like_us, 2),
                          "like_frac": round(g, 3), "like_over_this": round(g / f, 2)})

    @staticmethod
    def variants(make, nbytes):
        """Enough copies of an input that a round through them exceeds L2."""
        return [make() for _ in range(max(2, min(48, int(4e8 / nbytes) + 1)))]


def _kernel_table(torch, z: dict, peaks: dict, batch: int, ctx_len: int) -> list[dict]:
    """Microseconds and fraction of the roofline (measured copy bandwidth or burst bf16 throughput) of every kernel of the
    design at this layer size, each next to the like kernel of Qwen3 on the same sizes.  Inputs rotate through more than L2."""
    from flash_attn import flash_attn_varlen_func, flash_attn_with_kvcache
    from nanovllm_b200 import _abi, ops
    from nanovllm_b200.rowpar_microbench import time_in_graph
    dev, bf, W, S = "cuda", torch.bfloat16, z["width"], VEKERAX_STREAMS
    H, G, d, ff, win, keep = z["heads"], z["kv_heads"], z["dim"], z["ff"], VEKERAX_WINDOW, VEKERAX_KEEP
    table = KernelTable(peaks)
    rows, add, variants = table.rows, table.add, table.variants

    for M in (batch, 8192):
        # residual: streams against add + RMSNorm
        nb = M * W * (8 * S + 4)
        vs = variants(lambda: (torch.randn(M, S, W, device=dev), torch.randn(M, W, device=dev).to(bf)), nb)
        mix, so, si, nw = torch.eye(S, device=dev), torch.ones(S, device=dev), torch.ones(S, device=dev) / S, torch.ones(W, device=dev)
        us = time_in_graph(lambda i: ops.stream_step(vs[i][0], vs[i][1], mix, so, 0.1, si, nw, 1e-6, W), len(vs), 4 * len(vs))
        nl = M * W * 8
        ls = variants(lambda: (torch.randn(M, W, device=dev).to(bf), torch.randn(M, W, device=dev).to(bf)), nl)
        nwb = nw.to(bf)
        lus = time_in_graph(lambda i: ops.add_rmsnorm(ls[i][0], ls[i][1], nwb, 1e-6), len(ls), 4 * len(ls))
        add(f"stream_step M={M}", "add_rmsnorm", nb, us, nl, lus, "hbm")
        del vs, ls
        # gated norm against RMSNorm of the same row length
        n = H * d
        nb = M * n * 8
        vs = variants(lambda: (torch.randn(M, n, device=dev), torch.randn(M, n, device=dev).to(bf)), nb)
        w = torch.ones(n, device=dev)
        us = time_in_graph(lambda i: ops.gated_norm(vs[i][0], vs[i][1], w, 1e-6, n), len(vs), 4 * len(vs))
        ls = variants(lambda: torch.randn(M, n, device=dev).to(bf), M * n * 4)
        wb = w.to(bf)
        lus = time_in_graph(lambda i: ops.rmsnorm(ls[i], wb, 1e-6), len(ls), 4 * len(ls))
        add(f"gated_norm M={M}", "rmsnorm", nb, us, M * n * 4, lus, "hbm")
        del vs, ls
        # projections: the same GEMM with other epilogues
        def gemm_pair(name, like, mine, theirs, N, out_cols, K):
            ws = [(torch.randn(N, K, device=dev) * 0.02).to(bf) for _ in range(max(2, min(12, int(3e8 / (N * K * 2)) + 1)))]
            x = torch.randn(M, K, device=dev).to(bf)
            us = time_in_graph(lambda i: mine(x, ws[i]), len(ws), 4 * len(ws))
            lus = time_in_graph(lambda i: theirs(x, ws[i]), len(ws), 4 * len(ws))
            if M > 1000:
                add(f"{name} M={M}", like, 2.0 * M * N * K, us, 2.0 * M * N * K, lus, "tensor")
            else:
                nbytes = 2.0 * (N * K + M * K + M * out_cols)
                add(f"{name} M={M}", like, nbytes, us, nbytes, lus, "hbm")
        gemm_pair("gate_up + relu*mul", "gate_up + silu*mul", lambda x, w: ops.gemm_act_mul(x, w, _abi.ACT_RELU), ops.gemm_silu_mul, 2 * ff, ff, W)
        gemm_pair("lightning q|k|v|g + silu", "gemm", lambda x, w: ops.gemm(x, w, silu_cols=3 * H * d), ops.gemm, 4 * H * d, 4 * H * d, W)
        # o / down projection and what follows: GEMM, then the stream launch, against the fused row-parallel block
        for nm, K in (("o_proj", H * d), ("down_proj", ff)):
            ws = [(torch.randn(W, K, device=dev) * 0.02).to(bf) for _ in range(max(2, min(24, int(3e8 / (W * K * 2)) + 1)))]
            x, xs, r = torch.randn(M, K, device=dev).to(bf), torch.randn(M, S, W, device=dev), torch.randn(M, W, device=dev).to(bf)
            us = time_in_graph(lambda i: ops.stream_step(xs, ops.gemm(x, ws[i]), mix, so, 0.1, si, nw, 1e-6, W), len(ws), 4 * len(ws))
            lus = time_in_graph(lambda i: ops.rowpar_fused(x, ws[i], None, r, nwb, 1e-6), len(ws), 4 * len(ws))
            if M > 1000:
                # time at the two rooflines: the product, then the bytes of the streams (the like block: residual and outputs)
                roof = 2.0 * M * W * K / (peaks["bf16_tflops"] * 1e12) + M * W * (8.0 * S + 4) / (peaks["hbm_gbs"] * 1e9)
                lroof = 2.0 * M * W * K / (peaks["bf16_tflops"] * 1e12) + M * W * 8.0 / (peaks["hbm_gbs"] * 1e9)
            else:
                roof = (2.0 * (W * K + M * K) + M * W * (8.0 * S + 4)) / (peaks["hbm_gbs"] * 1e9)
                lroof = (2.0 * (W * K + M * K) + M * W * 8.0) / (peaks["hbm_gbs"] * 1e9)
            rows.append({"kernel": f"{nm} + stream_step M={M}", "us": round(us, 2), "bound": "sum", "frac": round(roof * 1e6 / us, 3),
                         "like": "rowpar_fused", "like_us": round(lus, 2), "like_frac": round(lroof * 1e6 / lus, 3),
                         "like_over_this": round((lroof / lus) / (roof / us), 2)})
            del ws, x, xs, r
        # head norm and scatter after the projection (decode: inside the projection launch for both models)
        N = (H + 2 * G) * d
        kc = torch.zeros(64, 256, G, d, dtype=bf, device=dev)
        vc = torch.zeros_like(kc)
        slots = torch.randperm(64 * 256, device=dev)[:M].int()
        pos = torch.arange(M, device=dev) % 2048
        cs = torch.randn(2048, d, device=dev)
        qw = torch.ones(d, device=dev).to(bf)
        nb = M * d * (2 * H + 2 * H + 2 * G + 2 * G + 2 * G + 2 * G + 2 * G)  # q in and out, k in and out, v in, both to the cache
        vs = variants(lambda: torch.randn(M, N, device=dev).to(bf), nb)
        us = time_in_graph(lambda i: ops.qk_norm_store(vs[i], H, G, d, d, d, d, qw, qw, 1e-6, kc, vc, slots), len(vs), 4 * len(vs))
        lus = time_in_graph(lambda i: ops.qk_norm_rope_store(vs[i], H, G, d, qw, qw, 1e-6, pos, cs, kc, vc, slots), len(vs), 4 * len(vs))
        add(f"qk_norm_store M={M}", "qk_norm_rope_store", nb, us, nb, lus, "hbm")
        del vs, kc, vc
    # attention, prefill: sequences of 2048 in a batch of 8192, the same window for both
    B, L = 4, 2048
    M = B * L
    kc = torch.randn(B * L // 256, 256, G, d, device=dev).to(bf)
    vc = torch.randn_like(kc)
    bt = torch.randperm(B * L // 256, device=dev).int().view(B, -1).contiguous()
    cu = torch.arange(0, M + 1, L, device=dev, dtype=torch.int32)
    kl = torch.full((B,), L, dtype=torch.int32, device=dev)
    q = torch.randn(M, H * d, device=dev).to(bf)
    sink = torch.zeros(H, device=dev)
    seen = sum(min(i + 1, win) for i in range(L)) * B
    flops = 4.0 * H * d * seen
    k, v = torch.randn(M, G, d, device=dev).to(bf), torch.randn(M, G, d, device=dev).to(bf)
    us = time_in_graph(lambda i: ops.window_attention(q, H, kc, vc, bt, cu, kl, L, L, d ** -0.5, 30.0, win, keep, sink), 4, 24)
    lus = time_in_graph(lambda i: flash_attn_varlen_func(q.view(M, H, d), k, v, cu, cu, L, L, softmax_scale=d ** -0.5, causal=True, window_size=(win - 1, 0)), 4, 24)
    add(f"window_attention prefill {B}x{L} window {win}", "flash-attn, same window, passed K/V", flops, us, flops, lus, "tensor")
    # linear attention, prefill
    D = torch.tensor([1.0 - 2.0 ** (-2 - 6 * h / H) for h in range(H)], dtype=torch.float64)
    dec, pw = D.float().to(dev), (D.unsqueeze(1) ** torch.arange(65)).float().to(dev)
    p = torch.randn(M, 4 * H * d, device=dev).to(bf)
    state = torch.zeros(max(batch, B), H, d, d, device=dev)
    sl = torch.arange(B, device=dev, dtype=torch.int32)
    lin_flops = 2.0 * M * H * (2 * d * d + 64 * d)  # state in and out, and the causal half of two 64-wide products
    us2 = time_in_graph(lambda i: ops.linear_attn(p, H, d, d, state, sl, cu, kl, L, dec, pw), 4, 24)
    full = 4.0 * H * d * B * L * (L + 1) / 2
    lus2 = time_in_graph(lambda i: flash_attn_varlen_func(q.view(M, H, d), k, v, cu, cu, L, L, softmax_scale=d ** -0.5, causal=True), 4, 24)
    # bound by memory: its bytes (q, k, v in bf16, o in fp32) take longer than its flops; the like kernel by the tensor pipe
    roof = max(M * H * d * (3 * 2 + 4.0) / (peaks["hbm_gbs"] * 1e9), lin_flops / (peaks["bf16_tflops"] * 1e12)) * 1e6
    lroof = full / (peaks["bf16_tflops"] * 1e12) * 1e6
    rows.append({"kernel": f"linear_attn prefill {B}x{L}", "us": round(us2, 2), "bound": "hbm", "frac": round(roof / us2, 3), "like": "flash-attn, full causal",
                 "like_us": round(lus2, 2), "like_frac": round(lroof / lus2, 3), "like_over_this": round((lroof / lus2) / (roof / us2), 2)})
    # decode
    nblk = -(-ctx_len // 256)
    n_layers = 6
    kcs = [torch.randn(batch * nblk, 256, G, d, device=dev).to(bf) for _ in range(n_layers)]
    vcs = [torch.randn(batch * nblk, 256, G, d, device=dev).to(bf) for _ in range(n_layers)]
    bt = torch.randperm(batch * nblk, device=dev).int().view(batch, nblk).contiguous()
    kl = torch.full((batch,), ctx_len, dtype=torch.int32, device=dev)
    q = torch.randn(batch, H * d, device=dev).to(bf)
    nb = 2.0 * batch * min(ctx_len, win) * G * d * 2
    us = time_in_graph(lambda i: ops.window_attention(q, H, kcs[i], vcs[i], bt, None, kl, 1, nblk * 256, d ** -0.5, 30.0, win, keep, sink), n_layers, 10 * n_layers)
    lus = time_in_graph(lambda i: flash_attn_with_kvcache(q.view(batch, 1, H, d), kcs[i], vcs[i], cache_seqlens=kl, block_table=bt, softmax_scale=d ** -0.5, causal=True),
                        n_layers, 10 * n_layers)
    add(f"window_attention decode {batch} x {ctx_len}", "flash-attn kvcache", nb, us, nb, lus, "hbm")
    sts = [torch.zeros(batch, H, d, d, device=dev) for _ in range(4)]
    sl = torch.arange(batch, device=dev, dtype=torch.int32)
    p = torch.randn(batch, 4 * H * d, device=dev).to(bf)
    us = time_in_graph(lambda i: ops.linear_attn(p, H, d, d, sts[i], sl, None, kl, 1, dec, pw), 4, 40)
    add(f"linear_attn decode {batch}", "flash-attn kvcache", 8.0 * batch * H * d * d, us, nb, lus, "hbm")
    return rows


def run_vekerax(args, peaks, clock_sampler_cls) -> None:
    torch, dist, rank, world, local = _setup(args)
    assert world == 1, "Vekerax runs on one GPU"
    from nanovllm_b200 import runtime as rt
    K, W = min(args.steps, 128), max(3, args.warmup)
    sizes = {}
    with clock_sampler_cls(local) as clocks:
        for name, z in VEKERAX_SIZES.items():
            res = {}
            for batch, prompt in ((64, 1024), (4, 4096)):
                key = f"batch {batch}, prompts of {prompt}"
                res[key] = {"vekerax": _model_throughput(torch, _vekerax_config(z), z["vocab"], batch, prompt, K, W),
                            "qwen3": _model_throughput(torch, _qwen_config(z), z["vocab"], batch, prompt, K, W)}
            rt.init_runtime(max_tokens=8192, hidden=z["width"], oneshot_tokens=1024)
            with torch.inference_mode():
                kernels = _kernel_table(torch, z, peaks, 64, 1024)
            rt.shutdown_runtime()
            torch.cuda.empty_cache()
            sizes[name] = {"layer_sizes": z, "throughput": res, "kernels": kernels}
    from nanovllm_b200 import _abi
    head = sizes["width4096"]["throughput"]["batch 64, prompts of 1024"]["vekerax"]
    print(json.dumps({"metric": "vekerax_decode_tokens_per_s", "value": head["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": K, "warmup": W,
                      "ms_per_step": head["decode_ms_per_step"], "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
                      "config": {"workload": f"Vekerax and Qwen3 with the same layer sizes, random weights; {VEKERAX_STREAMS} streams, window {VEKERAX_WINDOW} + {VEKERAX_KEEP}, "
                                             "attention and lightning layers in turn; value: width 4096, batch 64, 1024-token prompts, device-resident decode",
                                 "l2": "weights, caches and rotated kernel inputs exceed the 126 MB L2"},
                      "clocks": clocks.summary(), "gpu_launches": _abi.launch_count(), "sizes": sizes}), flush=True)
    dist.destroy_process_group()


# ---------------------------------------------------------------------------------------------------------------------
# mupulorn
# ---------------------------------------------------------------------------------------------------------------------
# the layer sizes above with latents; its feed-forward has two matrices instead of three, so ff is 1.5 times as wide
MUPULORN_SIZES = {
    "width1024": dict(VEKERAX_SIZES["width1024"], q_rank=512, kv_rank=256, rot_dim=64),
    "width4096": dict(VEKERAX_SIZES["width4096"], q_rank=1536, kv_rank=512, rot_dim=64),
}
MUPULORN_TAPS = 4


def _mupulorn_config(z: dict) -> dict:
    mixer = {"heads": z["heads"], "dim": z["dim"], "rot_dim": z["rot_dim"], "vdim": z["dim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"],
             "scale": (z["dim"] + z["rot_dim"]) ** -0.5, "rot": {"base": 10000.0, "dims": z["rot_dim"]}}
    layer = {"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": z["ff"] * 3 // 2}}
    return {"architecture": "Mupulorn", "canon": {"taps": MUPULORN_TAPS}, "layers": [layer] * z["layers"], "logit_scale": 0.5, "logit_softcap": 30.0,
            "norm": {"eps": 1e-6}, "vocab": z["vocab"], "width": z["width"]}


def _mupulorn_kernels(torch, z: dict, peaks: dict, batch: int, ctx_len: int) -> list[dict]:
    """Every kernel of the design at this layer size next to the like kernel of Qwen3."""
    from flash_attn import flash_attn_varlen_func, flash_attn_with_kvcache
    from nanovllm_b200 import ops
    from nanovllm_b200.layers.rotary_embedding import PairRotation
    from nanovllm_b200.rowpar_microbench import time_in_graph
    dev, bf, W, taps = "cuda", torch.bfloat16, z["width"], MUPULORN_TAPS
    H, G, d, rot, L, Q, ff = z["heads"], z["kv_heads"], z["dim"], z["rot_dim"], z["kv_rank"], z["q_rank"], z["ff"] * 3 // 2
    row, qh = L + rot, d + rot
    table = KernelTable(peaks)
    add, variants = table.add, table.variants
    hbm, tensor = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12
    rnd = lambda *s, k=1.0: (torch.randn(*s, device=dev) * k).to(bf)
    rope = PairRotation(rot, rot, 10000.0)
    rope.bind(8192, dev)
    one = torch.ones(1, device=dev)
    conv = rnd(taps, W, k=0.1)
    nwb = torch.ones(W, device=dev, dtype=bf)

    for M in (batch, 8192):
        seqs = batch if M == batch else 4
        slots = torch.arange(seqs, device=dev, dtype=torch.int32)
        lens = torch.full((seqs,), 1024 if M == batch else M // seqs, device=dev, dtype=torch.int32)
        cu = None if M == batch else torch.arange(0, M + 1, M // seqs, device=dev, dtype=torch.int32)
        per = 1 if M == batch else M // seqs
        cuts = (cu, lens, slots, per)
        states = [torch.zeros(seqs, taps - 1, W, device=dev, dtype=bf) for _ in range(8)]
        step = lambda x, y, i: ops.sandwich_step(x, y, one, one, 1e-6, W, cuts, conv, states[i % 8])
        # residual: x read and written in fp32, y in, h out (and the states of decoded rows)
        nb = M * W * (8 + 4) + (2 * (taps - 1) * seqs * W * 2)
        vs = variants(lambda: (torch.randn(M, W, device=dev), rnd(M, W)), nb)
        us = time_in_graph(lambda i: step(*vs[i], i), len(vs), 4 * len(vs))
        nl = M * W * 8
        ls = variants(lambda: (rnd(M, W), rnd(M, W)), nl)
        lus = time_in_graph(lambda i: ops.add_rmsnorm(ls[i][0], ls[i][1], nwb, 1e-6), len(ls), 4 * len(ls))
        add(f"sandwich_step M={M}", "add_rmsnorm", nb, us, nl, lus, "hbm")
        del vs, ls
        # PolyNorm (rows of ff) against RMSNorm (rows of the width)
        nb = M * ff * 4
        vs = variants(lambda: rnd(M, ff), nb)
        coef = torch.full((4,), 0.3, device=dev)
        us = time_in_graph(lambda i: ops.poly_norm(vs[i], coef, 1e-6, ff), len(vs), 4 * len(vs))
        ls = variants(lambda: rnd(M, W), M * W * 4)
        lus = time_in_graph(lambda i: ops.rmsnorm(ls[i], nwb, 1e-6), len(ls), 4 * len(ls))
        add(f"poly_norm M={M}", "rmsnorm", nb, us, M * W * 4, lus, "hbm")
        del vs, ls
        # latent norms, rotation and scatter against head norm, rotation and scatter
        N = Q + row + H * d
        cache = torch.zeros(64, 256, 1, row, dtype=bf, device=dev)
        sm = torch.randperm(64 * 256, device=dev)[:M].int()
        pos = torch.arange(M, device=dev) % 2048
        qw, kw = torch.ones(Q, device=dev), torch.ones(L, device=dev)
        nb = M * (2 * Q * 2 + 3 * row * 2)
        vs = variants(lambda: rnd(M, N), M * N * 2)
        us = time_in_graph(lambda i: ops.latent_store(vs[i], Q, Q, L, L, rot, qw, kw, 1e-6, pos, rope.table, cache, sm), len(vs), 4 * len(vs))
        del vs
        kc = torch.zeros(64, 256, G, d, dtype=bf, device=dev)
        vc, cs, hw = torch.zeros_like(kc), torch.randn(2048, d, device=dev), torch.ones(d, device=dev, dtype=bf)
        nl = M * d * (4 * H + 10 * G)
        ls = variants(lambda: rnd(M, (H + 2 * G) * d), nl)
        lus = time_in_graph(lambda i: ops.qk_norm_rope_store(ls[i], H, G, d, hw, hw, 1e-6, pos, cs, kc, vc, sm), len(ls), 4 * len(ls))
        add(f"latent_store M={M}", "qk_norm_rope_store", nb, us, nl, lus, "hbm")
        del ls, kc, vc, cache
        # o / down projection and what follows against the fused row-parallel block
        for nm, K in (("o_proj", H * d), ("down_proj", ff)):
            ws = [rnd(W, K, k=0.02) for _ in range(max(2, min(24, int(3e8 / (W * K * 2)) + 1)))]
            x, r, xs = rnd(M, K), rnd(M, W), torch.randn(M, W, device=dev)
            us = time_in_graph(lambda i: step(xs, ops.gemm(x, ws[i]), i), len(ws), 4 * len(ws))
            lus = time_in_graph(lambda i: ops.rowpar_fused(x, ws[i], None, r, nwb, 1e-6), len(ws), 4 * len(ws))
            if M > 1000:
                roof, lroof = 2.0 * M * W * K / tensor + M * W * 12.0 / hbm, 2.0 * M * W * K / tensor + M * W * 8.0 / hbm
            else:
                roof, lroof = (2.0 * (W * K + M * K) + M * W * 24.0) / hbm, (2.0 * (W * K + M * K) + M * W * 8.0) / hbm
            add(f"{nm} + sandwich_step M={M}", "rowpar_fused", roof, us, lroof, lus, "sum")
            del ws, x, r, xs
        # the design's other projections run on the same GEMM; a plain one of Qwen3's sizes beside them
        def gemm_us(N, K):
            ws = [rnd(N, K, k=0.02) for _ in range(max(2, min(24, int(3e8 / (N * K * 2)) + 1)))]
            x = rnd(M, K)
            return time_in_graph(lambda i: ops.gemm(x, ws[i]), len(ws), 4 * len(ws))
        # seconds at the slower of the two rooflines (a short K makes even a product of many tokens bound by its output)
        work = lambda N, K: max(2.0 * M * N * K / tensor, 2.0 * (N * K + M * K + M * N) / hbm)
        Nq = (H + 2 * G) * d
        qkv_us = gemm_us(Nq, W)
        for nm, N, K in (("in_proj", Q + row + H * d, W), ("q_proj", H * qh, Q), ("up_proj", ff, W)) + ((("kv_proj", H * 2 * d, L),) if M > 1000 else ()):
            add(f"{nm} M={M}", "qkv projection GEMM", work(N, K), gemm_us(N, K), work(Nq, W), qkv_us, "sum")
        if M == batch:  # per-head products of the absorbed form
            ws = [rnd(H, 2 * d, L, k=0.05) for _ in range(max(2, min(48, int(3e8 / (H * 2 * d * L * 2)) + 1)))]
            q, o, gate = rnd(M, H * qh), rnd(M, H * L), rnd(M, H * d)
            nb = 2.0 * (H * d * L + M * H * (qh + row))
            us = time_in_graph(lambda i: ops.heads_gemm(q, qh, ws[i][:, :d], True, row, rotate=(rot, pos, rope.table)), len(ws), 4 * len(ws))
            add(f"heads_gemm q Wk + rotation M={M}", "qkv projection GEMM", nb / hbm, us, work(Nq, W), qkv_us, "sum")
            nb = 2.0 * (H * d * L + M * H * (L + 2 * d))
            us = time_in_graph(lambda i: ops.heads_gemm(o, L, ws[i][:, d:], False, d, gate=gate, gate_head=d), len(ws), 4 * len(ws))
            add(f"heads_gemm Wv + gate M={M}", "qkv projection GEMM", nb / hbm, us, work(Nq, W), qkv_us, "sum")
            del ws
    sink = torch.zeros(H, device=dev)
    # prompts: 4 sequences of 2048, full causal
    B, T = 4, 2048
    M = B * T
    cu = torch.arange(0, M + 1, T, device=dev, dtype=torch.int32)
    q, kv, kr, gate = rnd(M, H * qh), rnd(M, H * 2 * d), rnd(M, rot), rnd(M, H * d)
    pairs = B * T * (T + 1) / 2
    us = time_in_graph(lambda i: ops.expanded_attention(q, H, kv, kr, cu, cu, T, d, rot, d, qh ** -0.5, sink, rope.table, gate), 4, 16)
    fq, fk, fv = rnd(M, H, d), rnd(M, G, d), rnd(M, G, d)
    lus = time_in_graph(lambda i: flash_attn_varlen_func(fq, fk, fv, cu, cu, T, T, softmax_scale=d ** -0.5, causal=True), 4, 16)
    add(f"expanded_attention {B}x{T}", "flash-attn, full causal", 2.0 * H * (qh + d) * pairs, us, 4.0 * H * d * pairs, lus, "tensor")
    # decoding, and a portion of 64 tokens (absorbed) against decoding / flash-attn on the cache
    nblk = -(-ctx_len // 256)
    layers = max(4, int(4e8 / (batch * nblk * 256 * row * 2)) + 1)
    caches = [rnd(batch * nblk, 256, 1, row) for _ in range(layers)]
    bt = torch.randperm(batch * nblk, device=dev).int().view(batch, nblk).contiguous()
    kl = torch.full((batch,), ctx_len, dtype=torch.int32, device=dev)
    q = rnd(batch, H * row)
    us = time_in_graph(lambda i: ops.latent_attention(q, H, caches[i], L, bt, None, kl, 1, nblk * 256, qh ** -0.5, sink), layers, 10 * layers)
    kcs = [rnd(batch * nblk, 256, G, d) for _ in range(4)]
    vcs = [rnd(batch * nblk, 256, G, d) for _ in range(4)]
    fq = rnd(batch, 1, H, d)
    lus = time_in_graph(lambda i: flash_attn_with_kvcache(fq, kcs[i], vcs[i], cache_seqlens=kl, block_table=bt, softmax_scale=d ** -0.5, causal=True), 4, 40)
    like = 2.0 * batch * ctx_len * G * d * 2
    add(f"latent_attention decode {batch} x {ctx_len}", "flash-attn kvcache", 2.0 * batch * (ctx_len * row + H * (row + L)), us, like, lus, "hbm")
    P = 64
    cu = torch.tensor([0, P], device=dev, dtype=torch.int32)
    big = bt.view(1, -1)
    n = min(16384, batch * nblk * 256)
    q, kl1 = rnd(P, H * row), torch.tensor([n], device=dev, dtype=torch.int32)
    us = time_in_graph(lambda i: ops.latent_attention(q, H, caches[i], L, big, cu, kl1, P, n, qh ** -0.5, sink), layers, 4 * layers)
    fq = rnd(P, H, d)
    cuk = torch.tensor([0, n], device=dev, dtype=torch.int32)
    lus = time_in_graph(lambda i: flash_attn_varlen_func(fq, kcs[i], vcs[i], cu, cuk, P, n, softmax_scale=d ** -0.5, causal=True, block_table=big), 4, 16)
    seen = P * (n - P / 2)
    add(f"latent_attention portion of {P} at {n}", "flash-attn, paged, the same portion", 2.0 * H * (row + L) * seen, us, 4.0 * H * d * seen, lus, "tensor")
    return table.rows


def run_mupulorn(args, peaks, clock_sampler_cls) -> None:
    torch, dist, rank, world, local = _setup(args)
    assert world == 1, "Mupulorn runs on one GPU"
    from nanovllm_b200 import runtime as rt
    K, W = min(args.steps, 128), max(3, args.warmup)
    sizes = {}
    with clock_sampler_cls(local) as clocks:
        for name, z in MUPULORN_SIZES.items():
            res = {}
            for batch, prompt in ((64, 1024), (4, 4096)):
                res[f"batch {batch}, prompts of {prompt}"] = {"mupulorn": _model_throughput(torch, _mupulorn_config(z), z["vocab"], batch, prompt, K, W),
                                                              "qwen3": _model_throughput(torch, _qwen_config(z), z["vocab"], batch, prompt, K, W)}
            rt.init_runtime(max_tokens=8192, hidden=z["width"], oneshot_tokens=1024)
            with torch.inference_mode():
                kernels = _mupulorn_kernels(torch, z, peaks, 64, 1024)
            rt.shutdown_runtime()
            torch.cuda.empty_cache()
            sizes[name] = {"layer_sizes": z, "throughput": res, "kernels": kernels}
    from nanovllm_b200 import _abi
    head = sizes["width4096"]["throughput"]["batch 64, prompts of 1024"]["mupulorn"]
    print(json.dumps({"metric": "mupulorn_decode_tokens_per_s", "value": head["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": K, "warmup": W,
                      "ms_per_step": head["decode_ms_per_step"], "higher_is_better": True, "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
                      "config": {"workload": "Mupulorn and Qwen3 with the same layer sizes, random weights; value: width 4096, batch 64, 1024-token prompts, "
                                             "device-resident decode", "l2": "weights, caches and rotated kernel inputs exceed the 126 MB L2"},
                      "clocks": clocks.summary(), "gpu_launches": _abi.launch_count(), "sizes": sizes}), flush=True)
    dist.destroy_process_group()
