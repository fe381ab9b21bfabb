"""Small Vekerax configurations and weights for the tests (sizes are the tests' own)."""
import torch

from oracle import vekerax as V


def attn(heads=6, kv_heads=2, dim=24, vdim=40, size=37, keep=3, cap=20.0, scale=0.3, ff=88):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap,
                                           "mask": {"size": size, "keep_first": keep}}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def light(heads=3, dim=20, vdim=28, decay=None, ff=104):
    decay = decay or [0.5 + 0.49 * (i + 1) / heads for i in range(heads)]
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=160, streams=3, loop=None, eps=1e-5, m=0.4, scale=1.7):
    c = {"architecture": "Vekerax", "embedding": {"scale": scale}, "layers": layers, "norm": {"eps": eps}, "residual_mult": m, "streams": streams,
         "vocab": vocab, "width": width}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


CASES = {
    # mixed layers, a loop over both kinds, head sizes that need padding, a layer without a feed-forward
    "mixed": config([attn(), light(), attn(heads=4, kv_heads=4, dim=16, vdim=16, size=9, keep=0, ff=0), light(heads=2, dim=64, vdim=72)], loop=(0, 2, 2)),
    # nothing looped, lightning first, one stream, vocabulary and width that are not multiples of 8
    "odd": config([light(heads=5, dim=12, vdim=9), attn(heads=5, kv_heads=1, dim=33, vdim=17, size=64, keep=65)], width=60, vocab=131, streams=1, m=1.0),
    # the sizes of the fused decode projection (128-wide heads) and a window of one token
    "wide": config([attn(heads=4, kv_heads=2, dim=128, vdim=128, size=50, keep=1, scale=0.09, ff=96), light(heads=2, dim=128, vdim=136, ff=0),
                    attn(heads=3, kv_heads=3, dim=128, vdim=64, size=1, keep=2, scale=0.09)], width=128, vocab=256, streams=4, loop=(1, 3, 2)),
}


def shapes(cfg):
    """Tensor names and shapes of a checkpoint, written down from the layer equations."""
    D, S, out = cfg["width"], cfg["streams"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (cfg["width"],)}
    for i, l in enumerate(cfg["layers"]):
        m, p = l["mixer"], f"l{i}."
        for q in ("1", "2") if l["mlp"] else ("1",):
            out |= {f"{p}norm{q}": (D,), f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)}
        g = m.get("kv_heads", m["heads"])
        out |= {p + "mix.q": (m["heads"] * m["dim"], D), p + "mix.k": (g * m["dim"], D), p + "mix.v": (g * m["vdim"], D), p + "mix.o": (D, m["heads"] * m["vdim"])}
        out |= {p + "mix.q.norm": (m["dim"],), p + "mix.k.norm": (m["dim"],), p + "mix.sink": (m["heads"],)} if l["type"] == "attention" else \
               {p + "mix.g": (m["heads"] * m["vdim"], D), p + "mix.norm": (m["heads"] * m["vdim"],)}
        if l["mlp"]:
            out |= {p + "mlp.gate": (l["mlp"]["ff"], D), p + "mlp.up": (l["mlp"]["ff"], D), p + "mlp.down": (D, l["mlp"]["ff"])}
    return out


def weights(cfg, seed=0):
    """bf16 weights with which scores, decays, sinks and streams all matter."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        if name.endswith("norm") or "norm" in name.split(".")[-1]:
            t = 1.0 + 0.3 * r
            if name.endswith(("q.norm", "k.norm")):
                t = 1.5 * t
        elif ".hc" in name:
            s = cfg["streams"]
            t = {"in": 1.0 / s + 0.3 * r, "out": 1.0 + 0.3 * r, "mix": (torch.eye(s) * 0.8 + 0.2 * r / s) if r.dim() == 2 else r}[name.rsplit(".", 1)[1]]
        elif name.endswith("sink"):
            t = 1.0 + r
        else:
            t = r / shape[-1] ** 0.5
        w[name] = t.bfloat16()
    return w


def save(folder, cfg, w):
    """config.json and model.safetensors (8-byte header length, JSON header, data)."""
    import json
    import os
    import struct
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


# root mean square of the logits' error over their own; bf16: what rounding does to these deliberately lively weights
TOL = {torch.float32: 2e-4, torch.bfloat16: 0.12}


class Model:
    """A test model behind the framework's engine, beside the plain implementation's logits for the same weights (GPU)."""

    def __init__(self, case, dtype, **kw):
        from tests.gpu_util import ensure_group
        ensure_group()
        from nanovllm_b200.engine.llm_engine import LLM
        self.cfg = CASES[case] if isinstance(case, str) else case
        w = weights(self.cfg, 5)
        self.w64 = {k: t.double() for k, t in w.items()}
        self.dtype = dtype
        self.llm = LLM(self.cfg, w, dtype=dtype, **({"max_num_seqs": 4, "max_model_len": 512, "max_num_batched_tokens": 512, "kvcache_block_size": 16,
                                                     "num_kvcache_blocks": 80} | kw))
        self.runner, self.cache = self.llm.runner, self.llm.cache
        self.memo = {}

    def want(self, toks):
        key = tuple(toks)
        if key not in self.memo:
            self.memo[key] = V.forward(self.cfg, self.w64, list(toks))[0]
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
        toks.append(int(V.forward(m.cfg, m.w64, toks)[0][-1].argmax()))
    return toks[len(prompt):]
