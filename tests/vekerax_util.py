"""Small Vekerax configurations and weights for the tests (sizes are the tests' own)."""
import torch

from oracle import vekerax as V
from tests.model_util import ServedModel


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


class Model(ServedModel):
    def __init__(self, case, dtype, **kw):
        cfg = CASES[case] if isinstance(case, str) else case
        super().__init__(V.forward, cfg, weights(cfg, 5), dtype, **kw)
