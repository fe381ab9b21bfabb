"""Small Mupulorn configurations and weights for the tests (sizes are the tests' own)."""
import torch

from oracle import mupulorn as P
from tests.model_util import ServedModel


def latent(heads=5, dim=20, rot=12, vdim=28, q=44, kv=52, scale=0.2, base=700.0, ff=104):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q, "kv_rank": kv, "scale": scale,
                                                  "rot": {"base": base, "dims": rot}}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def like(layers, j):
    """A layer that uses layer j's weights."""
    return dict(layers[j], weights_of=j)


def config(layers, width=72, vocab=160, taps=3, eps=1e-5, scale=0.7, cap=9.0):
    return {"architecture": "Mupulorn", "canon": {"taps": taps}, "layers": layers, "logit_scale": scale, "logit_softcap": cap, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


_mixed = [latent(), latent(heads=3, dim=16, rot=8, vdim=40, q=24, kv=32, scale=0.3, base=50.0, ff=0)]
_mixed += [like(_mixed, 0), latent(heads=2, dim=64, rot=10, vdim=9, q=40, kv=72, ff=72), like(_mixed, 1)]
_odd = [latent(heads=17, dim=40, rot=20, vdim=72, q=33, kv=136, scale=0.15, ff=57)]
_wide = [latent(heads=20, dim=128, rot=64, vdim=128, q=136, kv=264, scale=0.08, base=10000.0, ff=320)]
CASES = {
    # layers of different sizes, a layer without a feed-forward, shared weights; head sizes that need padding
    "mixed": config(_mixed),
    # more heads than one row tile, six taps, width and vocabulary that are not multiples of 8
    "odd": config(_odd + [like(_odd, 0)], width=60, vocab=131, taps=6, eps=1e-3),
    # the widest tiles
    "wide": config(_wide + [latent(heads=16, dim=96, rot=32, vdim=64, q=64, kv=128, scale=0.1, ff=0)], width=136, vocab=256, taps=4, scale=1.0, cap=20.0),
    # one head, one rotated pair, two taps
    "small": config([latent(heads=1, dim=7, rot=2, vdim=5, q=6, kv=9, scale=0.5, base=3.0, ff=16)] * 2, width=24, vocab=64, taps=2),
}


def shapes(cfg):
    """Tensor names and shapes of a checkpoint, written down from the layer equations."""
    D, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"]), "final.norm": (), "head": (cfg["vocab"], cfg["width"])}
    for i, l in enumerate(cfg["layers"]):
        if "weights_of" in l:
            continue
        m, p, H = l["mixer"], f"l{i}.", l["mixer"]["heads"]
        for n in "12" if l["mlp"] else "1":
            out |= {f"{p}norm{n}": (), f"{p}norm{n}b": (), f"{p}canon{n}": (D, cfg["canon"]["taps"])}
        p += "mix."
        out |= {p + "dq": (m["q_rank"], D), p + "dq.norm": (m["q_rank"],), p + "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]),
                p + "dkv": (m["kv_rank"] + m["rot_dim"], D), p + "dkv.norm": (m["kv_rank"],), p + "uk": (H * m["dim"], m["kv_rank"]),
                p + "uv": (H * m["vdim"], m["kv_rank"]), p + "sink": (H,), p + "g": (H * m["vdim"], D), p + "o": (D, H * m["vdim"])}
        if l["mlp"]:
            out |= {f"l{i}.mlp.up": (l["mlp"]["ff"], D), f"l{i}.mlp.down": (D, l["mlp"]["ff"]), f"l{i}.mlp.act": (4,)}
    return out


def weights(cfg, seed=0):
    """bf16 weights with which scores, sinks, gates, taps and every term of the activation matter."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in shapes(cfg).items():
        r = torch.randn(shape, generator=g)
        leaf = name.split(".")[-1]
        if "norm" in leaf:
            t = 1.0 + 0.3 * r
            if leaf.endswith("b"):
                t = 0.7 * t
        elif "canon" in leaf:
            t = 0.5 * r
        elif leaf == "act":
            t = 0.5 + 0.3 * r
        elif leaf == "sink":
            t = 1.0 + r
        elif leaf == "embed":
            t = r
        elif leaf == "uq":
            t = 1.5 * r / shape[-1] ** 0.5
        else:
            t = r / shape[-1] ** 0.5
        w[name] = t.bfloat16()
    return w


class Model(ServedModel):
    def __init__(self, case, dtype, **kw):
        cfg = CASES[case] if isinstance(case, str) else case
        super().__init__(P.forward, cfg, weights(cfg, 5), dtype, **kw)
