"""Plain, slow restatement of the Mupulorn decoder on the CPU (test infrastructure only).

One function per mechanism; it shares no code with the product path.  Everything runs in the dtype of the weights it is
given (the tests use float64).

A model is (config dict, weights dict); the weights are plain tensors under the checkpoint's names.
"""
from __future__ import annotations

import math

import torch


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gain_norm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    """RMSNorm; the weight is one number for all channels or one per channel."""
    return unit_rms(x, eps) * gain


def causal_conv(h: torch.Tensor, w: torch.Tensor, past: torch.Tensor | None = None) -> torch.Tensor:
    """h [T, D], w [D, taps]: y_t = sum_j w[:, j] h_(t - taps + 1 + j); `past` holds the taps - 1 inputs before h (zeros)."""
    taps = w.shape[1]
    past = torch.zeros(taps - 1, h.shape[1], dtype=h.dtype) if past is None else past
    seq = torch.cat((past, h))
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(taps):
            out[t] += w[:, j] * seq[t + j]
    return out


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, ..., n]: elements (2i, 2i + 1), 2i < dims, turn by position * base^(-2i / dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = (positions.to(x.dtype) * base ** (-2.0 * i / dims)).view(-1, *[1] * (x.dim() - 2))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Weights exp(s_j) / (exp(sink) + sum_j exp(s_j)) over the last dimension."""
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attend(qn: torch.Tensor, qr: torch.Tensor, kn: torch.Tensor, kr: torch.Tensor, v: torch.Tensor, scale: float, sink: torch.Tensor,
           first_pos: int = 0) -> torch.Tensor:
    """Unrotated parts qn [Tq, H, d], kn [Tk, H, d]; rotated parts qr [Tq, H, r], kr [Tk, r] (one for all heads); v [Tk, H, dv].
    Queries stand at first_pos, first_pos + 1, ...; keys at 0, 1, ..."""
    tq, heads = qn.shape[:2]
    out = torch.zeros(tq, heads, v.shape[2], dtype=qn.dtype)
    for t in range(tq):
        n = first_pos + t + 1
        for h in range(heads):
            s = (kn[:n, h] @ qn[t, h] + kr[:n] @ qr[t, h]) * scale
            out[t, h] = sink_softmax(s, sink[h]) @ v[:n, h]
    return out


def latents(h: torch.Tensor, w: dict, pre: str, c: dict, eps: float, first_pos: int = 0) -> tuple[torch.Tensor, torch.Tensor]:
    """What a token leaves in the cache: the normed latent and the rotated key part."""
    y = h @ w[pre + "dkv"].T
    pos = torch.arange(first_pos, first_pos + h.shape[0])
    return gain_norm(y[:, :c["kv_rank"]], w[pre + "dkv.norm"], eps), rotate_pairs(y[:, c["kv_rank"]:], pos, c["rot"]["dims"], c["rot"]["base"])


def queries(h: torch.Tensor, w: dict, pre: str, c: dict, eps: float, first_pos: int = 0) -> tuple[torch.Tensor, torch.Tensor]:
    q = gain_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T
    q = q.view(h.shape[0], c["heads"], c["dim"] + c["rot_dim"])
    pos = torch.arange(first_pos, first_pos + h.shape[0])
    return q[..., :c["dim"]], rotate_pairs(q[..., c["dim"]:], pos, c["rot"]["dims"], c["rot"]["base"])


def attention_mixer(h: torch.Tensor, w: dict, pre: str, c: dict, eps: float) -> torch.Tensor:
    t = h.shape[0]
    qn, qr = queries(h, w, pre, c, eps)
    lat, kr = latents(h, w, pre, c, eps)
    kn = (lat @ w[pre + "uk"].T).view(t, c["heads"], c["dim"])
    v = (lat @ w[pre + "uv"].T).view(t, c["heads"], c["vdim"])
    o = attend(qn, qr, kn, kr, v, c["scale"], w[pre + "sink"]).reshape(t, -1)
    return (o * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    a, b, c, e = coef
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def dense_ff(h: torch.Tensor, w: dict, pre: str, eps: float) -> torch.Tensor:
    return poly_norm(h @ w[pre + "up"].T, w[pre + "act"], eps) @ w[pre + "down"].T


def capped(logits: torch.Tensor, scale: float, cap: float) -> torch.Tensor:
    return cap * torch.tanh(logits * scale / cap)


def owner(cfg: dict, i: int) -> int:
    j = cfg["layers"][i].get("weights_of")
    return i if j is None else owner(cfg, j)


def forward(cfg: dict, w: dict, tokens: list[int]) -> tuple[torch.Tensor, list[torch.Tensor]]:
    """Logits [T, vocab] of a whole sequence and the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    trail = []
    for i, lc in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."

        def sublayer(x, n, f):
            h = gain_norm(x, w[p + "norm" + n], eps)
            return x + gain_norm(f(h + causal_conv(h, w[p + "canon" + n])), w[p + "norm" + n + "b"], eps)

        x = sublayer(x, "1", lambda h: attention_mixer(h, w, p + "mix.", lc["mixer"], eps))
        if lc["mlp"] is not None:
            x = sublayer(x, "2", lambda h: dense_ff(h, w, p + "mlp.", eps))
        trail.append(x)
    assert math.isfinite(x.abs().max())
    return capped(gain_norm(x, w["final.norm"], eps) @ w["head"].T, cfg["logit_scale"], cfg["logit_softcap"]), trail
