"""Plain, slow restatement of the Vekerax decoder on the CPU (test infrastructure only).

One function per mechanism, token by token where the mechanism is sequential; it shares no code with the
product path.  Everything runs in the dtype of the weights it is given (the tests use float64).

A model is (config dict, weights dict); the weights are plain tensors under the checkpoint's names.
"""
from __future__ import annotations

import math

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms(x, eps) * w


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def embedding(tokens: list[int], table: torch.Tensor, scale: float) -> torch.Tensor:
    return table[torch.tensor(tokens)] * scale


def window_allowed(i: int, j: int, size: int, keep_first: int) -> bool:
    """Does position i see position j: causal, and recent enough or among the kept first tokens."""
    return j <= i and (i - j < size or j < keep_first)


def softcap(score: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(score / cap)


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Weights exp(s_j) / (exp(sink) + sum_j exp(s_j)) over the last dimension."""
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention_core(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap: float, size: int, keep_first: int,
                   sink: torch.Tensor, first_pos: int = 0) -> torch.Tensor:
    """q [Tq, H, d] at positions first_pos .. first_pos + Tq - 1, k [Tk, G, d] and v [Tk, G, dv] at positions 0 .. Tk - 1."""
    tq, heads, _ = q.shape
    groups = k.shape[1]
    out = torch.zeros(tq, heads, v.shape[2], dtype=q.dtype)
    for t in range(tq):
        i = first_pos + t
        seen = torch.tensor([j for j in range(i + 1) if window_allowed(i, j, size, keep_first)])
        for h in range(heads):
            g = h // (heads // groups)
            s = softcap((k[seen, g] @ q[t, h]) * scale, cap)
            out[t, h] = sink_softmax(s, sink[h]) @ v[seen, g]
    return out


def attention_mixer(h: torch.Tensor, w: dict, pre: str, c: dict, eps: float) -> torch.Tensor:
    t = h.shape[0]
    q = (h @ w[pre + "q"].T).view(t, c["heads"], c["dim"])
    k = (h @ w[pre + "k"].T).view(t, c["kv_heads"], c["dim"])
    v = (h @ w[pre + "v"].T).view(t, c["kv_heads"], c["vdim"])
    q, k = rms_norm(q, w[pre + "q.norm"], eps), rms_norm(k, w[pre + "k.norm"], eps)
    o = attention_core(q, k, v, c["scale"], c["softcap"], c["mask"]["size"], c["mask"]["keep_first"], w[pre + "sink"])
    return o.reshape(t, -1) @ w[pre + "o"].T


def lightning_core(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: list[float], state: torch.Tensor | None = None):
    """S <- decay S + k v^T, o = S^T q, one token after the other; returns (o [T, H, dv], final state [H, d, dv])."""
    t, heads, d = q.shape
    s = torch.zeros(heads, d, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    dec = torch.tensor(decay, dtype=q.dtype).view(heads, 1, 1)
    o = torch.zeros(t, heads, v.shape[2], dtype=q.dtype)
    for i in range(t):
        s = dec * s + k[i].unsqueeze(2) * v[i].unsqueeze(1)
        o[i] = (s * q[i].unsqueeze(2)).sum(1)
    return o, s


def gated_norm(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_norm(o, w, eps) * torch.sigmoid(gate)


def lightning_mixer(h: torch.Tensor, w: dict, pre: str, c: dict, eps: float) -> torch.Tensor:
    t = h.shape[0]
    q = silu(h @ w[pre + "q"].T).view(t, c["heads"], c["dim"])
    k = silu(h @ w[pre + "k"].T).view(t, c["heads"], c["dim"])
    v = silu(h @ w[pre + "v"].T).view(t, c["heads"], c["vdim"])
    o, _ = lightning_core(q, k, v, c["decay"])
    return gated_norm(o.reshape(t, -1), h @ w[pre + "g"].T, w[pre + "norm"], eps) @ w[pre + "o"].T


def dense_ff(h: torch.Tensor, w: dict, pre: str) -> torch.Tensor:
    return (torch.relu(h @ w[pre + "gate"].T) * (h @ w[pre + "up"].T)) @ w[pre + "down"].T


def stream_input(x: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """x [T, S, D] -> sum_s in[s] x_s."""
    return torch.einsum("tsd,s->td", x, w_in)


def stream_update(x: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, w_out: torch.Tensor, m: float) -> torch.Tensor:
    """x_t <- sum_s mix[s, t] x_s + m out[t] y, all streams from the old ones."""
    return torch.einsum("nsd,st->ntd", x, mix) + m * w_out.view(1, -1, 1) * y.unsqueeze(1)


def layer_runs(cfg: dict) -> list[int]:
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


MIXERS = {"attention": attention_mixer, "lightning": lightning_mixer}


def forward(cfg: dict, w: dict, tokens: list[int]) -> tuple[torch.Tensor, list[torch.Tensor]]:
    """Logits [T, vocab] of a whole sequence and the residual stream (sum of the streams) after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embedding(tokens, w["embed"], cfg["embedding"]["scale"]).unsqueeze(1).repeat(1, cfg["streams"], 1)
    trail = []
    for i in layer_runs(cfg):
        lc, p = cfg["layers"][i], f"l{i}."
        y = MIXERS[lc["type"]](rms_norm(stream_input(x, w[p + "hc1.in"]), w[p + "norm1"], eps), w, p + "mix.", lc["mixer"], eps)
        x = stream_update(x, y, w[p + "hc1.mix"], w[p + "hc1.out"], m)
        if lc["mlp"] is not None:
            y = dense_ff(rms_norm(stream_input(x, w[p + "hc2.in"]), w[p + "norm2"], eps), w, p + "mlp.")
            x = stream_update(x, y, w[p + "hc2.mix"], w[p + "hc2.out"], m)
        trail.append(x.sum(1))
    return rms_norm(x.sum(1), w["final.norm"], eps) @ w["embed"].T, trail
