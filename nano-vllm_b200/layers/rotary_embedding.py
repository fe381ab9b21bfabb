"""Rotary position embedding (nanovllm/layers/rotary_embedding.py:17-59).

The decoder layer does not call `forward`: its rotation runs inside the qkv
projection's epilogue (or the q/k-norm + RoPE + KV-scatter kernel) on the same
cos||sin table.  `forward(positions, query, key)` keeps the reference's class
usable on its own (:37-48): it runs that kernel with the head norm and the
KV scatter switched off.
"""
from __future__ import annotations

from functools import lru_cache

import torch
from torch import nn

from .. import ops


class RotaryEmbedding(nn.Module):

    def __init__(self, head_size: int, rotary_dim: int, max_position_embeddings: int, base: float) -> None:
        super().__init__()
        assert rotary_dim == head_size
        self.head_size = head_size
        exponents = torch.arange(0, rotary_dim, 2, dtype=torch.float, device="cpu") / rotary_dim
        inv_freq = 1.0 / (base ** exponents)
        angles = torch.outer(torch.arange(max_position_embeddings, dtype=torch.float, device="cpu"), inv_freq)
        table = torch.cat((angles.cos(), angles.sin()), dim=-1)  # [max_pos, head_size], fp32
        self.register_buffer("cos_sin_cache", table.to(torch.get_default_device() if hasattr(torch, "get_default_device") else "cpu"), persistent=False)

    def forward(self, positions: torch.Tensor, query: torch.Tensor, key: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
        """query [T, heads, head_size], key [T, kv_heads, head_size] (or flattened over the heads); returns rotated
        copies, fp32 arithmetic and one rounding to bf16, as the reference's apply_rotary_emb (:6-14)."""
        hd = self.head_size
        t = positions.numel()
        q2, k2 = query.reshape(t, -1), key.reshape(t, -1)
        nq, nkv = q2.shape[1] // hd, k2.shape[1] // hd
        # the kernel works in place on a [T, (nq + 2 nkv) hd] row (q heads, k heads, v heads): the v part stays unused
        buf = torch.empty(t, (nq + 2 * nkv) * hd, dtype=torch.bfloat16, device=query.device)
        buf[:, :nq * hd] = q2
        buf[:, nq * hd:(nq + nkv) * hd] = k2
        ops.qk_norm_rope_store(buf, nq, nkv, hd, None, None, 0.0, positions.reshape(-1).to(torch.int64), self.cos_sin_cache, None, None, None)
        return buf[:, :nq * hd].reshape(query.shape), buf[:, nq * hd:(nq + nkv) * hd].reshape(key.shape)


@lru_cache(1)
def get_rope(head_size: int, rotary_dim: int, max_position: int, base: float) -> RotaryEmbedding:
    return RotaryEmbedding(head_size, rotary_dim, max_position, base)


class PairRotation:
    """Rotation of adjacent pairs: (u, v) = elements 2i and 2i + 1 of a part of `dim` elements turn by position * base^(-2i / dims),
    i < dims / 2; the other pairs stay as they are.  `table` fp32 [positions, pad8(dim) / 2, 2] holds (cos, sin), the angles
    taken in fp64; bind() builds it, shared by all rotations of the same kind on a device."""
    _tables: dict = {}

    def __init__(self, dim: int, dims: int, base: float) -> None:
        if dims % 2 or not 0 <= dims <= dim:
            raise ValueError(f"{dims} rotated of {dim} elements")
        self.dim, self.dims, self.base = dim, dims, float(base)
        self.pairs = (dim + 7) // 8 * 4
        self.table: torch.Tensor | None = None

    def bind(self, positions: int, device) -> None:
        key = (self.pairs, self.dims, self.base, positions, torch.device(device))
        if key not in self._tables:
            i = torch.arange(self.dims // 2, dtype=torch.float64, device="cpu")
            angles = torch.outer(torch.arange(positions, dtype=torch.float64, device="cpu"), self.base ** (-2.0 * i / max(self.dims, 1)))
            table = torch.zeros(positions, self.pairs, 2, dtype=torch.float32, device="cpu")
            table[..., 0] = 1.0
            table[:, :self.dims // 2, 0], table[:, :self.dims // 2, 1] = angles.cos().float(), angles.sin().float()
            self._tables[key] = table.to(device)
        self.table = self._tables[key]
