"""Multi-head latent attention: the paged cache holds one latent and one rotated key part per token, shared by all heads.

Decoding (and short portions of long sequences) attend to the cached latents themselves, with Wk folded into the query and Wv
applied to the mixed latents ("absorbed"); prompts expand the latents to per-head keys and values ("expanded").
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .linear import HeadsLinear, MergeHeadsLinear, pad8
from .rotary_embedding import PairRotation

EXPANDED_MAX_BYTES = 4 << 30  # of one layer's temporary keys and values


class PagedLatent:
    """One layer run's rows [latent | rotated key part] in the paged cache, bound by the runner; there is no separate V."""
    num_kv_heads = 1
    v_dim = 0

    def __init__(self, row: int):
        self.k_dim = row
        self.k_cache = self.v_cache = torch.tensor([])


def expansion_pays(tokens: int, keys: int, pairs: float, lat: int, rot: int, dim: int, vdim: int) -> bool:
    """Is it cheaper to expand `keys` latents and attend to keys and values than to attend to latents directly?  Per head, in
    multiply-adds; a plain matrix product runs several times faster than attention's."""
    gemm = 1.0 / 4
    expanded = keys * lat * (dim + vdim) * gemm + pairs * (dim + rot + vdim)
    absorbed = tokens * lat * (dim + vdim) + pairs * (2 * lat + rot)
    return expanded <= absorbed


class LatentAttention(nn.Module):
    """c_q = norm(Wdq h), q = Wuq c_q; [latent, rotated key part] = Wdkv h, the latent normed; k = [Wuk latent, rotated part],
    v = Wuv latent; softmax with a learned sink per head; heads gated by sigmoid(Wg h) before the output projection."""
    form = None  # None: chosen by cost; "absorbed" / "expanded" / "any" (tests)

    def __init__(self, hidden_size: int, num_heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int, scale: float, rot_dims: int,
                 rot_base: float, eps: float) -> None:
        super().__init__()
        self.num_heads, self.dim, self.rot_dim, self.vdim, self.q_rank, self.kv_rank = num_heads, dim, rot_dim, vdim, q_rank, kv_rank
        self.scale, self.eps = scale, eps
        self.dim_pad, self.rot_pad, self.v_pad, self.q_pad, self.lat_pad = map(pad8, (dim, rot_dim, vdim, q_rank, kv_rank))
        self.rotation = PairRotation(rot_dim, rot_dims, rot_base)
        # [query latent | latent | rotated key part | gate] in one product
        self.in_proj = HeadsLinear(hidden_size, [(1, q_rank), (1, kv_rank), (1, rot_dim), (num_heads, vdim)])
        self.q_proj = HeadsLinear(q_rank, [(num_heads, (dim, rot_dim))])
        self.kv_proj = HeadsLinear(kv_rank, [(num_heads, (dim, vdim))])
        self.o_proj = MergeHeadsLinear(num_heads, vdim, hidden_size)
        self.q_norm = nn.Parameter(torch.zeros(self.q_pad, dtype=torch.float32), requires_grad=False)
        self.kv_norm = nn.Parameter(torch.zeros(self.lat_pad, dtype=torch.float32), requires_grad=False)
        self.sink = nn.Parameter(torch.zeros(num_heads, dtype=torch.float32), requires_grad=False)

    def new_cache(self) -> PagedLatent:
        return PagedLatent(self.lat_pad + self.rot_pad)

    # ---- weights -----------------------------------------------------------
    def weight_shapes(self, width: int) -> dict[str, tuple[int, ...]]:
        h = self.num_heads
        return {"dq": (self.q_rank, width), "dq.norm": (self.q_rank,), "uq": (h * (self.dim + self.rot_dim), self.q_rank),
                "dkv": (self.kv_rank + self.rot_dim, width), "dkv.norm": (self.kv_rank,), "uk": (h * self.dim, self.kv_rank),
                "uv": (h * self.vdim, self.kv_rank), "sink": (h,), "g": (h * self.vdim, width), "o": (width, h * self.vdim)}

    def load_weight(self, name: str, w: torch.Tensor) -> None:
        w = w.to(self.sink.device)
        into = self.in_proj.weight_loader
        if name == "dq":
            into(self.in_proj.weight, w, 0)
        elif name == "dkv":
            into(self.in_proj.weight, w[:self.kv_rank], 1)
            into(self.in_proj.weight, w[self.kv_rank:], 2)
        elif name == "g":
            into(self.in_proj.weight, w, 3)
        elif name == "uq":
            self.q_proj.weight_loader(self.q_proj.weight, w, 0)
        elif name in ("uk", "uv"):  # the key and value rows of a head lie side by side
            at, n = (0, self.dim) if name == "uk" else (self.dim_pad, self.vdim)
            self._head_weights()[:, at:at + n, :self.kv_rank].copy_(w.view(self.num_heads, n, self.kv_rank))
        elif name == "o":
            self.o_proj.weight_loader(self.o_proj.weight, w)
        else:
            param = {"dq.norm": self.q_norm, "dkv.norm": self.kv_norm, "sink": self.sink}[name]
            param.data[:w.numel()].copy_(w)

    def _head_weights(self) -> torch.Tensor:
        """[heads, dim_pad key rows | v_pad value rows, latent]"""
        return self.kv_proj.weight.data.view(self.num_heads, self.dim_pad + self.v_pad, self.lat_pad)

    # ---- forward -----------------------------------------------------------
    def forward(self, x: torch.Tensor, positions: torch.Tensor, cache: PagedLatent) -> torch.Tensor:
        ctx = get_context()
        q0, l0, g0 = 0, self.q_pad, self.q_pad + self.lat_pad + self.rot_pad
        p = self.in_proj(x)
        ops.latent_store(p, self.q_rank, self.q_pad, self.kv_rank, self.lat_pad, self.rot_pad, self.q_norm, self.kv_norm, self.eps, positions,
                         self.rotation.table, cache.k_cache, ctx.slot_mapping)
        q, gate = self.q_proj(p[:, q0:l0]), p[:, g0:]
        attend = self._expanded if self._expands(x, ctx) else self._absorbed
        return self.o_proj(attend(q, p[:, l0:g0], gate, positions, cache, ctx))

    def _expands(self, x: torch.Tensor, ctx) -> bool:
        if not ctx.is_prefill or x.dtype != torch.bfloat16 or self.form in ("absorbed", "any"):
            return False
        if self.dim_pad > 128 or self.rot_pad > 64 or self.v_pad > 128 or self.scale <= 0:  # the kernel's tiles
            return False
        if self.form == "expanded":
            return True
        tokens, keys = x.shape[0], ctx.num_keys
        if 2 * keys * self.num_heads * (self.dim_pad + self.v_pad) > EXPANDED_MAX_BYTES:
            return False
        # (query, key) pairs: every token sees its sequence's earlier tokens and on average half of the step's own
        pairs = tokens * max(1.0, ctx.max_seqlen_k - ctx.max_seqlen_q / 2)
        return expansion_pays(tokens, keys, pairs, self.kv_rank, self.rot_dim, self.dim, self.vdim)

    def _expanded(self, q, rows, gate, positions, cache: PagedLatent, ctx) -> torch.Tensor:
        if ctx.num_keys != rows.shape[0]:  # earlier tokens' rows come from the cache
            rows = ops.latent_gather(cache.k_cache, ctx.block_tables, ctx.cu_seqlens_k, ctx.max_seqlen_k, ctx.num_keys)
        kv = self.kv_proj(rows[:, :self.lat_pad])
        return ops.expanded_attention(q, self.num_heads, kv, rows[:, self.lat_pad:], ctx.cu_seqlens_q, ctx.cu_seqlens_k, ctx.max_seqlen_q, self.dim_pad,
                                      self.rot_pad, self.v_pad, self.scale, self.sink, self.rotation.table, gate)

    def _absorbed(self, q, rows, gate, positions, cache: PagedLatent, ctx) -> torch.Tensor:
        w = self._head_weights()
        q = ops.heads_gemm(q, self.dim_pad + self.rot_pad, w[:, :self.dim_pad], True, self.lat_pad + self.rot_pad,
                           rotate=(self.rot_pad, positions, self.rotation.table))
        o = ops.latent_attention(q, self.num_heads, cache.k_cache, self.lat_pad, ctx.block_tables, ctx.cu_seqlens_q if ctx.is_prefill else None,
                                 ctx.context_lens, ctx.max_seqlen_q if ctx.is_prefill else 1, ctx.max_seqlen_k if ctx.is_prefill else 2 ** 31 - 1,
                                 self.scale, self.sink, form=1 if self.form == "any" else 0)
        return ops.heads_gemm(o, self.lat_pad, w[:, self.dim_pad:], False, self.v_pad, gate=gate, gate_head=self.v_pad)
