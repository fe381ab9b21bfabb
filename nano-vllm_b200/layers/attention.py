"""Paged-KV scatter on a hand-written CUDA kernel, and the attention call.

`store_kvcache` has the signature and preconditions of
nanovllm/layers/attention.py:33-40 (the Triton kernel at :10-30 is replaced by
b2_store_kvcache: 16-byte vector copies, several tokens per CTA, bit-exact).
`Attention` keeps the reference's interface (:43-75).  The attention
arithmetic itself stays a library call, as in the reference: flash-attn's
varlen kernel for prefill and its paged kv-cache kernel for decode.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .linear import HeadsLinear, MergeHeadsLinear, pad8

try:  # the attention library is outside this path; it is only called, never re-implemented
    from flash_attn import flash_attn_varlen_func, flash_attn_with_kvcache
except Exception:  # pragma: no cover
    flash_attn_varlen_func = flash_attn_with_kvcache = None


def store_kvcache(key: torch.Tensor, value: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, slot_mapping: torch.Tensor):
    ops.store_kvcache(key, value, k_cache, v_cache, slot_mapping)


def _sdpa_paged(q, k_cache, v_cache, context_lens, block_tables, scale, q_lens=None):
    """Plain-PyTorch attention over the paged cache: a slow stand-in for the
    library call, used for small shapes when flash-attn cannot run."""
    nh, hd = q.shape[-2], q.shape[-1]
    nkv = k_cache.shape[-2]
    bs = k_cache.shape[1]
    outs = []
    off = 0
    lens = context_lens.tolist()
    for i, n_ctx in enumerate(lens):
        tq = 1 if q_lens is None else q_lens[i]
        if n_ctx == 0:
            outs.append(torch.zeros(tq, nh, hd, dtype=q.dtype, device=q.device))
            off += tq
            continue
        nblk = (n_ctx + bs - 1) // bs
        blocks = block_tables[i, :nblk].long()
        k = k_cache[blocks].reshape(-1, nkv, hd)[:n_ctx]
        v = v_cache[blocks].reshape(-1, nkv, hd)[:n_ctx]
        qi = q[off:off + tq]
        mask = None
        if tq > 1:
            qpos = torch.arange(tq, device=q.device).unsqueeze(1) + (n_ctx - tq)
            mask = torch.arange(n_ctx, device=q.device).unsqueeze(0) <= qpos
        o = torch.nn.functional.scaled_dot_product_attention(qi.transpose(0, 1).unsqueeze(0), k.transpose(0, 1).unsqueeze(0),
                                                             v.transpose(0, 1).unsqueeze(0), attn_mask=mask, scale=scale, enable_gqa=True)
        outs.append(o.squeeze(0).transpose(0, 1))
        off += tq
    return torch.cat(outs)


class Attention(nn.Module):
    # "flash_attn" (the reference's library call) or "sdpa" (plain PyTorch, for tests on small shapes when flash-attn cannot run)
    backend = "flash_attn"

    def __init__(self, num_heads, head_dim, scale, num_kv_heads):
        super().__init__()
        self.num_heads, self.head_dim, self.scale, self.num_kv_heads = num_heads, head_dim, scale, num_kv_heads
        self.k_dim = self.v_dim = head_dim
        self.k_cache = self.v_cache = torch.tensor([])

    def attend(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
        """Attention over K/V that are already in the paged cache (decode, or
        prefill with a cached prefix) or passed in (plain prefill)."""
        ctx = get_context()
        k_cache, v_cache = self.k_cache, self.v_cache
        if Attention.backend == "sdpa":
            if ctx.is_prefill:
                cu_q, cu_k = ctx.cu_seqlens_q.tolist(), ctx.cu_seqlens_k.tolist()
                q_lens = [b - a for a, b in zip(cu_q[:-1], cu_q[1:])]
                k_lens = torch.tensor([b - a for a, b in zip(cu_k[:-1], cu_k[1:])])
                if ctx.block_tables is None:  # no cache bound (warm-up) or no prefix: attend over the passed K/V
                    outs = []
                    for i, (a, b) in enumerate(zip(cu_q[:-1], cu_q[1:])):
                        o = torch.nn.functional.scaled_dot_product_attention(
                            q[a:b].transpose(0, 1).unsqueeze(0), k[a:b].transpose(0, 1).unsqueeze(0), v[a:b].transpose(0, 1).unsqueeze(0),
                            is_causal=True, scale=self.scale, enable_gqa=True)
                        outs.append(o.squeeze(0).transpose(0, 1))
                    return torch.cat(outs)
                return _sdpa_paged(q, k_cache, v_cache, k_lens, ctx.block_tables, self.scale, q_lens)
            return _sdpa_paged(q, k_cache, v_cache, ctx.context_lens, ctx.block_tables, self.scale)
        if flash_attn_varlen_func is None:
            raise RuntimeError("flash-attn is not importable; set Attention.backend = 'sdpa' for small test shapes")
        if ctx.is_prefill:
            if ctx.block_tables is not None:  # prefix cache / chunked prefill: read K/V from the cache
                k, v = k_cache, v_cache
            return flash_attn_varlen_func(q, k, v, max_seqlen_q=ctx.max_seqlen_q, cu_seqlens_q=ctx.cu_seqlens_q,
                                          max_seqlen_k=ctx.max_seqlen_k, cu_seqlens_k=ctx.cu_seqlens_k,
                                          softmax_scale=self.scale, causal=True, block_table=ctx.block_tables)
        return flash_attn_with_kvcache(q.unsqueeze(1), k_cache, v_cache, cache_seqlens=ctx.context_lens,
                                       block_table=ctx.block_tables, softmax_scale=self.scale, causal=True).squeeze(1)

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor) -> torch.Tensor:
        """Reference behaviour: scatter this step's K/V into the cache (when one is bound), then attend."""
        if self.k_cache.numel() and self.v_cache.numel():
            store_kvcache(k, v, self.k_cache, self.v_cache, get_context().slot_mapping)
        return self.attend(q, k, v)


class PagedKV:
    """One layer run's K and V in the paged cache, bound by the runner; K and V heads may differ in size."""

    def __init__(self, num_kv_heads: int, k_dim: int, v_dim: int):
        self.num_kv_heads, self.k_dim, self.v_dim = num_kv_heads, k_dim, v_dim
        self.k_cache = self.v_cache = torch.tensor([])


class WindowAttention(nn.Module):
    """Grouped-query attention without rotation: q/k head norm, soft-capped scores, a sliding window that keeps the first
    tokens, a learned sink per head in the softmax's denominator.  Always reads K and V from the paged cache."""

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, dim: int, vdim: int, scale: float, softcap: float, window: int,
                 keep_first: int, eps: float) -> None:
        super().__init__()
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} query heads do not divide over {num_kv_heads} key/value heads")
        self.num_heads, self.num_kv_heads, self.dim, self.vdim = num_heads, num_kv_heads, dim, vdim
        self.qk_pad, self.v_pad = pad8(dim), pad8(vdim)
        self.scale, self.softcap, self.window, self.keep_first, self.eps = scale, softcap, window, keep_first, eps
        self.qkv_proj = HeadsLinear(hidden_size, [(num_heads, dim), (num_kv_heads, dim), (num_kv_heads, vdim)])
        self.o_proj = MergeHeadsLinear(num_heads, vdim, hidden_size)
        self.q_norm = nn.Parameter(torch.zeros(self.qk_pad), requires_grad=False)
        self.k_norm = nn.Parameter(torch.zeros(self.qk_pad), requires_grad=False)
        self.sink = nn.Parameter(torch.zeros(num_heads, dtype=torch.float32), requires_grad=False)
        for p in (self.q_norm, self.k_norm):
            p.weight_loader = self._load_norm

    def _load_norm(self, param: nn.Parameter, loaded_weight: torch.Tensor):
        param.data[:self.dim].copy_(loaded_weight)

    def forward(self, x: torch.Tensor, cache: PagedKV) -> torch.Tensor:
        ctx = get_context()
        if x.dtype == torch.bfloat16 and self.dim == self.vdim == 128:  # one launch for decode-sized batches
            qkv = ops.qkv_fused(x, self.qkv_proj.weight, None, self.num_heads, self.num_kv_heads, 128, self.q_norm, self.k_norm, self.eps,
                                None, None, cache.k_cache, cache.v_cache, ctx.slot_mapping)
        else:
            qkv = self.qkv_proj(x)
            ops.qk_norm_store(qkv, self.num_heads, self.num_kv_heads, self.dim, self.qk_pad, self.vdim, self.v_pad, self.q_norm, self.k_norm,
                              self.eps, cache.k_cache, cache.v_cache, ctx.slot_mapping)
        o = ops.window_attention(qkv, self.num_heads, cache.k_cache, cache.v_cache, ctx.block_tables, ctx.cu_seqlens_q if ctx.is_prefill else None,
                                 ctx.context_lens, ctx.max_seqlen_q if ctx.is_prefill else 1, ctx.max_seqlen_k if ctx.is_prefill else 2 ** 31 - 1,
                                 self.scale, self.softcap, self.window, self.keep_first, self.sink)
        return self.o_proj(o)
