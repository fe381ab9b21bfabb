"""Tensor-level wrappers over the C ABI: they check dtypes and layouts, pick
the current CUDA stream, allocate outputs with torch and pass raw pointers."""
from __future__ import annotations

import ctypes as C

import torch

from . import _abi
from .runtime import get_runtime

_lib = _abi.lib


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


def _bf16_rows(t: torch.Tensor, what: str) -> torch.Tensor:
    if t.dtype != torch.bfloat16 or not t.is_cuda:
        raise TypeError(f"{what}: expected a CUDA bf16 tensor, got {t.dtype} on {t.device}")
    if t.stride(-1) != 1:
        t = t.contiguous()
    return t


def _as2d(t: torch.Tensor) -> torch.Tensor:
    if t.dim() == 2:
        return t
    return t.reshape(-1, t.shape[-1])


def _dt(t: torch.Tensor) -> int:
    """The library's element-type code of a tensor."""
    if t.dtype == torch.bfloat16:
        return _abi.DT_BF16
    if t.dtype == torch.float32:
        return _abi.DT_F32
    raise TypeError(f"expected bf16 or fp32, got {t.dtype}")


def _ptr(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


def _gemm_f32(x: torch.Tensor, w: torch.Tensor, pair_act: int = _abi.ACT_NONE, silu_cols: int = 0) -> torch.Tensor:
    """The fp32 form of gemm / gemm_act_mul: true 32-bit products."""
    x2 = _as2d(x)
    if x2.stride(-1) != 1 or x2.stride(0) % 4 or x2.data_ptr() % 16:
        x2 = x2.contiguous()
    M, K = x2.shape
    N = w.shape[0]
    if w.dtype != torch.float32 or w.shape[1] != K:
        raise ValueError(f"fp32 gemm: input has {K} features, weight is {tuple(w.shape)} {w.dtype}")
    out = torch.empty(M, N // 2 if pair_act else N, dtype=torch.float32, device=x.device)
    _abi.check(_lib.b2_gemm_f32(x2.data_ptr(), x2.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0), M, N, K, pair_act,
                                silu_cols, _stream()), "b2_gemm_f32")
    return out.view(*x.shape[:-1], out.shape[1])


def gemm(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None = None, silu_cols: int = 0) -> torch.Tensor:
    """x[..., K] @ w[N, K]^T (+ bias); the first silu_cols output features leave as silu(x)."""
    if x.dtype == torch.float32:
        assert bias is None
        return _gemm_f32(x, w, silu_cols=silu_cols)
    lead = x.shape[:-1]
    x2 = _as2d(_bf16_rows(x, "gemm input"))
    if x2.stride(0) % 8 != 0 or x2.data_ptr() % 16 != 0:
        x2 = x2.contiguous()
    w = _bf16_rows(w, "gemm weight")
    M, K = x2.shape
    N = w.shape[0]
    if w.dim() != 2 or w.shape[1] != K:
        raise ValueError(f"gemm: input has {K} features, weight is {tuple(w.shape)}")
    out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    if M and silu_cols:
        assert bias is None
        _abi.check(_lib.b2_gemm_silu_cols(get_runtime().ctx, x2.data_ptr(), x2.stride(0), w.data_ptr(), w.stride(0), out.data_ptr(), out.stride(0),
                                          M, N, K, silu_cols, _stream()), "b2_gemm_silu_cols")
    elif M:
        _abi.check(_lib.b2_gemm(get_runtime().ctx, x2.data_ptr(), x2.stride(0), w.data_ptr(), w.stride(0),
                                bias.data_ptr() if bias is not None else None, out.data_ptr(), out.stride(0), M, N, K, _stream()), "b2_gemm")
    return out.view(*lead, N)


def qkv_fused(x: torch.Tensor, w: torch.Tensor, bias, nq: int, nkv: int, head_dim: int, q_norm_w, k_norm_w, eps: float,
              positions: torch.Tensor | None, cos_sin: torch.Tensor | None, k_cache, v_cache, slot_mapping) -> torch.Tensor:
    """qkv projection + q/k head norm + RoPE + KV scatter; returns the [M, (nq + 2 nkv) head_dim] tensor with q and k
    already normalised and rotated (cos_sin None: not rotated)."""
    x2 = _as2d(_bf16_rows(x, "qkv input"))
    if x2.stride(0) % 8 != 0 or x2.data_ptr() % 16 != 0:
        x2 = x2.contiguous()
    M, K = x2.shape
    N = w.shape[0]
    assert N == (nq + 2 * nkv) * head_dim and w.shape[1] == K
    assert cos_sin is None or (positions.dtype == torch.int64 and cos_sin.dtype == torch.float32 and cos_sin.is_contiguous())
    have_cache = k_cache is not None and k_cache.numel() > 0
    if have_cache:
        assert k_cache.stride(1) == nkv * head_dim and slot_mapping.dtype == torch.int32
    out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    if M:
        _abi.check(_lib.b2_qkv_fused(get_runtime().ctx, x2.data_ptr(), x2.stride(0), w.data_ptr(), w.stride(0),
                                     bias.data_ptr() if bias is not None else None, out.data_ptr(), out.stride(0), M, nq, nkv, head_dim, K,
                                     q_norm_w.data_ptr() if q_norm_w is not None else None, k_norm_w.data_ptr() if k_norm_w is not None else None,
                                     float(eps), _ptr(positions), _ptr(cos_sin), k_cache.data_ptr() if have_cache else None,
                                     v_cache.data_ptr() if have_cache else None, slot_mapping.data_ptr() if have_cache else None, _stream()),
                   "b2_qkv_fused")
    return out


def gemm_silu_mul(x: torch.Tensor, w_pairs: torch.Tensor) -> torch.Tensor:
    """silu(x @ gate^T) * (x @ up^T) where w_pairs interleaves gate and up rows (gate_0, up_0, gate_1, ...)."""
    return gemm_act_mul(x, w_pairs, _abi.ACT_SILU)


def gemm_act_mul(x: torch.Tensor, w_pairs: torch.Tensor, act: int) -> torch.Tensor:
    """act(x @ gate^T) * (x @ up^T), act one of _abi.ACT_SILU / ACT_RELU."""
    if x.dtype == torch.float32:
        return _gemm_f32(x, w_pairs, pair_act=act)
    lead = x.shape[:-1]
    x2 = _as2d(_bf16_rows(x, "gemm_act_mul input"))
    if x2.stride(0) % 8 != 0 or x2.data_ptr() % 16 != 0:
        x2 = x2.contiguous()
    M, K = x2.shape
    I = w_pairs.shape[0] // 2
    if w_pairs.shape[1] != K or w_pairs.shape[0] % 2:
        raise ValueError(f"gemm_act_mul: input has {K} features, paired weight is {tuple(w_pairs.shape)}")
    out = torch.empty(M, I, dtype=torch.bfloat16, device=x.device)
    if M:
        _abi.check(_lib.b2_gemm_act_mul(get_runtime().ctx, x2.data_ptr(), x2.stride(0), w_pairs.data_ptr(), w_pairs.stride(0),
                                        out.data_ptr(), out.stride(0), M, I, K, act, _stream()), "b2_gemm_act_mul")
    return out.view(*lead, I)


def rowpar_form(M: int, N: int) -> int:
    """Which form of the fused row-parallel block serves M tokens of N features on this runtime
    (_abi.FORM_ONESHOT / FORM_OWNER: b2_rowpar_fused; FORM_TWOSHOT: b2_rowpar_fused_twoshot).  The library decides."""
    form = _lib.b2_rowpar_form(get_runtime().ctx, M, N)
    if form < 0:
        raise _abi.B2Error(f"b2_rowpar_form({M}, {N}): bad argument")
    return form


def rowpar_fused(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None, residual: torch.Tensor | None,
                 norm_w: torch.Tensor | None, eps: float):
    """Row-parallel GEMM + all-reduce (+ residual add + RMSNorm when norm_w is given).
    Returns y, or (normed, new_residual).

    For many tokens at tensor-parallel size >= 2 (rowpar_form(M, N) == FORM_TWOSHOT) the two-shot kernel runs:
    `normed` is then a view of a buffer owned by the runtime (valid until the next such call) and `new_residual`
    holds only the rows this rank owns (16-row blocks rank, rank + world, ...); the next fused call reads exactly
    those rows."""
    x2 = _as2d(_bf16_rows(x, "row-parallel input"))
    if x2.stride(0) % 8 != 0 or x2.data_ptr() % 16 != 0:
        x2 = x2.contiguous()
    M, Kr = x2.shape
    N = w.shape[0]
    rt = get_runtime()
    res_out = None
    if norm_w is not None:
        residual = _bf16_rows(residual, "residual")
        if not residual.is_contiguous():
            residual = residual.contiguous()
        res_out = torch.empty_like(residual)
    args_tail = (residual.data_ptr() if norm_w is not None else None, norm_w.data_ptr() if norm_w is not None else None, float(eps))
    if M and rowpar_form(M, N) == _abi.FORM_TWOSHOT:
        ptr = C.c_void_p()
        _abi.check(_lib.b2_rowpar_fused_twoshot(rt.ctx, x2.data_ptr(), x2.stride(0), w.data_ptr(), w.stride(0),
                                                bias.data_ptr() if bias is not None else None, M, N, Kr, *args_tail, C.byref(ptr),
                                                res_out.data_ptr() if res_out is not None else None, _stream()), "b2_rowpar_fused_twoshot")
        out = _library_view(ptr.value, (M, N), x.device)
        if norm_w is None:
            return out.clone().view(*x.shape[:-1], N)  # a plain forward hands out memory the caller may keep
        return out, res_out
    out = torch.empty(M, N, dtype=torch.bfloat16, device=x.device)
    if M:
        _abi.check(_lib.b2_rowpar_fused(rt.ctx, x2.data_ptr(), x2.stride(0), w.data_ptr(), w.stride(0),
                                        bias.data_ptr() if bias is not None else None, M, N, Kr, *args_tail, out.data_ptr(),
                                        res_out.data_ptr() if res_out is not None else None, _stream()), "b2_rowpar_fused")
    if norm_w is None:
        return out.view(*x.shape[:-1], N)
    return out, res_out


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    x = _bf16_rows(x, "rmsnorm input")
    dim = x.shape[-1]
    # rows with a common stride: [rows, dim] views (e.g. q heads inside the qkv output) are taken as they are
    if x.dim() == 2:
        x2 = x
    elif x.is_contiguous():
        x2 = x.view(-1, dim)
    else:
        x2 = x.contiguous().view(-1, dim)
    if x2.stride(0) % 8 != 0 or x2.data_ptr() % 16 != 0:
        x2 = x2.contiguous()
    out = torch.empty(x2.shape, dtype=torch.bfloat16, device=x.device)
    _abi.check(_lib.b2_rmsnorm(x2.data_ptr(), x2.stride(0), w.data_ptr(), float(eps), x2.shape[0], dim, out.data_ptr(), dim, _stream()), "b2_rmsnorm")
    return out.view(x.shape)


def add_rmsnorm(x: torch.Tensor, residual: torch.Tensor, w: torch.Tensor, eps: float):
    x = _bf16_rows(x, "add_rmsnorm input").contiguous()
    residual = _bf16_rows(residual, "residual").contiguous()
    dim = x.shape[-1]
    rows = x.numel() // dim
    out, res_out = torch.empty_like(x), torch.empty_like(x)
    _abi.check(_lib.b2_add_rmsnorm(x.data_ptr(), residual.data_ptr(), w.data_ptr(), float(eps), rows, dim, out.data_ptr(), res_out.data_ptr(), _stream()), "b2_add_rmsnorm")
    return out, res_out


def store_kvcache(key: torch.Tensor, value: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, slot_mapping: torch.Tensor) -> None:
    n, heads, hd = key.shape
    D = heads * hd
    # the reference's own preconditions (nanovllm/layers/attention.py:36-39)
    assert key.stride(-1) == 1 and value.stride(-1) == 1
    assert key.stride(1) == hd and value.stride(1) == hd
    assert k_cache.stride(1) == D and v_cache.stride(1) == D
    assert slot_mapping.numel() == n
    assert key.element_size() == 2 and k_cache.element_size() == 2 and slot_mapping.dtype == torch.int32
    _abi.check(_lib.b2_store_kvcache(key.data_ptr(), key.stride(0), value.data_ptr(), value.stride(0), k_cache.data_ptr(),
                                     v_cache.data_ptr(), slot_mapping.data_ptr(), n, D, _stream()), "b2_store_kvcache")


def silu_and_mul(x: torch.Tensor) -> torch.Tensor:
    x2 = _as2d(_bf16_rows(x, "silu_and_mul input"))
    M, two_i = x2.shape
    I = two_i // 2
    out = torch.empty(M, I, dtype=torch.bfloat16, device=x.device)
    _abi.check(_lib.b2_silu_and_mul(x2.data_ptr(), x2.stride(0), M, I, out.data_ptr(), _stream()), "b2_silu_and_mul")
    return out.view(*x.shape[:-1], I)


def qk_norm_rope_store(qkv: torch.Tensor, nq: int, nkv: int, head_dim: int, q_norm_w, k_norm_w, eps: float,
                       positions: torch.Tensor, cos_sin: torch.Tensor, k_cache, v_cache, slot_mapping) -> None:
    assert qkv.dim() == 2 and qkv.stride(1) == 1 and qkv.dtype == torch.bfloat16
    assert positions.dtype == torch.int64 and cos_sin.dtype == torch.float32 and cos_sin.is_contiguous()
    have_cache = k_cache is not None and k_cache.numel() > 0
    if have_cache:
        assert k_cache.stride(1) == nkv * head_dim and slot_mapping.dtype == torch.int32
    _abi.check(_lib.b2_qk_norm_rope_store(qkv.data_ptr(), qkv.stride(0), qkv.shape[0], nq, nkv, head_dim,
                                          q_norm_w.data_ptr() if q_norm_w is not None else None,
                                          k_norm_w.data_ptr() if k_norm_w is not None else None, float(eps),
                                          positions.data_ptr(), cos_sin.data_ptr(),
                                          k_cache.data_ptr() if have_cache else None, v_cache.data_ptr() if have_cache else None,
                                          slot_mapping.data_ptr() if have_cache else None, _stream()), "b2_qk_norm_rope_store")


def embed(ids: torch.Tensor, w: torch.Tensor, vocab_start: int, vocab_end: int, world: int) -> torch.Tensor:
    assert ids.dtype == torch.int64 and ids.is_cuda
    ids = ids.contiguous()
    M, H = ids.numel(), w.shape[1]
    out = torch.empty(M, H, dtype=w.dtype, device=w.device)
    ctx = get_runtime().ctx if world > 1 else None
    _abi.check(_lib.b2_embed(ctx, ids.data_ptr(), w.data_ptr(), vocab_start, vocab_end, M, H, out.data_ptr(), _stream()), "b2_embed")
    return out.view(*ids.shape, H)


class _DevicePtr:
    """Minimal __cuda_array_interface__ carrier so torch can view library-owned memory."""

    def __init__(self, ptr: int, shape: tuple[int, ...]):
        self.__cuda_array_interface__ = {"shape": shape, "typestr": "<u2", "data": (ptr, False), "version": 3, "strides": None}


_LOGIT_VIEWS: dict = {}


def _library_view(ptr: int, shape: tuple[int, int], device) -> torch.Tensor:
    """bf16 tensor over memory the library owns; built once per (address, shape), outside any graph capture."""
    key = (ptr, *shape)
    view = _LOGIT_VIEWS.get(key)
    if view is None:
        view = torch.as_tensor(_DevicePtr(ptr, shape), device=device).view(torch.bfloat16)
        _LOGIT_VIEWS[key] = view
    return view


def lm_head(h: torch.Tensor, w: torch.Tensor, row_index: torch.Tensor | None):
    """Returns the gathered [B, vocab] logits on rank 0 (a view of the runtime's
    buffer, valid until the next call) and None elsewhere."""
    rt = get_runtime()
    h2 = _as2d(_bf16_rows(h, "lm_head input"))
    if h2.stride(0) % 8 != 0 or h2.data_ptr() % 16 != 0:
        h2 = h2.contiguous()
    B = h2.shape[0] if row_index is None else row_index.numel()
    if row_index is not None:
        assert row_index.dtype == torch.int32 and row_index.is_cuda
    Vr, H = w.shape
    out = C.c_void_p()
    _abi.check(_lib.b2_lm_head(rt.ctx, h2.data_ptr(), h2.stride(0), row_index.data_ptr() if row_index is not None else None,
                               w.data_ptr(), w.stride(0), B, Vr, H, C.byref(out), _stream()), "b2_lm_head")
    if rt.rank != 0:
        return None
    vocab = Vr * rt.world
    key = (out.value, B, vocab)
    view = _LOGIT_VIEWS.get(key)
    if view is None:  # built once per shape (outside any graph capture: the first call of a shape is a warm-up)
        view = torch.as_tensor(_DevicePtr(out.value, (B, vocab)), device=h.device).view(torch.bfloat16)
        _LOGIT_VIEWS[key] = view
    return view


def lm_head_sample(h: torch.Tensor, w: torch.Tensor, row_index: torch.Tensor | None, temperatures: torch.Tensor | None,
                   seed: int, out: torch.Tensor | None = None, scale: float = 1.0, cap: float = 0.0) -> torch.Tensor:
    """LM head and sampler in one pass over the vocabulary shard (no logits in memory).  Returns int64 token ids
    [B], valid on rank 0 only.  temperatures: fp32 [B] on the device, or None for greedy decoding.  The sampled logits are
    cap tanh(scale logit / cap) (cap 0: scale logit)."""
    rt = get_runtime()
    h2 = _as2d(_bf16_rows(h, "lm_head input"))
    if h2.stride(0) % 8 != 0 or h2.data_ptr() % 16 != 0:
        h2 = h2.contiguous()
    B = h2.shape[0] if row_index is None else row_index.numel()
    if row_index is not None:
        assert row_index.dtype == torch.int32 and row_index.is_cuda
    if temperatures is not None:
        assert temperatures.dtype == torch.float32 and temperatures.is_cuda and temperatures.is_contiguous() and temperatures.numel() >= B
    if out is None:
        out = torch.empty(B, dtype=torch.int64, device=h.device)
    assert out.dtype == torch.int64 and out.is_cuda and out.numel() >= B
    Vr, H = w.shape
    _abi.check(_lib.b2_lm_head_sample_capped(rt.ctx, h2.data_ptr(), h2.stride(0), row_index.data_ptr() if row_index is not None else None,
                                             w.data_ptr(), w.stride(0), B, Vr, H, float(scale), float(cap),
                                             temperatures.data_ptr() if temperatures is not None else None,
                                             int(seed) & 0xFFFFFFFFFFFFFFFF, out.data_ptr(), _stream()), "b2_lm_head_sample")
    return out[:B]


def stream_step(x: torch.Tensor, y: torch.Tensor | None, mix, w_out, mult: float, w_in, norm_w: torch.Tensor, eps: float, dim: int,
                store: bool = True, embed: tuple | None = None, dtype: torch.dtype | None = None) -> torch.Tensor:
    """Everything between two sublayers on the fp32 residual streams x [M, S, D] (updated in place unless store is
    False): x <- mix^T x + mult w_out y, then RMSNorm(sum_s w_in[s] x_s) * norm_w, which is returned.  w_in None = all
    ones.  embed = (ids, table, scale) fills x from the embedding table instead of reading it."""
    M, S, D = x.shape
    assert x.dtype == torch.float32 and x.is_contiguous()
    if y is not None:
        assert y.shape == (M, D) and y.stride(1) == 1 and mix.dtype == torch.float32 and w_out.dtype == torch.float32
    assert norm_w.dtype == torch.float32 and norm_w.numel() == D and (w_in is None or w_in.dtype == torch.float32)
    ids, table, scale = embed if embed is not None else (None, None, 1.0)
    dtype = y.dtype if y is not None else table.dtype if table is not None else dtype
    normed = torch.empty(M, D, dtype=dtype, device=x.device)
    _abi.check(_lib.b2_stream_step(_dt(normed), x.data_ptr() if store else None, None if embed is not None else x.data_ptr(), _ptr(ids), _ptr(table),
                                   table.stride(0) if table is not None else 0, table.shape[0] if table is not None else 0, float(scale),
                                   _ptr(y), y.stride(0) if y is not None else 0, _ptr(mix) if y is not None else None,
                                   _ptr(w_out) if y is not None else None, float(mult), _ptr(w_in), norm_w.data_ptr(), float(eps),
                                   normed.data_ptr(), D, M, S, dim, D, _stream()), "b2_stream_step")
    return normed


def qk_norm_store(qkv: torch.Tensor, nq: int, nkv: int, qk_dim: int, qk_pad: int, v_dim: int, v_pad: int, q_norm_w, k_norm_w, eps: float,
                  k_cache, v_cache, slot_mapping) -> None:
    """q/k head RMSNorm (no rotation) in place on [q heads | k heads | v heads] rows and the scatter into the paged cache."""
    assert qkv.dim() == 2 and qkv.stride(1) == 1
    have_cache = k_cache is not None and k_cache.numel() > 0
    if have_cache:
        assert k_cache.dtype == qkv.dtype and k_cache.stride(1) == nkv * qk_pad and v_cache.stride(1) == nkv * v_pad and slot_mapping.dtype == torch.int32
    _abi.check(_lib.b2_qk_norm_store(_dt(qkv), qkv.data_ptr(), qkv.stride(0), qkv.shape[0], nq, nkv, qk_dim, qk_pad, v_dim, v_pad, _ptr(q_norm_w),
                                     _ptr(k_norm_w), float(eps), _ptr(k_cache) if have_cache else None, _ptr(v_cache) if have_cache else None,
                                     _ptr(slot_mapping) if have_cache else None, _stream()), "b2_qk_norm_store")


_WORKSPACES: dict = {}


def _workspace(kind: str, nbytes: int, device) -> torch.Tensor | None:
    """Scratch shared by the calls of one kind (stream-ordered); grows, never shrinks.  Starts as zeros.  A larger buffer
    replaces the old one, which stays alive because a captured graph may hold its address."""
    if nbytes <= 0:
        return None
    held = _WORKSPACES.setdefault((kind, device), [])
    if not held or held[-1].numel() < nbytes:
        held.append(torch.zeros(nbytes, dtype=torch.uint8, device=device))
    return held[-1]


def window_attention(q: torch.Tensor, out_heads: int, k_cache: torch.Tensor, v_cache: torch.Tensor, block_tables: torch.Tensor, cu_q, kv_len,
                     max_q: int, max_kv: int, scale: float, softcap: float, window: int, keep_first: int, sink, form: int = 0) -> torch.Tensor:
    """Attention of q [M, >= nq * qk_pad] over the paged cache [blocks, block_size, nkv, dim]; cu_q None = decode (one row
    per sequence).  Returns [M, nq * v_pad]."""
    nkv, qk_pad, v_pad = k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    M, B = q.shape[0], kv_len.numel() if cu_q is None else cu_q.numel() - 1
    assert q.stride(1) == 1 and q.dtype == k_cache.dtype and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert block_tables.dtype == torch.int32 and kv_len.dtype == torch.int32 and (sink is None or sink.dtype == torch.float32)
    out = torch.empty(M, out_heads * v_pad, dtype=q.dtype, device=q.device)
    max_kv = min(max_kv, block_tables.shape[1] * k_cache.shape[1])
    window = min(window, 2 ** 31 - 1)
    nbytes = _lib.b2_attention_workspace(_dt(q), B, max_q, max_kv, out_heads, nkv, qk_pad, v_pad, window, keep_first)
    ws = _workspace("attention", nbytes, q.device)
    _abi.check(_lib.b2_attention(_dt(q), q.data_ptr(), q.stride(0), out.data_ptr(), out.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                                 block_tables.data_ptr(), block_tables.stride(0), k_cache.shape[1], _ptr(cu_q), kv_len.data_ptr(), B, max_q, max_kv,
                                 out_heads, nkv, qk_pad, v_pad, float(scale), float(softcap), window, keep_first, _ptr(sink), _ptr(ws),
                                 ws.numel() if ws is not None else 0, form, _stream()), "b2_attention")
    return out


def linear_attn(qkv: torch.Tensor, heads: int, qk_pad: int, v_pad: int, state: torch.Tensor, slots: torch.Tensor, cu_q, kv_len: torch.Tensor,
                max_q: int, decay: torch.Tensor, decay_powers: torch.Tensor, form: int = 0) -> torch.Tensor:
    """Decayed linear attention on rows [q heads | k heads | v heads | ...]; returns o [M, heads * v_pad] in fp32 and leaves
    the new state in `state` [slots, heads, qk_pad, v_pad]."""
    assert qkv.dim() == 2 and qkv.stride(1) == 1 and qkv.shape[1] >= heads * (2 * qk_pad + v_pad)
    assert state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (heads, qk_pad, v_pad)
    assert slots.dtype == torch.int32 and kv_len.dtype == torch.int32
    assert decay.dtype == torch.float32 and decay_powers.shape == (heads, 65) and decay_powers.is_contiguous()
    M, B = qkv.shape[0], slots.numel()
    o = torch.empty(M, heads * v_pad, dtype=torch.float32, device=qkv.device)
    nbytes = _lib.b2_linear_attn_workspace(_dt(qkv), B, max_q, M, heads, qk_pad, v_pad) if cu_q is not None else 0
    ws = _workspace("linear_attn", nbytes, qkv.device)
    _abi.check(_lib.b2_linear_attn(_dt(qkv), qkv.data_ptr(), qkv.stride(0), o.data_ptr(), o.stride(0), state.data_ptr(), slots.data_ptr(), _ptr(cu_q),
                                   kv_len.data_ptr(), decay.data_ptr(), decay_powers.data_ptr(), B, max_q, M, heads, qk_pad, v_pad, _ptr(ws),
                                   ws.numel() if ws is not None else 0, form, _stream()), "b2_linear_attn")
    return o


def gated_norm(o: torch.Tensor, gate: torch.Tensor, w: torch.Tensor, eps: float, dim: int) -> torch.Tensor:
    """o / rms(o) * w * sigmoid(gate) per row, in the gate's dtype; o and w fp32, the mean over `dim` elements."""
    M, pad = o.shape
    assert o.dtype == torch.float32 and w.dtype == torch.float32 and gate.shape == (M, pad) and gate.stride(1) == 1
    out = torch.empty(M, pad, dtype=gate.dtype, device=o.device)
    _abi.check(_lib.b2_gated_norm(_dt(gate), o.data_ptr(), o.stride(0), gate.data_ptr(), gate.stride(0), w.data_ptr(), float(eps), M, dim, pad,
                                  out.data_ptr(), out.stride(0), _stream()), "b2_gated_norm")
    return out


def sandwich_step(x: torch.Tensor | None, y: torch.Tensor | None, post_w, norm_w: torch.Tensor, eps: float, dim: int, batch, conv_w=None, state=None,
                  store: bool = True, embed: tuple | None = None, run: int = 0) -> tuple[torch.Tensor | None, torch.Tensor]:
    """Everything between two sublayers: x <- x + post_w y / rms(y) (fp32 x [M, D]; embed = (ids, table): x = table[ids]),
    h = norm_w x / rms(x), out = h + causal convolution of h.  batch = (cu_q or None, kv_len, state slots, max_q).  Returns
    (new x or None when store is False, out)."""
    if embed is not None:
        ids, table = embed
        M, D, dtype, dev = ids.numel(), table.shape[1], table.dtype, table.device
    else:
        ids = table = None
        (M, D), dtype, dev = x.shape, y.dtype, x.device
        assert x.dtype == torch.float32 and x.is_contiguous() and y.shape == (M, D) and y.stride(1) == 1
        assert post_w.dtype == torch.float32 and post_w.numel() in (1, D)
    assert norm_w.dtype == torch.float32 and norm_w.numel() in (1, D)
    cu_q, kv_len, slots, max_q = batch
    taps = 0
    if conv_w is not None:
        taps = conv_w.shape[0]
        assert conv_w.shape == (taps, D) and conv_w.is_contiguous() and conv_w.dtype == dtype and state.dtype == dtype and state.is_contiguous()
        assert state.shape[1:] == (taps - 1, D) and slots.dtype == torch.int32 and kv_len.dtype == torch.int32
        B = kv_len.numel() if cu_q is None else cu_q.numel() - 1
    else:  # no neighbours: every row is on its own
        cu_q, B, max_q = None, M, 1
    x_out = torch.empty(M, D, dtype=torch.float32, device=dev) if store else None
    out = torch.empty(M, D, dtype=dtype, device=dev)
    _abi.check(_lib.b2_sandwich_step(_dt(out), _ptr(x) if embed is None else None, _ptr(x_out), _ptr(ids), _ptr(table),
                                     table.stride(0) if table is not None else 0, table.shape[0] if table is not None else 0, _ptr(y),
                                     y.stride(0) if y is not None else 0, _ptr(post_w), post_w.numel() if post_w is not None else 0, norm_w.data_ptr(),
                                     norm_w.numel(), float(eps), _ptr(conv_w), taps, _ptr(state), _ptr(slots), _ptr(cu_q), _ptr(kv_len), B, max_q,
                                     out.data_ptr(), D, dim, D, run, _stream()), "b2_sandwich_step")
    return x_out, out


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float, dim: int) -> torch.Tensor:
    """a N(z) + b N(z^2) + c N(z^3) + e with coef = (a, b, c, e) in fp32; N divides a row by its root mean square."""
    M, D = z.shape
    assert z.stride(1) == 1 and coef.dtype == torch.float32 and coef.numel() == 4
    out = torch.empty(M, D, dtype=z.dtype, device=z.device)
    _abi.check(_lib.b2_poly_norm(_dt(z), z.data_ptr(), z.stride(0), coef.data_ptr(), float(eps), M, dim, D, out.data_ptr(), D, _stream()), "b2_poly_norm")
    return out


def logit_cap(x: torch.Tensor, scale: float, cap: float) -> torch.Tensor:
    """fp32 cap tanh(scale x / cap); cap 0: scale x."""
    M, V = x.shape
    assert x.stride(1) == 1
    out = torch.empty(M, V, dtype=torch.float32, device=x.device)
    _abi.check(_lib.b2_logit_cap(_dt(x), x.data_ptr(), x.stride(0), float(scale), float(cap), M, V, out.data_ptr(), V, _stream()), "b2_logit_cap")
    return out


def latent_store(rows: torch.Tensor, q_dim: int, q_pad: int, kv_dim: int, kv_pad: int, rot_pad: int, q_norm, kv_norm, eps: float, positions: torch.Tensor,
                 cos_sin: torch.Tensor, cache, slot_mapping) -> None:
    """In place on rows [query latent | latent | rotated part | ...]: norms and rotation; the last two also to the cache."""
    assert rows.dim() == 2 and rows.stride(1) == 1 and positions.dtype == torch.int64
    assert cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and cos_sin.shape[1:] == (rot_pad // 2, 2)
    have = cache is not None and cache.numel() > 0
    if have:
        assert cache.dtype == rows.dtype and cache.is_contiguous() and cache.shape[-1] == kv_pad + rot_pad and slot_mapping.dtype == torch.int32
    _abi.check(_lib.b2_latent_store(_dt(rows), rows.data_ptr(), rows.stride(0), rows.shape[0], q_dim, q_pad, kv_dim, kv_pad, rot_pad, _ptr(q_norm),
                                    kv_norm.data_ptr(), float(eps), positions.data_ptr(), cos_sin.data_ptr(), cos_sin.shape[0],
                                    _ptr(cache) if have else None, _ptr(slot_mapping) if have else None, _stream()), "b2_latent_store")


def latent_gather(cache: torch.Tensor, block_tables: torch.Tensor, cu_k: torch.Tensor, max_kv: int, total: int) -> torch.Tensor:
    """The cached rows of every sequence, contiguous [total, row]; cache [blocks, block_size, 1, row]."""
    row = cache.shape[-1]
    assert cache.is_contiguous() and block_tables.dtype == torch.int32 and cu_k.dtype == torch.int32
    out = torch.empty(total, row, dtype=cache.dtype, device=cache.device)
    _abi.check(_lib.b2_latent_gather(_dt(cache), cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), cache.shape[1], cu_k.data_ptr(),
                                     cu_k.numel() - 1, max_kv, row, out.data_ptr(), _stream()), "b2_latent_gather")
    return out


def heads_gemm(x: torch.Tensor, x_head: int, w: torch.Tensor, kn: bool, out_head: int, gate: torch.Tensor | None = None, gate_head: int = 0,
               rotate: tuple | None = None) -> torch.Tensor:
    """One product per head: w [heads, N, K] (kn: [heads, K, N]; may be a view); x [M, heads * x_head], returns
    [M, heads * out_head].  rotate = (rot_pad, positions, cos_sin): the elements behind a head's K inputs, rotated, go behind
    its N outputs."""
    heads, N, K = w.shape[0], w.shape[2 if kn else 1], w.shape[1 if kn else 2]
    M = x.shape[0]
    rot_pad, positions, cos_sin = rotate if rotate is not None else (0, None, None)
    assert x.stride(1) == 1 and x.dtype == w.dtype and w.stride(2) == 1 and x.shape[1] >= heads * x_head
    assert gate is None or (gate.dtype == x.dtype and gate.stride(1) == 1 and gate.shape[0] == M)
    out = torch.empty(M, heads * out_head, dtype=x.dtype, device=x.device)
    _abi.check(_lib.b2_heads_gemm(_dt(x), x.data_ptr(), x.stride(0), x_head, w.data_ptr(), w.stride(1), w.stride(0), int(kn), out.data_ptr(), out.stride(0),
                                  out_head, M, heads, N, K, _ptr(gate), gate.stride(0) if gate is not None else 0, gate_head, rot_pad, _ptr(positions),
                                  _ptr(cos_sin), cos_sin.shape[0] if cos_sin is not None else 0, _stream()), "b2_heads_gemm")
    return out


def latent_attention(q: torch.Tensor, heads: int, cache: torch.Tensor, lat_pad: int, block_tables: torch.Tensor, cu_q, kv_len: torch.Tensor, max_q: int,
                     max_kv: int, scale: float, sink, form: int = 0) -> torch.Tensor:
    """Absorbed attention of q [M, heads * row] over cached rows [blocks, block_size, 1, row]; cu_q None = decode.  Returns the
    mixed latents [M, heads * lat_pad]."""
    row, block = cache.shape[-1], cache.shape[1]
    M, B = q.shape[0], kv_len.numel() if cu_q is None else cu_q.numel() - 1
    assert q.is_contiguous() and q.shape[1] == heads * row and q.dtype == cache.dtype and cache.is_contiguous()
    assert block_tables.dtype == torch.int32 and kv_len.dtype == torch.int32 and (sink is None or sink.dtype == torch.float32)
    out = torch.empty(M, heads * lat_pad, dtype=q.dtype, device=q.device)
    max_kv = min(max_kv, block_tables.shape[1] * block)
    nbytes = _lib.b2_latent_attention_workspace(_dt(q), B, max_q, max_kv, block, heads, lat_pad, row - lat_pad)
    ws = _workspace("latent_attention", nbytes, q.device)
    _abi.check(_lib.b2_latent_attention(get_runtime().ctx, _dt(q), q.data_ptr(), M, out.data_ptr(), out.stride(0), cache.data_ptr(),
                                        cache.shape[0] * block, block_tables.data_ptr(), block_tables.stride(0), block, _ptr(cu_q), kv_len.data_ptr(), B,
                                        max_q, max_kv, heads, lat_pad, row - lat_pad, float(scale), _ptr(sink), _ptr(ws),
                                        ws.numel() if ws is not None else 0, form, _stream()), "b2_latent_attention")
    return out


def expanded_attention(q: torch.Tensor, heads: int, kv: torch.Tensor, rot: torch.Tensor, cu_q: torch.Tensor, cu_k: torch.Tensor, max_q: int, dim_pad: int,
                       rot_pad: int, v_pad: int, scale: float, sink, cos_sin: torch.Tensor, gate: torch.Tensor | None) -> torch.Tensor:
    """Attention of the unrotated q [M, heads * (dim_pad + rot_pad)] over contiguous rows kv [keys, heads * (dim_pad + v_pad)]
    and rot [keys, rot_pad]; the output is multiplied by sigmoid(gate)."""
    M = q.shape[0]
    assert q.dtype == kv.dtype == rot.dtype == torch.bfloat16 and q.stride(1) == kv.stride(1) == rot.stride(1) == 1 and rot.shape[0] == kv.shape[0]
    assert cu_q.dtype == cu_k.dtype == torch.int32 and cos_sin.is_contiguous() and (sink is None or sink.dtype == torch.float32)
    assert gate is None or (gate.dtype == q.dtype and gate.stride(1) == 1)
    out = torch.empty(M, heads * v_pad, dtype=q.dtype, device=q.device)
    _abi.check(_lib.b2_expanded_attention(get_runtime().ctx, q.data_ptr(), q.stride(0), M, out.data_ptr(), out.stride(0), kv.data_ptr(), kv.stride(0),
                                          rot.data_ptr(), rot.stride(0), kv.shape[0], cu_q.data_ptr(), cu_k.data_ptr(), cu_q.numel() - 1, max_q, heads,
                                          dim_pad, rot_pad, v_pad, float(scale), _ptr(sink), cos_sin.data_ptr(), cos_sin.shape[0], _ptr(gate),
                                          gate.stride(0) if gate is not None else 0, _stream()), "b2_expanded_attention")
    return out


def argmax(logits: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    assert logits.dim() == 2 and logits.dtype == torch.bfloat16 and logits.stride(1) == 1
    if out is None:
        out = torch.empty(logits.shape[0], dtype=torch.int64, device=logits.device)
    assert out.dtype == torch.int64 and out.numel() >= logits.shape[0]
    _abi.check(_lib.b2_argmax(logits.data_ptr(), logits.stride(0), logits.shape[0], logits.shape[1], out.data_ptr(), _stream()), "b2_argmax")
    return out


def broadcast_tokens(buf: torch.Tensor) -> torch.Tensor:
    """Rank 0's int64 token ids into `buf` on every rank (in place)."""
    assert buf.dtype == torch.int64 and buf.is_cuda and buf.is_contiguous()
    _abi.check(_lib.b2_broadcast_tokens(get_runtime().ctx, buf.data_ptr(), buf.numel(), _stream()), "b2_broadcast_tokens")
    return buf


def advance_decode(tokens, input_ids, positions, context_lens, slot_mapping, block_tables, block_size: int, num_slots: int) -> None:
    """Device-side equivalent of building the next decode step's inputs.  num_slots = slots of the KV cache
    (blocks * block_size): a row whose next position has no block, or whose slot would lie outside the cache, is
    frozen (slot -1, position and length unchanged) instead of being sent outside the cache."""
    n = tokens.numel()
    assert tokens.dtype == torch.int64 and positions.dtype == torch.int64 and block_tables.dtype == torch.int32
    assert block_tables.dim() == 2 and block_tables.stride(1) == 1 and block_tables.shape[0] >= n
    _abi.check(_lib.b2_advance_decode(tokens.data_ptr(), input_ids.data_ptr(), positions.data_ptr(), context_lens.data_ptr(),
                                      slot_mapping.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), block_tables.shape[1],
                                      block_size, num_slots, n, _stream()), "b2_advance_decode")
