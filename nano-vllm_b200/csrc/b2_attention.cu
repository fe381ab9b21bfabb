// Attention with a sliding window that keeps the first tokens, a soft cap on the scores and a learned sink in the
// softmax's denominator, over the paged KV cache.  Position i sees position j when j <= i and
// (i - j < window or j < keep_first); window = INT_MAX is full causal attention, softcap <= 0 and a null sink
// switch those parts off.
//
//   qk_norm_store_kernel   q/k head RMSNorm and the scatter of K and V into the cache
//   attn_any_kernel        any head size, bf16 or fp32, prefill and decode (one warp per query head)
#include <algorithm>
#include <climits>

#include "b2_vec.cuh"

namespace {

// ---------------------------------------------------------------------------
// q/k head RMSNorm (q in place, k into the cache) and V into the cache.  LANES lanes per (token, head), 8 elements
// per lane and pass.  Head strides are padded to 8 elements; the padding is zero and stays zero.
// ---------------------------------------------------------------------------
template <typename T, int LANES>
__global__ void __launch_bounds__(256) qk_norm_store_kernel(T* __restrict__ qkv, int64_t ld, int M, int nq, int nkv, int qk_dim, int qk_pad,
                                                            int v_pad, const T* __restrict__ qw, const T* __restrict__ kw, float eps,
                                                            T* __restrict__ k_cache, T* __restrict__ v_cache,
                                                            const int32_t* __restrict__ slots) {
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int heads = nq + 2 * nkv;
  const int64_t item = (blockIdx.x * static_cast<int64_t>(blockDim.x) + threadIdx.x) / LANES;
  const int lane = threadIdx.x & (LANES - 1);
  const bool live = item < static_cast<int64_t>(M) * heads;
  const int token = live ? static_cast<int>(item / heads) : 0;
  const int head = live ? static_cast<int>(item - static_cast<int64_t>(token) * heads) : 0;
  const bool is_q = head < nq, is_k = !is_q && head < nq + nkv;
  const int slot = (live && !is_q && k_cache != nullptr) ? slots[token] : -1;
  T* row = qkv + token * ld;
  if (live && !is_q && !is_k) {
    if (slot >= 0) {
      const T* src = row + static_cast<int64_t>(nq + nkv) * qk_pad + static_cast<int64_t>(head - nq - nkv) * v_pad;
      T* dst = v_cache + (static_cast<int64_t>(slot) * nkv + (head - nq - nkv)) * v_pad;
      for (int c = lane * 8; c < v_pad; c += LANES * 8) {
        float f[8];
        b2::load8<T>(src + c, f);
        b2::store8<T>(dst + c, f);
      }
    }
  }
  const bool norm = live && (is_q || is_k);
  T* src = row + static_cast<int64_t>(head) * qk_pad;
  float ss = 0.f;
  if (norm) {
    for (int c = lane * 8; c < qk_pad; c += LANES * 8) {
      float f[8];
      b2::load8<T>(src + c, f);
#pragma unroll
      for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
    }
  }
  ss = b2::group_sum<LANES>(ss);
  if (!norm) return;
  const T* w = is_q ? qw : kw;
  const float rstd = w != nullptr ? 1.0f / sqrtf(ss / static_cast<float>(qk_dim) + eps) : 1.0f;
  T* dst = is_q ? src : (slot >= 0 ? k_cache + (static_cast<int64_t>(slot) * nkv + (head - nq)) * qk_pad : nullptr);
  for (int c = lane * 8; c < qk_pad; c += LANES * 8) {
    float f[8], wf[8];
    b2::load8<T>(src + c, f);
    if (w != nullptr) {
      b2::load8<T>(w + c, wf);
#pragma unroll
      for (int e = 0; e < 8; ++e) f[e] = f[e] * rstd * wf[e];
    }
    if (is_k) b2::store8<T>(src + c, f);
    if (dst != nullptr) b2::store8<T>(dst + c, f);
  }
}

struct AttnArgs {
  const void* q;
  int64_t ldq;
  void* out;
  int64_t ldo;
  const void* k_cache;
  const void* v_cache;
  const int32_t* block_tables;
  int64_t bt_stride;
  int block_size;
  const int32_t* cu_q;    // [B + 1] first query row of every sequence; null = one row per sequence (decode)
  const int32_t* kv_len;  // [B] keys of every sequence, the step's own included
  int B, nq, nkv, qk_pad, v_pad;
  int window, keep_first;
  float scale, softcap;
  const float* sink;  // [nq] or null
};

__device__ __forceinline__ bool visible(int i, int j, int window, int keep_first) {
  return j <= i && (i - j < window || j < keep_first);
}

// ---------------------------------------------------------------------------
// One warp per (query row, head); a lane scores one key at a time, the warp folds 32 keys into the running maximum,
// sum and output.  VPL = outputs per lane.
// ---------------------------------------------------------------------------
template <typename T, int VPL>
__global__ void __launch_bounds__(128) attn_any_kernel(const AttnArgs a, int rows_per_seq_max) {
  extern __shared__ float q_smem[];  // [warps][qk_pad]
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int b = blockIdx.z, head = blockIdx.y;
  const int local = blockIdx.x * 4 + warp;
  const int row0 = a.cu_q ? a.cu_q[b] : b;
  const int n_q = a.cu_q ? a.cu_q[b + 1] - row0 : 1;
  if (local >= n_q) return;
  const int row = row0 + local;
  const int klen = a.kv_len[b];
  T* out = static_cast<T*>(a.out) + row * a.ldo + static_cast<int64_t>(head) * a.v_pad;
  const int pos = klen - n_q + local;
  if (pos < 0) {  // padded row of a decode graph
    for (int c = lane; c < a.v_pad; c += 32) out[c] = b2::from_float<T>(0.f);
    return;
  }
  const int g = head / (a.nq / a.nkv);
  float* qs = q_smem + warp * a.qk_pad;
  const T* q = static_cast<const T*>(a.q) + row * a.ldq + static_cast<int64_t>(head) * a.qk_pad;
  for (int c = lane; c < a.qk_pad; c += 32) qs[c] = b2::to_float(q[c]);
  __syncwarp();
  const int32_t* bt = a.block_tables + b * a.bt_stride;
  const T* kc = static_cast<const T*>(a.k_cache);
  const T* vc = static_cast<const T*>(a.v_cache);
  float m = -INFINITY, l = 0.f, acc[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) acc[i] = 0.f;
  const int win_lo = a.window > pos ? 0 : pos - a.window + 1;
  int j0 = 0;
  while (j0 <= pos) {
    if (j0 >= a.keep_first && j0 + 31 < win_lo) {  // between the kept tokens and the window
      j0 = win_lo & ~31;
      continue;
    }
    const int j = j0 + lane;
    float s = -INFINITY;
    int64_t krow = 0;
    if (visible(pos, j, a.window, a.keep_first)) {
      krow = (static_cast<int64_t>(bt[j / a.block_size]) * a.block_size + j % a.block_size) * a.nkv + g;
      const T* k = kc + krow * a.qk_pad;
      float d = 0.f;
      for (int c = 0; c < a.qk_pad; c += 8) {
        float f[8];
        b2::load8<T>(k + c, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) d = fmaf(f[e], qs[c + e], d);
      }
      s = d * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if (mx > -INFINITY) {
      const float m_new = fmaxf(m, mx);
      const float corr = expf(m - m_new);  // 0 at the first keys
      const float p = expf(s - m_new);
      l = l * corr + b2::group_sum(p);
#pragma unroll
      for (int i = 0; i < VPL; ++i) acc[i] *= corr;
      for (int t = 0; t < 32; ++t) {
        const float pt = __shfl_sync(0xffffffffu, p, t);
        const int64_t vrow = __shfl_sync(0xffffffffu, krow, t);
        if (pt == 0.f) continue;  // the same in every lane
        const T* v = vc + vrow * a.v_pad;
#pragma unroll
        for (int i = 0; i < VPL; ++i)
          if (lane + 32 * i < a.v_pad) acc[i] = fmaf(pt, b2::to_float(v[lane + 32 * i]), acc[i]);
      }
      m = m_new;
    }
    j0 += 32;
  }
  if (a.sink != nullptr) {
    const float sk = a.sink[head];
    const float m_new = fmaxf(m, sk);
    const float corr = expf(m - m_new);
    l = l * corr + expf(sk - m_new);
#pragma unroll
    for (int i = 0; i < VPL; ++i) acc[i] *= corr;
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int i = 0; i < VPL; ++i)
    if (lane + 32 * i < a.v_pad) out[lane + 32 * i] = b2::from_float<T>(acc[i] * inv);
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
int launch_any(const AttnArgs& a, int max_q, cudaStream_t s) {
  const size_t smem = 4 * sizeof(float) * a.qk_pad;
  const dim3 grid((max_q + 3) / 4, a.nq, a.B);
  const int vpl = (a.v_pad + 31) / 32;
  if (vpl <= 2) B2_CUDA(b2_launch(attn_any_kernel<T, 2>, grid, dim3(128), smem, s, a, max_q));
  else if (vpl <= 4) B2_CUDA(b2_launch(attn_any_kernel<T, 4>, grid, dim3(128), smem, s, a, max_q));
  else if (vpl <= 8) B2_CUDA(b2_launch(attn_any_kernel<T, 8>, grid, dim3(128), smem, s, a, max_q));
  else B2_CUDA(b2_launch(attn_any_kernel<T, 32>, grid, dim3(128), smem, s, a, max_q));
  return B2_OK;
}

template <typename T>
int launch_store(T* qkv, int64_t ld, int M, int nq, int nkv, int qk_dim, int qk_pad, int v_pad, const T* qw, const T* kw, float eps, T* kc,
                 T* vc, const int32_t* slots, cudaStream_t s) {
  const int vecs = std::max(qk_pad, v_pad) / 8;
  const int lanes = vecs <= 4 ? 4 : vecs <= 8 ? 8 : vecs <= 16 ? 16 : 32;
  const int64_t threads = static_cast<int64_t>(M) * (nq + 2 * nkv) * lanes;
  const dim3 grid(static_cast<unsigned>((threads + 255) / 256));
#define B2_STORE(L) B2_CUDA(b2_launch(qk_norm_store_kernel<T, L>, grid, dim3(256), 0, s, qkv, ld, M, nq, nkv, qk_dim, qk_pad, v_pad, qw, kw, eps, kc, vc, slots))
  switch (lanes) {
    case 4: B2_STORE(4); break;
    case 8: B2_STORE(8); break;
    case 16: B2_STORE(16); break;
    default: B2_STORE(32); break;
  }
#undef B2_STORE
  return B2_OK;
}

}  // namespace

extern "C" {

int b2_qk_norm_store(int dtype, void* qkv, int64_t ld_qkv, int M, int nq, int nkv, int qk_dim, int qk_pad, int v_dim, int v_pad,
                     const void* q_norm_w, const void* k_norm_w, float eps, void* k_cache, void* v_cache, const int32_t* slot_mapping,
                     void* stream) {
  if (M < 0 || nq <= 0 || nkv <= 0 || qk_dim <= 0 || v_dim <= 0 || qk_pad < qk_dim || v_pad < v_dim || qk_pad % 8 != 0 || v_pad % 8 != 0) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!qkv || !aligned16(qkv) || ld_qkv % 8 != 0 || ld_qkv < static_cast<int64_t>(nq + nkv) * qk_pad + static_cast<int64_t>(nkv) * v_pad) return B2_ERR_ARG;
  if ((q_norm_w == nullptr) != (k_norm_w == nullptr) || (q_norm_w && (!aligned16(q_norm_w) || !aligned16(k_norm_w)))) return B2_ERR_ARG;
  if (k_cache != nullptr && (!v_cache || !slot_mapping || !aligned16(k_cache) || !aligned16(v_cache))) return B2_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_BF16)
    return launch_store<uint16_t>(static_cast<uint16_t*>(qkv), ld_qkv, M, nq, nkv, qk_dim, qk_pad, v_pad, static_cast<const uint16_t*>(q_norm_w),
                                  static_cast<const uint16_t*>(k_norm_w), eps, static_cast<uint16_t*>(k_cache), static_cast<uint16_t*>(v_cache),
                                  slot_mapping, s);
  return launch_store<float>(static_cast<float*>(qkv), ld_qkv, M, nq, nkv, qk_dim, qk_pad, v_pad, static_cast<const float*>(q_norm_w),
                             static_cast<const float*>(k_norm_w), eps, static_cast<float*>(k_cache), static_cast<float*>(v_cache), slot_mapping, s);
}

int64_t b2_attention_workspace(int dtype, int B, int max_q, int max_kv, int nq, int nkv, int qk_pad, int v_pad, int window, int keep_first) {
  return 0;
}

int b2_attention(int dtype, const void* q, int64_t ldq, void* out, int64_t ldo, const void* k_cache, const void* v_cache,
                 const int32_t* block_tables, int64_t bt_stride, int block_size, const int32_t* cu_q, const int32_t* kv_len, int B, int max_q,
                 int max_kv, int nq, int nkv, int qk_pad, int v_pad, float scale, float softcap, int window, int keep_first, const float* sink,
                 void* workspace, int64_t workspace_bytes, int form, void* stream) {
  if (B < 0 || max_q < 0 || nq <= 0 || nkv <= 0 || nq % nkv != 0 || qk_pad <= 0 || v_pad <= 0 || qk_pad % 8 != 0 || v_pad % 8 != 0) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (window < 1 || keep_first < 0 || block_size < 1 || (cu_q == nullptr && max_q > 1)) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if (!q || !out || !k_cache || !v_cache || !block_tables || !kv_len) return B2_ERR_ARG;
  if (!aligned16(q) || !aligned16(out) || !aligned16(k_cache) || !aligned16(v_cache) || ldq % 8 != 0 || ldo % 8 != 0) return B2_ERR_ARG;
  if (qk_pad > 2048 || v_pad > 1024 || B > 65535) return B2_ERR_SHAPE;
  AttnArgs a{};
  a.q = q; a.ldq = ldq; a.out = out; a.ldo = ldo; a.k_cache = k_cache; a.v_cache = v_cache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.block_size = block_size; a.cu_q = cu_q; a.kv_len = kv_len;
  a.B = B; a.nq = nq; a.nkv = nkv; a.qk_pad = qk_pad; a.v_pad = v_pad; a.window = window; a.keep_first = keep_first;
  a.scale = scale; a.softcap = softcap; a.sink = sink;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_F32) return launch_any<float>(a, max_q, s);
  return launch_any<uint16_t>(a, max_q, s);
}

}  // extern "C"
