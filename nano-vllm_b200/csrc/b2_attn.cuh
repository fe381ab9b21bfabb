// Shared parts of the attention kernels: the argument block and the kernel that serves any head size.
#pragma once

#include <algorithm>
#include <climits>

#include "b2_mma.cuh"
#include "b2_vec.cuh"

namespace {

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
  int k_row, v_row;  // elements from one (slot, key/value head) to the next: qk_pad and v_pad, or a row that holds more
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
      const T* k = kc + krow * a.k_row;
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
        const T* v = vc + vrow * a.v_row;
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

constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
inline int launch_any(const AttnArgs& a, int max_q, cudaStream_t s) {
  const size_t smem = 4 * sizeof(float) * a.qk_pad;
  const dim3 grid((max_q + 3) / 4, a.nq, a.B);
  const int vpl = (a.v_pad + 31) / 32;
  if (vpl <= 2) B2_CUDA(b2_launch(attn_any_kernel<T, 2>, grid, dim3(128), smem, s, a, max_q));
  else if (vpl <= 4) B2_CUDA(b2_launch(attn_any_kernel<T, 4>, grid, dim3(128), smem, s, a, max_q));
  else if (vpl <= 8) B2_CUDA(b2_launch(attn_any_kernel<T, 8>, grid, dim3(128), smem, s, a, max_q));
  else B2_CUDA(b2_launch(attn_any_kernel<T, 32>, grid, dim3(128), smem, s, a, max_q));
  return B2_OK;
}

}  // namespace
