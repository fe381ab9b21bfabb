// Shared parts of the attention kernels: the argument block, the key tiles a range of positions looks at, scores and the
// running softmax on tensor-core fragments, and the kernel that serves any head size.
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

// ---------------------------------------------------------------------------
// Tensor-core kernels, bf16, head sizes up to 128.  The query heads that share a key/value head are rows of one tile
// (row = token * rep + head), so K and V are read once per group.  Scores, softmax and weights are fp32; the weights
// enter the product with V as a sum of two bf16 numbers.
// ---------------------------------------------------------------------------
constexpr int BN = 64;  // keys per tile

// The key tiles a range of positions [pmin, pmax] looks at: those of the kept first tokens, then those of the window.
struct KeyTiles {
  int n_first, win0, total;
  __device__ __forceinline__ KeyTiles(int pmin, int pmax, int window, int keep_first) {
    const int lo = pmin - window + 1;
    win0 = (lo > 0 ? lo : 0) / BN;
    const int kept = min(keep_first, pmax + 1);
    n_first = min((kept + BN - 1) / BN, win0);
    total = n_first + pmax / BN - win0 + 1;
  }
  __device__ __forceinline__ int at(int i) const { return i < n_first ? i : win0 + (i - n_first); }
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Scores in units of log2: t = log2(e) * softcap(scale * s).  The three forms of the cap:
enum { CAP_NONE = 0, CAP_SHORT = 1, CAP_FULL = 2 };
struct ScoreScale {
  float a, b, c;  // NONE: t = a s.  SHORT: t = c - b / (1 + 2^(a s)).  FULL: see score()
};
__host__ __device__ inline ScoreScale score_scale(int cap_form, float scale, float cap) {
  constexpr float L = 1.4426950408889634f;
  if (cap_form == CAP_NONE) return {scale * L, 0.f, 0.f};
  return {2.0f * L * scale / cap, 2.0f * cap * L, cap * L};
}
// tanh(x) = 1 - 2 / (1 + e^2x) has an absolute error of about 1e-7, so the capped score is off by 1e-7 cap: below fp32
// rounding of the scores themselves for caps up to a few hundred (SHORT).  FULL adds the Taylor series where the
// difference would cancel, for any cap.
template <int CAP>
__device__ __forceinline__ float score(float s, const ScoreScale& k) {
  if (CAP == CAP_NONE) return s * k.a;
  const float z = s * k.a;  // 2 log2(e) x
  const float t = fmaf(-k.b, __fdividef(1.0f, 1.0f + fast_exp2(fminf(z, 120.0f))), k.c);
  if (CAP == CAP_SHORT) return t;
  const float x = z * 0.34657359027997264f, x2 = x * x;
  const float series = k.c * x * fmaf(x2, fmaf(x2, 0.13333333333f, -0.33333333333f), 1.0f);
  return fabsf(x) < 0.125f ? series : t;
}

constexpr float LOG2E = 1.4426950408889634f;

// One tile's scores of a warp: NT 8-key column tiles starting at key j0.  Scales, caps, masks (when `masked`), folds
// into the running maximum m and sum l, and leaves the weights in s.  Returns the factors for the old outputs.
template <int NT, int CAP>
__device__ __forceinline__ void softmax_tile(const AttnArgs& a, const ScoreScale& k, float (&s)[NT][4], int j0, const int (&pos)[2], bool masked,
                                             float (&m)[2], float (&l)[2], float (&corr)[2], int lane) {
  float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) s[n][e] = score<CAP>(s[n][e], k);
  if (masked) {
#pragma unroll
    for (int n = 0; n < NT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (!visible(pos[e >> 1], j0 + n * 8 + (lane & 3) * 2 + (e & 1), a.window, a.keep_first)) s[n][e] = -INFINITY;
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) mx[e >> 1] = fmaxf(mx[e >> 1], s[n][e]);
  float base[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
    mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
    const float m_new = fmaxf(m[h], mx[h]);
    base[h] = m_new == -INFINITY ? 0.f : m_new;  // nothing visible yet: every weight is 2^-inf = 0
    corr[h] = fast_exp2(m[h] - base[h]);
    m[h] = m_new;
  }
  float sum[2] = {0.f, 0.f};
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float p = fast_exp2(s[n][e] - base[e >> 1]);
      s[n][e] = p;
      sum[e >> 1] += p;
    }
#pragma unroll
  for (int h = 0; h < 2; ++h) l[h] = fmaf(l[h], corr[h], sum[h]);  // this lane's part; summed over the row's four lanes at the end
}

template <int DQ, int DV>
struct CfgTile {
  static constexpr int STAGE = BN * (DQ + DV) * 2;
  static constexpr int SMEM_PREFILL = 64 * DQ * 2 + 2 * STAGE + 128;
  static constexpr int DEC_STAGES = 3;
  static constexpr int SMEM_DECODE = 16 * DQ * 2 + DEC_STAGES * STAGE + 128;
};

// The key loop of a prefill CTA: 64 rows (token, head of the group), 16 per warp; the four warps share the key tiles.  The
// query tile's copies have been issued (not committed); load(tile, sk, sv) issues the copies of one key tile; once() runs
// after the first copies have been issued.  Leaves the running maximum, this lane's part of the sum and the outputs.
template <int DQ, int DV, int CAP, typename Load, typename Once>
__device__ __forceinline__ void prefill_tiles(const AttnArgs& a, int first_pos, int tile0, int rows, int rep, const KeyTiles& tiles, uint32_t sq,
                                              uint32_t skv, Load&& load, Once&& once, float (&m)[2], float (&l)[2], float (&o)[DV / 8][4]) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const ScoreScale sscale = score_scale(CAP, a.scale, a.softcap);
  load(tiles.at(0), skv, skv + BN * DQ * 2);
  b2::cp_async_commit();
  once();
  int pos[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) pos[h] = first_pos + min(tile0 + warp * 16 + (lane >> 2) + h * 8, rows - 1) / rep;
  const int wpmin = first_pos + min(tile0 + warp * 16, rows - 1) / rep;
  const int wpmax = first_pos + min(tile0 + warp * 16 + 15, rows - 1) / rep;
  m[0] = m[1] = -INFINITY;
  l[0] = l[1] = 0.f;
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  for (int it = 0; it < tiles.total; ++it) {
    const uint32_t sk = skv + (it & 1) * CfgTile<DQ, DV>::STAGE, sv = sk + BN * DQ * 2;
    b2::cp_async_wait<0>();
    __syncthreads();  // this tile has landed for everyone, and everyone has left the stage that is filled next
    if (it + 1 < tiles.total) {
      const uint32_t nk = skv + ((it + 1) & 1) * CfgTile<DQ, DV>::STAGE;
      load(tiles.at(it + 1), nk, nk + BN * DQ * 2);
    }
    b2::cp_async_commit();
    const int j0 = tiles.at(it) * BN;
    float s[BN / 8][4];
#pragma unroll
    for (int n = 0; n < BN / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll
    for (int k = 0; k < DQ / 16; ++k) {
      uint32_t qa[4];
      b2::frag_a<DQ>(sq, warp * 16, k * 16, lane, qa);
#pragma unroll
      for (int n = 0; n < BN / 16; ++n) {
        uint32_t kb[4];
        b2::frag_b<DQ>(sk, n * 16, k * 16, lane, kb);
        b2::mma16816(s[2 * n], qa, kb[0], kb[1]);
        b2::mma16816(s[2 * n + 1], qa, kb[2], kb[3]);
      }
    }
    const bool all_seen = j0 + BN - 1 <= wpmin && (wpmax - j0 < a.window || j0 + BN - 1 < a.keep_first);
    float corr[2];
    softmax_tile<BN / 8, CAP>(a, sscale, s, j0, pos, !all_seen, m, l, corr, lane);
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
      o[n][0] *= corr[0]; o[n][1] *= corr[0]; o[n][2] *= corr[1]; o[n][3] *= corr[1];
    }
#pragma unroll
    for (int k = 0; k < BN / 16; ++k) {
      uint32_t hi[4], lo[4];
      b2::split_bf16(s[2 * k][0], s[2 * k][1], hi[0], lo[0]);
      b2::split_bf16(s[2 * k][2], s[2 * k][3], hi[1], lo[1]);
      b2::split_bf16(s[2 * k + 1][0], s[2 * k + 1][1], hi[2], lo[2]);
      b2::split_bf16(s[2 * k + 1][2], s[2 * k + 1][3], hi[3], lo[3]);
#pragma unroll
      for (int n = 0; n < DV / 16; ++n) {
        uint32_t vb[4];
        b2::frag_b_t<DV>(sv, n * 16, k * 16, lane, vb);
        b2::mma16816(o[2 * n], hi, vb[0], vb[1]);
        b2::mma16816(o[2 * n + 1], hi, vb[2], vb[3]);
        b2::mma16816(o[2 * n], lo, vb[0], vb[1]);
        b2::mma16816(o[2 * n + 1], lo, vb[2], vb[3]);
      }
    }
  }
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
