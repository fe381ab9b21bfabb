// Latent attention: the cache holds one row [latent | rotated key part] per token, shared by all heads.  A head's key is
// [Wk latent | rotated key part] and its value Wv latent, so there are two ways to attend:
//   absorbed   the query is multiplied by Wk^T first and attends to the cached rows themselves; the output is a mixture of
//              latents that is multiplied by Wv afterwards.  Least memory traffic per query: decoding, short portions.
//   expanded   every token's keys and values are computed once and attended to as usual.  Least arithmetic per
//              (query, key) pair: prompts.
//
//   latent_store_kernel    RMSNorm of the query latent and of the cached latent, rotation of the key part, scatter
//   latent_gather_kernel   cached rows of a batch as contiguous rows (a portion whose sequence has earlier tokens)
//   heads_gemm_kernel      one small matrix product per head, with the rotation of the query part or an output gate
//   latent_attn_kernel     absorbed attention on the tensor cores: 16 or 32 (token, head) rows x 64 keys
//   expanded_attn_kernel   expanded attention, 64 tokens of one head x 64 keys; rotates the queries it loads, gates its output
#include <algorithm>

#include "b2_attn.cuh"

namespace {

using namespace b2;

// cos/sin of one rotated pair: table [max_pos][rot_pad / 2] of (cos, sin)
__device__ __forceinline__ float2 rot_at(const float2* cs, int max_pos, int half, int64_t pos, int pair) {
  const int64_t p = pos < 0 ? 0 : pos >= max_pos ? max_pos - 1 : pos;
  return __ldg(cs + p * half + pair);
}
// (u, v) -> (u cos - v sin, v cos + u sin) on the four pairs of 8 elements
__device__ __forceinline__ void rotate8(float (&f)[8], const float2* cs, int max_pos, int half, int64_t pos, int pair0) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 r = rot_at(cs, max_pos, half, pos, pair0 + i);
    const float u = f[2 * i], v = f[2 * i + 1];
    f[2 * i] = u * r.x - v * r.y;
    f[2 * i + 1] = v * r.x + u * r.y;
  }
}

// ---------------------------------------------------------------------------
// Rows [q latent | latent | rotated part | ...] in place; [latent | rotated part] also to the cache.  One warp per
// (token, part).
// ---------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void warp_rms(const T* src, int dim, int pad, const float* w, float eps, int lane, T* dst0, T* dst1) {
  float ss = 0.f;
  for (int c = lane * 8; c < pad; c += 256) {
    float f[8];
    load8<T>(src + c, f);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
  }
  ss = group_sum(ss);
  const float rstd = 1.0f / sqrtf(ss / static_cast<float>(dim) + eps);
  for (int c = lane * 8; c < pad; c += 256) {
    float f[8], g[8];
    load8<T>(src + c, f);
    load8<float>(w + c, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = f[e] * rstd * g[e];
    store8<T>(dst0 + c, f);
    if (dst1 != nullptr) store8<T>(dst1 + c, f);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_store_kernel(T* p, int64_t ld, int M, int q_dim, int q_pad, int kv_dim, int kv_pad, int rot_pad,
                                                           const float* qw, const float* kvw, float eps, const int64_t* positions,
                                                           const float2* cs, int max_pos, T* cache, const int32_t* slots) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t item = blockIdx.x * 8ll + (threadIdx.x >> 5);
  const int lane = threadIdx.x & 31;
  const int64_t token = item >> 1;
  if (token >= M) return;
  T* row = p + token * ld;
  if (item & 1) {
    if (q_pad > 0) warp_rms<T>(row, q_dim, q_pad, qw, eps, lane, row, nullptr);
    return;
  }
  const int slot = cache != nullptr ? slots[token] : -1;
  T* dst = slot >= 0 ? cache + static_cast<int64_t>(slot) * (kv_pad + rot_pad) : nullptr;
  row += q_pad;
  warp_rms<T>(row, kv_dim, kv_pad, kvw, eps, lane, row, dst);
  const int64_t pos = positions[token];
  for (int c = lane * 8; c < rot_pad; c += 256) {
    float f[8];
    load8<T>(row + kv_pad + c, f);
    rotate8(f, cs, max_pos, rot_pad >> 1, pos, c >> 1);
    store8<T>(row + kv_pad + c, f);
    if (dst != nullptr) store8<T>(dst + kv_pad + c, f);
  }
}

// Cached rows of every sequence, contiguous: row cu_k[b] + j of out is position j of sequence b.  One warp per row.
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* cache, const int32_t* block_tables, int64_t bt_stride, int block_size,
                                                            const int32_t* cu_k, int vecs, uint4* out) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, lane = threadIdx.x & 31;
  const int k0 = cu_k[b], n = cu_k[b + 1] - k0;
  for (int j = blockIdx.x * 8 + (threadIdx.x >> 5); j < n; j += gridDim.x * 8) {
    const int64_t slot = static_cast<int64_t>(block_tables[b * bt_stride + j / block_size]) * block_size + j % block_size;
    for (int c = lane; c < vecs; c += 32) out[static_cast<int64_t>(k0 + j) * vecs + c] = cache[slot * vecs + c];
  }
}

// ---------------------------------------------------------------------------
// out[m, h, n] = sum_k x[m, h, k] W_h[n, k], one product per head.  W_h rows are outputs ([N, K]) or, KN, inputs ([K, N]).
// One CTA column past the last output tile (rot_pad > 0) rotates the rot_pad elements behind x's K and puts them behind
// the N outputs.  gate: the outputs are multiplied by sigmoid(gate[m, h * gate_hs + n]).
// ---------------------------------------------------------------------------
struct HeadsArgs {
  const void* x;
  int64_t ldx;
  int x_hs;  // elements from one head to the next
  const void* w;
  int64_t ldw, w_hs;
  void* out;
  int64_t ldo;
  int out_hs;
  int M, N, K;
  const void* gate;
  int64_t ldg;
  int gate_hs;
  int rot_pad;
  const int64_t* positions;
  const float2* cs;
  int max_pos;
};

template <typename T>
__device__ __forceinline__ void rotate_rows(const HeadsArgs& a, int m0, int h) {
  const int vecs = a.rot_pad >> 3;
  for (int i = threadIdx.x; i < 64 * vecs; i += blockDim.x) {
    const int m = m0 + i / vecs, c = (i % vecs) * 8;
    if (m >= a.M) break;
    float f[8];
    load8<T>(static_cast<const T*>(a.x) + m * a.ldx + static_cast<int64_t>(h) * a.x_hs + a.K + c, f);
    rotate8(f, a.cs, a.max_pos, a.rot_pad >> 1, a.positions[m], c >> 1);
    store8<T>(static_cast<T*>(a.out) + m * a.ldo + static_cast<int64_t>(h) * a.out_hs + a.N + c, f);
  }
}

template <bool KN>
__global__ void __launch_bounds__(128) heads_gemm_kernel(const HeadsArgs a) {
  __shared__ __align__(128) unsigned char smem[2][2][64 * 64 * 2];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64, h = blockIdx.z;
  if (n0 >= a.N) {
    rotate_rows<uint16_t>(a, m0, h);
    return;
  }
  const uint16_t* x = static_cast<const uint16_t*>(a.x) + static_cast<int64_t>(h) * a.x_hs;
  const uint16_t* w = static_cast<const uint16_t*>(a.w) + h * a.w_hs;
  auto load = [&](int st, int k0) {
    const uint32_t sa = smem_u32(smem[st][0]), sw = smem_u32(smem[st][1]);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx >> 3, p = idx & 7;
      const bool ok = m0 + r < a.M && k0 + p * 8 < a.K;
      cp_async16(tile_addr<64>(sa, r, p), ok ? x + (m0 + r) * a.ldx + k0 + p * 8 : x, ok);
      const int wr = (KN ? k0 : n0) + r, wc = (KN ? n0 : k0) + p * 8;
      const bool wok = wr < (KN ? a.K : a.N) && wc < (KN ? a.N : a.K);
      cp_async16(tile_addr<64>(sw, r, p), wok ? w + wr * a.ldw + wc : w, wok);
    }
  };
  float acc[8][4];
#pragma unroll
  for (int n = 0; n < 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  load(0, 0);
  cp_async_commit();
  for (int k0 = 0, it = 0; k0 < a.K; k0 += 64, ++it) {
    cp_async_wait<0>();
    __syncthreads();
    if (k0 + 64 < a.K) load((it + 1) & 1, k0 + 64);
    cp_async_commit();
    const uint32_t sa = smem_u32(smem[it & 1][0]), sw = smem_u32(smem[it & 1][1]);
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t qa[4];
      frag_a<64>(sa, warp * 16, k * 16, lane, qa);
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        uint32_t kb[4];
        if (KN) frag_b_t<64>(sw, n * 16, k * 16, lane, kb);
        else frag_b<64>(sw, n * 16, k * 16, lane, kb);
        mma16816(acc[2 * n], qa, kb[0], kb[1]);
        mma16816(acc[2 * n + 1], qa, kb[2], kb[3]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int m = m0 + warp * 16 + (lane >> 2) + e * 8;
    if (m >= a.M) continue;
    uint16_t* dst = static_cast<uint16_t*>(a.out) + m * a.ldo + static_cast<int64_t>(h) * a.out_hs;
    const uint16_t* g = a.gate != nullptr ? static_cast<const uint16_t*>(a.gate) + m * a.ldg + static_cast<int64_t>(h) * a.gate_hs : nullptr;
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int c = n0 + n * 8 + (lane & 3) * 2;
      if (c >= a.N) continue;
      float u = acc[n][2 * e], v = acc[n][2 * e + 1];
      if (g != nullptr) {
        const uint32_t gv = *reinterpret_cast<const uint32_t*>(g + c);
        u *= sigmoid_fast(bf16_lo(gv));
        v *= sigmoid_fast(bf16_hi(gv));
      }
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(u, v);
    }
  }
}

// fp32, CUDA cores: 64 x 64 outputs, 4 x 4 per thread
template <bool KN>
__global__ void __launch_bounds__(256) heads_gemm_f32_kernel(const HeadsArgs a) {
  constexpr int TK = 16;
  __shared__ float sa[TK][64 + 4], sw[TK][64 + 4];
  pdl_launch_dependents();
  pdl_wait();
  const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64, h = blockIdx.z;
  if (n0 >= a.N) {
    rotate_rows<float>(a, m0, h);
    return;
  }
  const float* x = static_cast<const float*>(a.x) + static_cast<int64_t>(h) * a.x_hs;
  const float* w = static_cast<const float*>(a.w) + h * a.w_hs;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += TK) {
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 256;
      const int xr = idx / TK, xk = idx % TK;
      sa[xk][xr] = (m0 + xr < a.M && k0 + xk < a.K) ? x[(m0 + xr) * a.ldx + k0 + xk] : 0.f;
      const int wn = KN ? idx % 64 : idx / TK, wk = KN ? idx / 64 : idx % TK;
      const bool ok = n0 + wn < a.N && k0 + wk < a.K;
      sw[wk][wn] = ok ? (KN ? w[(k0 + wk) * a.ldw + n0 + wn] : w[(n0 + wn) * a.ldw + k0 + wk]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float av[4], wv[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        av[i] = sa[k][ty * 4 + i];
        wv[i] = sw[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= a.M) break;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= a.N) break;
      float v = acc[i][j];
      if (a.gate != nullptr) v *= sigmoid(static_cast<const float*>(a.gate)[m * a.ldg + static_cast<int64_t>(h) * a.gate_hs + n]);
      static_cast<float*>(a.out)[m * a.ldo + static_cast<int64_t>(h) * a.out_hs + n] = v;
    }
  }
}

// ---------------------------------------------------------------------------
// Absorbed attention.  16 MT rows (token, head) per CTA; 8 warps.  Scores: the warps share the tile's keys (and the MT row
// groups); values: each warp owns DL / 8 columns of the latent for all rows.  Softmax weights pass through shared memory
// as a sum of two bf16 numbers.  Key tiles are dealt to `splits` CTAs whose parts the last one to arrive combines.
// ---------------------------------------------------------------------------
constexpr int LAT_ROT = 64;           // columns kept for the rotated part
constexpr int LAT_MAX_SPLITS = 64;
constexpr int LAT_MAX_GROUPS = 65536;  // arrival counters at the front of the workspace

template <int DL, int MT>
struct CfgLatent {
  static constexpr int DK = DL + LAT_ROT;
  static constexpr int ROWS = 16 * MT;
  static constexpr int STAGE = BN * DK * 2;
  static constexpr int Q_BYTES = ROWS * DK * 2;
  static constexpr int P_BYTES = ROWS * BN * 2;
  static constexpr int SMEM = Q_BYTES + 2 * STAGE + 2 * P_BYTES + 128;
  static constexpr int PART = ROWS * (DL + 2);  // floats of one split's part
};

// a row [lat_pad | rot_pad] into columns [0, lat_pad) and [DL, DL + rot_pad) of a tile row, zeros elsewhere; one warp per row
template <int DL>
__device__ __forceinline__ void load_latent_row(uint32_t tile, int r, const uint16_t* src, bool ok, int lat8, int rot8, int lane) {
  constexpr int P = (DL + LAT_ROT) / 8;
#pragma unroll
  for (int i = 0; i < (P + 31) / 32; ++i) {
    const int p = lane + i * 32;
    if (p >= P) break;
    const bool rot = p >= DL / 8;
    const bool in = ok && (rot ? p - DL / 8 < rot8 : p < lat8);
    cp_async16(tile_addr<DL + LAT_ROT>(tile, r, p), in ? src + (rot ? lat8 + p - DL / 8 : p) * 8 : src, in);
  }
}

template <int DL, int MT>
__global__ void __launch_bounds__(256, 1) latent_attn_kernel(const AttnArgs a, int rot_pad, int row_tiles, int splits, int* counters, float* part) {
  using C = CfgLatent<DL, MT>;
  constexpr int DK = C::DK, ROWS = C::ROWS, KG = 8 / MT, WC = DL / 8;  // KG key groups; WC value columns of a warp
  extern __shared__ unsigned char smem_raw[];
  __shared__ float s_max[KG][ROWS], s_corr[ROWS], s_ml[ROWS][2];
  __shared__ int s_last;
  const uint32_t base = (smem_u32(smem_raw) + 127) & ~127u;
  const uint32_t sq = base, skv = base + C::Q_BYTES, sp = skv + 2 * C::STAGE, sp_lo = sp + C::P_BYTES;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.z, split = blockIdx.x, r_base = blockIdx.y * ROWS;
  const int row0 = a.cu_q ? a.cu_q[b] : b;
  const int n_q = a.cu_q ? a.cu_q[b + 1] - row0 : 1;
  const int rows = n_q * a.nq;
  if (r_base >= rows) return;
  const int nrows = min(ROWS, rows - r_base);
  const int klen = a.kv_len[b];
  uint16_t* out = static_cast<uint16_t*>(a.out);
  const auto out_row = [&](int r) {
    const int gr = r_base + r, tok = gr / a.nq;
    return out + (row0 + tok) * a.ldo + static_cast<int64_t>(gr - tok * a.nq) * a.v_pad;
  };
  if (klen <= 0) {  // padded row of a decode graph
    if (split == 0)
      for (int i = threadIdx.x; i < nrows * a.v_pad; i += 256) out_row(i / a.v_pad)[i % a.v_pad] = 0;
    return;
  }
  const int first_pos = klen - n_q;
  const int pmin = first_pos + r_base / a.nq, pmax = first_pos + (r_base + nrows - 1) / a.nq;
  const int total = pmax / BN + 1, per = (total + splits - 1) / splits;
  const int t0 = split * per, t1 = min(total, t0 + per);
  const int lat8 = a.v_pad >> 3, rot8 = rot_pad >> 3;
  const int32_t* bt = a.block_tables + b * a.bt_stride;
  const uint16_t* cache = static_cast<const uint16_t*>(a.k_cache);
  auto load_tile = [&](int tile, uint32_t dst) {
#pragma unroll 2
    for (int r = warp; r < BN; r += 8) {
      const int j = tile * BN + r;
      const bool ok = j <= pmax;
      const int blk = ok ? j / a.block_size : 0;
      const int64_t slot = ok ? static_cast<int64_t>(__ldg(bt + blk)) * a.block_size + (j - blk * a.block_size) : 0;
      load_latent_row<DL>(dst, r, cache + slot * a.k_row, ok, lat8, rot8, lane);
    }
  };
  for (int r = warp; r < ROWS; r += 8) {
    const int gr = r_base + r, tok = r < nrows ? gr / a.nq : 0, h = r < nrows ? gr - tok * a.nq : 0;
    load_latent_row<DL>(sq, r, static_cast<const uint16_t*>(a.q) + (row0 + tok) * a.ldq + static_cast<int64_t>(h) * a.qk_pad, r < nrows, lat8, rot8, lane);
  }
  if (t0 < t1) load_tile(t0, skv);
  cp_async_commit();
  const int mt = warp % MT, kg = warp / MT;  // this warp's rows and keys of the score tile
  int pos[2];
#pragma unroll
  for (int e = 0; e < 2; ++e) pos[e] = first_pos + (r_base + min(mt * 16 + (lane >> 2) + e * 8, nrows - 1)) / a.nq;
  const float scale = a.scale * LOG2E;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[MT][WC / 8][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int n = 0; n < WC / 8; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[i][n][e] = 0.f;
  for (int t = t0; t < t1; ++t) {
    const uint32_t sk = skv + ((t - t0) & 1) * C::STAGE;
    cp_async_wait<0>();
    __syncthreads();  // this tile has landed, and everyone has left the stage that is filled next
    if (t + 1 < t1) load_tile(t + 1, skv + ((t + 1 - t0) & 1) * C::STAGE);
    cp_async_commit();
    // scores of 16 rows x 8 MT keys, even and odd steps of the product in separate accumulators
    float s[2][MT][4];
#pragma unroll
    for (int p = 0; p < 2; ++p)
#pragma unroll
      for (int n = 0; n < MT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) s[p][n][e] = 0.f;
#pragma unroll 4
    for (int k = 0; k < DK / 32; ++k) {
      uint32_t qa[2][4];
      frag_a<DK>(sq, mt * 16, k * 32, lane, qa[0]);
      frag_a<DK>(sq, mt * 16, k * 32 + 16, lane, qa[1]);
      if (MT == 1) {
        uint32_t kb[4];  // 8 keys, 32 columns
        ldsm_x4(tile_addr<DK>(sk, kg * 8 + (lane & 7), k * 4 + (lane >> 3)), kb);
        mma16816(s[0][0], qa[0], kb[0], kb[1]);
        mma16816(s[1][0], qa[1], kb[2], kb[3]);
      } else {
#pragma unroll
        for (int p = 0; p < 2; ++p) {
          uint32_t kb[4];
          frag_b<DK>(sk, kg * 16, k * 32 + p * 16, lane, kb);
          mma16816(s[p][0], qa[p], kb[0], kb[1]);
          mma16816(s[p][MT - 1], qa[p], kb[2], kb[3]);
        }
      }
    }
    const int j0 = t * BN + kg * 8 * MT;
    const bool masked = j0 + 8 * MT - 1 > pmin;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < MT; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        float v = (s[0][n][e] + s[1][n][e]) * scale;
        if (masked && j0 + n * 8 + (lane & 3) * 2 + (e & 1) > pos[e >> 1]) v = -INFINITY;
        s[0][n][e] = v;
        mx[e >> 1] = fmaxf(mx[e >> 1], v);
      }
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 1));
      mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], 2));
      if ((lane & 3) == 0) s_max[kg][mt * 16 + (lane >> 2) + e * 8] = mx[e];
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = mt * 16 + (lane >> 2) + e * 8;
      float m_new = m[e];
#pragma unroll
      for (int i = 0; i < KG; ++i) m_new = fmaxf(m_new, s_max[i][r]);
      const float ref = m_new == -INFINITY ? 0.f : m_new;
      const float corr = fast_exp2(m[e] - ref);
      m[e] = m_new;
      if (kg == 0 && (lane & 3) == 0) s_corr[r] = corr;
      float sum = 0.f;
#pragma unroll
      for (int n = 0; n < MT; ++n) {
        const float x = fast_exp2(s[0][n][2 * e] - ref), y = fast_exp2(s[0][n][2 * e + 1] - ref);
        sum += x + y;
        uint32_t hi, lo;
        split_bf16(x, y, hi, lo);
        const uint32_t at = tile_addr<64>(0, r, kg * MT + n) + (lane & 3) * 4;
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(sp + at), "r"(hi) : "memory");
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(sp_lo + at), "r"(lo) : "memory");
      }
      l[e] = fmaf(l[e], corr, sum);  // this lane's keys
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const float c0 = s_corr[i * 16 + (lane >> 2)], c1 = s_corr[i * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int n = 0; n < WC / 8; ++n) {
        o[i][n][0] *= c0; o[i][n][1] *= c0; o[i][n][2] *= c1; o[i][n][3] *= c1;
      }
    }
#pragma unroll
    for (int k = 0; k < BN / 16; ++k) {
      uint32_t hi[MT][4], lo[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        frag_a<64>(sp, i * 16, k * 16, lane, hi[i]);
        frag_a<64>(sp_lo, i * 16, k * 16, lane, lo[i]);
      }
#pragma unroll
      for (int n = 0; n < WC / 16; ++n) {
        uint32_t vb[4];
        frag_b_t<DK>(sk, warp * WC + n * 16, k * 16, lane, vb);
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma16816(o[i][2 * n], hi[i], vb[0], vb[1]);
          mma16816(o[i][2 * n + 1], hi[i], vb[2], vb[3]);
          mma16816(o[i][2 * n], lo[i], vb[0], vb[1]);
          mma16816(o[i][2 * n + 1], lo[i], vb[2], vb[3]);
        }
      }
    }
  }
  cp_async_wait<0>();
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int r = mt * 16 + (lane >> 2) + e * 8;
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
    if ((lane & 3) == 0) s_max[kg][r] = l[e];
    if (kg == 0 && (lane & 3) == 0) s_ml[r][0] = m[e];
  }
  __syncthreads();
  if (threadIdx.x < ROWS) {
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < KG; ++i) sum += s_max[i][threadIdx.x];
    s_ml[threadIdx.x][1] = sum;
  }
  __syncthreads();
  const int group = b * row_tiles + blockIdx.y;
  float* my = part + (static_cast<int64_t>(group) * splits + split) * C::PART;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = i * 16 + (lane >> 2) + e * 8;
      if (r >= nrows) continue;
      if (splits == 1) {
        float f = 1.0f, sum = s_ml[r][1];
        if (a.sink != nullptr) {
          const float mr = s_ml[r][0], sk = a.sink[(r_base + r) % a.nq] * LOG2E, m_new = fmaxf(mr, sk);
          f = fast_exp2(mr - m_new);
          sum = sum * f + fast_exp2(sk - m_new);
        }
        f /= sum;
        uint16_t* dst = out_row(r);
#pragma unroll
        for (int n = 0; n < WC / 8; ++n) {
          const int c = warp * WC + n * 8 + (lane & 3) * 2;
          if (c < a.v_pad) *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(o[i][n][2 * e] * f, o[i][n][2 * e + 1] * f);
        }
      } else {
#pragma unroll
        for (int n = 0; n < WC / 8; ++n)
          *reinterpret_cast<float2*>(my + 2 * ROWS + r * DL + warp * WC + n * 8 + (lane & 3) * 2) = make_float2(o[i][n][2 * e], o[i][n][2 * e + 1]);
      }
    }
  if (splits == 1) return;
  if (threadIdx.x < nrows) {
    my[threadIdx.x] = s_ml[threadIdx.x][0];
    my[ROWS + threadIdx.x] = s_ml[threadIdx.x][1];
  }
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(counters + group, 1) == splits - 1;
  __syncthreads();
  if (!s_last) return;
  if (threadIdx.x == 0) counters[group] = 0;
  __threadfence();
  const float* all = part + static_cast<int64_t>(group) * splits * C::PART;
  float* s_f = reinterpret_cast<float*>(smem_raw);  // [splits][ROWS] factors of the parts
  if (threadIdx.x < nrows) {
    const int r = threadIdx.x;
    const float sk = a.sink != nullptr ? a.sink[(r_base + r) % a.nq] * LOG2E : -INFINITY;
    float mt_ = sk;
    for (int s = 0; s < splits; ++s) mt_ = fmaxf(mt_, ld_cg_f32(all + static_cast<int64_t>(s) * C::PART + r));
    float lt = fast_exp2(sk - mt_);
    for (int s = 0; s < splits; ++s) {
      const float ms = ld_cg_f32(all + static_cast<int64_t>(s) * C::PART + r);
      const float f = ms > -INFINITY ? fast_exp2(ms - mt_) : 0.f;
      s_f[s * ROWS + r] = f;
      if (f > 0.f) lt += f * ld_cg_f32(all + static_cast<int64_t>(s) * C::PART + ROWS + r);
    }
    for (int s = 0; s < splits; ++s) s_f[s * ROWS + r] /= lt;
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < nrows * (DL / 4); idx += 256) {
    const int r = idx / (DL / 4), c = (idx % (DL / 4)) * 4;
    if (c >= a.v_pad) continue;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int s = 0; s < splits; ++s) {
      const float f = s_f[s * ROWS + r];
      if (f == 0.f) continue;  // a split without keys for this row may hold anything
      const uint4 v = ld_cg_v4(all + static_cast<int64_t>(s) * C::PART + 2 * ROWS + r * DL + c);
      acc.x += f * __uint_as_float(v.x); acc.y += f * __uint_as_float(v.y);
      acc.z += f * __uint_as_float(v.z); acc.w += f * __uint_as_float(v.w);
    }
    *reinterpret_cast<uint2*>(out_row(r) + c) = make_uint2(pack_bf16(acc.x, acc.y), pack_bf16(acc.z, acc.w));
  }
}

bool latent_tiled(int dtype, int lat_pad, int rot_pad) { return dtype == B2_DT_BF16 && lat_pad <= 512 && rot_pad <= LAT_ROT; }
int latent_width(int lat_pad) { return lat_pad <= 128 ? 128 : lat_pad <= 256 ? 256 : 512; }

struct LatentPlan {
  int rows, row_tiles, splits;
  int64_t groups, bytes;
};
// Rows per CTA and how many CTAs share a group's key tiles: as few rounds of one CTA per SM as possible, counting a part's
// combine as about two tiles.
LatentPlan latent_plan(int B, int max_q, int max_kv, int heads, int lat_pad) {
  LatentPlan p{};
  const int64_t all = static_cast<int64_t>(max_q) * heads;
  p.rows = all > 16 ? 32 : 16;
  p.row_tiles = static_cast<int>((all + p.rows - 1) / p.rows);
  p.groups = static_cast<int64_t>(B) * p.row_tiles;
  const int64_t tiles = std::max<int64_t>(1, (static_cast<int64_t>(max_kv) + BN - 1) / BN);
  p.splits = 1;
  if (p.groups <= LAT_MAX_GROUPS && p.groups < 4 * 148) {
    int64_t best = INT64_MAX;
    for (int s = 1; s <= std::min<int64_t>(LAT_MAX_SPLITS, tiles); ++s) {
      const int64_t cost = ((p.groups * s + 147) / 148) * ((tiles + s - 1) / s + 1 + (s > 1 ? 2 : 0)) + s / 8;
      if (cost < best) {
        best = cost;
        p.splits = s;
      }
    }
  }
  p.bytes = p.splits > 1 ? LAT_MAX_GROUPS * 4ll + p.groups * p.splits * p.rows * (latent_width(lat_pad) + 2) * 4ll : 0;
  return p;
}

template <int DL, int MT>
int launch_latent(const AttnArgs& a, int rot_pad, const LatentPlan& p, void* ws, cudaStream_t s) {
  using C = CfgLatent<DL, MT>;
  static const cudaError_t set = cudaFuncSetAttribute(latent_attn_kernel<DL, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
  B2_CUDA(set);
  float* part = ws != nullptr ? reinterpret_cast<float*>(static_cast<unsigned char*>(ws) + LAT_MAX_GROUPS * 4ll) : nullptr;
  B2_CUDA(b2_launch(latent_attn_kernel<DL, MT>, dim3(p.splits, p.row_tiles, a.B), dim3(256), C::SMEM, s, a, rot_pad, p.row_tiles, p.splits,
                    static_cast<int*>(ws), part));
  return B2_OK;
}

// ---------------------------------------------------------------------------
// Expanded attention
// ---------------------------------------------------------------------------
struct ExpandedArgs {
  const uint16_t* kv;  // rows [heads][dim_pad key | v_pad value], row cu_k[b] + j = position j
  int64_t ld_kv;
  const uint16_t* rot;  // rotated key parts of the same rows
  int64_t ld_rot;
  const int32_t* cu_k;
  int dim_pad, rot_pad;
  const float2* cs;
  int max_pos;
  const uint16_t* gate;  // [M][heads][v_pad] or null
  int64_t ldg;
};

template <int DQ, int DV>
__global__ void __launch_bounds__(128, 2) expanded_attn_kernel(const AttnArgs a, const ExpandedArgs e) {
  extern __shared__ unsigned char smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 127) & ~127u;
  const uint32_t sq = base, skv = base + 64 * DQ * 2;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int row0 = a.cu_q[b], rows = a.cu_q[b + 1] - row0;
  const int tile0 = (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * 64;  // the longest rows first
  if (tile0 >= rows) return;
  const int key0 = e.cu_k[b], first_pos = e.cu_k[b + 1] - key0 - rows;
  const int pmin = first_pos + tile0, pmax = first_pos + min(tile0 + 63, rows - 1);
  const KeyTiles tiles(pmin, pmax, a.window, a.keep_first);
  constexpr int PQ = DQ / 8, PV = DV / 8;
  const uint16_t* q = static_cast<const uint16_t*>(a.q) + row0 * a.ldq + static_cast<int64_t>(h) * a.qk_pad;
#pragma unroll 4
  for (int i = 0; i < 64 * PQ / 128; ++i) {
    const int idx = threadIdx.x + i * 128, r = idx / PQ, p = idx % PQ;
    const bool ok = tile0 + r < rows && p * 8 < a.qk_pad;
    cp_async16(tile_addr<DQ>(sq, r, p), ok ? q + (tile0 + r) * a.ldq + p * 8 : q, ok);
  }
  const int dim8 = e.dim_pad >> 3, all8 = dim8 + (e.rot_pad >> 3), v8 = a.v_pad >> 3;
  const uint16_t* kvh = e.kv + key0 * e.ld_kv + static_cast<int64_t>(h) * (e.dim_pad + a.v_pad);
  const uint16_t* rot = e.rot + key0 * e.ld_rot;
  auto load = [&](int tile, uint32_t sk, uint32_t sv) {
#pragma unroll 4
    for (int i = 0; i < 64 * PQ / 128; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx / PQ, p = idx % PQ, j = tile * BN + r;
      const bool ok = p < all8 && j <= pmax;
      const uint16_t* src = p < dim8 ? kvh + j * e.ld_kv + p * 8 : rot + j * e.ld_rot + (p - dim8) * 8;
      cp_async16(tile_addr<DQ>(sk, r, p), ok ? src : kvh, ok);
    }
#pragma unroll 4
    for (int i = 0; i < 64 * PV / 128; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx / PV, p = idx % PV, j = tile * BN + r;
      const bool ok = p < v8 && j <= pmax;
      cp_async16(tile_addr<DV>(sv, r, p), ok ? kvh + j * e.ld_kv + e.dim_pad + p * 8 : kvh, ok);
    }
  };
  auto rotate_q = [&] {
    cp_async_wait<0>();
    __syncthreads();
    const int rot8 = e.rot_pad >> 3;
    for (int idx = threadIdx.x; idx < 64 * rot8; idx += 128) {
      const int r = idx / rot8, p = idx % rot8;
      uint16_t* at = reinterpret_cast<uint16_t*>(smem_raw + (tile_addr<DQ>(sq, r, dim8 + p) - smem_u32(smem_raw)));
      float f[8];
      load8<uint16_t>(at, f);
      rotate8(f, e.cs, e.max_pos, e.rot_pad >> 1, first_pos + tile0 + r, p * 4);
      store8<uint16_t>(at, f);
    }
  };
  float m[2], l[2], o[DV / 8][4];
  prefill_tiles<DQ, DV, CAP_NONE>(a, first_pos, tile0, rows, 1, tiles, sq, skv, load, rotate_q, m, l, o);
  uint16_t* out = static_cast<uint16_t*>(a.out) + static_cast<int64_t>(h) * a.v_pad;
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
    l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
    const int r = tile0 + warp * 16 + (lane >> 2) + i * 8;
    if (r >= rows) continue;
    float f = 1.0f;
    if (a.sink != nullptr) {
      const float sk = a.sink[h] * LOG2E, m_new = fmaxf(m[i], sk);
      f = fast_exp2(m[i] - m_new);
      l[i] = l[i] * f + fast_exp2(sk - m_new);
    }
    f /= l[i];
    uint16_t* dst = out + (row0 + r) * a.ldo;
    const uint16_t* g = e.gate != nullptr ? e.gate + (row0 + r) * e.ldg + static_cast<int64_t>(h) * a.v_pad : nullptr;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
      const int c = n * 8 + (lane & 3) * 2;
      if (c >= a.v_pad) continue;
      float u = o[n][2 * i] * f, v = o[n][2 * i + 1] * f;
      if (g != nullptr) {
        const uint32_t gv = *reinterpret_cast<const uint32_t*>(g + c);
        u *= sigmoid_fast(bf16_lo(gv));
        v *= sigmoid_fast(bf16_hi(gv));
      }
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(u, v);
    }
  }
}

template <int DQ, int DV>
int launch_expanded(const AttnArgs& a, const ExpandedArgs& e, int max_q, cudaStream_t s) {
  constexpr int SMEM = CfgTile<DQ, DV>::SMEM_PREFILL;
  static const cudaError_t set = cudaFuncSetAttribute(expanded_attn_kernel<DQ, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM);
  B2_CUDA(set);
  B2_CUDA(b2_launch(expanded_attn_kernel<DQ, DV>, dim3((max_q + 63) / 64, a.nq, a.B), dim3(128), SMEM, s, a, e));
  return B2_OK;
}

bool bad_dtype(int dtype) { return dtype != B2_DT_BF16 && dtype != B2_DT_F32; }

}  // namespace

extern "C" {

int b2_latent_store(int dtype, void* rows, int64_t ld, int M, int q_dim, int q_pad, int kv_dim, int kv_pad, int rot_pad, const float* q_norm_w,
                    const float* kv_norm_w, float eps, const int64_t* positions, const float* cos_sin, int max_pos, void* cache,
                    const int32_t* slot_mapping, void* stream) {
  if (M < 0 || bad_dtype(dtype) || q_dim < 0 || q_pad < q_dim || kv_dim <= 0 || kv_pad < kv_dim || rot_pad < 0 || max_pos <= 0) return B2_ERR_ARG;
  if (q_pad % 8 != 0 || kv_pad % 8 != 0 || rot_pad % 8 != 0 || ld % 8 != 0 || ld < q_pad + kv_pad + rot_pad) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!rows || !aligned16(rows) || (q_dim > 0 && (!q_norm_w || !aligned16(q_norm_w))) || !kv_norm_w || !aligned16(kv_norm_w) || !positions) return B2_ERR_ARG;
  if (rot_pad > 0 && !cos_sin) return B2_ERR_ARG;
  if (cache != nullptr && (!slot_mapping || !aligned16(cache))) return B2_ERR_ARG;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid(static_cast<unsigned>((2ll * M + 7) / 8));
  const float2* cs = reinterpret_cast<const float2*>(cos_sin);
  if (dtype == B2_DT_BF16)
    B2_CUDA(b2_launch(latent_store_kernel<uint16_t>, grid, dim3(256), 0, s, static_cast<uint16_t*>(rows), ld, M, q_dim, q_pad, kv_dim, kv_pad, rot_pad,
                      q_norm_w, kv_norm_w, eps, positions, cs, max_pos, static_cast<uint16_t*>(cache), slot_mapping));
  else
    B2_CUDA(b2_launch(latent_store_kernel<float>, grid, dim3(256), 0, s, static_cast<float*>(rows), ld, M, q_dim, q_pad, kv_dim, kv_pad, rot_pad,
                      q_norm_w, kv_norm_w, eps, positions, cs, max_pos, static_cast<float*>(cache), slot_mapping));
  return B2_OK;
}

int b2_latent_gather(int dtype, const void* cache, const int32_t* block_tables, int64_t bt_stride, int block_size, const int32_t* cu_k, int B,
                     int max_kv, int row, void* out, void* stream) {
  if (B < 0 || bad_dtype(dtype) || max_kv < 0 || row <= 0 || row % 8 != 0 || block_size < 1) return B2_ERR_ARG;
  if (B == 0 || max_kv == 0) return B2_OK;
  if (!cache || !block_tables || !cu_k || !out || !aligned16(cache) || !aligned16(out)) return B2_ERR_ARG;
  if (B > 65535) return B2_ERR_SHAPE;
  const int vecs = row * (dtype == B2_DT_BF16 ? 2 : 4) / 16;
  B2_CUDA(b2_launch(latent_gather_kernel, dim3(std::min((max_kv + 7) / 8, 1024), B), dim3(256), 0, static_cast<cudaStream_t>(stream),
                    static_cast<const uint4*>(cache), block_tables, bt_stride, block_size, cu_k, vecs, static_cast<uint4*>(out)));
  return B2_OK;
}

int b2_heads_gemm(int dtype, const void* x, int64_t ldx, int x_head, const void* w, int64_t ldw, int64_t w_head, int w_is_kn, void* out, int64_t ldo,
                  int out_head, int M, int heads, int N, int K, const void* gate, int64_t ldg, int gate_head, int rot_pad, const int64_t* positions,
                  const float* cos_sin, int max_pos, void* stream) {
  if (M < 0 || bad_dtype(dtype) || heads <= 0 || N <= 0 || K <= 0 || N % 8 != 0 || K % 8 != 0 || rot_pad < 0 || rot_pad % 8 != 0) return B2_ERR_ARG;
  if (ldx % 8 != 0 || ldw % 8 != 0 || ldo % 8 != 0 || x_head % 8 != 0 || w_head % 8 != 0 || out_head % 8 != 0) return B2_ERR_ARG;
  if (x_head < K + rot_pad || out_head < N + rot_pad || ldw < (w_is_kn ? N : K)) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!x || !w || !out || !aligned16(x) || !aligned16(w) || !aligned16(out)) return B2_ERR_ARG;
  if (gate != nullptr && (!aligned16(gate) || ldg % 8 != 0 || gate_head % 8 != 0)) return B2_ERR_ARG;
  if (rot_pad > 0 && (!positions || !cos_sin || max_pos <= 0)) return B2_ERR_ARG;
  if (heads > 65535 || (M + 63) / 64 > 65535) return B2_ERR_SHAPE;
  HeadsArgs a{};
  a.x = x; a.ldx = ldx; a.x_hs = x_head; a.w = w; a.ldw = ldw; a.w_hs = w_head; a.out = out; a.ldo = ldo; a.out_hs = out_head;
  a.M = M; a.N = N; a.K = K; a.gate = gate; a.ldg = ldg; a.gate_hs = gate_head; a.rot_pad = rot_pad; a.positions = positions;
  a.cs = reinterpret_cast<const float2*>(cos_sin); a.max_pos = max_pos;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const dim3 grid((N + 63) / 64 + (rot_pad > 0 ? 1 : 0), (M + 63) / 64, heads);
  if (dtype == B2_DT_BF16) {
    if (w_is_kn) B2_CUDA(b2_launch(heads_gemm_kernel<true>, grid, dim3(128), 0, s, a));
    else B2_CUDA(b2_launch(heads_gemm_kernel<false>, grid, dim3(128), 0, s, a));
  } else {
    if (w_is_kn) B2_CUDA(b2_launch(heads_gemm_f32_kernel<true>, grid, dim3(256), 0, s, a));
    else B2_CUDA(b2_launch(heads_gemm_f32_kernel<false>, grid, dim3(256), 0, s, a));
  }
  return B2_OK;
}

int64_t b2_latent_attention_workspace(int dtype, int B, int max_q, int max_kv, int heads, int lat_pad, int rot_pad) {
  if (B <= 0 || max_q <= 0 || heads <= 0 || !latent_tiled(dtype, lat_pad, rot_pad)) return 0;
  return latent_plan(B, max_q, max_kv, heads, lat_pad).bytes;
}

int b2_latent_attention(int dtype, const void* q, int64_t ldq, void* out, int64_t ldo, const void* cache, const int32_t* block_tables,
                        int64_t bt_stride, int block_size, const int32_t* cu_q, const int32_t* kv_len, int B, int max_q, int max_kv, int heads,
                        int lat_pad, int rot_pad, float scale, const float* sink, void* workspace, int64_t workspace_bytes, int form, void* stream) {
  if (B < 0 || max_q < 0 || bad_dtype(dtype) || heads <= 0 || lat_pad <= 0 || rot_pad < 0 || lat_pad % 8 != 0 || rot_pad % 8 != 0) return B2_ERR_ARG;
  if (block_size < 1 || (cu_q == nullptr && max_q > 1)) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if (!q || !out || !cache || !block_tables || !kv_len) return B2_ERR_ARG;
  if (!aligned16(q) || !aligned16(out) || !aligned16(cache) || ldq % 8 != 0 || ldo % 8 != 0) return B2_ERR_ARG;
  if (lat_pad + rot_pad > 2048 || lat_pad > 1024 || B > 65535 || heads > 65535) return B2_ERR_SHAPE;
  AttnArgs a{};
  a.q = q; a.ldq = ldq; a.out = out; a.ldo = ldo; a.k_cache = a.v_cache = cache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.block_size = block_size; a.cu_q = cu_q; a.kv_len = kv_len;
  a.B = B; a.nq = heads; a.nkv = 1; a.qk_pad = lat_pad + rot_pad; a.v_pad = lat_pad; a.k_row = a.v_row = lat_pad + rot_pad;
  a.window = INT_MAX; a.scale = scale; a.sink = sink;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_F32) return launch_any<float>(a, max_q, s);
  if (form == 1 || !latent_tiled(dtype, lat_pad, rot_pad)) return launch_any<uint16_t>(a, max_q, s);
  const LatentPlan p = latent_plan(B, max_q, max_kv, heads, lat_pad);
  if (p.row_tiles > 65535) return B2_ERR_SHAPE;
  if (p.splits > 1 && (workspace == nullptr || workspace_bytes < p.bytes))
    return set_error(B2_ERR_SHAPE, "b2_latent_attention: workspace of %lld bytes, %lld needed", static_cast<long long>(workspace_bytes),
                     static_cast<long long>(p.bytes));
  switch (latent_width(lat_pad)) {
    case 128: return p.rows == 16 ? launch_latent<128, 1>(a, rot_pad, p, workspace, s) : launch_latent<128, 2>(a, rot_pad, p, workspace, s);
    case 256: return p.rows == 16 ? launch_latent<256, 1>(a, rot_pad, p, workspace, s) : launch_latent<256, 2>(a, rot_pad, p, workspace, s);
    default: return p.rows == 16 ? launch_latent<512, 1>(a, rot_pad, p, workspace, s) : launch_latent<512, 2>(a, rot_pad, p, workspace, s);
  }
}

int b2_expanded_attention(const void* q, int64_t ldq, void* out, int64_t ldo, const void* kv, int64_t ld_kv, const void* rot, int64_t ld_rot,
                          const int32_t* cu_q, const int32_t* cu_k, int B, int max_q, int heads, int dim_pad, int rot_pad, int v_pad, float scale,
                          const float* sink, const float* cos_sin, int max_pos, const void* gate, int64_t ldg, void* stream) {
  if (B < 0 || max_q < 0 || heads <= 0 || dim_pad < 0 || rot_pad < 0 || v_pad <= 0 || dim_pad % 8 != 0 || rot_pad % 8 != 0 || v_pad % 8 != 0) return B2_ERR_ARG;
  if (dim_pad + rot_pad <= 0) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if (!q || !out || !kv || !cu_q || !cu_k || !aligned16(q) || !aligned16(out) || !aligned16(kv)) return B2_ERR_ARG;
  if (ldq % 8 != 0 || ldo % 8 != 0 || ld_kv % 8 != 0 || ld_rot % 8 != 0) return B2_ERR_ARG;
  if (rot_pad > 0 && (!rot || !aligned16(rot) || !cos_sin || max_pos <= 0)) return B2_ERR_ARG;
  if (gate != nullptr && (!aligned16(gate) || ldg % 8 != 0)) return B2_ERR_ARG;
  if (dim_pad + rot_pad > 192 || v_pad > 128 || B > 65535 || heads > 65535) return B2_ERR_SHAPE;
  AttnArgs a{};
  a.q = q; a.ldq = ldq; a.out = out; a.ldo = ldo; a.cu_q = cu_q; a.B = B; a.nq = heads; a.nkv = heads;
  a.qk_pad = dim_pad + rot_pad; a.v_pad = v_pad; a.window = INT_MAX; a.scale = scale; a.sink = sink;
  ExpandedArgs e{};
  e.kv = static_cast<const uint16_t*>(kv); e.ld_kv = ld_kv;
  e.rot = rot_pad > 0 ? static_cast<const uint16_t*>(rot) : e.kv; e.ld_rot = ld_rot;
  e.cu_k = cu_k; e.dim_pad = dim_pad; e.rot_pad = rot_pad; e.cs = reinterpret_cast<const float2*>(cos_sin); e.max_pos = max_pos;
  e.gate = static_cast<const uint16_t*>(gate); e.ldg = ldg;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  const int dq = dim_pad + rot_pad;
  if (v_pad <= 64) return dq <= 64 ? launch_expanded<64, 64>(a, e, max_q, s) : dq <= 128 ? launch_expanded<128, 64>(a, e, max_q, s) : launch_expanded<192, 64>(a, e, max_q, s);
  return dq <= 64 ? launch_expanded<64, 128>(a, e, max_q, s) : dq <= 128 ? launch_expanded<128, 128>(a, e, max_q, s) : launch_expanded<192, 128>(a, e, max_q, s);
}

}  // extern "C"
