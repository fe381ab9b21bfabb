// Attention with a sliding window that keeps the first tokens, a soft cap on the scores and a learned sink in the
// softmax's denominator, over the paged KV cache.  Position i sees position j when j <= i and
// (i - j < window or j < keep_first); window = INT_MAX is full causal attention, softcap <= 0 and a null sink
// switch those parts off.
//
//   qk_norm_store_kernel   q/k head RMSNorm and the scatter of K and V into the cache
//   attn_prefill_kernel    bf16, head sizes up to 128: 64 rows x 64 keys on the tensor cores
//   attn_decode_kernel     the same for one query row per sequence, keys split over warps and CTAs
//   attn_any_kernel        any head size, bf16 or fp32, prefill and decode (one warp per query head)
#include "b2_attn.cuh"

namespace {

// ---------------------------------------------------------------------------
// q/k head RMSNorm (q in place, k into the cache) and V into the cache.  LANES lanes per (token, head), 8 elements
// per lane and pass.  Head strides are padded to 8 elements; the padding is zero and stays zero.
// ---------------------------------------------------------------------------
template <typename T, int LANES>
__global__ void __launch_bounds__(256) qk_norm_store_kernel(T* qkv, int64_t ld, int M, int nq, int nkv, int qk_dim, int qk_pad,
                                                            int v_pad, const T* __restrict__ qw, const T* __restrict__ kw, float eps,
                                                            T* k_cache, T* v_cache, const int32_t* slots) {
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

// The slot of key j of a sequence
__device__ __forceinline__ int64_t slot_of(const AttnArgs& a, const int32_t* bt, int j) {
  const int blk = j / a.block_size;
  return static_cast<int64_t>(__ldg(bt + blk)) * a.block_size + (j - blk * a.block_size);
}
// One tile of one operand, D columns of which `pad` exist: 128 threads, 16 bytes per copy.  base = first row's address
// when the tile lies in one block (`whole`), else every row is looked up.
template <int D>
__device__ __forceinline__ void load_rows(const AttnArgs& a, const uint16_t* cache, const int32_t* bt, bool whole, int64_t slot0, int g, int pad,
                                          int tile, int last, uint32_t dst) {
  constexpr int P = D / 8, STEP = 128 / P;
  const int r0 = threadIdx.x / P, p = threadIdx.x % P;
  const bool piece = p * 8 < pad;
  const int64_t stride = static_cast<int64_t>(a.nkv) * pad;
  const uint16_t* col = cache + static_cast<int64_t>(g) * pad + (piece ? p * 8 : 0);
  if (whole) {
    const uint16_t* src = col + (slot0 + r0) * stride;
#pragma unroll
    for (int i = 0; i < BN / STEP; ++i, src += STEP * stride) {
      const int r = r0 + i * STEP;
      const bool ok = piece && tile * BN + r <= last;
      b2::cp_async16(b2::tile_addr<D>(dst, r, p), ok ? src : cache, ok);
    }
  } else {
#pragma unroll
    for (int i = 0; i < BN / STEP; ++i) {
      const int r = r0 + i * STEP, j = tile * BN + r;
      const bool ok = piece && j <= last;
      b2::cp_async16(b2::tile_addr<D>(dst, r, p), ok ? col + slot_of(a, bt, j) * stride : cache, ok);
    }
  }
}
template <int DQ, int DV>
__device__ __forceinline__ void load_kv_tile(const AttnArgs& a, const int32_t* bt, bool whole, int g, int tile, int last, uint32_t sk, uint32_t sv) {
  const int64_t slot0 = whole ? slot_of(a, bt, tile * BN) : 0;
  load_rows<DQ>(a, static_cast<const uint16_t*>(a.k_cache), bt, whole, slot0, g, a.qk_pad, tile, last, sk);
  load_rows<DV>(a, static_cast<const uint16_t*>(a.v_cache), bt, whole, slot0, g, a.v_pad, tile, last, sv);
}

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

// Prefill: 64 rows (token, head of the group) per CTA, 16 per warp; the four warps share the key tiles.
template <int DQ, int DV, int CAP>
__global__ void __launch_bounds__(128, 2) attn_prefill_kernel(const AttnArgs a, int rep, bool whole) {
  extern __shared__ unsigned char smem_raw[];
  const uint32_t base = (b2::smem_u32(smem_raw) + 127) & ~127u;
  const uint32_t sq = base, skv = base + 64 * DQ * 2;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int b = blockIdx.z, g = blockIdx.y;
  const int row0 = a.cu_q[b];
  const int n_q = a.cu_q[b + 1] - row0;
  const int rows = n_q * rep;
  const int tile0 = (static_cast<int>(gridDim.x) - 1 - static_cast<int>(blockIdx.x)) * 64;  // the longest rows first
  if (tile0 >= rows) return;
  const int klen = a.kv_len[b];
  const int first_pos = klen - n_q;
  const int32_t* bt = a.block_tables + b * a.bt_stride;
  const int pmin = first_pos + tile0 / rep, pmax = first_pos + min(tile0 + 63, rows - 1) / rep;
  const KeyTiles tiles(pmin, pmax, a.window, a.keep_first);
  const ScoreScale sscale = score_scale(CAP, a.scale, a.softcap);
  const uint16_t* q = static_cast<const uint16_t*>(a.q);
#pragma unroll
  for (int i = 0; i < 64 * (DQ / 8) / 128; ++i) {
    const int idx = threadIdx.x + i * 128, r = idx / (DQ / 8), p = idx % (DQ / 8);
    const int gr = tile0 + r;
    const bool ok = gr < rows && p * 8 < a.qk_pad;
    const int tok = ok ? gr / rep : 0, hh = ok ? gr - tok * rep : 0;
    b2::cp_async16(b2::tile_addr<DQ>(sq, r, p), q + (row0 + tok) * a.ldq + static_cast<int64_t>(g * rep + hh) * a.qk_pad + (ok ? p * 8 : 0), ok);
  }
  load_kv_tile<DQ, DV>(a, bt, whole, g, tiles.at(0), pmax, skv, skv + BN * DQ * 2);
  b2::cp_async_commit();
  int pos[2];
#pragma unroll
  for (int h = 0; h < 2; ++h) pos[h] = first_pos + min(tile0 + warp * 16 + (lane >> 2) + h * 8, rows - 1) / rep;
  const int wpmin = first_pos + min(tile0 + warp * 16, rows - 1) / rep;
  const int wpmax = first_pos + min(tile0 + warp * 16 + 15, rows - 1) / rep;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[DV / 8][4];
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
      load_kv_tile<DQ, DV>(a, bt, whole, g, tiles.at(it + 1), pmax, nk, nk + BN * DQ * 2);
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
  uint16_t* out = static_cast<uint16_t*>(a.out);
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    const int gr = tile0 + warp * 16 + (lane >> 2) + h * 8;
    if (gr >= rows) continue;
    const int tok = gr / rep, head = g * rep + (gr - tok * rep);
    float f = 1.0f;
    if (a.sink != nullptr) {
      const float sk = a.sink[head] * LOG2E, m_new = fmaxf(m[h], sk);
      f = fast_exp2(m[h] - m_new);
      l[h] = l[h] * f + fast_exp2(sk - m_new);
    }
    f /= l[h];
    uint16_t* dst = out + (row0 + tok) * a.ldo + static_cast<int64_t>(head) * a.v_pad;
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
      const int c = n * 8 + (lane & 3) * 2;
      if (c < a.v_pad) *reinterpret_cast<uint32_t*>(dst + c) = b2::pack_bf16(o[n][2 * h] * f, o[n][2 * h + 1] * f);
    }
  }
}

// Decode: up to 16 query heads of one key/value head are the rows; the keys of a tile are dealt to the four warps and
// the tiles to `splits` CTAs, whose partial results the last one to arrive combines.
constexpr int DEC_MAX_SPLITS = 64;
constexpr int DEC_MAX_GROUPS = 65536;  // arrival counters at the front of the workspace

template <int DQ, int DV, int CAP>
__global__ void __launch_bounds__(128) attn_decode_kernel(const AttnArgs a, int rep, int row_tiles, bool whole, int splits, int* counters,
                                                          float* part) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ float s_ml[4][16][2];
  __shared__ float s_fin[16][2];
  __shared__ int s_last;
  constexpr int STAGES = CfgTile<DQ, DV>::DEC_STAGES;
  const uint32_t base = (b2::smem_u32(smem_raw) + 127) & ~127u;
  const uint32_t sq = base, skv = base + 16 * DQ * 2;
  float* o_buf = reinterpret_cast<float*>(smem_raw + (skv - b2::smem_u32(smem_raw)));  // [4][16][DV], after the last tile
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int b = blockIdx.z, g = blockIdx.y / row_tiles, h0 = (blockIdx.y % row_tiles) * 16, split = blockIdx.x;
  const int nrows = min(16, rep - h0);
  const int klen = a.kv_len[b];
  uint16_t* out = static_cast<uint16_t*>(a.out) + b * a.ldo + static_cast<int64_t>(g * rep + h0) * a.v_pad;
  if (klen <= 0) {  // padded row of a decode graph
    if (split == 0)
      for (int i = threadIdx.x; i < nrows * a.v_pad; i += 128) out[i] = 0;
    return;
  }
  const int p = klen - 1;
  const int32_t* bt = a.block_tables + b * a.bt_stride;
  const KeyTiles tiles(p, p, a.window, a.keep_first);
  const int per = (tiles.total + splits - 1) / splits;
  const int t0 = split * per, t1 = min(tiles.total, t0 + per);
  const ScoreScale sscale = score_scale(CAP, a.scale, a.softcap);
  const uint16_t* q = static_cast<const uint16_t*>(a.q) + b * a.ldq + static_cast<int64_t>(g * rep + h0) * a.qk_pad;
  for (int idx = threadIdx.x; idx < 16 * (DQ / 8); idx += 128) {
    const int r = idx / (DQ / 8), pc = idx % (DQ / 8);
    const bool ok = r < nrows && pc * 8 < a.qk_pad;
    b2::cp_async16(b2::tile_addr<DQ>(sq, r, pc), q + (ok ? r * a.qk_pad + pc * 8 : 0), ok);
  }
#pragma unroll
  for (int i = 0; i < STAGES - 1; ++i) {
    if (t0 + i < t1) {
      const uint32_t sk = skv + i * CfgTile<DQ, DV>::STAGE;
      load_kv_tile<DQ, DV>(a, bt, whole, g, tiles.at(t0 + i), p, sk, sk + BN * DQ * 2);
    }
    b2::cp_async_commit();
  }
  const int pos[2] = {p, p};
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float o[DV / 8][4];
#pragma unroll
  for (int n = 0; n < DV / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
  for (int t = t0; t < t1; ++t) {
    const uint32_t sk = skv + ((t - t0) % STAGES) * CfgTile<DQ, DV>::STAGE, sv = sk + BN * DQ * 2;
    b2::cp_async_wait<STAGES - 2>();
    __syncthreads();
    if (t + STAGES - 1 < t1) {
      const uint32_t nk = skv + ((t - t0 + STAGES - 1) % STAGES) * CfgTile<DQ, DV>::STAGE;
      load_kv_tile<DQ, DV>(a, bt, whole, g, tiles.at(t + STAGES - 1), p, nk, nk + BN * DQ * 2);
    }
    b2::cp_async_commit();
    const int j0 = tiles.at(t) * BN + warp * 16;  // this warp's 16 keys
    float s[2][4] = {};
#pragma unroll
    for (int k = 0; k < DQ / 16; ++k) {
      uint32_t qa[4], kb[4];
      b2::frag_a<DQ>(sq, 0, k * 16, lane, qa);
      b2::frag_b<DQ>(sk, warp * 16, k * 16, lane, kb);
      b2::mma16816(s[0], qa, kb[0], kb[1]);
      b2::mma16816(s[1], qa, kb[2], kb[3]);
    }
    float corr[2];
    softmax_tile<2, CAP>(a, sscale, s, j0, pos, j0 + 15 > p || (p - j0 >= a.window && j0 + 15 >= a.keep_first), m, l, corr, lane);
#pragma unroll
    for (int n = 0; n < DV / 8; ++n) {
      o[n][0] *= corr[0]; o[n][1] *= corr[0]; o[n][2] *= corr[1]; o[n][3] *= corr[1];
    }
    uint32_t hi[4], lo[4];
    b2::split_bf16(s[0][0], s[0][1], hi[0], lo[0]);
    b2::split_bf16(s[0][2], s[0][3], hi[1], lo[1]);
    b2::split_bf16(s[1][0], s[1][1], hi[2], lo[2]);
    b2::split_bf16(s[1][2], s[1][3], hi[3], lo[3]);
#pragma unroll
    for (int n = 0; n < DV / 16; ++n) {
      uint32_t vb[4];
      b2::frag_b_t<DV>(sv, n * 16, warp * 16, lane, vb);
      b2::mma16816(o[2 * n], hi, vb[0], vb[1]);
      b2::mma16816(o[2 * n + 1], hi, vb[2], vb[3]);
      b2::mma16816(o[2 * n], lo, vb[0], vb[1]);
      b2::mma16816(o[2 * n + 1], lo, vb[2], vb[3]);
    }
  }
  b2::cp_async_wait<0>();
  __syncthreads();  // the stages become the combine buffer
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    const int r = (lane >> 2) + h * 8;
    if ((lane & 3) == 0) {
      s_ml[warp][r][0] = m[h];
      s_ml[warp][r][1] = l[h];
    }
#pragma unroll
    for (int n = 0; n < DV / 8; ++n)
      *reinterpret_cast<float2*>(o_buf + (warp * 16 + r) * DV + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * h], o[n][2 * h + 1]);
  }
  __syncthreads();
  const int group = (b * a.nkv + g) * row_tiles + blockIdx.y % row_tiles;
  float* my = part + (static_cast<int64_t>(group) * splits + split) * 16 * (DV + 2);
  for (int idx = threadIdx.x; idx < nrows * DV; idx += 128) {
    const int r = idx / DV, c = idx % DV;
    float mt = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mt = fmaxf(mt, s_ml[w][r][0]);
    float lt = 0.f, ot = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = s_ml[w][r][0] == -INFINITY ? 0.f : fast_exp2(s_ml[w][r][0] - mt);
      lt += f * s_ml[w][r][1];
      ot += f * o_buf[(w * 16 + r) * DV + c];
    }
    if (splits == 1) {
      if (a.sink != nullptr) {
        const float sk = a.sink[g * rep + h0 + r] * LOG2E, m_new = fmaxf(mt, sk);
        const float f = fast_exp2(mt - m_new);
        lt = lt * f + fast_exp2(sk - m_new);
        ot *= f;
      }
      if (c < a.v_pad) out[r * a.v_pad + c] = b2::from_float<uint16_t>(ot / lt);
    } else {
      my[32 + r * DV + c] = ot;
      if (c == 0) {
        my[r] = mt;
        my[16 + r] = lt;
      }
    }
  }
  if (splits == 1) return;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(counters + group, 1) == splits - 1;
  __syncthreads();
  if (!s_last) return;
  if (threadIdx.x == 0) counters[group] = 0;
  __threadfence();
  const float* all = part + static_cast<int64_t>(group) * splits * 16 * (DV + 2);
  if (threadIdx.x < nrows) {  // the rows' maximum over the splits, and the denominator
    const int r = threadIdx.x;
    const float sk = a.sink != nullptr ? a.sink[g * rep + h0 + r] * LOG2E : -INFINITY;
    float mt = sk;
    for (int s = 0; s < splits; ++s) mt = fmaxf(mt, b2::ld_cg_f32(all + static_cast<int64_t>(s) * 16 * (DV + 2) + r));
    float lt = fast_exp2(sk - mt);
    for (int s = 0; s < splits; ++s) {
      const float* ps = all + static_cast<int64_t>(s) * 16 * (DV + 2);
      const float ms = b2::ld_cg_f32(ps + r);
      if (ms > -INFINITY) lt += fast_exp2(ms - mt) * b2::ld_cg_f32(ps + 16 + r);
    }
    s_fin[r][0] = mt;
    s_fin[r][1] = 1.0f / lt;
  }
  __syncthreads();
  for (int idx = threadIdx.x; idx < nrows * DV; idx += 128) {
    const int r = idx / DV, c = idx % DV;
    float ot = 0.f;
    for (int s = 0; s < splits; ++s) {
      const float* ps = all + static_cast<int64_t>(s) * 16 * (DV + 2);
      const float ms = b2::ld_cg_f32(ps + r);
      if (ms > -INFINITY) ot += fast_exp2(ms - s_fin[r][0]) * b2::ld_cg_f32(ps + 32 + r * DV + c);
    }
    if (c < a.v_pad) out[r * a.v_pad + c] = b2::from_float<uint16_t>(ot * s_fin[r][1]);
  }
}

bool tiled_form(int dtype, int qk_pad, int v_pad) { return dtype == B2_DT_BF16 && qk_pad <= 128 && v_pad <= 128; }

// CTAs a decode step's keys are dealt to, per (sequence, key/value head, 16 query heads)
int decode_splits(int B, int max_kv, int nq, int nkv, int window, int keep_first) {
  const int64_t groups = static_cast<int64_t>(B) * nkv * ((nq / nkv + 15) / 16);
  const int64_t all = (static_cast<int64_t>(max_kv) + BN - 1) / BN;
  const int64_t seen = (static_cast<int64_t>(keep_first) + BN - 1) / BN + (static_cast<int64_t>(window) + BN - 2) / BN + 1;
  const int64_t tiles = std::max<int64_t>(1, std::min(all, seen));
  // two CTAs per SM fit: about four rounds of them, so that the last one is short; a CTA should have several tiles
  const int64_t want = (4 * 2 * 148 + groups - 1) / groups;
  return static_cast<int>(std::max<int64_t>(1, std::min({want, tiles / 4, static_cast<int64_t>(DEC_MAX_SPLITS)})));
}

template <int DQ, int DV, int CAP>
int launch_tiled_cap(const AttnArgs& a, int max_q, int max_kv, void* ws, int64_t ws_bytes, cudaStream_t s) {
  using C = CfgTile<DQ, DV>;
  const int rep = a.nq / a.nkv;
  const bool whole = a.block_size % BN == 0;
  if (a.cu_q != nullptr) {
    static const cudaError_t set = cudaFuncSetAttribute(attn_prefill_kernel<DQ, DV, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_PREFILL);
    B2_CUDA(set);
    const int64_t tiles = (static_cast<int64_t>(max_q) * rep + 63) / 64;
    B2_CUDA(b2_launch(attn_prefill_kernel<DQ, DV, CAP>, dim3(static_cast<unsigned>(tiles), a.nkv, a.B), dim3(128), C::SMEM_PREFILL, s, a, rep, whole));
    return B2_OK;
  }
  static const cudaError_t set = cudaFuncSetAttribute(attn_decode_kernel<DQ, DV, CAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM_DECODE);
  B2_CUDA(set);
  const int row_tiles = (rep + 15) / 16;
  const int64_t groups = static_cast<int64_t>(a.B) * a.nkv * row_tiles;
  int splits = decode_splits(a.B, max_kv, a.nq, a.nkv, a.window, a.keep_first);
  const int64_t need = DEC_MAX_GROUPS * 4ll + groups * splits * 16 * (DV + 2) * 4;
  if (groups > DEC_MAX_GROUPS) splits = 1;
  if (splits > 1 && (ws == nullptr || ws_bytes < need)) return b2::set_error(B2_ERR_SHAPE, "b2_attention: workspace of %lld bytes, %lld needed",
                                                                             static_cast<long long>(ws_bytes), static_cast<long long>(need));
  B2_CUDA(b2_launch(attn_decode_kernel<DQ, DV, CAP>, dim3(splits, a.nkv * row_tiles, a.B), dim3(128), C::SMEM_DECODE, s, a, rep, row_tiles, whole,
                    splits, static_cast<int*>(ws), reinterpret_cast<float*>(static_cast<unsigned char*>(ws) + DEC_MAX_GROUPS * 4ll)));
  return B2_OK;
}

template <int DQ, int DV>
int launch_tiled(const AttnArgs& a, int max_q, int max_kv, void* ws, int64_t ws_bytes, cudaStream_t s) {
  if (!(a.softcap > 0.f)) return launch_tiled_cap<DQ, DV, CAP_NONE>(a, max_q, max_kv, ws, ws_bytes, s);
  if (a.softcap <= 256.f) return launch_tiled_cap<DQ, DV, CAP_SHORT>(a, max_q, max_kv, ws, ws_bytes, s);
  return launch_tiled_cap<DQ, DV, CAP_FULL>(a, max_q, max_kv, ws, ws_bytes, s);
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
  if (max_q > 1 || B <= 0 || nkv <= 0 || nq < nkv || !tiled_form(dtype, qk_pad, v_pad)) return 0;
  const int64_t groups = static_cast<int64_t>(B) * nkv * ((nq / nkv + 15) / 16);
  const int splits = decode_splits(B, max_kv, nq, nkv, window, keep_first);
  return splits > 1 ? DEC_MAX_GROUPS * 4ll + groups * splits * 16 * ((v_pad <= 64 ? 64 : 128) + 2) * 4 : 0;
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
  a.B = B; a.nq = nq; a.nkv = nkv; a.qk_pad = qk_pad; a.v_pad = v_pad; a.k_row = qk_pad; a.v_row = v_pad; a.window = window; a.keep_first = keep_first;
  a.scale = scale; a.softcap = softcap; a.sink = sink;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_F32) return launch_any<float>(a, max_q, s);
  if (form == 1 || !tiled_form(dtype, qk_pad, v_pad)) return launch_any<uint16_t>(a, max_q, s);
  if (qk_pad <= 64) return v_pad <= 64 ? launch_tiled<64, 64>(a, max_q, max_kv, workspace, workspace_bytes, s)
                                       : launch_tiled<64, 128>(a, max_q, max_kv, workspace, workspace_bytes, s);
  return v_pad <= 64 ? launch_tiled<128, 64>(a, max_q, max_kv, workspace, workspace_bytes, s)
                     : launch_tiled<128, 128>(a, max_q, max_kv, workspace, workspace_bytes, s);
}

}  // extern "C"
