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
//   latent_tc_kernel       absorbed attention on tcgen05: 16 or 32 (token, head) rows, 128 keys per tile
//   latent_combine_kernel  the parts of its key ranges
// (The expanded form is in b2_expanded.cu.)
#include <algorithm>

#include "b2_attn.cuh"

namespace {

using namespace b2;

// ---------------------------------------------------------------------------
// Rows [q latent | latent | rotated part | ...] in place; [latent | rotated part] also to the cache.  One warp per
// (token, part).
// ---------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ void warp_rms(const T* src, int dim, int pad, const float* w, float eps, int lane, T* dst0, T* dst1) {
  constexpr int KEEP = sizeof(T) == 2 ? 6 : 3;  // vectors of 8 a lane keeps in registers; longer rows are read again
  float f[KEEP][8], ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[i][e] = 0.f;
    const int c = (lane + 32 * i) * 8;
    if (c < pad) load8<T>(src + c, f[i]);
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += f[i][e] * f[i][e];
  for (int c = (lane + 32 * KEEP) * 8; c < pad; c += 256) {
    float g[8];
    load8<T>(src + c, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += g[e] * g[e];
  }
  ss = group_sum(ss);
  const float rstd = 1.0f / sqrtf(ss / static_cast<float>(dim) + eps);
  auto finish = [&](int c, float (&v)[8]) {
    float g[8];
    load8<float>(w + c, g);
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] = v[e] * rstd * g[e];
    store8<T>(dst0 + c, v);
    if (dst1 != nullptr) store8<T>(dst1 + c, v);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i)
    if ((lane + 32 * i) * 8 < pad) finish((lane + 32 * i) * 8, f[i]);
  for (int c = (lane + 32 * KEEP) * 8; c < pad; c += 256) {
    float g[8];
    load8<T>(src + c, g);
    finish(c, g);
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

// Output tiles of 64 x NT; K in steps of 64, STAGES of them in flight
template <bool KN, int STAGES>
struct CfgHeads {
  static constexpr int NT = KN ? 64 : 32;
  static constexpr int A_BYTES = 64 * 64 * 2, STAGE = A_BYTES + 64 * NT * 2;
  static constexpr int SMEM = STAGES * STAGE + 128;
};
template <bool KN, int STAGES>
__global__ void __launch_bounds__(128) heads_gemm_kernel(const HeadsArgs a) {
  using C = CfgHeads<KN, STAGES>;
  constexpr int NT = C::NT;
  extern __shared__ unsigned char smem_raw[];
  const uint32_t base = (smem_u32(smem_raw) + 127) & ~127u;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * NT, m0 = blockIdx.y * 64, h = blockIdx.z;
  pdl_launch_dependents();
  const uint16_t* x = static_cast<const uint16_t*>(a.x) + static_cast<int64_t>(h) * a.x_hs;
  const uint16_t* w = static_cast<const uint16_t*>(a.w) + h * a.w_hs;
  auto load_w = [&](int st, int k0) {
    const uint32_t sw = base + st * C::STAGE + C::A_BYTES;
#pragma unroll
    for (int i = 0; i < NT / 16; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx >> 3, p = idx & 7;
      const int wr = (KN ? k0 : n0) + r, wc = (KN ? n0 : k0) + p * 8;
      const bool ok = wr < (KN ? a.K : a.N) && wc < (KN ? a.N : a.K);
      cp_async16(tile_addr<64>(sw, r, p), ok ? w + wr * a.ldw + wc : w, ok);
    }
  };
  auto load_x = [&](int st, int k0) {
    const uint32_t sa = base + st * C::STAGE;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx >> 3, p = idx & 7;
      const bool ok = m0 + r < a.M && k0 + p * 8 < a.K;
      cp_async16(tile_addr<64>(sa, r, p), ok ? x + (m0 + r) * a.ldx + k0 + p * 8 : x, ok);
    }
  };
  const bool product = n0 < a.N;
  // weights do not depend on an earlier kernel: the first ones are fetched before the wait
  if (product)
    for (int i = 0; i < STAGES && i * 64 < a.K; ++i) load_w(i, i * 64);
  pdl_wait();
  if (!product) {
    rotate_rows<uint16_t>(a, m0, h);
    return;
  }
  for (int i = 0; i < STAGES; ++i) {
    if (i * 64 < a.K) load_x(i, i * 64);
    cp_async_commit();
  }
  float acc[NT / 8][4];
#pragma unroll
  for (int n = 0; n < NT / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
  for (int k0 = 0, st = 0; k0 < a.K; k0 += 64, st = st + 1 == STAGES ? 0 : st + 1) {
    cp_async_wait<STAGES - 1>();
    __syncthreads();  // this step has landed for everyone
    const uint32_t sa = base + st * C::STAGE, sw = sa + C::A_BYTES;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t qa[4];
      frag_a<64>(sa, warp * 16, k * 16, lane, qa);
#pragma unroll
      for (int n = 0; n < NT / 16; ++n) {
        uint32_t kb[4];
        if (KN) frag_b_t<64>(sw, n * 16, k * 16, lane, kb);
        else frag_b<64>(sw, n * 16, k * 16, lane, kb);
        mma16816(acc[2 * n], qa, kb[0], kb[1]);
        mma16816(acc[2 * n + 1], qa, kb[2], kb[3]);
      }
    }
    if (k0 + 64 * STAGES < a.K) {
      __syncthreads();  // everyone has left the stage
      load_w(st, k0 + 64 * STAGES);
      load_x(st, k0 + 64 * STAGES);
    }
    cp_async_commit();
  }
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int m = m0 + warp * 16 + (lane >> 2) + e * 8;
    if (m >= a.M) continue;
    uint16_t* dst = static_cast<uint16_t*>(a.out) + m * a.ldo + static_cast<int64_t>(h) * a.out_hs;
    const uint16_t* g = a.gate != nullptr ? static_cast<const uint16_t*>(a.gate) + m * a.ldg + static_cast<int64_t>(h) * a.gate_hs : nullptr;
#pragma unroll
    for (int n = 0; n < NT / 8; ++n) {
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

template <bool KN, int STAGES>
int launch_heads(const HeadsArgs& a, int heads, cudaStream_t s) {
  using C = CfgHeads<KN, STAGES>;
  static const cudaError_t set = cudaFuncSetAttribute(heads_gemm_kernel<KN, STAGES>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM);
  B2_CUDA(set);
  const dim3 grid((a.N + C::NT - 1) / C::NT + (a.rot_pad > 0 ? 1 : 0), (a.M + 63) / 64, heads);
  B2_CUDA(b2_launch(heads_gemm_kernel<KN, STAGES>, grid, dim3(128), C::SMEM, s, a));
  return B2_OK;
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
// Absorbed attention on tcgen05.  A CTA holds NR (token, head) rows and walks key tiles of 128 cached rows, which TMA brings
// into shared memory as boxes of 128 keys x 64 columns.  Both products have the big operand on the 128-row side:
//   scores   S^T [128 keys x NR]   = rows (K-major)           x Q^T
//   outputs  O^T [128 dims x NR]  += latents^T (M contiguous) x P^T, one accumulator per 128 latent columns
// from the same boxes.  Warps 0-3: softmax, a thread per key; the weights go back through shared memory as a sum of two bf16
// numbers that lie side by side in the N dimension of one product.  Warp 4: TMA.  Warp 5: MMA.  Key tiles are dealt to
// `splits` CTAs; a second kernel combines their parts.
// ---------------------------------------------------------------------------
constexpr int LT_KEYS = 128;                 // keys per tile
constexpr int LT_BOX = LT_KEYS * 64 * 2;     // bytes of one box
constexpr int LT_THREADS = 192;
constexpr int LT_MAX_PAIRS = 4;              // latents up to 512 wide
constexpr int LT_MAX_STAGES = 3;
constexpr int LT_MAX_SPLITS = 64;
constexpr uint64_t LT_LIMIT_NS = 1000000000ull;
constexpr int LT_SMEM_MAX = 227 * 1024, LT_SMEM_STATIC = 2048;  // per CTA, and what of it the kernel declares statically
constexpr float LT_RESCALE = 8.0f;           // the running maximum may be exceeded by 2^8 before the outputs are rescaled

struct LatentTcArgs {
  uint16_t* out;
  int64_t ldo;
  const int32_t* block_tables;
  int64_t bt_stride;
  int block_size;
  const int32_t* cu_q;
  const int32_t* kv_len;
  int heads, v_pad, boxes, rot;  // boxes: 64-column boxes of the latent; rot: 1 = there is a rotated part
  int stages, row_tiles, splits;
  float scale;
  const float* sink;
  float* part;  // [group][split]: maxima [NR], sums [NR], outputs [NR / 4][128 pairs][4 rows]
  B2Status* status;
};
__host__ __device__ constexpr int64_t latent_part_floats(int nr, int pairs) { return 2 * nr + static_cast<int64_t>(nr) * 128 * pairs; }

// v over the warp's 32 lanes, one result per column: lane l gets column l & (NR - 1).  Destroys v.
template <int NR, typename Op>
__device__ __forceinline__ float reduce_columns(float (&v)[NR], int lane, Op op) {
  if (NR == 16) {
#pragma unroll
    for (int j = 0; j < NR; ++j) v[j] = op(v[j], __shfl_xor_sync(0xffffffffu, v[j], 16));
  }
#pragma unroll
  for (int o = NR / 2; o >= 1; o >>= 1) {
    const bool upper = (lane & o) != 0;
#pragma unroll
    for (int j = 0; j < o; ++j) {
      const float send = upper ? v[j] : v[j + o], keep = upper ? v[j + o] : v[j];
      v[j] = op(keep, __shfl_xor_sync(0xffffffffu, send, o));
    }
  }
  return v[0];
}
// all 128 softmax threads meet; true when every one brought true
__device__ __forceinline__ bool softmax_meet(bool ok) {
  uint32_t r;
  asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbarrier.cta.red.and.pred q, 1, 128, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
               : "=r"(r) : "r"(static_cast<uint32_t>(ok)) : "memory");
  return r != 0;
}
template <int NR>
__device__ __forceinline__ void tmem_load(uint32_t addr, uint32_t (&r)[NR]) {
  if constexpr (NR == 32) tmem_ld_32x32(addr, r);
  else tmem_ld_32x16(addr, r);
  tc_wait_ld();
}

template <int NR>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_tc_kernel(const __grid_constant__ CUtensorMap tm_lat, const __grid_constant__ CUtensorMap tm_rot, const __grid_constant__ CUtensorMap tm_ql,
                 const __grid_constant__ CUtensorMap tm_qr, const LatentTcArgs a) {
  constexpr uint32_t TMEM_COLS = NR == 32 ? 512 : 256;  // S^T: NR columns, O^T: 2 NR (leading and trailing parts) per pair of boxes
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t s_bars[2 * LT_MAX_STAGES * (LT_MAX_PAIRS + 1) + 4];
  __shared__ float s_red[4][32];
  __shared__ int64_t s_out[NR];  // offset of every row's output
  __shared__ int s_pos[NR];      // its position
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  volatile int* abort_flag = &s_abort;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int pairs = (a.boxes + 1) >> 1, stage_bytes = (2 * pairs + a.rot) * LT_BOX;
  const uint32_t q_bytes = (a.boxes + a.rot) * NR * 128;
  const uint32_t sq = (smem_u32(smem_raw) + 1023u) & ~1023u;
  const uint32_t sp = sq + ((q_bytes + 1023u) & ~1023u);  // P: [two halves of 64 keys][NR leading, NR trailing rows of 128 bytes]
  const uint32_t sk = sp + NR * 512;
  const uint32_t bar_full = smem_u32(s_bars), bar_empty = bar_full + LT_MAX_STAGES * (LT_MAX_PAIRS + 1) * 8;
  const uint32_t bar_q = bar_empty + LT_MAX_STAGES * (LT_MAX_PAIRS + 1) * 8, bar_s = bar_q + 8, bar_p = bar_q + 16, bar_o = bar_q + 24;
  const auto full = [&](int st, int i) { return bar_full + (st * (LT_MAX_PAIRS + 1) + i) * 8; };
  const auto empty = [&](int st, int i) { return bar_empty + (st * (LT_MAX_PAIRS + 1) + i) * 8; };
  if (threadIdx.x == 0) {
    for (int i = 0; i < LT_MAX_STAGES * (LT_MAX_PAIRS + 1); ++i) {
      mbar_init(bar_full + i * 8, 1);
      mbar_init(bar_empty + i * 8, 1);
    }
    mbar_init(bar_q, 1);
    mbar_init(bar_s, 1);
    mbar_init(bar_p, 4);
    mbar_init(bar_o, 1);
    s_abort = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_lat);
    tma_prefetch_desc(&tm_rot);
    tma_prefetch_desc(&tm_ql);
    tma_prefetch_desc(&tm_qr);
  }
  if (warp == 5) {
    tmem_alloc(smem_u32(&s_tmem), TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm_s = s_tmem, tm_o = s_tmem + NR;
  pdl_launch_dependents();  // only now: a later kernel must not take the tensor memory that a CTA of this one still needs
  pdl_wait();

  const int b = blockIdx.z, split = blockIdx.x, r_base = blockIdx.y * NR;
  const int row0 = a.cu_q ? a.cu_q[b] : b;
  const int n_q = a.cu_q ? a.cu_q[b + 1] - row0 : 1;
  const int rows = n_q * a.heads, klen = a.kv_len[b];
  const int nrows = max(0, min(NR, rows - r_base));
  const int first_pos = klen - n_q;
  const int pmin = first_pos + r_base / a.heads, pmax = first_pos + (r_base + max(nrows, 1) - 1) / a.heads;
  const int total = nrows > 0 && klen > 0 ? pmax / LT_KEYS + 1 : 0, per = (total + a.splits - 1) / a.splits;
  const int t0 = split * per, t1 = min(total, t0 + per);

  if (warp == 4) {
    // ---------------- TMA ----------------
    if (lane == 0 && t0 < t1) {
      mbar_arrive_expect_tx(bar_q, q_bytes);
      const int qrow = row0 * a.heads + r_base;
      for (int i = 0; i < a.boxes; ++i) tma_load_2d(sq + i * NR * 128, &tm_ql, bar_q, i * 64, qrow, kEvictFirst);
      if (a.rot) tma_load_2d(sq + a.boxes * NR * 128, &tm_qr, bar_q, 0, qrow, kEvictFirst);
      int st = 0;
      uint32_t phase = 0;
      const int per_block = a.block_size / LT_KEYS;
      bool ok = true;
      for (int t = t0; ok && t < t1; ++t) {
        const int slot = a.block_tables[b * a.bt_stride + t / per_block] * a.block_size + (t % per_block) * LT_KEYS;
        const uint32_t base = sk + st * stage_bytes;
        if (a.rot) {  // free first, read first
          if (!(ok = mbar_wait(empty(st, pairs), phase ^ 1, abort_flag, LT_LIMIT_NS, B2_WAIT_SMEM_EMPTY))) break;
          mbar_arrive_expect_tx(full(st, pairs), LT_BOX);
          tma_load_2d(base + 2 * pairs * LT_BOX, &tm_rot, full(st, pairs), 0, slot, kEvictNormal);
        }
        for (int p = 0; p < pairs; ++p) {
          if (!(ok = mbar_wait(empty(st, p), phase ^ 1, abort_flag, LT_LIMIT_NS, B2_WAIT_SMEM_EMPTY))) break;
          const int n = min(2, a.boxes - 2 * p);
          mbar_arrive_expect_tx(full(st, p), n * LT_BOX);
          for (int i = 0; i < n; ++i) tma_load_2d(base + (2 * p + i) * LT_BOX, &tm_lat, full(st, p), (2 * p + i) * 64, slot, kEvictNormal);
        }
        if (++st == a.stages) { st = 0; phase ^= 1; }
      }
    }
  } else if (warp == 5) {
    // ---------------- MMA ----------------
    if (lane == 0 && t0 < t1) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(NR), idesc_o = umma_idesc_bf16(2 * NR) | UMMA_A_MN;
      int st = 0;
      uint32_t phase = 0;
      bool ok = mbar_wait(bar_q, 0, abort_flag, LT_LIMIT_NS, B2_WAIT_SMEM_FULL);
      for (int t = t0; ok && t < t1; ++t) {
        const uint32_t base = sk + st * stage_bytes;
        const auto scores = [&](int box, bool first) {
          const uint64_t dk = umma_smem_desc(base + box * LT_BOX), dq = umma_smem_desc(sq + (box < a.boxes ? box : a.boxes) * NR * 128);
#pragma unroll
          for (int k = 0; k < 4; ++k) umma_bf16(tm_s, dk + 2 * k, dq + 2 * k, idesc_s, (first && k == 0) ? 0u : 1u);
        };
        bool first = true;
        if (a.rot) {
          if (!(ok = mbar_wait(full(st, pairs), phase, abort_flag, LT_LIMIT_NS, B2_WAIT_SMEM_FULL))) break;
          tc_fence_after();
          scores(2 * pairs, true);
          first = false;
          umma_commit(empty(st, pairs));
        }
        for (int p = 0; p < pairs; ++p) {
          if (!(ok = mbar_wait(full(st, p), phase, abort_flag, LT_LIMIT_NS, B2_WAIT_SMEM_FULL))) break;
          tc_fence_after();
          for (int i = 2 * p; i < min(a.boxes, 2 * p + 2); ++i) {
            scores(i, first);
            first = false;
          }
        }
        if (!ok) break;
        umma_commit(bar_s);  // also says that the outputs of the previous tile are complete
        if (!(ok = mbar_wait(bar_p, (t - t0) & 1, abort_flag, LT_LIMIT_NS, B2_WAIT_TMEM_EMPTY))) break;
        tc_fence_after();
        for (int p = 0; p < pairs; ++p) {
#pragma unroll
          for (int k = 0; k < LT_KEYS / 16; ++k) {
            const uint64_t dv = umma_smem_desc_mn(base + 2 * p * LT_BOX + k * 2048, LT_BOX);
            const uint64_t dp = umma_smem_desc(sp + (k >> 2) * NR * 256) + 2 * (k & 3);
            umma_bf16(tm_o + p * 2 * NR, dv, dp, idesc_o, (t > t0 || k > 0) ? 1u : 0u);
          }
          umma_commit(empty(st, p));
        }
        if (++st == a.stages) { st = 0; phase ^= 1; }
      }
      if (ok) umma_commit(bar_o);
    }
  } else {
    // ---------------- softmax: thread = key of the tile ----------------
    const uint32_t lanes = static_cast<uint32_t>(warp * 32) << 16;
    const int col = lane & (NR - 1);  // the row whose maximum, sum and factors this lane keeps
    const float scale = a.scale * LOG2E;
    if (threadIdx.x < NR) {
      const int gr = r_base + min(static_cast<int>(threadIdx.x), max(nrows, 1) - 1), tok = gr / a.heads;
      s_pos[threadIdx.x] = first_pos + tok;
      s_out[threadIdx.x] = (row0 + tok) * a.ldo + static_cast<int64_t>(gr - tok * a.heads) * a.v_pad;
    }
    softmax_meet(true);
    float m_col = -INFINITY;
    float l[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) l[r] = 0.f;
    bool ok = true;
    for (int t = t0; ok && t < t1; ++t) {
      ok = mbar_wait(bar_s, (t - t0) & 1, abort_flag, LT_LIMIT_NS, B2_WAIT_TMEM_FULL);
      __syncwarp();
      tc_fence_after();
      uint32_t raw[NR];
      tmem_load<NR>(tm_s + lanes, raw);
      float v[NR], w[NR];
#pragma unroll
      for (int r = 0; r < NR; ++r) v[r] = __uint_as_float(raw[r]) * scale;
      if (t * LT_KEYS + LT_KEYS - 1 > pmin) {
        const int j = t * LT_KEYS + threadIdx.x;
#pragma unroll
        for (int r = 0; r < NR; ++r)
          if (j > s_pos[r]) v[r] = -INFINITY;
      }
#pragma unroll
      for (int r = 0; r < NR; ++r) w[r] = v[r];
      s_red[warp][lane] = reduce_columns<NR>(w, lane, [](float x, float y) { return fmaxf(x, y); });
      if (!(ok = softmax_meet(ok))) break;
      const float m_tile = fmaxf(fmaxf(s_red[0][col], s_red[1][col]), fmaxf(s_red[2][col], s_red[3][col]));
      const bool grow = m_tile > m_col + LT_RESCALE || m_col == -INFINITY;
      const float m_new = grow ? fmaxf(m_tile, m_col) : m_col;
      const float corr = grow && m_col > -INFINITY ? fast_exp2(m_col - m_new) : 1.0f;
      if (__any_sync(0xffffffffu, corr != 1.0f)) {  // the same in all four warps; never in the first tile
#pragma unroll
        for (int r = 0; r < NR; ++r) l[r] *= __shfl_sync(0xffffffffu, corr, r);
        for (int p = 0; p < 2 * pairs; ++p) {
          tmem_load<NR>(tm_o + p * NR + lanes, raw);
#pragma unroll
          for (int r = 0; r < NR; ++r) raw[r] = __float_as_uint(__uint_as_float(raw[r]) * __shfl_sync(0xffffffffu, corr, r));
#pragma unroll
          for (int h = 0; h < NR / 16; ++h) {
            uint32_t part[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) part[i] = raw[16 * h + i];
            tmem_st_32x16(tm_o + p * NR + 16 * h + lanes, part);
          }
        }
        tc_wait_st();
      }
      m_col = m_new;
      const float ref = m_col == -INFINITY ? 0.f : m_col;
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        v[r] = fast_exp2(v[r] - __shfl_sync(0xffffffffu, ref, r));
        l[r] += v[r];
      }
      // neighbours exchange: an even lane stores row r of keys (lane, lane + 1), an odd one row r + 1
      const int odd = lane & 1, key2 = (warp & 1) * 32 + (lane & ~1);  // first of the two keys inside the half tile
      const uint32_t at = sp + (warp >> 1) * NR * 256 + (key2 & 7) * 2;
#pragma unroll
      for (int r = 0; r < NR; r += 2) {
        const float other = __shfl_xor_sync(0xffffffffu, odd ? v[r] : v[r + 1], 1);
        const int rr = r + odd;
        uint32_t hi, lo;
        split_bf16(odd ? other : v[r], odd ? v[r + 1] : other, hi, lo);
        const uint32_t dst = at + rr * 128 + (((key2 >> 3) ^ (rr & 7)) << 4);  // NR is a multiple of 8: the same for both parts
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst), "r"(hi) : "memory");
        asm volatile("st.shared.u32 [%0], %1;" ::"r"(dst + NR * 128), "r"(lo) : "memory");
      }
      fence_proxy_async();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_p);
    }
    if (ok && t0 < t1) ok = mbar_wait(bar_o, 0, abort_flag, LT_LIMIT_NS, B2_WAIT_TMEM_FULL);
    __syncwarp();
    tc_fence_after();
    s_red[warp][lane] = reduce_columns<NR>(l, lane, [](float x, float y) { return x + y; });
    ok = softmax_meet(ok);
    if (ok && nrows > 0) {
      const float l_col = s_red[0][col] + s_red[1][col] + s_red[2][col] + s_red[3][col];
      float* my = a.part + (static_cast<int64_t>(b * a.row_tiles + blockIdx.y) * a.splits + split) * latent_part_floats(NR, pairs);
      float f = 0.f;
      if (a.splits > 1) {
        if (warp == 0 && lane < NR) {
          my[lane] = m_col;
          my[NR + lane] = l_col;
        }
      } else if (klen > 0) {
        const float sk_ = a.sink != nullptr ? a.sink[(r_base + col) % a.heads] * LOG2E : -INFINITY, m_new = fmaxf(m_col, sk_);
        f = fast_exp2(m_col - m_new);
        f /= l_col * f + fast_exp2(sk_ - m_new);
      }
      if (t0 < t1 || a.splits == 1) {
        for (int p = 0; p < pairs; ++p) {
          uint32_t raw[NR], low[NR];
          float o[NR];
          if (t0 < t1) {
            tmem_load<NR>(tm_o + p * 2 * NR + lanes, raw);
            tmem_load<NR>(tm_o + p * 2 * NR + NR + lanes, low);
          }
#pragma unroll
          for (int r = 0; r < NR; ++r) o[r] = t0 < t1 ? __uint_as_float(raw[r]) + __uint_as_float(low[r]) : 0.f;  // nothing seen: a padded row
          const int dim = p * 128 + threadIdx.x;
          if (a.splits > 1) {
#pragma unroll
            for (int r = 0; r < NR; r += 4)
              *reinterpret_cast<float4*>(my + 2 * NR + ((r >> 2) * 128 * pairs + dim) * 4) = make_float4(o[r], o[r + 1], o[r + 2], o[r + 3]);
          } else {
#pragma unroll
            for (int r = 0; r < NR; ++r) {
              const float x = o[r] * __shfl_sync(0xffffffffu, f, r);
              if (r < nrows && dim < a.v_pad) a.out[s_out[r] + dim] = from_float<uint16_t>(x);
            }
          }
        }
      }
    }
  }
  __syncwarp();
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (s_abort) {  // let bulk copies that may still be in flight land before the CTA leaves
    for (int i = 0; i < 100; ++i) __nanosleep(2000);
    if (threadIdx.x == 0) report_timeout(a.status, s_abort);
  }
  if (warp == 5) tmem_dealloc(s_tmem, TMEM_COLS);
}

// The splits' parts of 4 rows -> their outputs.  One thread per latent column.
template <int NR>
__global__ void __launch_bounds__(512) latent_combine_kernel(const LatentTcArgs a) {
  __shared__ float s_fac[4][LT_MAX_SPLITS];
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.z, r_base = blockIdx.y * NR, r4 = blockIdx.x;
  const int row0 = a.cu_q ? a.cu_q[b] : b;
  const int rows = (a.cu_q ? a.cu_q[b + 1] - row0 : 1) * a.heads;
  if (r_base + r4 * 4 >= rows) return;
  const int pairs = (a.boxes + 1) >> 1, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t floats = latent_part_floats(NR, pairs);
  const float* all = a.part + static_cast<int64_t>(b * a.row_tiles + blockIdx.y) * a.splits * floats;
  const bool live = a.kv_len[b] > 0;
  if (warp < 4) {  // a warp per row: the factors of its parts
    const int r = r4 * 4 + warp;
    const float sk = a.sink != nullptr ? a.sink[(r_base + r) % a.heads] * LOG2E : -INFINITY;
    float ms[LT_MAX_SPLITS / 32], ls[LT_MAX_SPLITS / 32], top = sk, sum = 0.f;
#pragma unroll
    for (int i = 0; i < LT_MAX_SPLITS / 32; ++i) {
      const int s = lane + 32 * i;
      ms[i] = s < a.splits && live ? all[s * floats + r] : -INFINITY;
      ls[i] = s < a.splits && live ? all[s * floats + NR + r] : 0.f;
      top = fmaxf(top, ms[i]);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
#pragma unroll
    for (int i = 0; i < LT_MAX_SPLITS / 32; ++i) {
      ms[i] = ms[i] > -INFINITY ? fast_exp2(ms[i] - top) : 0.f;
      sum += ms[i] * ls[i];
    }
    sum = group_sum(sum) + (sk > -INFINITY ? fast_exp2(sk - top) : 0.f);
#pragma unroll
    for (int i = 0; i < LT_MAX_SPLITS / 32; ++i)
      if (lane + 32 * i < a.splits) s_fac[warp][lane + 32 * i] = sum > 0.f ? ms[i] / sum : 0.f;
  }
  __syncthreads();
  const int dim = threadIdx.x;
  if (dim >= a.v_pad) return;
  float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
  for (int s = 0; s < a.splits; ++s) {
    const float f[4] = {s_fac[0][s], s_fac[1][s], s_fac[2][s], s_fac[3][s]};
    if (f[0] == 0.f && f[1] == 0.f && f[2] == 0.f && f[3] == 0.f) continue;  // a part without keys may hold anything
    const float4 x = *reinterpret_cast<const float4*>(all + s * floats + 2 * NR + (static_cast<int64_t>(r4) * 128 * pairs + dim) * 4);
    o[0] += f[0] * x.x; o[1] += f[1] * x.y; o[2] += f[2] * x.z; o[3] += f[3] * x.w;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int gr = r_base + r4 * 4 + i, tok = gr / a.heads;
    if (gr < rows) a.out[(row0 + tok) * a.ldo + static_cast<int64_t>(gr - tok * a.heads) * a.v_pad + dim] = from_float<uint16_t>(o[i]);
  }
}

struct LatentPlan {
  int rows, row_tiles, splits, boxes, rot, pairs, stages, smem;
  int64_t groups, bytes;
};
bool latent_tiled(int dtype, int block_size, int lat_pad, int rot_pad) {
  return dtype == B2_DT_BF16 && lat_pad <= 128 * LT_MAX_PAIRS && rot_pad <= 64 && block_size % LT_KEYS == 0;
}
// Rows per CTA, tiles in shared memory, and how many CTAs share a group's key tiles: as few rounds of one CTA per SM as
// possible, where a CTA's start and end cost about two tiles and a combine one more.
LatentPlan latent_plan(int B, int max_q, int max_kv, int heads, int lat_pad, int rot_pad) {
  LatentPlan p{};
  const int64_t all = static_cast<int64_t>(max_q) * heads;
  p.rows = all > 16 ? 32 : 16;
  p.row_tiles = static_cast<int>(std::min<int64_t>((all + p.rows - 1) / p.rows, INT_MAX));
  p.boxes = (lat_pad + 63) / 64;
  p.rot = rot_pad > 0;
  p.pairs = (p.boxes + 1) / 2;
  const int fixed = 1024 + (((p.boxes + p.rot) * p.rows * 128 + 1023) & ~1023) + p.rows * 512 + LT_SMEM_STATIC;
  const int stage = (2 * p.pairs + p.rot) * LT_BOX;
  // two CTAs on an SM with one tile each hide each other's waits better than one with several tiles
  const int per_sm = p.rows == 16 && 2 * (fixed + stage + 1024) <= LT_SMEM_MAX + 1024 ? 2 : 1;
  p.stages = per_sm == 2 ? 1 : std::max(1, std::min(LT_MAX_STAGES, (LT_SMEM_MAX - fixed) / stage));
  p.smem = fixed - LT_SMEM_STATIC + p.stages * stage;
  p.groups = static_cast<int64_t>(B) * p.row_tiles;
  const int64_t tiles = std::max<int64_t>(1, (static_cast<int64_t>(max_kv) + LT_KEYS - 1) / LT_KEYS);
  p.splits = 1;
  const int64_t at_once = 148 * per_sm;
  if (p.groups < 4 * at_once) {
    int64_t best = INT64_MAX;
    for (int s = 1; s <= std::min<int64_t>(LT_MAX_SPLITS, tiles); ++s) {
      const int64_t cost = ((p.groups * s + at_once - 1) / at_once) * (8 * ((tiles + s - 1) / s) + 16) + (s > 1 ? 8 : 0) + s / 2;
      if (cost < best) {
        best = cost;
        p.splits = s;
      }
    }
  }
  p.bytes = p.splits > 1 ? p.groups * p.splits * latent_part_floats(p.rows, p.pairs) * 4 : 0;
  return p;
}

template <int NR>
int launch_latent(const b2_ctx* ctx, const AttnArgs& a, int64_t slots, int64_t q_rows, int rot_pad, const LatentPlan& p, void* ws, cudaStream_t s) {
  static const cudaError_t set = cudaFuncSetAttribute(latent_tc_kernel<NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, LT_SMEM_MAX - LT_SMEM_STATIC);
  B2_CUDA(set);
  CUtensorMap maps[4];
  const uint16_t* cache = static_cast<const uint16_t*>(a.k_cache);
  const uint16_t* q = static_cast<const uint16_t*>(a.q);
  int rc = encode_tmap_2d(&maps[0], cache, a.v_pad, slots, a.k_row, 64, LT_KEYS);
  if (rc == B2_OK) rc = encode_tmap_2d(&maps[2], q, a.v_pad, q_rows, a.qk_pad, 64, NR);
  if (rc == B2_OK && p.rot) rc = encode_tmap_2d(&maps[1], cache + a.v_pad, rot_pad, slots, a.k_row, 64, LT_KEYS);
  if (rc == B2_OK && p.rot) rc = encode_tmap_2d(&maps[3], q + a.v_pad, rot_pad, q_rows, a.qk_pad, 64, NR);
  if (rc != B2_OK) return rc;
  if (!p.rot) {
    maps[1] = maps[0];
    maps[3] = maps[2];
  }
  LatentTcArgs t{};
  t.out = static_cast<uint16_t*>(a.out); t.ldo = a.ldo; t.block_tables = a.block_tables; t.bt_stride = a.bt_stride; t.block_size = a.block_size;
  t.cu_q = a.cu_q; t.kv_len = a.kv_len; t.heads = a.nq; t.v_pad = a.v_pad; t.boxes = p.boxes; t.rot = p.rot; t.stages = p.stages;
  t.row_tiles = p.row_tiles; t.splits = p.splits; t.scale = a.scale; t.sink = a.sink;
  t.part = static_cast<float*>(ws);
  t.status = ctx->status_dev;
  B2_CUDA(b2_launch(latent_tc_kernel<NR>, dim3(p.splits, p.row_tiles, a.B), dim3(LT_THREADS), p.smem, s, maps[0], maps[1], maps[2], maps[3], t));
  if (p.splits > 1)
    B2_CUDA(b2_launch(latent_combine_kernel<NR>, dim3(NR / 4, p.row_tiles, a.B), dim3(std::max(128, (a.v_pad + 31) / 32 * 32)), 0, s, t));
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
  if (dtype == B2_DT_BF16) {
    if (K <= 128) return w_is_kn ? launch_heads<true, 2>(a, heads, s) : launch_heads<false, 2>(a, heads, s);
    return w_is_kn ? launch_heads<true, 8>(a, heads, s) : launch_heads<false, 8>(a, heads, s);
  }
  const dim3 grid((N + 63) / 64 + (rot_pad > 0 ? 1 : 0), (M + 63) / 64, heads);
  if (w_is_kn) B2_CUDA(b2_launch(heads_gemm_f32_kernel<true>, grid, dim3(256), 0, s, a));
  else B2_CUDA(b2_launch(heads_gemm_f32_kernel<false>, grid, dim3(256), 0, s, a));
  return B2_OK;
}

int64_t b2_latent_attention_workspace(int dtype, int B, int max_q, int max_kv, int block_size, int heads, int lat_pad, int rot_pad) {
  if (B <= 0 || max_q <= 0 || heads <= 0 || block_size < 1 || !latent_tiled(dtype, block_size, lat_pad, rot_pad)) return 0;
  return latent_plan(B, max_q, max_kv, heads, lat_pad, rot_pad).bytes;
}

int b2_latent_attention(b2_ctx* ctx, int dtype, const void* q, int64_t q_rows, void* out, int64_t ldo, const void* cache, int64_t cache_slots,
                        const int32_t* block_tables, int64_t bt_stride, int block_size, const int32_t* cu_q, const int32_t* kv_len, int B, int max_q,
                        int max_kv, int heads, int lat_pad, int rot_pad, float scale, const float* sink, void* workspace, int64_t workspace_bytes,
                        int form, void* stream) {
  if (B < 0 || max_q < 0 || bad_dtype(dtype) || heads <= 0 || lat_pad <= 0 || rot_pad < 0 || lat_pad % 8 != 0 || rot_pad % 8 != 0) return B2_ERR_ARG;
  if (block_size < 1 || (cu_q == nullptr && max_q > 1) || q_rows < 0 || cache_slots < 0) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if (!q || !out || !cache || !block_tables || !kv_len) return B2_ERR_ARG;
  if (!aligned16(q) || !aligned16(out) || !aligned16(cache) || ldo % 8 != 0) return B2_ERR_ARG;
  if (lat_pad + rot_pad > 2048 || lat_pad > 1024 || B > 65535 || heads > 65535 || cache_slots > INT_MAX || q_rows * heads > INT_MAX) return B2_ERR_SHAPE;
  AttnArgs a{};
  a.q = q; a.ldq = static_cast<int64_t>(heads) * (lat_pad + rot_pad); a.out = out; a.ldo = ldo; a.k_cache = a.v_cache = cache;
  a.block_tables = block_tables; a.bt_stride = bt_stride; a.block_size = block_size; a.cu_q = cu_q; a.kv_len = kv_len;
  a.B = B; a.nq = heads; a.nkv = 1; a.qk_pad = lat_pad + rot_pad; a.v_pad = lat_pad; a.k_row = a.v_row = lat_pad + rot_pad;
  a.window = INT_MAX; a.scale = scale; a.sink = sink;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_F32) return launch_any<float>(a, max_q, s);
  if (form == 1 || !latent_tiled(dtype, block_size, lat_pad, rot_pad)) return launch_any<uint16_t>(a, max_q, s);
  if (ctx == nullptr) return B2_ERR_ARG;
  const LatentPlan p = latent_plan(B, max_q, max_kv, heads, lat_pad, rot_pad);
  if (p.row_tiles > 65535) return B2_ERR_SHAPE;
  if (p.splits > 1 && (workspace == nullptr || workspace_bytes < p.bytes))
    return set_error(B2_ERR_SHAPE, "b2_latent_attention: workspace of %lld bytes, %lld needed", static_cast<long long>(workspace_bytes),
                     static_cast<long long>(p.bytes));
  return p.rows == 16 ? launch_latent<16>(ctx, a, cache_slots, q_rows * heads, rot_pad, p, workspace, s)
                      : launch_latent<32>(ctx, a, cache_slots, q_rows * heads, rot_pad, p, workspace, s);
}

}  // extern "C"
