// Attention over keys and values that have been expanded from latents for one step: rows [key | value] per head, a rotated key
// part shared by all heads, queries [unrotated | not yet rotated].  Causal, a learned sink, an output gate.
//
// A CTA walks 256 query tokens of one head as two tiles of 128 rows against key tiles of 128.  Warps 0-3 and 4-7 are the two
// tiles' softmax, a thread per row; warp 8 issues the copies, warp 9 the products:
//     S = Q K^T       128 x 128 fp32 in tensor memory
//     O += P V        P in tensor memory where S was, as a leading and a trailing bf16 part; V rows are used as they lie
// While one tile's softmax runs, the tensor cores work for the other tile: P0 V, S0 of the next keys, P1 V, S1 ...
// Copies land in boxes of 128 rows x 64 columns (16 KB).  Key and value boxes share a ring of three pairs (keys of tile t,
// values of t, keys of t + 1, ...); the rotated key part has two boxes of its own, copied together with the keys: the slot that
// keys of tile t go to held the values of tile t - 2, whose last use comes after the last use of the keys of tile t - 2.
#include <algorithm>

#include "b2_attn.cuh"

namespace {

using namespace b2;

constexpr int EX_BOX = 128 * 64 * 2;
constexpr int EX_THREADS = 320;
constexpr int EX_SMEM = 14 * EX_BOX + 1024;  // 6 query boxes, 3 pairs, 2 rotated key parts
constexpr uint64_t EX_LIMIT_NS = 1000000000ull;
constexpr float EX_RESCALE = 8.0f;  // the running maximum may be exceeded by 2^8 before the outputs are rescaled

struct ExpandedArgs {
  uint16_t* out;
  int64_t ldo;
  const int32_t* cu_q;
  const int32_t* cu_k;
  int nd, nv, rot, v_pad;  // boxes of the unrotated part and of the value; elements of the rotated part (padded) and value
  float scale;
  const float* sink;
  const float2* cs;
  int max_pos;
  const uint16_t* gate;
  int64_t ldg;
  B2Status* status;
};

__global__ void __launch_bounds__(EX_THREADS, 1)
expanded_attn_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_qr, const __grid_constant__ CUtensorMap tm_k,
                     const __grid_constant__ CUtensorMap tm_kr, const __grid_constant__ CUtensorMap tm_v, const ExpandedArgs a) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t s_bars[16];
  __shared__ uint32_t s_tmem;
  __shared__ int s_abort;
  volatile int* abort_flag = &s_abort;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t sq = (smem_u32(smem_raw) + 1023u) & ~1023u, s_pair = sq + 6 * EX_BOX, s_one = s_pair + 6 * EX_BOX;
  const uint32_t bars = smem_u32(s_bars);
  // per pair slot: full, empty; per query tile: copied, rotated, scores, weights, outputs
  const auto full = [&](int i) { return bars + i * 8; };
  const auto empty = [&](int i) { return bars + (3 + i) * 8; };
  const auto q_full = [&](int g) { return bars + (6 + g) * 8; };
  const auto q_ready = [&](int g) { return bars + (8 + g) * 8; };
  const auto s_full = [&](int g) { return bars + (10 + g) * 8; };
  const auto p_full = [&](int g) { return bars + (12 + g) * 8; };
  const auto o_full = [&](int g) { return bars + (14 + g) * 8; };
  if (threadIdx.x == 0) {
    for (int i = 0; i < 16; ++i) mbar_init(bars + i * 8, (i == 8 || i == 9 || i == 12 || i == 13) ? 4 : 1);  // softmax: a lane per warp arrives
    s_abort = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tm_q);
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  if (warp == 9) {
    tmem_alloc(smem_u32(&s_tmem), 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tm = s_tmem;  // S / P of tile g at 128 g, O at 256 + 128 g
  pdl_launch_dependents();     // only now: a later kernel must not take the tensor memory that a CTA of this one still needs
  pdl_wait();

  const int b = blockIdx.y, h = blockIdx.x;
  const int row0 = a.cu_q[b], rows = a.cu_q[b + 1] - row0;
  const int key0 = a.cu_k[b], first_pos = a.cu_k[b + 1] - key0 - rows;
  const int tile0 = (static_cast<int>(gridDim.z) - 1 - static_cast<int>(blockIdx.z)) * 256;  // the longest rows first
  int nr[2], nt[2];  // rows and key tiles of the two query tiles
#pragma unroll
  for (int g = 0; g < 2; ++g) {
    nr[g] = max(0, min(128, rows - tile0 - 128 * g));
    nt[g] = nr[g] > 0 ? (first_pos + tile0 + 128 * g + nr[g] - 1) / 128 + 1 : 0;
  }
  const int tiles = max(nt[0], nt[1]), last = nt[1] > 0 ? 1 : 0;  // the tile that uses keys and values last

  if (warp == 8) {
    // ---------------- copies ----------------
    if (lane == 0 && tiles > 0) {
      for (int g = 0; g <= last; ++g) {
        mbar_arrive_expect_tx(q_full(g), (a.nd + (a.rot > 0)) * EX_BOX);
        const int row = row0 + tile0 + 128 * g;
        for (int i = 0; i < a.nd; ++i) tma_load_3d(sq + (3 * g + i) * EX_BOX, &tm_q, q_full(g), 64 * i, h, row, kEvictFirst);
        if (a.rot > 0) tma_load_3d(sq + (3 * g + 2) * EX_BOX, &tm_qr, q_full(g), 0, h, row, kEvictFirst);
      }
      bool ok = true;
      for (int t = 0; ok && t < tiles; ++t) {
        const int key = key0 + t * 128;
        for (int half = 0; half < 2; ++half) {  // keys, then values
          const int u = 2 * t + half, slot = u % 3, n = half ? a.nv : a.nd;
          if (!(ok = mbar_wait(empty(slot), ((u / 3) & 1) ^ 1, abort_flag, EX_LIMIT_NS, B2_WAIT_SMEM_EMPTY))) break;
          const bool r = half == 0 && a.rot > 0;
          mbar_arrive_expect_tx(full(slot), (n + r) * EX_BOX);
          for (int i = 0; i < n; ++i)
            tma_load_3d(s_pair + (2 * slot + i) * EX_BOX, half ? &tm_v : &tm_k, full(slot), 64 * i, h, key, kEvictNormal);
          if (r) tma_load_2d(s_one + (t & 1) * EX_BOX, &tm_kr, full(slot), 0, key, kEvictNormal);
        }
      }
    }
  } else if (warp == 9) {
    // ---------------- products ----------------
    if (lane == 0 && tiles > 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(128);
      const uint32_t idesc_o = umma_idesc_bf16(64 * a.nv) | UMMA_B_MN;
      bool ok = true;
      for (int t = 0; ok && t <= tiles; ++t) {
        for (int g = 0; ok && g < 2; ++g) {
          if (t > 0 && t - 1 < nt[g]) {  // O_g += P_g V of tile t - 1
            const int u = 2 * (t - 1) + 1, slot = u % 3;
            if (!(ok = mbar_wait(full(slot), (u / 3) & 1, abort_flag, EX_LIMIT_NS, B2_WAIT_SMEM_FULL))) break;
            if (!(ok = mbar_wait(p_full(g), (t - 1) & 1, abort_flag, EX_LIMIT_NS, B2_WAIT_TMEM_EMPTY))) break;
            tc_fence_after();
#pragma unroll
            for (int half = 0; half < 2; ++half)
#pragma unroll
              for (int k = 0; k < 8; ++k)
                umma_bf16_ts(tm + 256 + 128 * g, tm + 128 * g + 64 * half + 8 * k, umma_smem_desc_mn(s_pair + 2 * slot * EX_BOX + k * 2048, EX_BOX), idesc_o,
                             (t > 1 || half > 0 || k > 0) ? 1u : 0u);
            if (g == last) umma_commit(empty(slot));
            if (t == nt[g]) umma_commit(o_full(g));
          }
          if (t < nt[g]) {  // S_g = Q_g K^T of tile t, over the weights that have just been used
            const int u = 2 * t, slot = u % 3;
            if (t == 0 && !(ok = mbar_wait(q_ready(g), 0, abort_flag, EX_LIMIT_NS, B2_WAIT_SMEM_FULL))) break;
            if (!(ok = mbar_wait(full(slot), (u / 3) & 1, abort_flag, EX_LIMIT_NS, B2_WAIT_SMEM_FULL))) break;
            tc_fence_after();
            for (int i = 0; i < a.nd + (a.rot > 0); ++i) {
              const bool r = i == a.nd;
              const uint64_t dq = umma_smem_desc(sq + (3 * g + (r ? 2 : i)) * EX_BOX);
              const uint64_t dk = umma_smem_desc(r ? s_one + (t & 1) * EX_BOX : s_pair + (2 * slot + i) * EX_BOX);
#pragma unroll
              for (int k = 0; k < 4; ++k) umma_bf16(tm + 128 * g, dq + 2 * k, dk + 2 * k, idesc_s, (i > 0 || k > 0) ? 1u : 0u);
            }
            umma_commit(s_full(g));  // also says that this tile's outputs so far are complete
            if (g == last) umma_commit(empty(slot));
          }
        }
      }
    }
  } else {
    // ---------------- softmax: thread = row of query tile g ----------------
    const int g = warp >> 2, r = threadIdx.x & 127, tiles_g = nt[g];
    const uint32_t lanes = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t ts = tm + 128 * g + lanes, to = tm + 256 + 128 * g + lanes;
    const int pos = first_pos + tile0 + 128 * g + min(r, max(nr[g], 1) - 1), pmin = first_pos + tile0 + 128 * g;
    const float scale = a.scale * LOG2E;
    bool ok = true;
    if (tiles_g > 0) {
      // the row's angles are on their way while the queries are copied
      float4 cs[16];
      const int64_t at_pos = min(pos, a.max_pos - 1);
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (4 * i < a.rot) cs[i] = __ldg(reinterpret_cast<const float4*>(a.cs + at_pos * (a.rot >> 1)) + i);  // two pairs
      ok = mbar_wait(q_full(g), 0, abort_flag, EX_LIMIT_NS, B2_WAIT_SMEM_FULL);
      if (ok && a.rot > 0) {
        unsigned char* box = smem_raw + (sq - smem_u32(smem_raw)) + (3 * g + 2) * EX_BOX + r * 128;
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          if (c * 8 >= a.rot) break;
          uint16_t* at = reinterpret_cast<uint16_t*>(box + ((c ^ (r & 7)) << 4));
          float f[8], o[8];
          load8<uint16_t>(at, f);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float4 w = cs[2 * c + i];
            o[4 * i] = f[4 * i] * w.x - f[4 * i + 1] * w.y;
            o[4 * i + 1] = f[4 * i + 1] * w.x + f[4 * i] * w.y;
            o[4 * i + 2] = f[4 * i + 2] * w.z - f[4 * i + 3] * w.w;
            o[4 * i + 3] = f[4 * i + 3] * w.z + f[4 * i + 2] * w.w;
          }
          store8<uint16_t>(at, o);
        }
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(q_ready(g));
    }
    float m = -INFINITY, l = 0.f;
    for (int t = 0; t < tiles_g; ++t) {
      ok = mbar_wait(s_full(g), t & 1, abort_flag, EX_LIMIT_NS, B2_WAIT_TMEM_FULL);
      if (!__all_sync(0xffffffffu, ok)) {
        ok = false;
        break;
      }
      tc_fence_after();
      uint32_t raw[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld_32x32(ts + 32 * c, raw[c]);
      tc_wait_ld();
      if (t * 128 + 127 > pmin) {
        const int seen = pos - t * 128;
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (32 * c + i > seen) raw[c][i] = 0xFF800000u;  // -inf
      }
      float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < 32; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) mx[c] = fmaxf(mx[c], __uint_as_float(raw[c][i]));
      const float m_tile = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * scale;  // the scale is positive
      const bool grow = m_tile > m + EX_RESCALE || m == -INFINITY;
      const float m_new = grow ? fmaxf(m_tile, m) : m;
      const float corr = grow && m > -INFINITY ? fast_exp2(m - m_new) : 1.0f;
      if (__any_sync(0xffffffffu, corr != 1.0f)) {  // never in the first tile
        l *= corr;
#pragma unroll 1
        for (int c = 0; c < 4 * a.nv; ++c) {
          uint32_t o[16];
          tmem_ld_32x16(to + 16 * c, o);
          tc_wait_ld();
#pragma unroll
          for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
          tmem_st_32x16(to + 16 * c, o);
        }
      }
      m = m_new;
      const float ref = m == -INFINITY ? 0.f : m;
      float sum[2] = {0.f, 0.f};
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t hi[16], lo[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float x = fast_exp2(fmaf(__uint_as_float(raw[c][2 * i]), scale, -ref)), y = fast_exp2(fmaf(__uint_as_float(raw[c][2 * i + 1]), scale, -ref));
          sum[0] += x;
          sum[1] += y;
          split_bf16(x, y, hi[i], lo[i]);
        }
        tmem_st_32x16(ts + 16 * c, hi);
        tmem_st_32x16(ts + 64 + 16 * c, lo);
      }
      l += sum[0] + sum[1];
      tc_wait_st();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full(g));
    }
    const bool write = ok && r < nr[g];
    const int64_t row = row0 + tile0 + 128 * g + r;
    uint4 gate[16];  // the row's gates are on their way while the last product runs
    if (a.gate != nullptr && write) {
      const uint16_t* src = a.gate + row * a.ldg + static_cast<int64_t>(h) * a.v_pad;
#pragma unroll
      for (int i = 0; i < 16; ++i)
        if (8 * i < a.v_pad) gate[i] = *reinterpret_cast<const uint4*>(src + 8 * i);
    }
    if (ok && tiles_g > 0) ok = mbar_wait(o_full(g), 0, abort_flag, EX_LIMIT_NS, B2_WAIT_TMEM_FULL);
    if (__all_sync(0xffffffffu, ok) && tiles_g > 0) {
      tc_fence_after();
      float f = 1.0f;
      if (a.sink != nullptr) {
        const float sk = a.sink[h] * LOG2E, m_new = fmaxf(m, sk);
        f = fast_exp2(m - m_new);
        l = l * f + fast_exp2(sk - m_new);
      }
      f /= l;
      uint16_t* dst = a.out + row * a.ldo + static_cast<int64_t>(h) * a.v_pad;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        if (32 * c >= a.v_pad) break;
        uint32_t o[32];
        tmem_ld_32x32(to + 32 * c, o);
        tc_wait_ld();
        if (!write) continue;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (32 * c + 8 * i >= a.v_pad) break;
          float x[8];
#pragma unroll
          for (int e = 0; e < 8; ++e) x[e] = __uint_as_float(o[8 * i + e]) * f;
          if (a.gate != nullptr) {
            const uint4 s = gate[4 * c + i];
            const float y[8] = {bf16_lo(s.x), bf16_hi(s.x), bf16_lo(s.y), bf16_hi(s.y), bf16_lo(s.z), bf16_hi(s.z), bf16_lo(s.w), bf16_hi(s.w)};
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] *= sigmoid_fast(y[e]);
          }
          store8<uint16_t>(dst + 32 * c + 8 * i, x);
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
  if (warp == 9) tmem_dealloc(tm, 512);
}

}  // namespace

extern "C" {

int b2_expanded_attention(b2_ctx* ctx, const void* q, int64_t ldq, int64_t q_rows, void* out, int64_t ldo, const void* kv, int64_t ld_kv,
                          const void* rot, int64_t ld_rot, int64_t k_rows, const int32_t* cu_q, const int32_t* cu_k, int B, int max_q, int heads,
                          int dim_pad, int rot_pad, int v_pad, float scale, const float* sink, const float* cos_sin, int max_pos, const void* gate,
                          int64_t ldg, void* stream) {
  if (ctx == nullptr || B < 0 || max_q < 0 || heads <= 0 || dim_pad <= 0 || rot_pad < 0 || v_pad <= 0) return B2_ERR_ARG;
  if (dim_pad % 8 != 0 || rot_pad % 8 != 0 || v_pad % 8 != 0 || !(scale > 0.f) || q_rows < 0 || k_rows < 0) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if (!q || !out || !kv || !cu_q || !cu_k || !aligned16(q) || !aligned16(out) || !aligned16(kv)) return B2_ERR_ARG;
  if (ldq % 8 != 0 || ldo % 8 != 0 || ld_kv % 8 != 0 || ld_rot % 8 != 0) return B2_ERR_ARG;
  if (ldq < static_cast<int64_t>(heads) * (dim_pad + rot_pad) || ld_kv < static_cast<int64_t>(heads) * (dim_pad + v_pad)) return B2_ERR_ARG;
  if (rot_pad > 0 && (!rot || !aligned16(rot) || ld_rot < rot_pad || !cos_sin || !aligned16(cos_sin) || max_pos <= 0)) return B2_ERR_ARG;
  if (gate != nullptr && (!aligned16(gate) || ldg % 8 != 0)) return B2_ERR_ARG;
  if (dim_pad > 128 || rot_pad > 64 || v_pad > 128 || B > 65535 || (max_q + 255) / 256 > 65535 || q_rows > INT_MAX || k_rows > INT_MAX) return B2_ERR_SHAPE;
  static const cudaError_t set = cudaFuncSetAttribute(expanded_attn_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, EX_SMEM);
  B2_CUDA(set);
  const uint16_t* qp = static_cast<const uint16_t*>(q);
  const uint16_t* kp = static_cast<const uint16_t*>(kv);
  CUtensorMap m[5];
  const uint64_t qh = dim_pad + rot_pad, kh = dim_pad + v_pad;
  int rc = encode_tmap_heads(&m[0], qp, dim_pad, heads, qh, q_rows, ldq, 64, 128);
  if (rc == B2_OK) rc = encode_tmap_heads(&m[2], kp, dim_pad, heads, kh, k_rows, ld_kv, 64, 128);
  if (rc == B2_OK) rc = encode_tmap_heads(&m[4], kp + dim_pad, v_pad, heads, kh, k_rows, ld_kv, 64, 128);
  if (rot_pad > 0) {
    if (rc == B2_OK) rc = encode_tmap_heads(&m[1], qp + dim_pad, rot_pad, heads, qh, q_rows, ldq, 64, 128);
    if (rc == B2_OK) rc = encode_tmap_2d(&m[3], rot, rot_pad, k_rows, ld_rot, 64, 128);
  } else {
    m[1] = m[0];
    m[3] = m[2];
  }
  if (rc != B2_OK) return rc;
  ExpandedArgs a{};
  a.out = static_cast<uint16_t*>(out); a.ldo = ldo; a.cu_q = cu_q; a.cu_k = cu_k; a.nd = (dim_pad + 63) / 64; a.nv = (v_pad + 63) / 64;
  a.rot = rot_pad; a.v_pad = v_pad; a.scale = scale; a.sink = sink; a.cs = reinterpret_cast<const float2*>(cos_sin); a.max_pos = max_pos;
  a.gate = static_cast<const uint16_t*>(gate); a.ldg = ldg; a.status = ctx->status_dev;
  B2_CUDA(b2_launch(expanded_attn_kernel, dim3(heads, B, (max_q + 255) / 256), dim3(EX_THREADS), EX_SMEM, static_cast<cudaStream_t>(stream), m[0], m[1],
                    m[2], m[3], m[4], a));
  return B2_OK;
}

}  // extern "C"
