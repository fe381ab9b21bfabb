// Linear attention with a constant decay per head ("lightning attention"):
//     S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// The state S [dim, vdim] of every head lives in fp32, one slot per sequence; a sequence that starts at position 0
// starts from zero whatever its slot holds.
//
//   linear_attn_segment_kernel, linear_attn_scan_kernel
//                              prefill, bf16, heads up to 128: chunks of 64 tokens on the tensor cores
//   linear_attn_decode_kernel  one token per sequence, bf16
//   linear_attn_any_kernel     any size, bf16 or fp32, token by token (also decode)
//   gated_norm_kernel          RMSNorm over the concatenated heads times sigmoid(gate)
#include <algorithm>

#include "b2_mma.cuh"
#include "b2_vec.cuh"

namespace {

struct LinArgs {
  const void* qkv;  // rows [q heads | k heads | v heads | ...], activations already applied
  int64_t ld;
  float* o;         // [M, heads * v_pad] fp32
  int64_t ldo;
  float* state;     // [slots, heads, qk_pad, v_pad]
  const int32_t* slots;   // [B]; negative = no sequence (padded row of a decode graph)
  const int32_t* cu_q;    // [B + 1]; null = one row per sequence
  const int32_t* kv_len;  // [B] tokens of every sequence including this step's
  const float* decay;     // [heads]
  int B, heads, qk_pad, v_pad;
};

// ---------------------------------------------------------------------------
// Token by token.  A CTA owns 32 columns of one head's state in shared memory; 8 threads share a column's rows.
// ---------------------------------------------------------------------------
constexpr int ANY_COLS = 32;
template <typename T>
__global__ void __launch_bounds__(256) linear_attn_any_kernel(const LinArgs a) {
  extern __shared__ float sm[];
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int h = blockIdx.x, c0 = blockIdx.y * ANY_COLS, b = blockIdx.z;
  const int D = a.qk_pad;
  float* S = sm;                       // [D][ANY_COLS]
  float* qs = S + D * ANY_COLS;        // [D]
  float* ks = qs + D;                  // [D]
  float* part = ks + D;                // [8][ANY_COLS]
  const int col = threadIdx.x & 31, rg = threadIdx.x >> 5;
  const int row0 = a.cu_q ? a.cu_q[b] : b;
  const int n = a.cu_q ? a.cu_q[b + 1] - row0 : 1;
  const int slot = a.slots[b];
  const bool col_ok = c0 + col < a.v_pad;
  if (slot < 0) {
    for (int t = 0; t < n; ++t)
      if (rg == 0 && col_ok) a.o[(row0 + t) * a.ldo + static_cast<int64_t>(h) * a.v_pad + c0 + col] = 0.f;
    return;
  }
  const bool fresh = a.kv_len[b] == n;
  const float dec = a.decay[h];
  float* st = a.state + (static_cast<int64_t>(slot) * a.heads + h) * D * a.v_pad;
  for (int r = rg; r < D; r += 8) S[r * ANY_COLS + col] = (fresh || !col_ok) ? 0.f : st[static_cast<int64_t>(r) * a.v_pad + c0 + col];
  for (int t = 0; t < n; ++t) {
    const T* row = static_cast<const T*>(a.qkv) + (row0 + t) * a.ld;
    __syncthreads();
    for (int i = threadIdx.x; i < D; i += blockDim.x) {
      qs[i] = b2::to_float(row[static_cast<int64_t>(h) * D + i]);
      ks[i] = b2::to_float(row[static_cast<int64_t>(a.heads + h) * D + i]);
    }
    const float v = col_ok ? b2::to_float(row[2ll * a.heads * D + static_cast<int64_t>(h) * a.v_pad + c0 + col]) : 0.f;
    __syncthreads();
    float acc = 0.f;
    for (int r = rg; r < D; r += 8) {
      const float s = fmaf(ks[r], v, dec * S[r * ANY_COLS + col]);
      S[r * ANY_COLS + col] = s;
      acc = fmaf(s, qs[r], acc);
    }
    part[rg * ANY_COLS + col] = acc;
    __syncthreads();
    if (rg == 0 && col_ok) {
      float o = 0.f;
#pragma unroll
      for (int i = 0; i < 8; ++i) o += part[i * ANY_COLS + col];
      a.o[(row0 + t) * a.ldo + static_cast<int64_t>(h) * a.v_pad + c0 + col] = o;
    }
  }
  if (col_ok)
    for (int r = rg; r < D; r += 8) st[static_cast<int64_t>(r) * a.v_pad + c0 + col] = S[r * ANY_COLS + col];
}

// ---------------------------------------------------------------------------
// Decode, bf16: one token per sequence.  A CTA owns 32 columns of one head's state: 8 threads cover a 128-byte piece
// of a state row, 32 rows at a time; every state word is read and written once.
// ---------------------------------------------------------------------------
constexpr int DEC_COLS = 32, DEC_BATCH = 4;
__global__ void __launch_bounds__(256) linear_attn_decode_kernel(const LinArgs a) {
  __shared__ float4 part[8][8];
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int tiles = (a.v_pad + DEC_COLS - 1) / DEC_COLS;
  const int h = blockIdx.x / tiles, c0 = (blockIdx.x % tiles) * DEC_COLS, b = blockIdx.y;
  const int D = a.qk_pad;
  const int c = c0 + (threadIdx.x & 7) * 4, rl = threadIdx.x >> 3;
  const bool col_ok = c < a.v_pad;
  float* orow = a.o + b * a.ldo + static_cast<int64_t>(h) * a.v_pad;
  const int slot = a.slots[b];
  if (slot < 0) {
    if (rl == 0 && col_ok) *reinterpret_cast<float4*>(orow + c) = make_float4(0.f, 0.f, 0.f, 0.f);
    return;
  }
  const bool fresh = a.kv_len[b] == 1;
  const float dec = a.decay[h];
  const uint16_t* row = static_cast<const uint16_t*>(a.qkv) + b * a.ld;
  const uint16_t* q = row + static_cast<int64_t>(h) * D;
  const uint16_t* k = row + static_cast<int64_t>(a.heads + h) * D;
  float* st = a.state + (static_cast<int64_t>(slot) * a.heads + h) * D * a.v_pad;
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f), acc = v;
  if (col_ok) v = b2::load4<uint16_t>(row + 2ll * a.heads * D + static_cast<int64_t>(h) * a.v_pad + c);
  for (int r0 = 0; r0 < D; r0 += 32 * DEC_BATCH) {
    float4 s[DEC_BATCH];
    float kf[DEC_BATCH], qf[DEC_BATCH];
#pragma unroll
    for (int i = 0; i < DEC_BATCH; ++i) {
      const int r = r0 + rl + i * 32;
      const bool ok = r < D && col_ok;
      s[i] = ok && !fresh ? *reinterpret_cast<const float4*>(st + static_cast<int64_t>(r) * a.v_pad + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      kf[i] = ok ? b2::to_float(k[r]) : 0.f;
      qf[i] = ok ? b2::to_float(q[r]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < DEC_BATCH; ++i) {
      const int r = r0 + rl + i * 32;
      s[i].x = fmaf(kf[i], v.x, dec * s[i].x); s[i].y = fmaf(kf[i], v.y, dec * s[i].y);
      s[i].z = fmaf(kf[i], v.z, dec * s[i].z); s[i].w = fmaf(kf[i], v.w, dec * s[i].w);
      acc.x = fmaf(s[i].x, qf[i], acc.x); acc.y = fmaf(s[i].y, qf[i], acc.y);
      acc.z = fmaf(s[i].z, qf[i], acc.z); acc.w = fmaf(s[i].w, qf[i], acc.w);
      if (r < D && col_ok) *reinterpret_cast<float4*>(st + static_cast<int64_t>(r) * a.v_pad + c) = s[i];
    }
  }
#pragma unroll
  for (int o = 8; o <= 16; o <<= 1) {
    acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o); acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
    acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o); acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
  }
  if ((threadIdx.x & 31) < 8) part[threadIdx.x >> 5][threadIdx.x & 7] = acc;
  __syncthreads();
  if (threadIdx.x < 8 && col_ok) {
    acc = part[0][threadIdx.x];
#pragma unroll
    for (int w = 1; w < 8; ++w) {
      const float4 p = part[w][threadIdx.x];
      acc.x += p.x; acc.y += p.y; acc.z += p.z; acc.w += p.w;
    }
    *reinterpret_cast<float4*>(orow + c) = acc;
  }
}

// ---------------------------------------------------------------------------
// Prefill, bf16, heads up to 128 wide, on the tensor cores.  A sequence is walked in chunks of 64 tokens; where there
// are too few heads and sequences to fill the SMs it is cut into segments that run side by side.  With P_n = decay^n, inside a chunk that starts from state S:
//     o_i = P_(i+1) S^T q_i + sum_(j <= i) P_(i-j) (q_i . k_j) v_j
//     S'  = P_n S + sum_j k_j (P_(n-1-j) v_j)^T
// q, k, v are exact bf16; S, the decayed scores and the decayed values are fp32 and enter the products as a sum of two
// bf16 numbers.  Sequences of several segments take three launches: every segment's own contribution (SUMS), a scan
// that turns those into the states the segments start from, and the outputs.
// ---------------------------------------------------------------------------
constexpr int CH = 64, SEG = 512, VT = 64;

struct SegArgs {
  LinArgs a;
  const float* powers;  // [heads][65]
  float* seg_state;     // [segments][heads][qk_pad][v_pad]; sequence b's segments start at cu_q[b] / seg + b
  int seg;              // tokens per segment, a multiple of 64
  int multi;            // some sequence has several segments: their start states are in seg_state
};

template <int DQ>
struct CfgSeg {
  static constexpr int STAGE = CH * (2 * DQ + VT) * 2;  // q, k, v
  static constexpr int SMEM = 2 * STAGE + 2 * DQ * VT * 2 + 128;
};

template <int DQ, bool SUMS>
__global__ void __launch_bounds__(128, 2) linear_attn_segment_kernel(const SegArgs sa) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ float pw[CH + 1];
  const LinArgs& a = sa.a;
  constexpr int MT = DQ / 64;  // 16-row tiles of the state per warp
  const uint32_t base = (b2::smem_u32(smem_raw) + 127) & ~127u;
  const uint32_t s_hi = base + 2 * CfgSeg<DQ>::STAGE, s_lo = s_hi + DQ * VT * 2;  // state, later the decayed values
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  b2::pdl_launch_dependents();
  const int vtiles = (a.v_pad + VT - 1) / VT;
  const int h = blockIdx.y / vtiles, v0 = (blockIdx.y % vtiles) * VT, b = blockIdx.z, seg = blockIdx.x;
  for (int i = threadIdx.x; i <= CH; i += 128) pw[i] = sa.powers[h * (CH + 1) + i];
  b2::pdl_wait();
  const int row0 = a.cu_q[b];
  const int n_q = a.cu_q[b + 1] - row0;
  const int t_begin = seg * sa.seg, t_end = min(n_q, t_begin + sa.seg);
  if (t_begin >= n_q) return;
  const bool final_seg = t_end == n_q;
  if (SUMS && final_seg) return;  // no segment starts from its sum
  const int slot = a.slots[b];
  const int D = a.qk_pad;
  const int64_t head_state = static_cast<int64_t>(D) * a.v_pad;
  float* slot_state = slot >= 0 ? a.state + (static_cast<int64_t>(slot) * a.heads + h) * head_state : nullptr;
  float* seg_state = sa.seg_state + (static_cast<int64_t>(row0 / sa.seg + b + seg) * a.heads + h) * head_state;

  const uint16_t* qkv = static_cast<const uint16_t*>(a.qkv);
  const int64_t off_q = static_cast<int64_t>(h) * D, off_k = static_cast<int64_t>(a.heads + h) * D;
  const int64_t off_v = 2ll * a.heads * D + static_cast<int64_t>(h) * a.v_pad + v0;
  auto load_chunk = [&](int t0, int stage) {
    const uint32_t sq = base + stage * CfgSeg<DQ>::STAGE, sk = sq + CH * DQ * 2, sv = sk + CH * DQ * 2;
    constexpr int QP = DQ / 8, VP = VT / 8;
#pragma unroll
    for (int i = 0; i < CH * QP / 128; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx / QP, p = idx % QP;
      const bool ok = t0 + r < t_end && p * 8 < D;
      const uint16_t* src = qkv + (row0 + (ok ? t0 + r : 0)) * a.ld + (ok ? p * 8 : 0);
      if (!SUMS) b2::cp_async16(b2::tile_addr<DQ>(sq, r, p), src + off_q, ok);
      b2::cp_async16(b2::tile_addr<DQ>(sk, r, p), src + off_k, ok);
    }
#pragma unroll
    for (int i = 0; i < CH * VP / 128; ++i) {
      const int idx = threadIdx.x + i * 128, r = idx / VP, p = idx % VP;
      const bool ok = t0 + r < t_end && v0 + p * 8 < a.v_pad;
      b2::cp_async16(b2::tile_addr<VT>(sv, r, p), qkv + (row0 + (ok ? t0 + r : 0)) * a.ld + off_v + (ok ? p * 8 : 0), ok);
    }
    b2::cp_async_commit();
  };
  load_chunk(t_begin, 0);

  // this warp's rows of the state: 16-row tiles warp * MT .. , 64 columns
  float S[MT][VT / 8][4];
  auto state_at = [&](const float* src, int mt, int n, int half) {  // two neighbouring columns
    const int r = (warp * MT + mt) * 16 + (lane >> 2) + half * 8, c = v0 + n * 8 + (lane & 3) * 2;
    return (src != nullptr && r < D && c < a.v_pad) ? *reinterpret_cast<const float2*>(src + static_cast<int64_t>(r) * a.v_pad + c) : make_float2(0.f, 0.f);
  };
  const float* start = nullptr;
  if (!SUMS) start = sa.multi && n_q > sa.seg ? seg_state : (a.kv_len[b] == n_q ? nullptr : slot_state);
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < VT / 8; ++n) {
      const float2 lo = state_at(start, mt, n, 0), hi = state_at(start, mt, n, 1);
      S[mt][n][0] = lo.x; S[mt][n][1] = lo.y; S[mt][n][2] = hi.x; S[mt][n][3] = hi.y;
    }

  int stage = 0;
  for (int t0 = t_begin; t0 < t_end; t0 += CH, stage ^= 1) {
    const int nc = min(CH, t_end - t0);
    b2::cp_async_wait<0>();
    __syncthreads();
    if (t0 + CH < t_end) load_chunk(t0 + CH, stage ^ 1);
    const uint32_t sq = base + stage * CfgSeg<DQ>::STAGE, sk = sq + CH * DQ * 2, sv = sk + CH * DQ * 2;
    if (!SUMS) {
      // the state as two bf16 tiles [d][v]
#pragma unroll
      for (int mt = 0; mt < MT; ++mt)
#pragma unroll
        for (int n = 0; n < VT / 8; ++n)
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int r = (warp * MT + mt) * 16 + (lane >> 2) + half * 8;
            uint32_t hi, lo;
            b2::split_bf16(S[mt][n][2 * half], S[mt][n][2 * half + 1], hi, lo);
            const uint32_t off = b2::tile_addr<VT>(0, r, n) + (lane & 3) * 4;
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(s_hi + off), "r"(hi) : "memory");
            asm volatile("st.shared.b32 [%0], %1;" ::"r"(s_lo + off), "r"(lo) : "memory");
          }
      __syncthreads();
      float o[VT / 8][4], sc[CH / 8][4];
#pragma unroll
      for (int n = 0; n < VT / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
#pragma unroll
      for (int n = 0; n < CH / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[n][e] = 0.f;
#pragma unroll
      for (int k = 0; k < DQ / 16; ++k) {
        uint32_t qa[4];
        b2::frag_a<DQ>(sq, warp * 16, k * 16, lane, qa);
#pragma unroll
        for (int n = 0; n < VT / 16; ++n) {
          uint32_t bh[4], bl[4];
          b2::frag_b_t<VT>(s_hi, n * 16, k * 16, lane, bh);
          b2::frag_b_t<VT>(s_lo, n * 16, k * 16, lane, bl);
          b2::mma16816(o[2 * n], qa, bh[0], bh[1]);
          b2::mma16816(o[2 * n + 1], qa, bh[2], bh[3]);
          b2::mma16816(o[2 * n], qa, bl[0], bl[1]);
          b2::mma16816(o[2 * n + 1], qa, bl[2], bl[3]);
        }
#pragma unroll
        for (int n = 0; n < CH / 16; ++n) {
          if (n > warp) break;  // keys after the warp's last row
          uint32_t kb[4];
          b2::frag_b<DQ>(sk, n * 16, k * 16, lane, kb);
          b2::mma16816(sc[2 * n], qa, kb[0], kb[1]);
          b2::mma16816(sc[2 * n + 1], qa, kb[2], kb[3]);
        }
      }
      const int i0 = warp * 16 + (lane >> 2);
      const float p0 = pw[i0 + 1], p1 = pw[i0 + 9];
#pragma unroll
      for (int n = 0; n < VT / 8; ++n) {
        o[n][0] *= p0; o[n][1] *= p0; o[n][2] *= p1; o[n][3] *= p1;
      }
#pragma unroll
      for (int k = 0; k < CH / 16; ++k) {
        if (k > warp) break;
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int x = 0; x < 4; ++x) {  // operand register x: columns of tile 2k + (x >> 1), row half x & 1
          const int i = i0 + (x & 1) * 8, j = k * 16 + (x >> 1) * 8 + (lane & 3) * 2;
          const float w0 = j <= i ? sc[2 * k + (x >> 1)][(x & 1) * 2] * pw[i - j] : 0.f;
          const float w1 = j + 1 <= i ? sc[2 * k + (x >> 1)][(x & 1) * 2 + 1] * pw[i - j - 1] : 0.f;
          b2::split_bf16(w0, w1, hi[x], lo[x]);
        }
#pragma unroll
        for (int n = 0; n < VT / 16; ++n) {
          uint32_t vb[4];
          b2::frag_b_t<VT>(sv, n * 16, k * 16, lane, vb);
          b2::mma16816(o[2 * n], hi, vb[0], vb[1]);
          b2::mma16816(o[2 * n + 1], hi, vb[2], vb[3]);
          b2::mma16816(o[2 * n], lo, vb[0], vb[1]);
          b2::mma16816(o[2 * n + 1], lo, vb[2], vb[3]);
        }
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = i0 + half * 8;
        if (i >= nc) continue;
        float* dst = a.o + (row0 + t0 + i) * a.ldo + static_cast<int64_t>(h) * a.v_pad;
#pragma unroll
        for (int n = 0; n < VT / 8; ++n) {
          const int c = v0 + n * 8 + (lane & 3) * 2;
          if (c < a.v_pad) *reinterpret_cast<float2*>(dst + c) = make_float2(o[n][2 * half], o[n][2 * half + 1]);
        }
      }
      __syncthreads();  // the state tiles are free
    }
    // decayed values P_(nc-1-j) v_j as two bf16 tiles [j][v], where the state tiles were
#pragma unroll
    for (int i = 0; i < CH * (VT / 2) / 128; ++i) {
      const int idx = threadIdx.x + i * 128, j = idx / (VT / 2), c2 = idx % (VT / 2);
      const uint32_t off = b2::tile_addr<VT>(0, j, c2 >> 2) + (c2 & 3) * 4;
      uint32_t v, hi, lo;
      asm volatile("ld.shared.b32 %0, [%1];" : "=r"(v) : "r"(sv + off) : "memory");
      const float w = j < nc ? pw[nc - 1 - j] : 0.f;
      b2::split_bf16(b2::bf16_lo(v) * w, b2::bf16_hi(v) * w, hi, lo);
      asm volatile("st.shared.b32 [%0], %1;" ::"r"(s_hi + off), "r"(hi) : "memory");
      asm volatile("st.shared.b32 [%0], %1;" ::"r"(s_lo + off), "r"(lo) : "memory");
    }
    __syncthreads();
    const float pn = pw[nc];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int n = 0; n < VT / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][n][e] *= pn;
#pragma unroll
    for (int k = 0; k < CH / 16; ++k) {
      uint32_t ka[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) b2::frag_a_t<DQ>(sk, (warp * MT + mt) * 16, k * 16, lane, ka[mt]);
#pragma unroll
      for (int n = 0; n < VT / 16; ++n) {
        uint32_t bh[4], bl[4];
        b2::frag_b_t<VT>(s_hi, n * 16, k * 16, lane, bh);
        b2::frag_b_t<VT>(s_lo, n * 16, k * 16, lane, bl);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          b2::mma16816(S[mt][2 * n], ka[mt], bh[0], bh[1]);
          b2::mma16816(S[mt][2 * n + 1], ka[mt], bh[2], bh[3]);
          b2::mma16816(S[mt][2 * n], ka[mt], bl[0], bl[1]);
          b2::mma16816(S[mt][2 * n + 1], ka[mt], bl[2], bl[3]);
        }
      }
    }
    // (the next chunk's first barrier comes before anyone writes these tiles again)
  }
  float* dst = SUMS ? seg_state : (final_seg ? slot_state : nullptr);
  if (dst == nullptr) return;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int n = 0; n < VT / 8; ++n)
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int r = (warp * MT + mt) * 16 + (lane >> 2) + half * 8, c = v0 + n * 8 + (lane & 3) * 2;
        if (r < D && c < a.v_pad)
          *reinterpret_cast<float2*>(dst + static_cast<int64_t>(r) * a.v_pad + c) = make_float2(S[mt][n][2 * half], S[mt][n][2 * half + 1]);
      }
}

// seg_state[s] <- the state segment s starts from (it held segment s's own contribution)
__global__ void __launch_bounds__(256) linear_attn_scan_kernel(const SegArgs sa) {
  const LinArgs& a = sa.a;
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int b = blockIdx.z, h = blockIdx.y;
  const int row0 = a.cu_q[b], n_q = a.cu_q[b + 1] - row0;
  if (n_q <= sa.seg) return;
  const int segs = (n_q + sa.seg - 1) / sa.seg;
  const int64_t head_state = static_cast<int64_t>(a.qk_pad) * a.v_pad;
  const int64_t e = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) * 4;
  if (e >= head_state) return;
  float p = sa.powers[h * (CH + 1) + CH], ps = 1.0f;
  for (int i = 0; i < sa.seg / CH; ++i) ps *= p;
  const int slot = a.slots[b];
  float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
  if (slot >= 0 && a.kv_len[b] != n_q) s = *reinterpret_cast<const float4*>(a.state + (static_cast<int64_t>(slot) * a.heads + h) * head_state + e);
  float* at = sa.seg_state + (static_cast<int64_t>(row0 / sa.seg + b) * a.heads + h) * head_state + e;
  const int64_t step = a.heads * head_state;
  constexpr int AHEAD = 4;  // contributions in flight per thread
  for (int i0 = 0; i0 < segs; i0 += AHEAD) {
    float4 own[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
      own[i] = i0 + i + 1 < segs ? *reinterpret_cast<const float4*>(at + i * step) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < AHEAD; ++i, at += step) {
      if (i0 + i >= segs) return;
      *reinterpret_cast<float4*>(at) = s;
      s.x = fmaf(ps, s.x, own[i].x); s.y = fmaf(ps, s.y, own[i].y); s.z = fmaf(ps, s.z, own[i].z); s.w = fmaf(ps, s.w, own[i].w);
    }
  }
}

bool segment_form(int dtype, int qk_pad, int v_pad) { return dtype == B2_DT_BF16 && qk_pad <= 128; }

// Tokens per segment.  A sequence in one piece does no work twice, so it is cut only where the CTAs of whole sequences
// (total / longest of them run side by side, two on an SM) would leave SMs idle.
int segment_length(int max_q, int total_q, int heads, int v_pad) {
  const int64_t ctas = static_cast<int64_t>(heads) * ((v_pad + VT - 1) / VT) * std::max(total_q, 1) / std::max(max_q, 1);
  return max_q <= SEG || ctas >= 230 ? (max_q + CH - 1) / CH * CH : SEG;
}
int64_t segment_slots(int B, int total_q, int seg) { return static_cast<int64_t>(total_q) / seg + B + 1; }

template <int DQ>
int launch_segments(const SegArgs& sa, int max_q, cudaStream_t s) {
  const LinArgs& a = sa.a;
  static bool set = false;
  if (!set) {
    B2_CUDA(cudaFuncSetAttribute(linear_attn_segment_kernel<DQ, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, CfgSeg<DQ>::SMEM));
    B2_CUDA(cudaFuncSetAttribute(linear_attn_segment_kernel<DQ, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, CfgSeg<DQ>::SMEM));
    set = true;
  }
  const dim3 grid((max_q + sa.seg - 1) / sa.seg, a.heads * ((a.v_pad + VT - 1) / VT), a.B);
  if (sa.multi) {
    B2_CUDA(b2_launch(linear_attn_segment_kernel<DQ, true>, grid, dim3(128), CfgSeg<DQ>::SMEM, s, sa));
    const int64_t quads = static_cast<int64_t>(a.qk_pad) * a.v_pad / 4;
    B2_CUDA(b2_launch(linear_attn_scan_kernel, dim3(static_cast<unsigned>((quads + 255) / 256), a.heads, a.B), dim3(256), 0, s, sa));
  }
  B2_CUDA(b2_launch(linear_attn_segment_kernel<DQ, false>, grid, dim3(128), CfgSeg<DQ>::SMEM, s, sa));
  return B2_OK;
}

// ---------------------------------------------------------------------------
// out = o / sqrt(mean(o^2) + eps) * w * sigmoid(gate); o in fp32, the mean over `dim` true elements of a row of
// dim_pad (the padding of o is zero).  One CTA per row.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(1024) gated_norm_kernel(const float* o, int64_t ldo, const T* gate, int64_t ldg, const float* w, float eps, int dim,
                                                           int dim_pad, T* out, int64_t ld_out) {
  __shared__ float red[32];
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int row = blockIdx.x;
  const int nvec = dim_pad >> 2;
  const float* orow = o + row * ldo;
  constexpr int KEEP = 4;  // vectors of the row, and of the gate, a thread keeps in registers
  float4 kept[KEEP], gates[KEEP];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    gates[i] = v < nvec ? b2::load4<T>(gate + row * ldg + v * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    kept[i] = v < nvec ? *reinterpret_cast<const float4*>(orow + v * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += kept[i].x * kept[i].x + kept[i].y * kept[i].y + kept[i].z * kept[i].z + kept[i].w * kept[i].w;
  }
  for (int v = threadIdx.x + KEEP * blockDim.x; v < nvec; v += blockDim.x) {
    const float4 x = *reinterpret_cast<const float4*>(orow + v * 4);
    ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
  }
  ss = b2::block_sum(ss, red);
  const float rstd = 1.0f / sqrtf(ss / static_cast<float>(dim) + eps);
  auto sig = [](float x) { return sizeof(T) == 2 ? b2::sigmoid_fast(x) : b2::sigmoid(x); };
  auto finish = [&](int v, float4 x, const float4& g) {
    const float4 wv = __ldg(reinterpret_cast<const float4*>(w + v * 4));
    x.x *= rstd * wv.x * sig(g.x); x.y *= rstd * wv.y * sig(g.y);
    x.z *= rstd * wv.z * sig(g.z); x.w *= rstd * wv.w * sig(g.w);
    b2::store4<T>(out + row * ld_out + v * 4, x);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nvec) finish(v, kept[i], gates[i]);
  }
  for (int v = threadIdx.x + KEEP * blockDim.x; v < nvec; v += blockDim.x) finish(v, *reinterpret_cast<const float4*>(orow + v * 4), b2::load4<T>(gate + row * ldg + v * 4));
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T>
int launch_any(const LinArgs& a, cudaStream_t s) {
  const size_t smem = sizeof(float) * (static_cast<size_t>(a.qk_pad) * (ANY_COLS + 2) + 8 * ANY_COLS);
  if (smem > 48 * 1024) B2_CUDA(cudaFuncSetAttribute(linear_attn_any_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  B2_CUDA(b2_launch(linear_attn_any_kernel<T>, dim3(a.heads, (a.v_pad + ANY_COLS - 1) / ANY_COLS, a.B), dim3(256), smem, s, a));
  return B2_OK;
}

}  // namespace

extern "C" {

int64_t b2_linear_attn_workspace(int dtype, int B, int max_q, int total_q, int heads, int qk_pad, int v_pad) {
  if (max_q <= 0 || B <= 0 || heads <= 0 || !segment_form(dtype, qk_pad, v_pad)) return 0;
  const int seg = segment_length(max_q, total_q, heads, v_pad);
  return max_q <= seg ? 0 : segment_slots(B, total_q, seg) * heads * qk_pad * v_pad * 4;
}

int b2_linear_attn(int dtype, const void* qkv, int64_t ld_qkv, float* o, int64_t ldo, float* state, const int32_t* slots, const int32_t* cu_q,
                   const int32_t* kv_len, const float* decay, const float* decay_powers, int B, int max_q, int total_q, int heads, int qk_pad,
                   int v_pad, void* workspace, int64_t workspace_bytes, int form, void* stream) {
  if (B < 0 || max_q < 0 || heads <= 0 || qk_pad <= 0 || v_pad <= 0 || qk_pad % 8 != 0 || v_pad % 8 != 0) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (cu_q == nullptr && max_q > 1) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if (!qkv || !o || !state || !slots || !kv_len || !decay) return B2_ERR_ARG;
  if (!aligned16(qkv) || !aligned16(o) || !aligned16(state) || ld_qkv % 8 != 0 || ldo % 8 != 0) return B2_ERR_ARG;
  if (qk_pad > 1024 || B > 65535 || ldo < static_cast<int64_t>(heads) * v_pad) return B2_ERR_SHAPE;
  LinArgs a{};
  a.qkv = qkv; a.ld = ld_qkv; a.o = o; a.ldo = ldo; a.state = state; a.slots = slots; a.cu_q = cu_q; a.kv_len = kv_len; a.decay = decay;
  a.B = B; a.heads = heads; a.qk_pad = qk_pad; a.v_pad = v_pad;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_F32) return launch_any<float>(a, s);
  if (form == 1) return launch_any<uint16_t>(a, s);
  if (cu_q == nullptr) {
    B2_CUDA(b2_launch(linear_attn_decode_kernel, dim3(heads * ((v_pad + DEC_COLS - 1) / DEC_COLS), B), dim3(256), 0, s, a));
    return B2_OK;
  }
  if (!segment_form(dtype, qk_pad, v_pad)) return launch_any<uint16_t>(a, s);
  if (decay_powers == nullptr) return B2_ERR_ARG;
  SegArgs sa{};
  sa.a = a;
  sa.powers = decay_powers;
  sa.seg = segment_length(max_q, total_q, heads, v_pad);
  sa.multi = max_q > sa.seg;
  sa.seg_state = static_cast<float*>(workspace);
  if (sa.multi && (workspace == nullptr || workspace_bytes < segment_slots(B, total_q, sa.seg) * heads * qk_pad * v_pad * 4))
    return b2::set_error(B2_ERR_SHAPE, "b2_linear_attn: workspace of %lld bytes is too small", static_cast<long long>(workspace_bytes));
  return qk_pad <= 64 ? launch_segments<64>(sa, max_q, s) : launch_segments<128>(sa, max_q, s);
}

int b2_gated_norm(int dtype, const float* o, int64_t ldo, const void* gate, int64_t ldg, const float* w, float eps, int M, int dim, int dim_pad,
                  void* out, int64_t ld_out, void* stream) {
  if (M < 0 || dim <= 0 || dim_pad < dim || dim_pad % 8 != 0 || ldo % 4 != 0 || ldg % 8 != 0 || ld_out % 8 != 0) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!o || !gate || !w || !out || !aligned16(o) || !aligned16(gate) || !aligned16(w) || !aligned16(out)) return B2_ERR_ARG;
  if (ldo < dim_pad || ldg < dim_pad || ld_out < dim_pad) return B2_ERR_ARG;
  const int nvec = dim_pad / 4;
  const int threads = std::min(M <= 296 ? 1024 : 256, (nvec + 31) / 32 * 32);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_BF16)
    B2_CUDA(b2_launch(gated_norm_kernel<uint16_t>, dim3(M), dim3(threads), 0, s, o, ldo, static_cast<const uint16_t*>(gate), ldg, w, eps, dim,
                      dim_pad, static_cast<uint16_t*>(out), ld_out));
  else
    B2_CUDA(b2_launch(gated_norm_kernel<float>, dim3(M), dim3(threads), 0, s, o, ldo, static_cast<const float*>(gate), ldg, w, eps, dim, dim_pad,
                      static_cast<float*>(out), ld_out));
  return B2_OK;
}

}  // extern "C"
