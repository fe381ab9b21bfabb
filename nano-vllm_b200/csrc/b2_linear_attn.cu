// Linear attention with a constant decay per head ("lightning attention"):
//     S_t = decay_h S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t
// The state S [dim, vdim] of every head lives in fp32, one slot per sequence; a sequence that starts at position 0
// starts from zero whatever its slot holds.
//
//   linear_attn_any_kernel     any size, bf16 or fp32, token by token (also decode)
//   gated_norm_kernel          RMSNorm over the concatenated heads times sigmoid(gate)
#include <algorithm>

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
// out = o / sqrt(mean(o^2) + eps) * w * sigmoid(gate); o in fp32, the mean over `dim` true elements of a row of
// dim_pad (the padding of o is zero).  One CTA per row.
// ---------------------------------------------------------------------------
template <typename T>
__global__ void gated_norm_kernel(const float* __restrict__ o, int64_t ldo, const T* __restrict__ gate, int64_t ldg,
                                  const float* __restrict__ w, float eps, int dim, int dim_pad, T* __restrict__ out, int64_t ld_out) {
  __shared__ float red[32];
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int row = blockIdx.x;
  const int nvec = dim_pad >> 2;
  const float* orow = o + row * ldo;
  constexpr int KEEP = 4;  // vectors of the row a thread keeps in registers
  float4 kept[KEEP];
  float ss = 0.f;
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
  auto finish = [&](int v, float4 x) {
    const float4 g = b2::load4<T>(gate + row * ldg + v * 4);
    const float4 wv = __ldg(reinterpret_cast<const float4*>(w + v * 4));
    x.x *= rstd * wv.x * b2::sigmoid(g.x); x.y *= rstd * wv.y * b2::sigmoid(g.y);
    x.z *= rstd * wv.z * b2::sigmoid(g.z); x.w *= rstd * wv.w * b2::sigmoid(g.w);
    b2::store4<T>(out + row * ld_out + v * 4, x);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nvec) finish(v, kept[i]);
  }
  for (int v = threadIdx.x + KEEP * blockDim.x; v < nvec; v += blockDim.x) finish(v, *reinterpret_cast<const float4*>(orow + v * 4));
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

int64_t b2_linear_attn_workspace(int dtype, int B, int max_q, int total_q, int heads, int qk_pad, int v_pad) { return 0; }

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
  return dtype == B2_DT_BF16 ? launch_any<uint16_t>(a, s) : launch_any<float>(a, s);
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
