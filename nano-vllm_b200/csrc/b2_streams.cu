// Residual streams in fp32.  A decoder with hyper-connections keeps S copies of the residual; a sublayer reads one
// combination of them and its output is added to every copy after the copies have been mixed.  One launch covers
// everything between two sublayers:
//     x_t <- sum_s mix[s, t] x_s + m out[t] y           (skipped where there is no y)
//     u    = sum_s in[s] x_s                             (in = 1 for every s after the last sublayer)
//     normed = u / sqrt(mean(u^2) + eps) * w
// and the embedding lookup takes the place of the first line at the start of the model.
// The copies are read and written once per sublayer; u stays in shared memory.
#include <algorithm>

#include "b2_vec.cuh"

namespace {

struct StreamArgs {
  const float* x_in;
  float* x_out;  // may be x_in; null = not written
  const int64_t* ids;
  const void* table;
  int64_t ld_table, vocab;
  float scale;
  const void* y;
  int64_t ldy;
  const float* mix;
  const float* w_out;
  float m;
  const float* w_in;
  const float* norm_w;
  float eps;
  void* normed;
  int64_t ldn;
  int M, S, dim, dim_pad;
};

constexpr int MAX_STREAMS = 32;

// ST > 0: number of streams at compile time; ST = 0: a.S streams (at most MAX_STREAMS)
constexpr int MAX_THREADS = 512;

template <typename T, int ST>
__global__ void __launch_bounds__(MAX_THREADS) stream_step_kernel(const StreamArgs a) {
  extern __shared__ float u_row[];  // [dim_pad]
  __shared__ float coef[MAX_STREAMS * MAX_STREAMS + 2 * MAX_STREAMS];
  __shared__ float red[32];
  constexpr int CAP = ST > 0 ? ST : MAX_STREAMS;
  const int S = ST > 0 ? ST : a.S;
  b2::pdl_launch_dependents();
  float* c_mix = coef;
  float* c_out = coef + S * S;
  float* c_in = c_out + S;
  const bool update = a.y != nullptr;
  // the coefficients are weights: no earlier kernel writes them
  if (update) {
    for (int i = threadIdx.x; i < S * S; i += blockDim.x) c_mix[i] = a.mix[i];
    for (int i = threadIdx.x; i < S; i += blockDim.x) c_out[i] = a.m * a.w_out[i];
  }
  for (int i = threadIdx.x; i < S; i += blockDim.x) c_in[i] = a.w_in != nullptr ? a.w_in[i] : 1.0f;
  __syncthreads();
  b2::pdl_wait();
  const int row = blockIdx.x;
  const int nvec = a.dim_pad >> 2;
  const T* emb = nullptr;
  if (a.ids != nullptr) {
    int64_t id = a.ids[row];
    if (id < 0 || id >= a.vocab) id = 0;
    emb = static_cast<const T*>(a.table) + id * a.ld_table;
  }
  const float* xr = a.x_in + static_cast<int64_t>(row) * S * a.dim_pad;
  float* xw = a.x_out + static_cast<int64_t>(row) * S * a.dim_pad;
  const T* yr = update ? static_cast<const T*>(a.y) + row * a.ldy : nullptr;
  float ss = 0.f;
#pragma unroll 2
  for (int v = threadIdx.x; v < nvec; v += blockDim.x) {
    float4 x[CAP];
    if (emb != nullptr) {
      float4 e = b2::load4<T>(emb + v * 4);
      e.x *= a.scale; e.y *= a.scale; e.z *= a.scale; e.w *= a.scale;
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S) x[s] = e;
    } else {
#pragma unroll
      for (int s = 0; s < CAP; ++s)
        if (s < S) x[s] = *reinterpret_cast<const float4*>(xr + static_cast<int64_t>(s) * a.dim_pad + v * 4);
    }
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    if (update) y = b2::load4<T>(yr + v * 4);
    float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int t = 0; t < CAP; ++t) {
      if (t >= S) break;
      float4 n;
      if (update) {
        const float o = c_out[t];
        n = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
        for (int s = 0; s < CAP; ++s) {
          if (s >= S) break;
          const float c = c_mix[s * S + t];
          n.x += c * x[s].x; n.y += c * x[s].y; n.z += c * x[s].z; n.w += c * x[s].w;
        }
      } else {
        n = x[t];
      }
      if (a.x_out != nullptr) *reinterpret_cast<float4*>(xw + static_cast<int64_t>(t) * a.dim_pad + v * 4) = n;
      const float ci = c_in[t];
      u.x += ci * n.x; u.y += ci * n.y; u.z += ci * n.z; u.w += ci * n.w;
    }
    *reinterpret_cast<float4*>(u_row + v * 4) = u;
    ss += u.x * u.x + u.y * u.y + u.z * u.z + u.w * u.w;
  }
  if (a.normed == nullptr) return;
  ss = b2::block_sum(ss, red);
  const float rstd = 1.0f / sqrtf(ss / static_cast<float>(a.dim) + a.eps);
  T* nr = static_cast<T*>(a.normed) + row * a.ldn;
  for (int v = threadIdx.x; v < nvec; v += blockDim.x) {  // each thread reads back what it wrote itself
    float4 u = *reinterpret_cast<const float4*>(u_row + v * 4);
    const float4 w = __ldg(reinterpret_cast<const float4*>(a.norm_w + v * 4));
    u.x = u.x * rstd * w.x; u.y = u.y * rstd * w.y; u.z = u.z * rstd * w.z; u.w = u.w * rstd * w.w;
    b2::store4<T>(nr + v * 4, u);
  }
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, int ST>
int launch_step(const StreamArgs& a, cudaStream_t s) {
  const int nvec = a.dim_pad / 4;
  // few rows: more threads per row; many rows: 256 threads, so that several rows share an SM
  const int threads = std::min(a.M <= 296 ? MAX_THREADS : 256, (nvec + 31) / 32 * 32);
  const size_t smem = static_cast<size_t>(a.dim_pad) * sizeof(float);
  if (smem > 48 * 1024) B2_CUDA(cudaFuncSetAttribute(stream_step_kernel<T, ST>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  B2_CUDA(b2_launch(stream_step_kernel<T, ST>, dim3(a.M), dim3(threads), smem, s, a));
  return B2_OK;
}

template <typename T>
int dispatch_step(const StreamArgs& a, cudaStream_t s) {
  switch (a.S) {
    case 1: return launch_step<T, 1>(a, s);
    case 2: return launch_step<T, 2>(a, s);
    case 3: return launch_step<T, 3>(a, s);
    case 4: return launch_step<T, 4>(a, s);
    case 6: return launch_step<T, 6>(a, s);
    case 8: return launch_step<T, 8>(a, s);
    default: return launch_step<T, 0>(a, s);
  }
}

}  // namespace

extern "C" {

int b2_stream_step(int dtype, float* x_out, const float* x_in, const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab,
                   float embed_scale, const void* y, int64_t ldy, const float* mix, const float* w_out, float mult, const float* w_in,
                   const float* norm_w, float eps, void* normed, int64_t ldn, int M, int streams, int dim, int dim_pad, void* stream) {
  if (M < 0 || streams < 1 || streams > MAX_STREAMS || dim < 1 || dim_pad < dim || dim_pad % 8 != 0 || dim_pad > 49152) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if ((ids == nullptr) == (x_in == nullptr)) return B2_ERR_ARG;
  if (ids != nullptr && (!table || !aligned16(table) || vocab <= 0 || ld_table < dim_pad || ld_table % 8 != 0)) return B2_ERR_ARG;
  if (x_in != nullptr && !aligned16(x_in)) return B2_ERR_ARG;
  if (y != nullptr && (!mix || !w_out || !aligned16(y) || ldy < dim_pad || ldy % 8 != 0)) return B2_ERR_ARG;
  if (x_out != nullptr && !aligned16(x_out)) return B2_ERR_ARG;
  if (normed != nullptr && (!norm_w || !aligned16(norm_w) || !aligned16(normed) || ldn < dim_pad || ldn % 8 != 0)) return B2_ERR_ARG;
  StreamArgs a{};
  a.x_in = x_in; a.x_out = x_out; a.ids = ids; a.table = table; a.ld_table = ld_table; a.vocab = vocab; a.scale = embed_scale;
  a.y = y; a.ldy = ldy; a.mix = mix; a.w_out = w_out; a.m = mult; a.w_in = w_in; a.norm_w = norm_w; a.eps = eps;
  a.normed = normed; a.ldn = ldn; a.M = M; a.S = streams; a.dim = dim; a.dim_pad = dim_pad;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == B2_DT_BF16 ? dispatch_step<uint16_t>(a, s) : dispatch_step<float>(a, s);
}

}  // extern "C"
