// fp32 matrix product on the CUDA cores (no reduced-precision tensor mode), for models run in true 32-bit:
// C[M, N] = A[M, K] W[N, K]^T with the same epilogues as the bf16 GEMM (a leading range of SiLU columns, or
// gate/up row pairs).  64 x 64 tiles, 4 x 4 outputs per thread.
#include "b2_vec.cuh"

namespace {

constexpr int TM = 64, TN = 64, TK = 16;

__device__ __forceinline__ float act_pair(float g, float u, int act) {
  return (act == B2_ACT_RELU ? fmaxf(g, 0.f) : g * b2::sigmoid(g)) * u;
}

__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* A, int64_t lda, const float* __restrict__ W, int64_t ldw,
                                                       float* C, int64_t ldc, int M, int N, int K, int pair_act, int silu_cols) {
  __shared__ float sa[TK][TM + 4];
  __shared__ float sw[TK][TN + 4];
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int m0 = blockIdx.y * TM, n0 = blockIdx.x * TN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const int lr = threadIdx.x >> 2, lk = (threadIdx.x & 3) * 4;  // this thread's row and first k of the tile loads
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += TK) {
    float4 va = make_float4(0.f, 0.f, 0.f, 0.f), vw = va;
    if (k0 + lk < K) {  // K is a multiple of 8, so a vector of 4 never straddles its end
      if (m0 + lr < M) va = *reinterpret_cast<const float4*>(A + (m0 + lr) * lda + k0 + lk);
      if (n0 + lr < N) vw = *reinterpret_cast<const float4*>(W + (n0 + lr) * ldw + k0 + lk);
    }
    __syncthreads();
    sa[lk][lr] = va.x; sa[lk + 1][lr] = va.y; sa[lk + 2][lr] = va.z; sa[lk + 3][lr] = va.w;
    sw[lk][lr] = vw.x; sw[lk + 1][lr] = vw.y; sw[lk + 2][lr] = vw.z; sw[lk + 3][lr] = vw.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      const float4 a4 = *reinterpret_cast<const float4*>(&sa[k][ty * 4]);
      const float4 w4 = *reinterpret_cast<const float4*>(&sw[k][tx * 4]);
      const float av[4] = {a4.x, a4.y, a4.z, a4.w}, wv[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) break;
    const int n = n0 + tx * 4;
    if (pair_act != B2_ACT_NONE) {
#pragma unroll
      for (int j = 0; j < 4; j += 2)
        if (n + j < N) C[m * ldc + ((n + j) >> 1)] = act_pair(acc[i][j], acc[i][j + 1], pair_act);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n + j < N) C[m * ldc + n + j] = (n + j < silu_cols) ? acc[i][j] * b2::sigmoid(acc[i][j]) : acc[i][j];
    }
  }
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace

extern "C" {

int b2_gemm_f32(const float* A, int64_t lda, const float* W, int64_t ldw, float* C, int64_t ldc, int M, int N, int K, int pair_act,
                int silu_cols, void* stream) {
  if (M < 0 || N <= 0 || K <= 0 || K % 8 != 0 || N % 2 != 0 || lda % 4 != 0 || ldw % 4 != 0 || lda < K || ldw < K) return B2_ERR_ARG;
  if (pair_act != B2_ACT_NONE && pair_act != B2_ACT_SILU && pair_act != B2_ACT_RELU) return B2_ERR_ARG;
  if (ldc < (pair_act != B2_ACT_NONE ? N / 2 : N) || silu_cols < 0) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!A || !W || !C || !aligned16(A) || !aligned16(W)) return B2_ERR_ARG;
  const dim3 grid((N + TN - 1) / TN, (M + TM - 1) / TM);
  if (grid.y > 65535) return B2_ERR_SHAPE;
  B2_CUDA(b2_launch(gemm_f32_kernel, grid, dim3(256), 0, static_cast<cudaStream_t>(stream), A, lda, W, ldw, C, ldc, M, N, K, pair_act, silu_cols));
  return B2_OK;
}

}  // extern "C"
