// The residual of a decoder with norms before and after its sublayers and a short causal convolution on what a sublayer
// reads.  One launch covers everything between two sublayers (x fp32, all norms fp32):
//     x  <- x + post * y / rms(y)            (at the start of the model: x = table[id])
//     h   = norm * x / rms(x)                 rounded to the activations' type
//     out = h + sum_j w[j] h_(t - taps + 1 + j)   per channel, zeros before the sequence's first token
// A CTA walks a run of consecutive tokens of one sequence with the last taps - 1 values of h of its channels at hand.  What
// lies before the run is computed again from x and y (x is written to another buffer, so both are intact); before the step's
// first token it comes from the sequence's state slot, which the sequence's first CTA replaces with the step's last values.
#include <algorithm>

#include "b2_vec.cuh"

namespace {

struct SandwichArgs {
  const float* x_in;
  float* x_out;  // another buffer than x_in; null = not written
  const int64_t* ids;
  const void* table;
  int64_t ld_table, vocab;
  const void* y;
  int64_t ldy;
  const float* post_w;
  int post_vec;  // 1: one weight per channel; 0: a single number
  const float* norm_w;
  int norm_vec;
  float eps;
  const void* conv_w;  // [taps][dim_pad]
  int taps;            // 0 = no convolution
  void* state;         // [slots][taps - 1][dim_pad]
  const int32_t* slots;
  const int32_t* cu_q;    // null = one row per sequence
  const int32_t* kv_len;
  void* out;
  int64_t ldo;
  int dim, dim_pad, run;  // run: tokens per CTA
};

template <typename T>
struct Vec8;
template <>
struct Vec8<uint16_t> {
  uint4 v;
  __device__ __forceinline__ void zero() { v = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void load(const uint16_t* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void store(uint16_t* p) const { *reinterpret_cast<uint4*>(p) = v; }
  __device__ __forceinline__ void set(const float (&f)[8]) {
    v = make_uint4(b2::pack_bf16(f[0], f[1]), b2::pack_bf16(f[2], f[3]), b2::pack_bf16(f[4], f[5]), b2::pack_bf16(f[6], f[7]));
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = b2::bf16_lo(v.x); f[1] = b2::bf16_hi(v.x); f[2] = b2::bf16_lo(v.y); f[3] = b2::bf16_hi(v.y);
    f[4] = b2::bf16_lo(v.z); f[5] = b2::bf16_hi(v.z); f[6] = b2::bf16_lo(v.w); f[7] = b2::bf16_hi(v.w);
  }
};
template <>
struct Vec8<float> {
  float4 a, b;
  __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void load(const float* p) {
    a = *reinterpret_cast<const float4*>(p);
    b = *reinterpret_cast<const float4*>(p + 4);
  }
  __device__ __forceinline__ void store(float* p) const {
    *reinterpret_cast<float4*>(p) = a;
    *reinterpret_cast<float4*>(p + 4) = b;
  }
  __device__ __forceinline__ void set(const float (&f)[8]) {
    a = make_float4(f[0], f[1], f[2], f[3]);
    b = make_float4(f[4], f[5], f[6], f[7]);
  }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
};

// TAPS > 0: that many taps, history and weights in registers; 0: no convolution; -1: a.taps, history in shared memory.
// NV vectors of 8 channels per thread; RB tokens at a time, so that their loads are in flight together and share barriers.
template <typename T, int NV, int TAPS, int RB>
__global__ void __launch_bounds__(512, RB == 2 && sizeof(T) == 2 ? 2 : 1) sandwich_step_kernel(const SandwichArgs a) {
  extern __shared__ __align__(16) unsigned char hist_smem[];  // TAPS < 0: [taps - 1][dim_pad], a ring by row
  __shared__ __align__(16) float red[2][16][RB];
  constexpr bool CONV = TAPS != 0, REG = TAPS > 0;
  constexpr int HIST = REG && TAPS > 1 ? TAPS - 1 : 1;
  const int taps = REG ? TAPS : a.taps;
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int b = blockIdx.x, start = blockIdx.y * a.run;
  const int row0 = a.cu_q ? a.cu_q[b] : b;
  const int n_q = a.cu_q ? a.cu_q[b + 1] - row0 : 1;
  if (start >= n_q) return;
  const int stop = min(n_q, start + a.run);
  int nv[NV];  // this thread's first channel of every vector, -1 = none
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    nv[i] = c < a.dim_pad ? c : -1;
  }
  T* ring = reinterpret_cast<T*>(hist_smem);
  constexpr bool KEEP_W = REG && RB == 1;  // else the weights come from the L1 cache for every token
  Vec8<T> hist[HIST][NV], w[KEEP_W ? TAPS : 1][NV];
  int head = 0;  // the ring's oldest row
  if constexpr (KEEP_W) {
    const T* cw = static_cast<const T*>(a.conv_w);
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (nv[i] >= 0) w[j][i].load(cw + static_cast<int64_t>(j) * a.dim_pad + nv[i]);
  }
  const int slot = CONV && a.slots != nullptr ? a.slots[b] : -1;
  T* state = CONV && slot >= 0 ? static_cast<T*>(a.state) + static_cast<int64_t>(slot) * (taps - 1) * a.dim_pad : nullptr;
  if constexpr (CONV) {  // the history in front of the run: zeros, or the state where the run is the step's first
    const bool keep = start == 0 && state != nullptr && a.kv_len[b] - n_q > 0;
#pragma unroll
    for (int j = 0; j < (REG ? TAPS - 1 : taps - 1); ++j)
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (nv[i] < 0) continue;
        Vec8<T> v;
        v.zero();
        if (keep) v.load(state + static_cast<int64_t>(j) * a.dim_pad + nv[i]);
        if constexpr (REG) hist[j][i] = v;
        else v.store(ring + static_cast<int64_t>(j) * a.dim_pad + nv[i]);
      }
  }
  const int warps = (blockDim.x + 31) >> 5;
  int flip = 0;
  auto total = [&](float (&v)[RB]) {  // sums over the CTA; two buffers in turn, so one barrier per call is enough
#pragma unroll
    for (int r = 0; r < RB; ++r) v[r] = b2::group_sum(v[r]);
    if ((threadIdx.x & 31) == 0) {
#pragma unroll
      for (int r = 0; r < RB; ++r) red[flip][threadIdx.x >> 5][r] = v[r];
    }
    __syncthreads();
#pragma unroll
    for (int r = 0; r < RB; ++r) v[r] = 0.f;
    for (int i = 0; i < warps; ++i) {
      if constexpr (RB == 4) {
        const float4 q = *reinterpret_cast<const float4*>(red[flip][i]);
        v[0] += q.x; v[1] += q.y; v[2] += q.z; v[3] += q.w;
      } else {
#pragma unroll
        for (int r = 0; r < RB; ++r) v[r] += red[flip][i][r];
      }
    }
    flip ^= 1;
  };
  const float inv_dim = 1.0f / static_cast<float>(a.dim);

  // tokens t0 .. min(t0 + RB, end) - 1, of which those from `emit` on are written
  auto process = [&](int t0, int end, int emit) {
    float x[RB][NV][8], ss[RB];
    Vec8<T> y[RB][NV];
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      const bool live = t0 + r < end;
      const int64_t row = row0 + t0 + (live ? r : 0);
      const T* emb = nullptr;
      if (a.ids != nullptr) {
        int64_t id = a.ids[row];
        if (id < 0 || id >= a.vocab) id = 0;
        emb = static_cast<const T*>(a.table) + id * a.ld_table;
      }
#pragma unroll
      for (int i = 0; i < NV; ++i) {
#pragma unroll
        for (int e = 0; e < 8; ++e) x[r][i][e] = 0.f;
        y[r][i].zero();
        if (nv[i] < 0) continue;
        if (emb != nullptr) b2::load8<T>(emb + nv[i], x[r][i]);
        else b2::load8<float>(a.x_in + row * a.dim_pad + nv[i], x[r][i]);
        if (a.y != nullptr) y[r][i].load(static_cast<const T*>(a.y) + row * a.ldy + nv[i]);
      }
    }
    if (a.y != nullptr) {
#pragma unroll
      for (int r = 0; r < RB; ++r) {
        ss[r] = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          float f[8];
          y[r][i].get(f);
#pragma unroll
          for (int e = 0; e < 8; ++e) ss[r] += f[e] * f[e];
        }
      }
      total(ss);
      float g[8];
#pragma unroll
      for (int e = 0; e < 8; ++e) g[e] = a.post_w[0];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (nv[i] < 0) continue;
        if (a.post_vec) b2::load8<float>(a.post_w + nv[i], g);
#pragma unroll
        for (int r = 0; r < RB; ++r) {
          const float rstd = 1.0f / sqrtf(ss[r] * inv_dim + a.eps);
          float f[8];
          y[r][i].get(f);
#pragma unroll
          for (int e = 0; e < 8; ++e) x[r][i][e] += f[e] * (rstd * g[e]);
        }
      }
    }
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      const bool out = t0 + r >= emit && t0 + r < end;
      ss[r] = 0.f;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
#pragma unroll
        for (int e = 0; e < 8; ++e) ss[r] += x[r][i][e] * x[r][i][e];
        if (out && a.x_out != nullptr && nv[i] >= 0) b2::store8<float>(a.x_out + (row0 + t0 + r) * static_cast<int64_t>(a.dim_pad) + nv[i], x[r][i]);
      }
    }
    total(ss);
#pragma unroll
    for (int r = 0; r < RB; ++r) {
      if (t0 + r >= end) break;
      const int64_t row = row0 + t0 + r;
      const float rstd = 1.0f / sqrtf(ss[r] * inv_dim + a.eps);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (nv[i] < 0) continue;
        if (a.norm_vec) {
          float g[8];
          b2::load8<float>(a.norm_w + nv[i], g);
#pragma unroll
          for (int e = 0; e < 8; ++e) x[r][i][e] = x[r][i][e] * rstd * g[e];
        } else {
          const float g = rstd * a.norm_w[0];
#pragma unroll
          for (int e = 0; e < 8; ++e) x[r][i][e] *= g;
        }
        Vec8<T> h;
        h.set(x[r][i]);
        T* dst = static_cast<T*>(a.out) + row * a.ldo + nv[i];
        if constexpr (!CONV) {
          h.store(dst);
        } else {
          if (t0 + r >= emit) {
            float acc[8], hf[8], wf[8];
            h.get(hf);
            if constexpr (KEEP_W) w[TAPS - 1][i].get(wf);
            else b2::load8<T>(static_cast<const T*>(a.conv_w) + static_cast<int64_t>(taps - 1) * a.dim_pad + nv[i], wf);
#pragma unroll
            for (int e = 0; e < 8; ++e) acc[e] = fmaf(wf[e], hf[e], hf[e]);
#pragma unroll
            for (int j = 0; j < (REG ? TAPS - 1 : taps - 1); ++j) {
              float f[8];
              if constexpr (KEEP_W) w[j][i].get(wf);
              else b2::load8<T>(static_cast<const T*>(a.conv_w) + static_cast<int64_t>(j) * a.dim_pad + nv[i], wf);
              if constexpr (REG) {
                hist[j][i].get(f);
              } else {
                b2::load8<T>(ring + static_cast<int64_t>((head + j) % (taps - 1)) * a.dim_pad + nv[i], f);
              }
#pragma unroll
              for (int e = 0; e < 8; ++e) acc[e] = fmaf(wf[e], f[e], acc[e]);
            }
            b2::store8<T>(dst, acc);
          }
          if constexpr (REG) {
#pragma unroll
            for (int j = 0; j + 1 < TAPS - 1; ++j) hist[j][i] = hist[j + 1][i];
            if (TAPS > 1) hist[HIST - 1][i] = h;
          } else if (taps > 1) {
            h.store(ring + static_cast<int64_t>(head) * a.dim_pad + nv[i]);
          }
        }
      }
      if (!REG && CONV && taps > 1) head = (head + 1) % (taps - 1);
    }
  };

  // the tokens before a later run are part of the step (run >= taps - 1): computed again, not written
  for (int t = CONV && start > 0 ? start - (taps - 1) : start; t < stop; t += RB) process(t, stop, start);
  if constexpr (CONV) {
    if (start > 0 || state == nullptr) return;
    if (stop < n_q)
      for (int t = n_q - (taps - 1); t < n_q; t += RB) process(t, n_q, n_q);
#pragma unroll
    for (int j = 0; j < (REG ? TAPS - 1 : taps - 1); ++j)
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        if (nv[i] < 0) continue;
        T* dst = state + static_cast<int64_t>(j) * a.dim_pad + nv[i];
        if constexpr (REG) {
          hist[j][i].store(dst);
        } else {
          Vec8<T> v;
          v.load(ring + static_cast<int64_t>((head + j) % (taps - 1)) * a.dim_pad + nv[i]);
          v.store(dst);
        }
      }
  }
}

bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <typename T, int NV, int TAPS, int RB>
int launch(SandwichArgs a, int B, int max_q, int run, int threads, size_t smem, cudaStream_t s) {
  const auto kernel = sandwich_step_kernel<T, NV, TAPS, RB>;
  if (smem > 48 * 1024) B2_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)));
  const int back = a.taps > 0 ? a.taps - 1 : 0;
  if (max_q == 1) run = 1;
  if (run == 0) {
    // tokens per CTA: the fewest rounds of groups over all SMs, where a run also walks the tokens in front of it
    static int known_threads = -1, known = 1;  // of the last thread count asked for: a model has one
    if (threads != known_threads) {
      B2_CUDA(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&known, kernel, threads, smem));
      known_threads = threads;
    }
    const int resident = known;
    const int64_t at_once = 148ll * std::max(1, resident);
    int64_t best = INT64_MAX;
    for (int groups = 1; groups <= 16; ++groups) {
      const int r = groups * RB - back;
      if (r < 1) continue;
      const int64_t ctas = static_cast<int64_t>(B) * ((max_q + r - 1) / r);
      const int64_t cost = (ctas + at_once - 1) / at_once * groups;
      if (cost < best) {
        best = cost;
        run = r;
      }
      if (r >= max_q) break;
    }
  }
  a.run = std::max({run, back, (max_q + 65534) / 65535, 1});
  B2_CUDA(b2_launch(kernel, dim3(B, (max_q + a.run - 1) / a.run), dim3(threads), smem, s, a));
  return B2_OK;
}
template <typename T, int NV>
int dispatch_taps(const SandwichArgs& a, int B, int max_q, int run, int threads, cudaStream_t s) {
#define B2_STEP(TAPS) return max_q > 1 ? launch<T, NV, TAPS, 2>(a, B, max_q, run, threads, 0, s) : launch<T, NV, TAPS, 1>(a, B, max_q, run, threads, 0, s)
  if (a.taps == 0) return launch<T, NV, 0, 1>(a, B, max_q, run, threads, 0, s);
  if constexpr (NV == 1) {
    switch (a.taps) {
      case 2: B2_STEP(2);
      case 3: B2_STEP(3);
      case 4: B2_STEP(4);
      default: break;
    }
  }
#undef B2_STEP
  const size_t smem = static_cast<size_t>(a.taps - 1) * a.dim_pad * sizeof(T);
  if (smem > 200 * 1024) return b2::set_error(B2_ERR_SHAPE, "b2_sandwich_step: %d taps on %d channels do not fit in shared memory", a.taps, a.dim_pad);
  return launch<T, NV, -1, 1>(a, B, max_q, run, threads, smem, s);
}
template <typename T>
int dispatch(const SandwichArgs& a, int B, int max_q, int run, cudaStream_t s) {
  const int nvec = a.dim_pad / 8;
  if (nvec <= 512) return dispatch_taps<T, 1>(a, B, max_q, run, (nvec + 31) / 32 * 32, s);
  if (nvec <= 1024) return dispatch_taps<T, 2>(a, B, max_q, run, (nvec + 63) / 64 * 32, s);
  return dispatch_taps<T, 8>(a, B, max_q, run, 512, s);
}

// out = a N(z) + b N(z^2) + c N(z^3) + e, N dividing by the root mean square over the row's `dim` elements
// KEEP vectors of 8 per thread stay in registers, longer rows are read again: many for few rows, few where many rows share an SM
template <typename T, int KEEP>
__global__ void __launch_bounds__(512, KEEP <= 3 ? 3 : 1) poly_norm_kernel(const T* z, int64_t ldz, const float* coef, float eps, int dim, int dim_pad, T* out, int64_t ldo) {
  __shared__ float red[3][32];
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int64_t row = blockIdx.x;
  const T* zr = z + row * ldz;
  Vec8<T> kept[KEEP];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
  auto add = [&](const float (&f)[8]) {
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float q = f[e] * f[e], q2 = q * q;
      s1 += q;
      s2 += q2;
      s3 += q2 * q;
    }
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    kept[i].zero();
    if (c < dim_pad) kept[i].load(zr + c);
  }
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    float f[8];
    kept[i].get(f);
    add(f);
  }
  for (int c = (threadIdx.x + KEEP * blockDim.x) * 8; c < dim_pad; c += blockDim.x * 8) {
    float f[8];
    b2::load8<T>(zr + c, f);
    add(f);
  }
  s1 = b2::group_sum(s1);
  s2 = b2::group_sum(s2);
  s3 = b2::group_sum(s3);
  if ((threadIdx.x & 31) == 0) {
    red[0][threadIdx.x >> 5] = s1;
    red[1][threadIdx.x >> 5] = s2;
    red[2][threadIdx.x >> 5] = s3;
  }
  __syncthreads();
  s1 = s2 = s3 = 0.f;
  for (int i = 0; i < (static_cast<int>(blockDim.x) + 31) >> 5; ++i) {
    s1 += red[0][i];
    s2 += red[1][i];
    s3 += red[2][i];
  }
  const float inv = 1.0f / static_cast<float>(dim);
  const float p1 = coef[0] / sqrtf(s1 * inv + eps), p2 = coef[1] / sqrtf(s2 * inv + eps), p3 = coef[2] / sqrtf(s3 * inv + eps), p0 = coef[3];
  auto finish = [&](int c, const float (&f)[8]) {
    float r[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) r[e] = c + e < dim ? fmaf(f[e], fmaf(f[e], fmaf(f[e], p3, p2), p1), p0) : 0.f;
    b2::store8<T>(out + row * ldo + c, r);
  };
#pragma unroll
  for (int i = 0; i < KEEP; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 8;
    if (c >= dim_pad) break;
    float f[8];
    kept[i].get(f);
    finish(c, f);
  }
  for (int c = (threadIdx.x + KEEP * blockDim.x) * 8; c < dim_pad; c += blockDim.x * 8) {
    float f[8];
    b2::load8<T>(zr + c, f);
    finish(c, f);
  }
}

// fp32 logits = cap tanh(x scale / cap), or x scale without a cap
template <typename T>
__global__ void __launch_bounds__(256) logit_cap_kernel(const T* x, int64_t ldx, float scale, float cap, int cols, float* out, int64_t ldo) {
  b2::pdl_launch_dependents();
  b2::pdl_wait();
  const int64_t row = blockIdx.y;
  for (int c = (blockIdx.x * 256 + threadIdx.x) * 4; c < cols; c += gridDim.x * 1024) {
    float4 v = b2::load4<T>(x + row * ldx + c);
    v.x *= scale; v.y *= scale; v.z *= scale; v.w *= scale;
    if (cap > 0.f) {
      v.x = cap * tanhf(v.x / cap); v.y = cap * tanhf(v.y / cap);
      v.z = cap * tanhf(v.z / cap); v.w = cap * tanhf(v.w / cap);
    }
    *reinterpret_cast<float4*>(out + row * ldo + c) = v;
  }
}

}  // namespace

extern "C" {

int b2_sandwich_step(int dtype, const float* x_in, float* x_out, const int64_t* ids, const void* table, int64_t ld_table, int64_t vocab, const void* y,
                     int64_t ldy, const float* post_w, int post_len, const float* norm_w, int norm_len, float eps, const void* conv_w, int taps,
                     void* state, const int32_t* slots, const int32_t* cu_q, const int32_t* kv_len, int B, int max_q, void* out, int64_t ldo, int dim,
                     int dim_pad, int run, void* stream) {
  if (B < 0 || max_q < 0 || taps < 0 || dim < 1 || dim_pad < dim || dim_pad % 8 != 0 || (dtype != B2_DT_BF16 && dtype != B2_DT_F32)) return B2_ERR_ARG;
  if (run < 0 || (cu_q == nullptr && max_q > 1)) return B2_ERR_ARG;
  if (B == 0 || max_q == 0) return B2_OK;
  if ((ids == nullptr) == (x_in == nullptr) || !out || !norm_w || !aligned16(out) || ldo < dim_pad || ldo % 8 != 0) return B2_ERR_ARG;
  if ((norm_len != 1 && norm_len != dim_pad) || (norm_len != 1 && !aligned16(norm_w))) return B2_ERR_ARG;
  if (ids != nullptr && (!table || !aligned16(table) || vocab <= 0 || ld_table < dim_pad || ld_table % 8 != 0)) return B2_ERR_ARG;
  if (x_in != nullptr && (!aligned16(x_in) || (x_in == x_out && taps > 0 && cu_q != nullptr))) return B2_ERR_ARG;
  if (x_out != nullptr && !aligned16(x_out)) return B2_ERR_ARG;
  if (y != nullptr && (ids != nullptr || !aligned16(y) || ldy < dim_pad || ldy % 8 != 0 || !post_w || (post_len != 1 && post_len != dim_pad) ||
                       (post_len != 1 && !aligned16(post_w)))) return B2_ERR_ARG;
  if (taps > 0 && (!conv_w || !aligned16(conv_w) || !slots || !kv_len || (taps > 1 && (!state || !aligned16(state))))) return B2_ERR_ARG;
  if (dim_pad > 32768) return B2_ERR_SHAPE;
  SandwichArgs a{};
  a.x_in = x_in; a.x_out = x_out; a.ids = ids; a.table = table; a.ld_table = ld_table; a.vocab = vocab; a.y = y; a.ldy = ldy;
  a.post_w = post_w; a.post_vec = post_len != 1; a.norm_w = norm_w; a.norm_vec = norm_len != 1; a.eps = eps; a.conv_w = conv_w; a.taps = taps;
  a.state = state; a.slots = slots; a.cu_q = cu_q; a.kv_len = kv_len; a.out = out; a.ldo = ldo; a.dim = dim; a.dim_pad = dim_pad;
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  return dtype == B2_DT_BF16 ? dispatch<uint16_t>(a, B, max_q, run, s) : dispatch<float>(a, B, max_q, run, s);
}

int b2_poly_norm(int dtype, const void* z, int64_t ldz, const float* coef, float eps, int M, int dim, int dim_pad, void* out, int64_t ldo, void* stream) {
  if (M < 0 || dim < 1 || dim_pad < dim || dim_pad % 8 != 0 || ldz < dim_pad || ldo < dim_pad || ldz % 8 != 0 || ldo % 8 != 0) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!z || !out || !coef || !aligned16(z) || !aligned16(out)) return B2_ERR_ARG;
  const int nvec = dim_pad / 8;
  const bool many = M > 296;
  const int threads = std::min(512, std::max(32, (nvec + (many ? 3 : 0)) / (many ? 4 : 1) + 31) / 32 * 32);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
#define B2_POLY(T, KEEP) \
  B2_CUDA(b2_launch(poly_norm_kernel<T, KEEP>, dim3(M), dim3(threads), 0, s, static_cast<const T*>(z), ldz, coef, eps, dim, dim_pad, static_cast<T*>(out), ldo))
  if (dtype == B2_DT_BF16) {
    if (many) B2_POLY(uint16_t, 3);
    else B2_POLY(uint16_t, 6);
  } else {
    B2_POLY(float, 4);
  }
#undef B2_POLY
  return B2_OK;
}

int b2_logit_cap(int dtype, const void* x, int64_t ldx, float scale, float cap, int M, int cols, float* out, int64_t ldo, void* stream) {
  if (M < 0 || cols < 1 || cols % 8 != 0 || ldx < cols || ldo < cols || ldx % 8 != 0 || ldo % 4 != 0) return B2_ERR_ARG;
  if (dtype != B2_DT_BF16 && dtype != B2_DT_F32) return B2_ERR_ARG;
  if (M == 0) return B2_OK;
  if (!x || !out || !aligned16(x) || !aligned16(out)) return B2_ERR_ARG;
  if (M > 65535) return B2_ERR_SHAPE;
  const dim3 grid(std::min((cols + 1023) / 1024, 64), M);
  cudaStream_t s = static_cast<cudaStream_t>(stream);
  if (dtype == B2_DT_BF16) B2_CUDA(b2_launch(logit_cap_kernel<uint16_t>, grid, dim3(256), 0, s, static_cast<const uint16_t*>(x), ldx, scale, cap, cols, out, ldo));
  else B2_CUDA(b2_launch(logit_cap_kernel<float>, grid, dim3(256), 0, s, static_cast<const float*>(x), ldx, scale, cap, cols, out, ldo));
  return B2_OK;
}

}  // extern "C"
