// Element-type helpers of the kernels that serve bf16 and fp32 activations: vectors of 4 and 8 elements to and
// from fp32 registers, warp and block sums, and the per-sequence batch description.
#pragma once

#include "b2_common.cuh"

namespace b2 {

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&f)[8]);
template <>
__device__ __forceinline__ void load8<uint16_t>(const uint16_t* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  f[0] = bf16_lo(v.x); f[1] = bf16_hi(v.x); f[2] = bf16_lo(v.y); f[3] = bf16_hi(v.y);
  f[4] = bf16_lo(v.z); f[5] = bf16_hi(v.z); f[6] = bf16_lo(v.w); f[7] = bf16_hi(v.w);
}
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&f)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&f)[8]);
template <>
__device__ __forceinline__ void store8<uint16_t>(uint16_t* p, const float (&f)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(f[0], f[1]), pack_bf16(f[2], f[3]), pack_bf16(f[4], f[5]), pack_bf16(f[6], f[7]));
}
template <>
__device__ __forceinline__ void store8<float>(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(f[0], f[1], f[2], f[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(f[4], f[5], f[6], f[7]);
}

template <typename T>
__device__ __forceinline__ float4 load4(const T* p);
template <>
__device__ __forceinline__ float4 load4<uint16_t>(const uint16_t* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  return make_float4(bf16_lo(v.x), bf16_hi(v.x), bf16_lo(v.y), bf16_hi(v.y));
}
template <>
__device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <typename T>
__device__ __forceinline__ void store4(T* p, const float4& f);
template <>
__device__ __forceinline__ void store4<uint16_t>(uint16_t* p, const float4& f) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(f.x, f.y), pack_bf16(f.z, f.w));
}
template <>
__device__ __forceinline__ void store4<float>(float* p, const float4& f) { *reinterpret_cast<float4*>(p) = f; }

__device__ __forceinline__ float to_float(uint16_t v) { return __uint_as_float(static_cast<uint32_t>(v) << 16); }
__device__ __forceinline__ float to_float(float v) { return v; }
template <typename T>
__device__ __forceinline__ T from_float(float v);
template <>
__device__ __forceinline__ uint16_t from_float<uint16_t>(float v) { return static_cast<uint16_t>(pack_bf16(v, 0.f) & 0xFFFF); }
template <>
__device__ __forceinline__ float from_float<float>(float v) { return v; }

template <int LANES = 32>
__device__ __forceinline__ float group_sum(float v) {
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// sum over the block; `red` holds one float per warp (at most 32); every thread returns the total
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = group_sum(v);
  const int warps = (blockDim.x + 31) >> 5;
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  v = 0.f;
  for (int i = 0; i < warps; ++i) v += red[i];
  return v;
}

__device__ __forceinline__ float sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
// a few units in the last place of fp32: for values that are rounded to bf16
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }

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

}  // namespace b2
