// Element access shared by kernels that exist for bf16 and for fp32 activations.
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace eredu {

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

// Four consecutive elements (16-byte aligned fp32, 8-byte aligned bf16).
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const __nv_bfloat16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xFFFF0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xFFFF0000u));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&a);
  u.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

__device__ __forceinline__ float sigmoid_f32(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f32(float x) { return x / (1.f + expf(-x)); }
// The same from the approximate exponential and reciprocal (a few units in the last place), for bf16 results or inputs.
__device__ __forceinline__ float sigmoid_fast(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
__device__ __forceinline__ float silu_fast(float x) { return x * sigmoid_fast(x); }
// log(sigmoid(x)) without overflow for either sign
__device__ __forceinline__ float log_sigmoid_f32(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }

// xIELU: above z^2 + z / 2 for z > 0, below (e^z - 1 - z) + z / 2 elsewhere. Near zero e^z - 1 - z comes from its power series, where the
// difference would cancel. FAST: the approximate exponential, for bf16 results.
template <bool FAST>
__device__ __forceinline__ float xielu(float z, float above, float below) {
  const float n = fminf(z, 0.f);
  const float series = n * n * fmaf(n, fmaf(n, fmaf(n, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f);
  const float tail = n > -0.0625f ? series : (FAST ? __expf(n) : expf(n)) - 1.f - n;
  return fmaf(0.5f, z, z > 0.f ? above * z * z : below * tail);
}

__device__ __forceinline__ float warp_sum_f32(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over the block (every thread gets it); `red` holds one float per warp, and may be used again after the call.
__device__ __forceinline__ float block_sum_f32(float v, float* red) {
  v = warp_sum_f32(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < static_cast<int>((blockDim.x + 31) >> 5); ++w) t += red[w];
  __syncthreads();
  return t;
}

}  // namespace eredu
