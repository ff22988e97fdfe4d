// Element access and reductions shared by the kernels around token mixers (bf16 and fp32 activations).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace mixer {

using bf16 = __nv_bfloat16;

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(bf16 x) { return __bfloat162float(x); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16(v); }
// four consecutive elements (16-byte aligned fp32, 8-byte aligned bf16)
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 u = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<uint32_t*>(&a);
  u.y = *reinterpret_cast<uint32_t*>(&b);
  *reinterpret_cast<uint2*>(p) = u;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// sum over the block, returned to every thread; `red` holds one float per warp plus the total
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) t += red[w];
  __syncthreads();
  return t;
}
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.f + expf(-x)); }
// the same for values that came from, or end in, bf16: the hardware exponential and reciprocal (a few ulp of fp32)
template <typename T>
__device__ __forceinline__ float sigmoid_t(float x) { return sigmoid_f(x); }
template <>
__device__ __forceinline__ float sigmoid_t<bf16>(float x) { return __fdividef(1.f, 1.f + __expf(-x)); }
template <typename T>
__device__ __forceinline__ float silu_t(float x) { return x * sigmoid_t<T>(x); }
template <>
__device__ __forceinline__ float silu_t<float>(float x) { return silu_f(x); }

// sequence that owns token t (cu[0] = 0 .. cu[B] = T)
__device__ __forceinline__ int sequence_of(const int* __restrict__ cu, int B, int t) {
  if (t < B && cu[t] <= t && cu[t + 1] > t) return t;       // one token per sequence up to here: decode steps
  int lo = 0, hi = B - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu[mid] <= t) lo = mid;
    else hi = mid - 1;
  }
  return lo;
}

}  // namespace mixer
