// Vectors of 8 elements (bf16: 16 bytes, fp32: 32 bytes) as floats, for kernels that are instantiated for both types.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace ksana {

typedef __nv_bfloat16 bf16;

// 8 consecutive elements as floats
__device__ __forceinline__ void load8(const bf16* p, float (&f)[8]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) { const float2 t = __bfloat1622float2(h[i]); f[2 * i] = t.x; f[2 * i + 1] = t.y; }
}
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
  *reinterpret_cast<float4*>(&f[0]) = *reinterpret_cast<const float4*>(p);
  *reinterpret_cast<float4*>(&f[4]) = *reinterpret_cast<const float4*>(p + 4);
}
__device__ __forceinline__ void store8(bf16* p, const float (&f)[8]) {
  uint4 v;
  __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&v);
#pragma unroll
  for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = v;
}
__device__ __forceinline__ void store8(float* p, const float (&f)[8]) {
  *reinterpret_cast<float4*>(p) = *reinterpret_cast<const float4*>(&f[0]);
  *reinterpret_cast<float4*>(p + 4) = *reinterpret_cast<const float4*>(&f[4]);
}
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
__device__ __forceinline__ float sigmoid_f(float x) { return 1.f / (1.f + __expf(-x)); }

static inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

}  // namespace ksana
