// Two floats in one 64-bit register: additions, products and fused products of pairs are single instructions on sm_100a.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace ksana {

struct F2 { unsigned long long v; };
__device__ __forceinline__ F2 f2(float x, float y) { F2 r; asm("mov.b64 %0, {%1, %2};" : "=l"(r.v) : "f"(x), "f"(y)); return r; }
__device__ __forceinline__ F2 f2(float x) { return f2(x, x); }
__device__ __forceinline__ void split(F2 p, float& x, float& y) { asm("mov.b64 {%0, %1}, %2;" : "=f"(x), "=f"(y) : "l"(p.v)); }
__device__ __forceinline__ F2 operator*(F2 a, F2 b) { F2 r; asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v)); return r; }
__device__ __forceinline__ F2 operator+(F2 a, F2 b) { F2 r; asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v)); return r; }
__device__ __forceinline__ F2 fma2(F2 a, F2 b, F2 c) {
  F2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.v) : "l"(a.v), "l"(b.v), "l"(c.v));
  return r;
}
__device__ __forceinline__ float sum2(F2 p) { float x, y; split(p, x, y); return x + y; }

}  // namespace ksana
