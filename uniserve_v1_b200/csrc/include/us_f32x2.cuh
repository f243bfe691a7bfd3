// Packed FP32 pairs: one instruction on two values.
#pragma once
#include <stdint.h>

namespace us {
namespace f32x2 {

typedef unsigned long long f2;
__device__ __forceinline__ f2 pack2(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float lo2(f2 r) { return __uint_as_float((uint32_t)r); }
__device__ __forceinline__ float hi2(f2 r) { return __uint_as_float((uint32_t)(r >> 32)); }
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ f2 add2(f2 a, f2 b) {
  f2 d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
// four consecutive floats as two pairs
__device__ __forceinline__ void lds_vec(f2 (&o)[2], const float* p) {
  const ulonglong2 v = *reinterpret_cast<const ulonglong2*>(p);
  o[0] = v.x;
  o[1] = v.y;
}

}  // namespace f32x2
}  // namespace us
