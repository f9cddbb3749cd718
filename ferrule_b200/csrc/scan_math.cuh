// Functions of recurrences: bf16 models take the hardware exponential and logarithm (a few 1e-7 relative), fp32 models the
// full-precision functions.
#pragma once
#include "act_type.cuh"

namespace fb {

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <typename T>
__device__ __forceinline__ float scan_exp2(float x) { return sizeof(T) == 4 ? exp2f(x) : exp2_approx(x); }
template <typename T>
__device__ __forceinline__ float scan_softplus(float z) {
  if constexpr (sizeof(T) == 4) return softplus_f(z);
  const float e = __expf(-fabsf(z)), w = 1.f + e;
  // log1p(e) = log(w) * e / (w - 1): the quotient restores what rounding w lost
  const float l = w == 1.f ? e : __logf(w) * __fdividef(e, w - 1.f);
  return fmaxf(z, 0.f) + l;
}
template <typename T>
__device__ __forceinline__ float scan_silu(float z) {
  if constexpr (sizeof(T) == 4) return z / (1.f + expf(-z));
  return __fdividef(z, 1.f + __expf(-z));
}

}  // namespace fb
