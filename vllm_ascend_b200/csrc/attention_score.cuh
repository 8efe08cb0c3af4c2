// Transformations of attention scores shared by the tcgen05 kernels: capping and the log2-domain form that the
// softmax works on.
#pragma once
#include "dtypes.cuh"

namespace b200 {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float score_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float sigmoid_f(float x) { return __fdividef(1.f, 1.f + score_exp2(-x * kLog2e)); }

// tanh by one exponential and one division; absolute error about one part in 2^23 of the range
__device__ __forceinline__ float tanh_by_exp(float t) {
  return 1.f - __fdividef(2.f, 1.f + score_exp2(2.f * kLog2e * t));
}

// cap * tanh(scale * s / cap) * log2(e) for raw products s.  |t| <= kSmall takes an odd polynomial (least
// squares in the relative error, 9e-8), which leaves the special-function unit to the softmax.
struct SoftCap {
  static constexpr float kSmall = 0.6f;
  float to_t, to_z, w, c1, c2, c3, c4;
  __device__ __forceinline__ SoftCap(float scale, float cap) {
    to_t = scale / cap;
    to_z = cap * kLog2e;
    w = scale * kLog2e;
    const float k = to_t * to_t;
    c1 = -0.33332622f * k;
    c2 = 0.13313521f * k * k;
    c3 = -0.05223110f * k * k * k;
    c4 = 0.01564047f * k * k * k * k;
  }
  __device__ __forceinline__ float any(float s) const { return to_z * tanh_by_exp(s * to_t); }
  __device__ __forceinline__ f32x2 small2(f32x2 s) const {
    const f32x2 r = mul2(s, s);
    const f32x2 p = fma2(fma2(fma2(pack2(c4, c4), r, pack2(c3, c3)), r, pack2(c2, c2)), r, pack2(c1, c1));
    const f32x2 z = mul2(s, pack2(w, w));
    return fma2(mul2(z, r), p, z);
  }
};

}  // namespace b200
