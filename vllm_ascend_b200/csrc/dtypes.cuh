// Element-type helpers of the kernels that are templated over bf16 / fp32 storage: conversion, short
// vector loads and stores (up to 16 bytes), packed fp32 arithmetic.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

namespace b200 {

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16(v); }

inline bool aligned16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

template <int BYTES> struct RawVec;
template <> struct RawVec<2> { using type = uint16_t; };
template <> struct RawVec<4> { using type = uint32_t; };
template <> struct RawVec<8> { using type = uint2; };
template <> struct RawVec<16> { using type = uint4; };

// N elements from an address aligned to N * sizeof(T)
template <typename T, int N>
__device__ __forceinline__ void load_raw(const T* p, T* v) {
  using V = typename RawVec<N * (int)sizeof(T)>::type;
  union { V raw; T e[N]; } u;
  u.raw = *reinterpret_cast<const V*>(p);
#pragma unroll
  for (int i = 0; i < N; i++) v[i] = u.e[i];
}
template <typename T, int N>
__device__ __forceinline__ void load_vec(const T* p, float* v) {
  T e[N];
  load_raw<T, N>(p, e);
#pragma unroll
  for (int i = 0; i < N; i++) v[i] = to_f(e[i]);
}
template <typename T, int N>
__device__ __forceinline__ void store_vec(T* p, const float* v) {
  using V = typename RawVec<N * (int)sizeof(T)>::type;
  union { V raw; T e[N]; } u;
#pragma unroll
  for (int i = 0; i < N; i++) u.e[i] = from_f<T>(v[i]);
  *reinterpret_cast<V*>(p) = u.raw;
}

// SiLU: the fast exponential where the result is rounded to bf16
template <typename T> __device__ __forceinline__ float silu_f(float v) {
  if constexpr (sizeof(T) == 2) return v / (1.f + __expf(-v));
  return v / (1.f + expf(-v));
}
// gate of a gated MLP: silu(g) u, or with alpha > 0 the clamped min(g, limit) sigmoid(alpha .) (clamp(u, -limit, limit) + 1)
__device__ __forceinline__ float glu_f(float g, float u, float alpha, float limit) {
  if (alpha > 0.f) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.f + expf(-alpha * g)) * (u + 1.f);
  }
  return g / (1.f + expf(-g)) * u;
}
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return 0.5f * z * (1.f + tanhf(u));
}

// two fp32 values in one 64-bit register, and the packed operations on them
using f32x2 = unsigned long long;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
  return d;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

}  // namespace b200
