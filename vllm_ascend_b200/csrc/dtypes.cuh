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
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float u = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return 0.5f * z * (1.f + tanhf(u));
}

// packed pair of fp32 operations
__device__ __forceinline__ float2 fma2(float2 a, float2 b, float2 c) {
  float2 d;
  asm("{\n\t.reg .b64 A, B, C, D;\n\t"
      "mov.b64 A, {%2, %3};\n\tmov.b64 B, {%4, %5};\n\tmov.b64 C, {%6, %7};\n\t"
      "fma.rn.f32x2 D, A, B, C;\n\tmov.b64 {%0, %1}, D;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y), "f"(c.x), "f"(c.y));
  return d;
}
__device__ __forceinline__ float2 mul2(float2 a, float2 b) {
  float2 d;
  asm("{\n\t.reg .b64 A, B, D;\n\t"
      "mov.b64 A, {%2, %3};\n\tmov.b64 B, {%4, %5};\n\t"
      "mul.rn.f32x2 D, A, B;\n\tmov.b64 {%0, %1}, D;\n\t}"
      : "=f"(d.x), "=f"(d.y)
      : "f"(a.x), "f"(a.y), "f"(b.x), "f"(b.y));
  return d;
}

// R consecutive elements held as they are stored (fetched one token ahead), R even
template <typename T, int R>
struct RawSlice {
  T e[R];
  // VEC: 16-byte loads, ``left`` (elements up to the end of the row) is a multiple of the vector
  template <bool VEC>
  __device__ __forceinline__ void load(const T* p, int left) {
    constexpr int V = 16 / (int)sizeof(T);
    if constexpr (VEC && R % V == 0) {
#pragma unroll
      for (int i = 0; i < R; i += V) {
        if (i < left) load_raw<T, V>(p + i, e + i);
        else
#pragma unroll
          for (int j = 0; j < V; j++) e[i + j] = from_f<T>(0.f);
      }
    } else {
#pragma unroll
      for (int i = 0; i < R; i++) e[i] = i < left ? p[i] : from_f<T>(0.f);
    }
  }
  __device__ __forceinline__ void unpack(float2* v) const {
#pragma unroll
    for (int i = 0; i < R / 2; i++) v[i] = make_float2(to_f(e[2 * i]), to_f(e[2 * i + 1]));
  }
};

}  // namespace b200
