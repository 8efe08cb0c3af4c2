// RMS norm of equal parts of a row, in one pass behind a recurrence or an attention layer:
//   x   = y                   (per-head norm of a linear-attention read-out)
//       = y * silu(z)         (Mamba-2: the gate comes before the norm)
//       = y - lam * y2        (difference of two softmax maps)
//   out = scale * w * x / sqrt(mean(x^2) + eps)      per part, w per channel, shared by the parts, or absent
// A group of LANES threads owns one part of one row and keeps the first KEEP vectors of it in registers; everything is
// fp32 between load and store.  Rows bf16 or fp32 (template), also fp32 rows with a bf16 result.  The reference fuses
// gate and norm the same way (vllm_ascend/ops/layernorm.py:110-197).
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

struct GroupNormArgs {
  const void* y;              // part g of row t at t * y_stride + g * y_group
  const void* y2;             // null, or subtracted lam times; strides of y
  const void* z;              // null, or gate: row stride z_stride, parts side by side
  const void* w;              // null, or w_len channels: size (shared by the parts) or groups * size
  void* out;                  // row stride out_stride, parts side by side
  long rows, y_stride, y_group, z_stride, out_stride, w_len;
  int groups, size, in_f32, dtype;
  float lam, eps, scale;
};

template <typename TI, typename T, int VEC, int LANES>
__global__ void __launch_bounds__(256) group_norm_kernel(const GroupNormArgs p) {
  constexpr int KEEP = 4;
  __shared__ float red[8];
  const long unit = ((long)blockIdx.x * 256 + threadIdx.x) / LANES;
  const bool on = unit < p.rows * p.groups;          // others only take part in the reductions
  const int lane = threadIdx.x % LANES;
  const long t = on ? unit / p.groups : 0;
  const int g = on ? (int)(unit - t * p.groups) : 0;
  const int size = on ? p.size : 0;
  const long at = t * p.y_stride + g * p.y_group;
  const TI* y = (const TI*)p.y + at;
  const TI* y2 = p.y2 ? (const TI*)p.y2 + at : nullptr;
  const T* z = p.z ? (const T*)p.z + t * p.z_stride + (long)g * p.size : nullptr;
  auto input = [&](int c, float* v) {
    load_vec<TI, VEC>(y + c, v);
    if (y2) {
      float u[VEC];
      load_vec<TI, VEC>(y2 + c, u);
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] -= p.lam * u[e];
    }
    if (z) {
      float u[VEC];
      load_vec<T, VEC>(z + c, u);
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] *= silu_f<T>(u[e]);
    }
  };
  float kept[KEEP][VEC], ss = 0.f;
#pragma unroll
  for (int k = 0; k < KEEP; k++) {
    const int c = (k * LANES + lane) * VEC;
    if (c >= size) continue;
    input(c, kept[k]);
#pragma unroll
    for (int e = 0; e < VEC; e++) ss = fmaf(kept[k][e], kept[k][e], ss);
  }
  for (int c = (KEEP * LANES + lane) * VEC; c < size; c += LANES * VEC) {
    float v[VEC];
    input(c, v);
#pragma unroll
    for (int e = 0; e < VEC; e++) ss = fmaf(v[e], v[e], ss);
  }
#pragma unroll
  for (int o = (LANES < 32 ? LANES : 32) / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if constexpr (LANES > 32) {
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; i++) ss += red[i];
  }
  const float inv = p.scale / sqrtf(ss / (float)p.size + p.eps);
  const T* w = p.w ? (const T*)p.w + (p.w_len > p.size ? (long)g * p.size : 0) : nullptr;
  T* out = (T*)p.out + t * p.out_stride + (long)g * p.size;
  auto store = [&](int c, float* v) {
    float u[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) u[e] = 1.f;
    if (w) load_vec<T, VEC>(w + c, u);
#pragma unroll
    for (int e = 0; e < VEC; e++) v[e] *= inv * u[e];
    store_vec<T, VEC>(out + c, v);
  };
#pragma unroll
  for (int k = 0; k < KEEP; k++) {
    const int c = (k * LANES + lane) * VEC;
    if (c < size) store(c, kept[k]);
  }
  for (int c = (KEEP * LANES + lane) * VEC; c < size; c += LANES * VEC) {
    float v[VEC];
    input(c, v);
    store(c, v);
  }
}

template <typename TI, typename T, int VEC, int LANES>
static int launch_group_norm(const GroupNormArgs& p, cudaStream_t stream) {
  const long blocks = (p.rows * p.groups * LANES + 255) / 256;
  if (blocks > 0x7fffffffL) return 9771;
  group_norm_kernel<TI, T, VEC, LANES><<<(unsigned)blocks, 256, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

template <typename TI, typename T>
static int group_norm_t(const GroupNormArgs& p, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(TI);
  const bool vec = p.size % V == 0 && p.y_stride % V == 0 && p.y_group % V == 0 && p.z_stride % V == 0 &&
                   p.out_stride % V == 0 && aligned16(p.y) && aligned16(p.y2) && aligned16(p.z) && aligned16(p.w) &&
                   aligned16(p.out);
  const int n = p.size / (vec ? V : 1);
  if (vec) {
    if (n <= 16) return launch_group_norm<TI, T, V, 8>(p, stream);
    if (n <= 128) return launch_group_norm<TI, T, V, 32>(p, stream);
    return launch_group_norm<TI, T, V, 256>(p, stream);
  }
  if (n <= 16) return launch_group_norm<TI, T, 1, 8>(p, stream);
  if (n <= 256) return launch_group_norm<TI, T, 1, 32>(p, stream);
  return launch_group_norm<TI, T, 1, 256>(p, stream);
}

}  // namespace b200

using namespace b200;

// dtype: 0 bf16, 1 fp32 (z, w, out; y and y2 unless in_f32)
B200_API int b200_group_norm(const GroupNormArgs* a, cudaStream_t stream) {
  if (a->rows <= 0) return 0;
  if (a->groups < 1 || a->size < 1 || (a->w && a->w_len != a->size && a->w_len != (long)a->size * a->groups)) return 9770;
  if (a->dtype) return group_norm_t<float, float>(*a, stream);
  return a->in_f32 ? group_norm_t<float, __nv_bfloat16>(*a, stream) : group_norm_t<__nv_bfloat16, __nv_bfloat16>(*a, stream);
}
