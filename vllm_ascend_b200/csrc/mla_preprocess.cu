// MLA pre-processing of one step, fused: what lies between the down-projections and the attention
// kernel of a multi-head-latent-attention layer.
//
//   kv  [T, dc + dr]  (output of the joint KV down-projection)
//     latent = RMSNorm(kv[:, :dc]) * w          -> latent cache slot of the token (and an optional copy)
//     k_pe   = RoPE(kv[:, dc:])                  -> rope-key cache slot of the token (and an optional copy)
//   q   [T, H, dn + dr]
//     q[..., dn:] = RoPE(q[..., dn:])            in place
//
// RoPE is the interleaved (GPT-J) pairing (2j, 2j+1) of DeepSeek's rope slice, angles from a
// [max_pos, dr] fp32 table (cos in the first half of a row, sin in the second).  One CTA per
// token; values are computed in fp32 and rounded once to the storage type (bf16 or fp32), like the separate
// norm / rope / scatter steps they replace.  Layers whose queries go through a latent as well, with both
// down-projections in one product, take the same work in two kernels around the query's up-projection:
//   latent_prep   [cq | c | kr] rows: RMSNorm(cq) dense, RMSNorm(c) and RoPE(kr) to their cache slots
//   latent_query  q: rotary part of every head in place, the rest as head-major rows
// Tokens with slot < 0 (padding, or tokens another rank stores) do the
// q rotation only.  The reference runs this stage as one fused op as well (csrc/mla_preprocess/,
// registered as npu_mla_process in csrc/torch_binding.cpp:1987-1997), there together with the
// projections.
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

template <typename T>
struct MlaPreParams {
  T* q;
  long q_stride;           // elements between tokens
  int H, dn, dr;
  const T* kv;
  long kv_stride;
  int dc;
  const T* norm_w;
  float eps;
  const long* positions;
  const float* cos_sin;    // [max_pos, dr]
  long max_pos;
  const long* slot_mapping;
  T* lat_cache;            // [num_slots, dc]
  T* pe_cache;             // [num_slots, dr]
  long num_slots;
  T* latent_out;           // optional [T, dc]
  T* kpe_out;              // optional [T, dr]
  int* status;
};

// PAIR: every rotary pair of q is one aligned access
template <typename T, bool PAIR>
__global__ void __launch_bounds__(256) mla_preprocess_kernel(const MlaPreParams<T> p) {
  __shared__ float red[8];
  __shared__ float s_inv;
  const long t = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  long pos = p.positions[t];
  bool bad = pos < 0 || pos >= p.max_pos;
  if (bad) pos = 0;
  long slot = p.slot_mapping ? p.slot_mapping[t] : -1;
  if (slot >= p.num_slots) {
    bad = true;
    slot = -1;
  }
  if (bad && tid == 0 && p.status) atomicCAS(p.status, 0, B200_BAD_INDEX);
  const float* cs = p.cos_sin + pos * (long)p.dr;
  const int half = p.dr >> 1;

  // ---- latent: RMSNorm over dc
  const T* kvrow = p.kv + t * p.kv_stride;
  const bool want_latent = slot >= 0 || p.latent_out != nullptr;
  if (want_latent) {
    float ss = 0.f;
    for (int i = tid; i < p.dc; i += blockDim.x) {
      const float v = to_f(kvrow[i]);
      ss += v * v;
    }
    ss = warp_reduce_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (warp == 0) {
      float v = lane < (int)(blockDim.x >> 5) ? red[lane] : 0.f;
      v = warp_reduce_sum(v);
      if (lane == 0) s_inv = rsqrtf(v / (float)p.dc + p.eps);
    }
    __syncthreads();
    const float inv = s_inv;
    for (int i = tid; i < p.dc; i += blockDim.x) {
      const T o = from_f<T>(to_f(kvrow[i]) * inv * to_f(p.norm_w[i]));
      if (slot >= 0) p.lat_cache[slot * p.dc + i] = o;
      if (p.latent_out) p.latent_out[t * p.dc + i] = o;
    }
    // ---- rope key
    for (int j = tid; j < half; j += blockDim.x) {
      const float x1 = to_f(kvrow[p.dc + 2 * j]);
      const float x2 = to_f(kvrow[p.dc + 2 * j + 1]);
      const float c = cs[j], s = cs[half + j];
      const T o1 = from_f<T>(x1 * c - x2 * s);
      const T o2 = from_f<T>(x2 * c + x1 * s);
      if (slot >= 0) {
        p.pe_cache[slot * p.dr + 2 * j] = o1;
        p.pe_cache[slot * p.dr + 2 * j + 1] = o2;
      }
      if (p.kpe_out) {
        p.kpe_out[t * p.dr + 2 * j] = o1;
        p.kpe_out[t * p.dr + 2 * j + 1] = o2;
      }
    }
  }
  // ---- rope slice of every query head, in place
  T* qrow = p.q + t * p.q_stride;
  const int D = p.dn + p.dr;
  const int pairs = p.H * half;
  for (int i = tid; i < pairs; i += blockDim.x) {
    const int h = i / half, j = i - h * half;
    T* ptr = qrow + (long)h * D + p.dn + 2 * j;
    float x[2];
    if (PAIR) load_vec<T, 2>(ptr, x);
    else {
      x[0] = to_f(ptr[0]);
      x[1] = to_f(ptr[1]);
    }
    const float c = cs[j], s = cs[half + j];
    const float y[2] = {x[0] * c - x[1] * s, x[1] * c + x[0] * s};
    if (PAIR) store_vec<T, 2>(ptr, y);
    else {
      ptr[0] = from_f<T>(y[0]);
      ptr[1] = from_f<T>(y[1]);
    }
  }
}

struct LatentPrepParams {
  const void* down;        // [T, stride]: rq | dc | dr columns
  long stride;
  int rq, dc, dr;          // dc = dr = 0: the query latent only
  const void *q_norm, *kv_norm;
  float eps;
  const long* positions;
  const float* cos_sin;    // [max_pos, dr]
  long max_pos;
  const long* slot_mapping;
  void* cq;                // [T, rq]
  void *lat_cache, *pe_cache;
  long num_slots;
  int* status;
};

template <typename T, int VEC>
__device__ __forceinline__ void scaled_row(const T* x, const T* w, T* out, int n, float inv) {
  for (int c = (int)threadIdx.x * VEC; c < n; c += (int)blockDim.x * VEC) {
    float v[VEC], wv[VEC];
    load_vec<T, VEC>(x + c, v);
    load_vec<T, VEC>(w + c, wv);
#pragma unroll
    for (int e = 0; e < VEC; e++) v[e] = v[e] * inv * wv[e];
    store_vec<T, VEC>(out + c, v);
  }
}

template <typename T, int VEC>
__global__ void __launch_bounds__(128) latent_prep_kernel(const LatentPrepParams p) {
  __shared__ float red[2][4];
  const long t = blockIdx.x;
  const T* row = (const T*)p.down + t * p.stride;
  long slot = p.dc > 0 && p.slot_mapping ? p.slot_mapping[t] : -1;
  long pos = slot >= 0 ? p.positions[t] : 0;
  if (slot >= p.num_slots || pos < 0 || (slot >= 0 && pos >= p.max_pos)) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, B200_BAD_INDEX);
    slot = -1;
  }
  float s[2] = {0.f, 0.f};
  const int width = p.rq + (slot >= 0 ? p.dc : 0);
  for (int c = (int)threadIdx.x * VEC; c < width; c += (int)blockDim.x * VEC) {
    float v[VEC], a = 0.f;
    load_vec<T, VEC>(row + c, v);
#pragma unroll
    for (int e = 0; e < VEC; e++) a = fmaf(v[e], v[e], a);
    if (c < p.rq) s[0] += a; else s[1] += a;
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
#pragma unroll
  for (int k = 0; k < 2; k++) {
    s[k] = warp_reduce_sum(s[k]);
    if (lane == 0) red[k][warp] = s[k];
  }
  __syncthreads();
#pragma unroll
  for (int k = 0; k < 2; k++) s[k] = red[k][0] + red[k][1] + red[k][2] + red[k][3];
  scaled_row<T, VEC>(row, (const T*)p.q_norm, (T*)p.cq + t * p.rq, p.rq, 1.f / sqrtf(s[0] / (float)p.rq + p.eps));
  if (slot < 0) return;
  scaled_row<T, VEC>(row + p.rq, (const T*)p.kv_norm, (T*)p.lat_cache + slot * p.dc, p.dc,
                     1.f / sqrtf(s[1] / (float)p.dc + p.eps));
  const float* cs = p.cos_sin + pos * (long)p.dr;
  const T* kr = row + p.rq + p.dc;
  T* dst = (T*)p.pe_cache + slot * p.dr;
  const int half = p.dr >> 1;
  for (int j = threadIdx.x; j < half; j += blockDim.x) {
    const float a = to_f(kr[2 * j]), b = to_f(kr[2 * j + 1]), c = cs[j], sn = cs[half + j];
    dst[2 * j] = from_f<T>(a * c - b * sn);
    dst[2 * j + 1] = from_f<T>(b * c + a * sn);
  }
}

struct LatentQueryParams {
  void* q;                 // [T, H, dn + dr]
  long T;
  int H, dn, dr;
  const long* positions;
  const float* cos_sin;
  long max_pos;
  void* nope;              // [H, T, dn]
  int* status;
};

// VEC: elements of a unit of work (1: single elements of the unrotated part, pairs of the rotated one)
template <typename T, int VEC>
__global__ void __launch_bounds__(256) latent_query_kernel(const LatentQueryParams p) {
  const long t = blockIdx.x;
  long pos = p.positions[t];
  if (pos < 0 || pos >= p.max_pos) {
    if (threadIdx.x == 0 && blockIdx.y == 0 && p.status) atomicCAS(p.status, 0, B200_BAD_INDEX);
    pos = 0;
  }
  const float* cs = p.cos_sin + pos * (long)p.dr;
  constexpr int RV = VEC > 1 ? VEC : 2;              // rotated elements of a unit
  const int un = p.dn / VEC, ur = p.dr / RV, units = un + ur, half = p.dr >> 1, D = p.dn + p.dr;
  T* row = (T*)p.q + t * (long)p.H * D;
  for (int i = (int)(blockIdx.y * blockDim.x + threadIdx.x); i < p.H * units; i += (int)(gridDim.y * blockDim.x)) {
    const int h = i / units, u = i - h * units;
    T* head = row + (long)h * D;
    if (u < un) {
      T raw[VEC];
      load_raw<T, VEC>(head + u * VEC, raw);
      float v[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] = to_f(raw[e]);
      store_vec<T, VEC>((T*)p.nope + ((long)h * p.T + t) * p.dn + u * VEC, v);
      continue;
    }
    const int r = (u - un) * RV;
    T* ptr = head + p.dn + r;
    float v[RV];
    if constexpr (VEC > 1) load_vec<T, RV>(ptr, v);
    else {
      v[0] = to_f(ptr[0]);
      v[1] = to_f(ptr[1]);
    }
#pragma unroll
    for (int e = 0; e < RV; e += 2) {
      const float c = cs[(r + e) >> 1], sn = cs[half + ((r + e) >> 1)], a = v[e], b = v[e + 1];
      v[e] = a * c - b * sn;
      v[e + 1] = b * c + a * sn;
    }
    if constexpr (VEC > 1) store_vec<T, RV>(ptr, v);
    else {
      ptr[0] = from_f<T>(v[0]);
      ptr[1] = from_f<T>(v[1]);
    }
  }
}

template <typename T>
static int launch_latent_prep(const LatentPrepParams& p, long tokens, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool vec = p.rq % V == 0 && p.dc % V == 0 && p.stride % V == 0 && aligned16(p.down) && aligned16(p.q_norm) &&
                   aligned16(p.kv_norm) && aligned16(p.cq) && aligned16(p.lat_cache);
  if (vec) latent_prep_kernel<T, V><<<(unsigned)tokens, 128, 0, stream>>>(p);
  else latent_prep_kernel<T, 1><<<(unsigned)tokens, 128, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int launch_latent_query(const LatentQueryParams& p, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool vec = p.dn % V == 0 && p.dr % V == 0 && aligned16(p.q) && aligned16(p.nope);
  const long units = (long)p.H * (p.dn + p.dr) / (vec ? V : 1);
  long parts = (units + 255) / 256;                  // blocks per token: more of them for few tokens
  const long want = (4L * num_sms() + p.T - 1) / p.T;
  if (parts > want) parts = want;
  const dim3 grid((unsigned)p.T, (unsigned)(parts < 1 ? 1 : parts));
  if (vec) latent_query_kernel<T, V><<<grid, 256, 0, stream>>>(p);
  else latent_query_kernel<T, 1><<<grid, 256, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int launch_mla_preprocess(void* q, long q_stride, int tokens, int H, int dn, int dr, const void* kv,
                                 long kv_stride, int dc, const void* norm_w, float eps, const void* positions,
                                 const void* cos_sin, long max_pos, const void* slot_mapping, void* lat_cache,
                                 void* pe_cache, long num_slots, void* latent_out, void* kpe_out, int* status,
                                 cudaStream_t stream) {
  MlaPreParams<T> p{(T*)q, q_stride, H, dn, dr, (const T*)kv, kv_stride, dc, (const T*)norm_w, eps,
                    (const long*)positions, (const float*)cos_sin, max_pos, (const long*)slot_mapping,
                    (T*)lat_cache, (T*)pe_cache, num_slots, (T*)latent_out, (T*)kpe_out, status};
  const bool pair = dn % 2 == 0 && q_stride % 2 == 0 && (reinterpret_cast<uintptr_t>(q) % (2 * sizeof(T))) == 0;
  if (pair) mla_preprocess_kernel<T, true><<<tokens, 256, 0, stream>>>(p);
  else mla_preprocess_kernel<T, false><<<tokens, 256, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

}  // namespace b200

using namespace b200;

// dr even; every stride is free.  dtype: 0 bf16, 1 fp32.  lat_cache / pe_cache: dense [num_slots, dc] /
// [num_slots, dr].
B200_API int b200_mla_preprocess(void* q, long q_stride, int T, int H, int dn, int dr, const void* kv,
                                 long kv_stride, int dc, const void* norm_w, float eps,
                                 const void* positions, const void* cos_sin, long max_pos,
                                 const void* slot_mapping, void* lat_cache, void* pe_cache,
                                 long num_slots, void* latent_out, void* kpe_out, int dtype, int* status,
                                 cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((dr & 1) || dr <= 0 || dc <= 0 || H <= 0) return 9400;
  if (slot_mapping && (!lat_cache || !pe_cache)) return 9402;
  return (dtype ? launch_mla_preprocess<float> : launch_mla_preprocess<__nv_bfloat16>)(
      q, q_stride, T, H, dn, dr, kv, kv_stride, dc, norm_w, eps, positions, cos_sin, max_pos, slot_mapping,
      lat_cache, pe_cache, num_slots, latent_out, kpe_out, status, stream);
}

// down [T, stride] = rq | dc | dr columns (dc = dr = 0: no key part, caches unused); cq [T, rq]; caches dense
// [num_slots, dc] / [num_slots, dr].  dtype: 0 bf16, 1 fp32
B200_API int b200_latent_prep(const void* down, long stride, long T, int rq, const void* q_norm, void* cq, int dc, int dr,
                              const void* kv_norm, float eps, const void* positions, const void* cos_sin, long max_pos,
                              const void* slot_mapping, void* lat_cache, void* pe_cache, long num_slots, int dtype,
                              int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rq < 1 || dc < 0 || dr < 0 || (dr & 1) || (dc > 0) != (dr > 0) || stride < rq + dc + dr) return 9410;
  if (dc > 0 && (!kv_norm || !positions || !cos_sin || !lat_cache || !pe_cache)) return 9411;
  LatentPrepParams p{down, stride, rq, dc, dr, q_norm, kv_norm, eps, (const long*)positions, (const float*)cos_sin,
                     max_pos, (const long*)slot_mapping, cq, dc > 0 ? lat_cache : nullptr, dc > 0 ? pe_cache : nullptr,
                     num_slots, status};
  return dtype ? launch_latent_prep<float>(p, T, stream) : launch_latent_prep<__nv_bfloat16>(p, T, stream);
}

// q [T, H, dn + dr] dense, rotated in place; nope [H, T, dn].  dtype: 0 bf16, 1 fp32
B200_API int b200_latent_query(void* q, long T, int H, int dn, int dr, const void* positions, const void* cos_sin,
                               long max_pos, void* nope, int dtype, int* status, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H < 1 || dn < 1 || dr < 2 || (dr & 1) || max_pos < 1) return 9412;
  LatentQueryParams p{q, T, H, dn, dr, (const long*)positions, (const float*)cos_sin, max_pos, nope, status};
  return dtype ? launch_latent_query<float>(p, stream) : launch_latent_query<__nv_bfloat16>(p, stream);
}
