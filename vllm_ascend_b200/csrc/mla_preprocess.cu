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
// norm / rope / scatter steps they replace.  Tokens with slot < 0 (padding, or tokens another rank stores) do the
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
