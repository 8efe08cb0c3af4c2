// Paged grouped-query attention with options (AttnVariantArgs) on the CUDA cores, for every size and storage
// type the tcgen05 kernels of attention_tc.cu, attention_decode_tc.cu and attention_wide.cu do not take: fp32 caches,
// head sizes that are no multiple of 8 elements or too large, more than 128 query heads on one value head.
//
// One warp per (query row, head): the head dimension is spread over the lanes, four keys are in flight at a
// time.  Row r sees the keys [row_kv_len - window, row_kv_len) of its sequence and the first keep_first ones.
#include "attention.h"
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

constexpr int VAR_KEYS = 4;            // keys in flight

// the query and a key take NK x 32 dimensions at most, a value NV x 32; TO: type of the output
template <typename T, typename TO, int NK, int NV>
__global__ void __launch_bounds__(128) attention_variant_kernel(const AttnVariantArgs p, int* status) {
  const long row = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const int h = (int)blockIdx.y * 4 + (threadIdx.x >> 5);
  if (h >= p.Hq) return;
  const int g = h / (p.Hq / p.Hkv), gk = g * p.key_heads / p.Hkv;
  const int kv_len = p.row_kv_len[row];
  const int first = p.window > 0 ? max(0, kv_len - p.window) : 0;
  const int kept = min(p.keep_first, first);        // keys before the window
  const int n = kept + kv_len - first;
  const int* bt = p.block_table + (long)p.row_seq[row] * p.max_blocks;
  const T* qr = (const T*)p.q + row * p.q_stride + (long)h * p.D;
  const float* bias = p.bias ? p.bias + (long)h * p.bias_len : nullptr;
  float q[NK], acc[NV];
#pragma unroll
  for (int i = 0; i < NK; i++) {
    const int d = i * 32 + lane;
    q[i] = d < p.D ? to_f(qr[d]) : 0.f;
  }
#pragma unroll
  for (int i = 0; i < NV; i++) acc[i] = 0.f;
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < n; k0 += VAR_KEYS) {
    float s[VAR_KEYS];
    long off[VAR_KEYS];
#pragma unroll
    for (int j = 0; j < VAR_KEYS; j++) {
      const int idx = min(k0 + j, n - 1);
      const int key = idx < kept ? idx : first + idx - kept;
      const int blk = bt[key / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        if (lane == 0 && status) atomicExch(status, B200_BAD_INDEX);
        return;
      }
      const int slot = key % p.block_size;
      const T* kr = (const T*)p.k_cache + blk * p.k_block + slot * p.k_tok + gk * p.k_head;
      off[j] = blk * p.v_block + slot * p.v_tok + g * p.v_head;
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < NK; i++) {
        const int d = i * 32 + lane;
        if (d < p.D) a = fmaf(q[i], to_f(kr[d]), a);
      }
      a = warp_reduce_sum(a) * p.scale;
      if (p.softcap > 0.f) a = p.softcap * tanhf(a / p.softcap);
      if (bias) a += bias[min(kv_len - 1 - key, p.bias_len - 1)];
      s[j] = k0 + j < n ? a : -INFINITY;
    }
    float mn = m;
#pragma unroll
    for (int j = 0; j < VAR_KEYS; j++) mn = fmaxf(mn, s[j]);
    const float alpha = expf(m - mn);               // 0 for the first group (m = -inf)
    m = mn;
    l *= alpha;
#pragma unroll
    for (int i = 0; i < NV; i++) acc[i] *= alpha;
#pragma unroll
    for (int j = 0; j < VAR_KEYS; j++) {
      const float w = expf(s[j] - m);
      l += w;
      const T* vr = (const T*)p.v_cache + off[j];
#pragma unroll
      for (int i = 0; i < NV; i++) {
        const int d = i * 32 + lane;
        if (d < p.Dv) acc[i] = fmaf(w, to_f(vr[d]), acc[i]);
      }
    }
  }
  float f = 1.f;
  if (p.sink) {
    const float sk = p.sink[h], top = fmaxf(m, sk);
    f = expf(m - top);
    l = l * f + expf(sk - top);
  }
  float inv = l > 0.f ? f / l : 0.f;
  if (p.gate) inv *= 1.f / (1.f + expf(-to_f(((const T*)p.gate)[row * p.gate_stride + h])));
  inv *= p.out_scale;
  TO* o = (TO*)p.out + row * p.out_stride + (long)h * p.Dv;
#pragma unroll
  for (int i = 0; i < NV; i++) {
    const int d = i * 32 + lane;
    if (d < p.Dv) o[d] = from_f<TO>(acc[i] * inv);
  }
}

template <typename T, typename TO>
static int launch_variant(const AttnVariantArgs& p, int* status, cudaStream_t stream) {
  const dim3 grid((unsigned)p.tokens, (unsigned)((p.Hq + 3) / 4));
  const int d = p.D > p.Dv ? p.D : p.Dv;
  if (d <= 64) attention_variant_kernel<T, TO, 2, 2><<<grid, 128, 0, stream>>>(p, status);
  else if (d <= 128) attention_variant_kernel<T, TO, 4, 4><<<grid, 128, 0, stream>>>(p, status);
  else if (d <= 256) attention_variant_kernel<T, TO, 8, 8><<<grid, 128, 0, stream>>>(p, status);
  else if (d <= 512) attention_variant_kernel<T, TO, 16, 16><<<grid, 128, 0, stream>>>(p, status);
  else if (p.D <= 1024 && p.Dv <= 256) attention_variant_kernel<T, TO, 32, 8><<<grid, 128, 0, stream>>>(p, status);
  else if (p.D <= 2048 && p.Dv <= 256) attention_variant_kernel<T, TO, 64, 8><<<grid, 128, 0, stream>>>(p, status);
  else return 9850;
  return B200_CHECK_LAUNCH();
}

}  // namespace b200

using namespace b200;

B200_API int b200_attention_variant(const AttnVariantArgs* a, int* status, cudaStream_t stream) {
  if (a->tokens <= 0) return 0;
  if (a->D < 1 || a->Dv < 1 || a->Hkv < 1 || a->Hq < 1 || a->Hq % a->Hkv || a->block_size < 1) return 9851;
  if ((a->bias && a->bias_len < 1) || !a->row_seq || !a->row_kv_len || a->keep_first < 0) return 9852;
  if (a->key_heads < 1 || a->Hkv % a->key_heads) return 9853;
  if (a->dtype) return launch_variant<float, float>(*a, status, stream);
  return a->out_f32 ? launch_variant<__nv_bfloat16, float>(*a, status, stream)
                    : launch_variant<__nv_bfloat16, __nv_bfloat16>(*a, status, stream);
}
