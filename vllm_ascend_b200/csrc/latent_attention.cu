// Latent attention on the CUDA cores, for every size and storage type the tcgen05 kernel of
// attention_mla_decode.cu does not take (fp32 caches, widths that are no multiple of 8 elements).
//
// Query rows with absorbed up-projections attend to the paged latent ‖ rotated-key cache; the latent is also
// the value.  Row r sees the keys [row_kv_len[r] - window, row_kv_len[r]) of its sequence (window 0: all
// row_kv_len[r] of them).  With a sink the softmax denominator also holds exp(sink[h]).  One warp per (row,
// head): the latent is spread over the lanes, four keys are in flight at a time.
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

struct LatentParams {
  const void* q_lat;      // [R, H, dc]
  long ql_row, ql_head;   // strides in elements
  const void* q_pe;       // [R, H, dr]
  long qp_row, qp_head;
  const void* lat_cache;  // [blocks, block_size, dc]
  const void* pe_cache;   // [blocks, block_size, dr]
  long num_blocks;
  int block_size;
  const int *row_seq, *row_kv_len, *block_table;
  int max_blocks;
  const float* sink;      // [H] or null
  float scale;
  int window;
  void* out;              // [R, H, dc]
  long o_row, o_head;
  int H, dc, dr;
  int* status;
};

constexpr int LAT_ROPE_REGS = 4;       // rotated part: up to 128 dimensions
constexpr int LAT_KEYS = 4;            // keys in flight

template <typename T, int NACC>
__global__ void __launch_bounds__(128) latent_attention_kernel(const LatentParams p) {
  const long row = blockIdx.x;
  const int lane = threadIdx.x & 31;
  const int h = (int)blockIdx.y * 4 + (threadIdx.x >> 5);
  if (h >= p.H) return;
  const int kv_len = p.row_kv_len[row];
  const int first = p.window > 0 ? max(0, kv_len - p.window) : 0;
  const int* bt = p.block_table + (long)p.row_seq[row] * p.max_blocks;
  const T* ql = (const T*)p.q_lat + row * p.ql_row + (long)h * p.ql_head;
  const T* qp = (const T*)p.q_pe + row * p.qp_row + (long)h * p.qp_head;
  float q[NACC], qr[LAT_ROPE_REGS], acc[NACC];
#pragma unroll
  for (int i = 0; i < NACC; i++) {
    const int d = i * 32 + lane;
    q[i] = d < p.dc ? to_f(ql[d]) : 0.f;
    acc[i] = 0.f;
  }
#pragma unroll
  for (int i = 0; i < LAT_ROPE_REGS; i++) {
    const int d = i * 32 + lane;
    qr[i] = d < p.dr ? to_f(qp[d]) : 0.f;
  }
  float m = -INFINITY, l = 0.f;
  for (int k0 = first; k0 < kv_len; k0 += LAT_KEYS) {
    float kv[LAT_KEYS][NACC], s[LAT_KEYS];
#pragma unroll
    for (int j = 0; j < LAT_KEYS; j++) {
      const int key = min(k0 + j, kv_len - 1);
      const int blk = bt[key / p.block_size];
      if (blk < 0 || blk >= p.num_blocks) {
        if (lane == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
        return;
      }
      const long slot = (long)blk * p.block_size + key % p.block_size;
      const T* lat = (const T*)p.lat_cache + slot * p.dc;
      const T* pe = (const T*)p.pe_cache + slot * p.dr;
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < NACC; i++) {
        const int d = i * 32 + lane;
        kv[j][i] = d < p.dc ? to_f(lat[d]) : 0.f;
        a = fmaf(q[i], kv[j][i], a);
      }
#pragma unroll
      for (int i = 0; i < LAT_ROPE_REGS; i++) {
        const int d = i * 32 + lane;
        if (d < p.dr) a = fmaf(qr[i], to_f(pe[d]), a);
      }
      s[j] = a;
    }
    float mn = m;
#pragma unroll
    for (int j = 0; j < LAT_KEYS; j++) {
      s[j] = k0 + j < kv_len ? warp_reduce_sum(s[j]) * p.scale : -INFINITY;
      mn = fmaxf(mn, s[j]);
    }
    const float alpha = expf(m - mn);            // 0 for the first group (m = -inf)
    m = mn;
    l *= alpha;
#pragma unroll
    for (int i = 0; i < NACC; i++) acc[i] *= alpha;
#pragma unroll
    for (int j = 0; j < LAT_KEYS; j++) {
      const float w = expf(s[j] - m);
      l += w;
#pragma unroll
      for (int i = 0; i < NACC; i++) acc[i] = fmaf(w, kv[j][i], acc[i]);
    }
  }
  float f = 1.f;
  if (p.sink) {
    const float sk = p.sink[h], top = fmaxf(m, sk);
    f = expf(m - top);
    l = l * f + expf(sk - top);
  }
  const float inv = l > 0.f ? f / l : 0.f;
  T* o = (T*)p.out + row * p.o_row + (long)h * p.o_head;
#pragma unroll
  for (int i = 0; i < NACC; i++) {
    const int d = i * 32 + lane;
    if (d < p.dc) o[d] = from_f<T>(acc[i] * inv);
  }
}

template <typename T>
static int launch_latent(const LatentParams& p, long R, cudaStream_t stream) {
  const dim3 grid((unsigned)R, (unsigned)((p.H + 3) / 4));
  if (p.dc <= 128) latent_attention_kernel<T, 4><<<grid, 128, 0, stream>>>(p);
  else if (p.dc <= 256) latent_attention_kernel<T, 8><<<grid, 128, 0, stream>>>(p);
  else if (p.dc <= 512) latent_attention_kernel<T, 16><<<grid, 128, 0, stream>>>(p);
  else if (p.dc <= 1024) latent_attention_kernel<T, 32><<<grid, 128, 0, stream>>>(p);
  else return 9520;
  return B200_CHECK_LAUNCH();
}

}  // namespace b200

using namespace b200;

// dtype: 0 bf16, 1 fp32 (queries, caches, output); strides in elements, the innermost dimension dense
B200_API int b200_latent_attention(const void* q_lat, long ql_row, long ql_head, const void* q_pe, long qp_row,
                                   long qp_head, long R, int H, int dc, int dr, const void* lat_cache,
                                   const void* pe_cache, long num_blocks, int block_size, const void* row_seq,
                                   const void* row_kv_len, const void* block_table, int max_blocks, const void* sink,
                                   float scale, int window, void* out, long o_row, long o_head, int dtype,
                                   int* status, cudaStream_t stream) {
  if (R <= 0) return 0;
  if (dc < 1 || dr < 1 || dr > 32 * LAT_ROPE_REGS || H < 1 || block_size < 1) return 9521;
  LatentParams p{q_lat, ql_row, ql_head, q_pe, qp_row, qp_head, lat_cache, pe_cache, num_blocks, block_size,
                 (const int*)row_seq, (const int*)row_kv_len, (const int*)block_table, max_blocks,
                 (const float*)sink, scale, window, out, o_row, o_head, H, dc, dr, status};
  return dtype ? launch_latent<float>(p, R, stream) : launch_latent<__nv_bfloat16>(p, R, stream);
}
