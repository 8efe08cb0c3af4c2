// Kernels around an fp32 residual stream (decoders that normalise a sub-layer's input and its output):
//   stream_norm      one pass over a token's row between two sub-layers:
//                      r  = scale * embed[id]                    (start of the stream), or
//                      r += m norm_post(y) (+ scale * embed[id]) (a sub-layer's output joins; a looped
//                                                                 stack is fed the embedding again)
//                      x  = norm_next(r), or r rounded to the activation type
//   stream_mix       the same pass over S parallel streams per token (hyper-connections):
//                      x_t = sum_s mix[s, t] x_s + out[t] post(y)          (a sub-layer's output joins), or
//                      x_t = scale * embed[id] + pos[position] for all t   (start of the streams)
//                      u   = sum_s in[s] x_s (no weights: their sum);  x = norm_next(u)
//   side_gate        g = gelu_tanh(a) * side_embed[id, slice]    (per-layer token input)
//   gated_head_norm  o = rms_norm(o) * w * silu(z) per head      (delta-rule read-out)
// Either norm is a layer norm (weight, bias) or an RMS norm (in stream_norm also of equal parts of the row, each by
// itself), statistics in fp32.  Activations, weights and
// tables are bf16 or fp32.  The reference fuses add + norm the same way on a 16-bit residual
// (vllm_ascend/ops/layernorm.py:63-85).
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

enum : int { NORM_NONE = 0, NORM_LAYER = 1, NORM_RMS = 2, NORM_PLAIN = 3 };
enum : int { EMB_NONE = 0, EMB_SET = 1, EMB_ADD = 2 };

struct StreamParams {
  float* r;               // [T, W]
  const void* y;          // [T, W] sub-layer output (post != NONE)
  long y_stride;
  int post;
  const void *post_w, *post_b;
  float post_scale;       // m
  int emb;
  const long* ids;        // [T]; null: row t of the table
  const void* table;      // [rows, W]
  long table_rows;
  float emb_scale;
  int next;
  const void *next_w, *next_b;
  void* x;                // [T, W]
  int W;
  int post_groups, next_groups;      // RMS norms: equal parts of the row, each by itself
  int part_threads;                  // > 0: threads of each part of the next norm (and of no other norm in parts)
  float eps;
  int* status;
};

__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_reduce_sum(v);
  const int warps = (blockDim.x + 31) >> 5;
  if (warps == 1) return v;
  __syncthreads();                     // the previous use of red is over
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = (threadIdx.x & 31) < warps ? red[threadIdx.x & 31] : 0.f;
  return warp_reduce_sum(t);
}

template <typename T, int VEC, int PER>
__device__ __forceinline__ void row_norm(float (&v)[PER][VEC], int kind, const T* w, const T* b, int W, float eps,
                                         float* red) {
  const int nvec = W / VEC;
  float mean = 0.f;
  if (kind == NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < PER; i++)
#pragma unroll
      for (int e = 0; e < VEC; e++) s += v[i][e];      // slots beyond the row hold zero
    mean = block_sum(s, red) / (float)W;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < PER; i++)
    if ((int)threadIdx.x + i * (int)blockDim.x < nvec)
#pragma unroll
      for (int e = 0; e < VEC; e++) {
        const float d = v[i][e] - mean;
        ss += d * d;
      }
  const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)W + eps);
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int c = (int)threadIdx.x + i * (int)blockDim.x;
    if (c >= nvec) continue;
    float wv[VEC], bv[VEC];
    load_vec<T, VEC>(w + (long)c * VEC, wv);
#pragma unroll
    for (int e = 0; e < VEC; e++) bv[e] = 0.f;
    if (b) load_vec<T, VEC>(b + (long)c * VEC, bv);
#pragma unroll
    for (int e = 0; e < VEC; e++) v[i][e] = (v[i][e] - mean) * inv * wv[e] + bv[e];
  }
}

constexpr int GROUP_BATCH = 4;         // parts reduced together

// RMS norm of ``groups`` equal parts of the row; a vector lies in one part
template <typename T, int VEC, int PER>
__device__ __forceinline__ void row_group_norm(float (&v)[PER][VEC], const T* w, int W, int groups, float eps,
                                               float (*red)[32]) {
  const int nvec = W / VEC, per = nvec / groups, warps = (blockDim.x + 31) >> 5;
  for (int g0 = 0; g0 < groups; g0 += GROUP_BATCH) {
    float ss[GROUP_BATCH];
#pragma unroll
    for (int k = 0; k < GROUP_BATCH; k++) ss[k] = 0.f;
#pragma unroll
    for (int i = 0; i < PER; i++) {
      const int c = (int)threadIdx.x + i * (int)blockDim.x;
      if (c >= nvec) continue;
      const int k = c / per - g0;
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; e++) s = fmaf(v[i][e], v[i][e], s);
#pragma unroll
      for (int j = 0; j < GROUP_BATCH; j++) ss[j] += j == k ? s : 0.f;
    }
#pragma unroll
    for (int k = 0; k < GROUP_BATCH; k++) ss[k] = warp_reduce_sum(ss[k]);
    if (warps > 1) {
      __syncthreads();                 // the previous use of red is over
      if ((threadIdx.x & 31) == 0)
#pragma unroll
        for (int k = 0; k < GROUP_BATCH; k++) red[k][threadIdx.x >> 5] = ss[k];
      __syncthreads();
#pragma unroll
      for (int k = 0; k < GROUP_BATCH; k++)
        ss[k] = warp_reduce_sum((threadIdx.x & 31) < warps ? red[k][threadIdx.x & 31] : 0.f);
    }
    const float n = (float)(per * VEC);
#pragma unroll
    for (int i = 0; i < PER; i++) {
      const int c = (int)threadIdx.x + i * (int)blockDim.x;
      if (c >= nvec) continue;
      const int k = c / per - g0;
      if (k < 0 || k >= GROUP_BATCH) continue;
      float s = 0.f, wv[VEC];
#pragma unroll
      for (int j = 0; j < GROUP_BATCH; j++) s = j == k ? ss[j] : s;
      const float inv = 1.f / sqrtf(s / n + eps);
      load_vec<T, VEC>(w + (long)c * VEC, wv);
#pragma unroll
      for (int e = 0; e < VEC; e++) v[i][e] = v[i][e] * inv * wv[e];
    }
  }
}

// the sum over the threads that share a part: part_threads (a multiple of 32) neighbours each
__device__ __forceinline__ float part_sum(float v, float* red, int part_threads) {
  v = warp_reduce_sum(v);
  const int warps = part_threads >> 5;
  if (warps == 1) return v;
  __syncthreads();                     // the previous use of red is over
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  const int first = (int)threadIdx.x / part_threads * warps;
  return warp_reduce_sum((threadIdx.x & 31) < warps ? red[first + (threadIdx.x & 31)] : 0.f);
}

// GROUPED: RMS norms may come in several parts.  With part_threads every part has threads of its own, which reduce it as
// plain norms reduce a row.
template <typename T, int VEC, int PER, bool GROUPED>
__global__ void stream_norm_kernel(const StreamParams p) {
  __shared__ float red[GROUPED ? GROUP_BATCH : 1][32];
  const int nvec = p.W / VEC, pt = GROUPED ? p.part_threads : 0;
  const int part = GROUPED && pt ? (int)threadIdx.x / pt : 0, per = GROUPED && pt ? nvec / p.next_groups : nvec;
  const int base = GROUPED && pt ? part * per + (int)threadIdx.x - part * pt : (int)threadIdx.x;
  const int step = GROUPED && pt ? pt : (int)blockDim.x, end = GROUPED && pt ? (part + 1) * per : nvec;
  auto norm = [&](float (&v)[PER][VEC], int kind, const void* w, const void* b, int groups) {
    if (GROUPED && pt) {
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < PER; i++)
        if (base + i * step < end)
#pragma unroll
          for (int e = 0; e < VEC; e++) ss = fmaf(v[i][e], v[i][e], ss);
      const float inv = 1.f / sqrtf(part_sum(ss, red[0], pt) / (float)(per * VEC) + p.eps);
#pragma unroll
      for (int i = 0; i < PER; i++) {
        const int c = base + i * step;
        if (c >= end) continue;
        float wv[VEC];
        load_vec<T, VEC>((const T*)w + (long)c * VEC, wv);
#pragma unroll
        for (int e = 0; e < VEC; e++) v[i][e] *= inv * wv[e];
      }
    } else if (GROUPED && groups > 1) row_group_norm<T, VEC, PER>(v, (const T*)w, p.W, groups, p.eps, red);
    else row_norm<T, VEC, PER>(v, kind, (const T*)w, (const T*)b, p.W, p.eps, red[0]);
  };
  const long t = blockIdx.x;
  float v[PER][VEC];
  float* rrow = p.r + t * p.W;
  if (p.post != NORM_NONE) {
    const T* yrow = (const T*)p.y + t * p.y_stride;
#pragma unroll
    for (int i = 0; i < PER; i++) {
      const int c = base + i * step;
      if (c < end) load_vec<T, VEC>(yrow + (long)c * VEC, v[i]);
      else
#pragma unroll
        for (int e = 0; e < VEC; e++) v[i][e] = 0.f;
    }
    if (p.post != NORM_PLAIN) norm(v, p.post, p.post_w, p.post_b, p.post_groups);
  } else {
#pragma unroll
    for (int i = 0; i < PER; i++)
#pragma unroll
      for (int e = 0; e < VEC; e++) v[i][e] = 0.f;
  }
  const T* erow = nullptr;
  if (p.emb != EMB_NONE) {
    const long id = p.ids ? p.ids[t] : t;
    if (id >= 0 && id < p.table_rows) erow = (const T*)p.table + id * p.W;
    else if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, B200_BAD_INDEX);
  }
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int c = base + i * step;
    if (c >= end) continue;
    if (p.emb != EMB_SET) {
      float rv[VEC];
      load_vec<float, VEC>(rrow + (long)c * VEC, rv);
#pragma unroll
      for (int e = 0; e < VEC; e++) v[i][e] = fmaf(v[i][e], p.post_scale, rv[e]);
    }
    if (erow) {
      float ev[VEC];
      load_vec<T, VEC>(erow + (long)c * VEC, ev);
#pragma unroll
      for (int e = 0; e < VEC; e++) v[i][e] += ev[e] * p.emb_scale;
    }
    if (p.post != NORM_NONE || p.emb != EMB_NONE) store_vec<float, VEC>(rrow + (long)c * VEC, v[i]);
  }
  if (p.next == NORM_NONE) return;
  if (p.next != NORM_PLAIN) norm(v, p.next, p.next_w, p.next_b, p.next_groups);
  T* xrow = (T*)p.x + t * p.W;
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int c = base + i * step;
    if (c < end) store_vec<T, VEC>(xrow + (long)c * VEC, v[i]);
  }
}

struct MixParams {
  float* r;               // [T, S, W]
  const void* y;          // [T, W] sub-layer output (post != NONE)
  long y_stride;
  int post;
  const void *post_w, *post_b;
  const float* mix;       // [S, S] from, to
  const float* out;       // [S]
  int emb;                // EMB_NONE or EMB_SET
  const long* ids;        // [T]; null: row t of the table
  const void* table;      // [rows, W]
  long table_rows;
  float emb_scale;
  const long* positions;  // [T]
  const void* pos_table;  // [pos_rows, W] or null
  long pos_rows;
  const float* in;        // [S] or null: ones
  int next;
  const void *next_w, *next_b;
  void* x;                // [T, W]
  int W, S, store;        // store: the streams are written back
  float eps;
  int* status;
};

// MAXS >= S streams of a column live in registers; one thread block per token
template <typename T, int VEC, int PER, int MAXS>
__global__ void __launch_bounds__(512) stream_mix_kernel(const MixParams p) {
  __shared__ float red[32];
  __shared__ float cf[MAXS * MAXS + 2 * MAXS];      // mix, out, in
  const long t = blockIdx.x;
  const int nvec = p.W / VEC, S = p.S;
  for (int i = threadIdx.x; i < S * S + 2 * S; i += blockDim.x) {
    if (i < S * S) cf[i / S * MAXS + i % S] = p.mix ? p.mix[i] : 0.f;
    else if (i < S * S + S) cf[MAXS * MAXS + i - S * S] = p.out ? p.out[i - S * S] : 0.f;
    else cf[MAXS * MAXS + MAXS + i - S * S - S] = p.in ? p.in[i - S * S - S] : 1.f;
  }
  float v[PER][VEC];
#pragma unroll
  for (int i = 0; i < PER; i++)
#pragma unroll
    for (int e = 0; e < VEC; e++) v[i][e] = 0.f;
  const T *erow = nullptr, *prow = nullptr;
  if (p.emb == EMB_SET) {
    const long id = p.ids ? p.ids[t] : t;
    if (id >= 0 && id < p.table_rows) erow = (const T*)p.table + id * p.W;
    const long pos = p.pos_table ? p.positions[t] : 0;
    if (p.pos_table && pos >= 0 && pos < p.pos_rows) prow = (const T*)p.pos_table + pos * p.W;
    if (threadIdx.x == 0 && p.status && (!erow || (p.pos_table && !prow))) atomicCAS(p.status, 0, B200_BAD_INDEX);
  } else if (p.post != NORM_NONE) {
    const T* yrow = (const T*)p.y + t * p.y_stride;
#pragma unroll
    for (int i = 0; i < PER; i++) {
      const int c = (int)threadIdx.x + i * (int)blockDim.x;
      if (c < nvec) load_vec<T, VEC>(yrow + (long)c * VEC, v[i]);
    }
    if (p.post != NORM_PLAIN)
      row_norm<T, VEC, PER>(v, p.post, (const T*)p.post_w, (const T*)p.post_b, p.W, p.eps, red);
  }
  __syncthreads();                                  // the coefficients are there
  float* rrow = p.r + t * (long)S * p.W;
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int c = (int)threadIdx.x + i * (int)blockDim.x;
    if (c >= nvec) continue;
    float* rc = rrow + (long)c * VEC;
    float xs[MAXS][VEC], u[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) u[e] = 0.f;
    if (p.emb == EMB_SET) {
      float ev[VEC], pv[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) ev[e] = pv[e] = 0.f;
      if (erow) load_vec<T, VEC>(erow + (long)c * VEC, ev);
      if (prow) load_vec<T, VEC>(prow + (long)c * VEC, pv);
#pragma unroll
      for (int e = 0; e < VEC; e++) ev[e] = ev[e] * p.emb_scale + pv[e];
      float w = 0.f;
#pragma unroll
      for (int s = 0; s < MAXS; s++)
        if (s < S) {
          w += cf[MAXS * MAXS + MAXS + s];
          if (p.store) store_vec<float, VEC>(rc + (long)s * p.W, ev);
        }
#pragma unroll
      for (int e = 0; e < VEC; e++) v[i][e] = w * ev[e];
      continue;
    }
#pragma unroll
    for (int s = 0; s < MAXS; s++)
      if (s < S) load_vec<float, VEC>(rc + (long)s * p.W, xs[s]);
#pragma unroll
    for (int to = 0; to < MAXS; to++) {
      if (to >= S) break;
      float nv[VEC];
      if (p.post != NORM_NONE) {
        const float o = cf[MAXS * MAXS + to];
#pragma unroll
        for (int e = 0; e < VEC; e++) nv[e] = o * v[i][e];
#pragma unroll
        for (int s = 0; s < MAXS; s++)
          if (s < S) {
            const float m = cf[s * MAXS + to];
#pragma unroll
            for (int e = 0; e < VEC; e++) nv[e] = fmaf(m, xs[s][e], nv[e]);
          }
        if (p.store) store_vec<float, VEC>(rc + (long)to * p.W, nv);
      } else {
#pragma unroll
        for (int e = 0; e < VEC; e++) nv[e] = xs[to][e];
      }
      const float w = cf[MAXS * MAXS + MAXS + to];
#pragma unroll
      for (int e = 0; e < VEC; e++) u[e] = fmaf(w, nv[e], u[e]);
    }
#pragma unroll
    for (int e = 0; e < VEC; e++) v[i][e] = u[e];
  }
  if (p.next == NORM_NONE) return;
  if (p.next != NORM_PLAIN)
    row_norm<T, VEC, PER>(v, p.next, (const T*)p.next_w, (const T*)p.next_b, p.W, p.eps, red);
  T* xrow = (T*)p.x + t * p.W;
#pragma unroll
  for (int i = 0; i < PER; i++) {
    const int c = (int)threadIdx.x + i * (int)blockDim.x;
    if (c < nvec) store_vec<T, VEC>(xrow + (long)c * VEC, v[i]);
  }
}

// a [T, D] -> out [T, D]; the table row holds one D-wide slice per layer
template <typename T, int VEC>
__global__ void side_gate_kernel(const T* __restrict__ a, long a_stride, const long* __restrict__ ids,
                                 const T* __restrict__ table, long table_stride, long table_rows, long offset,
                                 T* __restrict__ out, long tokens, int D, int* status) {
  const int nvec = D / VEC;
  const long i = (long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= tokens * nvec) return;
  const long t = i / nvec;
  const int c = (int)(i - t * nvec) * VEC;
  const long id = ids[t];
  float av[VEC], ev[VEC];
  load_vec<T, VEC>(a + t * a_stride + c, av);
  if (id >= 0 && id < table_rows) load_vec<T, VEC>(table + id * table_stride + offset + c, ev);
  else {
#pragma unroll
    for (int e = 0; e < VEC; e++) ev[e] = 0.f;
    if (c == 0 && status) atomicCAS(status, 0, B200_BAD_INDEX);
  }
#pragma unroll
  for (int e = 0; e < VEC; e++) av[e] = gelu_tanh_f(av[e]) * ev[e];
  store_vec<T, VEC>(out + t * D + c, av);
}

// one warp per (token, head): o [T, H, D] dense, z rows with a stride, out dense
template <typename T, int VEC>
__global__ void gated_head_norm_kernel(const T* __restrict__ o, const T* __restrict__ z, long z_stride,
                                       const T* __restrict__ w, T* __restrict__ out, long rows, int H, int D,
                                       float eps) {
  const long r = (long)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int lane = threadIdx.x & 31;
  const long t = r / H;
  const int h = (int)(r - t * H);
  const T* orow = o + r * D;
  const T* zrow = z + t * z_stride + (long)h * D;
  float ss = 0.f;
  for (int c = lane * VEC; c < D; c += 32 * VEC) {
    float v[VEC];
    load_vec<T, VEC>(orow + c, v);
#pragma unroll
    for (int e = 0; e < VEC; e++) ss += v[e] * v[e];
  }
  const float inv = 1.f / sqrtf(warp_reduce_sum(ss) / (float)D + eps);
  for (int c = lane * VEC; c < D; c += 32 * VEC) {
    float v[VEC], zv[VEC], wv[VEC];
    load_vec<T, VEC>(orow + c, v);
    load_vec<T, VEC>(zrow + c, zv);
    load_vec<T, VEC>(w + c, wv);
#pragma unroll
    for (int e = 0; e < VEC; e++) v[e] = v[e] * inv * wv[e] * silu_f<T>(zv[e]);
    store_vec<T, VEC>(out + r * D + c, v);
  }
}

template <typename T, int VEC>
static int launch_stream(StreamParams& p, long tokens, cudaStream_t stream) {
  const int nvec = p.W / VEC;
  int threads = (((nvec + 1) / 2 + 31) / 32) * 32;
  if (threads > 1024) threads = 1024;
  int per = (nvec + threads - 1) / threads;
  const dim3 grid((unsigned)tokens);
  const bool grouped = p.post_groups > 1 || p.next_groups > 1;
  p.part_threads = 0;
  if (p.next_groups > 1 && (p.post == NORM_NONE || p.post == NORM_PLAIN)) {
    const int own = nvec / p.next_groups, pt = (((own + 1) / 2 + 31) / 32) * 32;
    if (pt * p.next_groups <= 1024) {
      p.part_threads = pt;
      threads = pt * p.next_groups;
      per = (own + pt - 1) / pt;
    }
  }
#define LAUNCH_STREAM(PER)                                                                    \
  if (grouped) stream_norm_kernel<T, VEC, PER, true><<<grid, threads, 0, stream>>>(p);        \
  else stream_norm_kernel<T, VEC, PER, false><<<grid, threads, 0, stream>>>(p)
  if (per <= 1) { LAUNCH_STREAM(1); }
  else if (per <= 2) { LAUNCH_STREAM(2); }
  else if (per <= 4) { LAUNCH_STREAM(4); }
  else if (per <= 8) { LAUNCH_STREAM(8); }
  else return 9710;
#undef LAUNCH_STREAM
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int stream_norm_t(StreamParams& p, long tokens, cudaStream_t stream) {
  const bool vec = p.W % 4 == 0 && p.y_stride % 4 == 0 && aligned16(p.r) && aligned16(p.y) && aligned16(p.x) &&
                   aligned16(p.table) && aligned16(p.post_w) && aligned16(p.post_b) && aligned16(p.next_w) &&
                   aligned16(p.next_b) && p.W / p.post_groups % 4 == 0 && p.W / p.next_groups % 4 == 0;
  return vec ? launch_stream<T, 4>(p, tokens, stream) : launch_stream<T, 1>(p, tokens, stream);
}

template <typename T, int VEC, int MAXS>
static int launch_mix(const MixParams& p, long tokens, cudaStream_t stream) {
  const int nvec = p.W / VEC;
  int threads = (((nvec + 1) / 2 + 31) / 32) * 32;
  if (threads > 512) threads = 512;
  const int per = (nvec + threads - 1) / threads;
  const dim3 grid((unsigned)tokens);
  if (per <= 1) stream_mix_kernel<T, VEC, 1, MAXS><<<grid, threads, 0, stream>>>(p);
  else if (per <= 2) stream_mix_kernel<T, VEC, 2, MAXS><<<grid, threads, 0, stream>>>(p);
  else if (per <= 4) stream_mix_kernel<T, VEC, 4, MAXS><<<grid, threads, 0, stream>>>(p);
  else if (per <= 16) stream_mix_kernel<T, VEC, 16, MAXS><<<grid, threads, 0, stream>>>(p);
  else return 9740;
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int stream_mix_t(const MixParams& p, long tokens, cudaStream_t stream) {
  const bool vec = p.W % 4 == 0 && p.y_stride % 4 == 0 && aligned16(p.r) && aligned16(p.y) && aligned16(p.x) &&
                   aligned16(p.table) && aligned16(p.pos_table) && aligned16(p.post_w) && aligned16(p.post_b) &&
                   aligned16(p.next_w) && aligned16(p.next_b);
  if (vec)
    return p.S <= 2 ? launch_mix<T, 4, 2>(p, tokens, stream)
                    : p.S <= 4 ? launch_mix<T, 4, 4>(p, tokens, stream) : launch_mix<T, 4, 16>(p, tokens, stream);
  return p.S <= 4 ? launch_mix<T, 1, 4>(p, tokens, stream) : launch_mix<T, 1, 16>(p, tokens, stream);
}

template <typename T>
static int side_gate_t(const void* a, long a_stride, const void* ids, const void* table, long table_stride,
                       long table_rows, long offset, void* out, long tokens, int D, int* status, cudaStream_t stream) {
  const bool vec = D % 4 == 0 && a_stride % 4 == 0 && table_stride % 4 == 0 && offset % 4 == 0 && aligned16(a) &&
                   aligned16(table) && aligned16(out);
  const long n = tokens * (D / (vec ? 4 : 1));
  const unsigned blocks = (unsigned)((n + 255) / 256);
  if (vec)
    side_gate_kernel<T, 4><<<blocks, 256, 0, stream>>>((const T*)a, a_stride, (const long*)ids, (const T*)table,
                                                       table_stride, table_rows, offset, (T*)out, tokens, D, status);
  else
    side_gate_kernel<T, 1><<<blocks, 256, 0, stream>>>((const T*)a, a_stride, (const long*)ids, (const T*)table,
                                                       table_stride, table_rows, offset, (T*)out, tokens, D, status);
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int gated_head_norm_t(const void* o, const void* z, long z_stride, const void* w, void* out, long tokens,
                             int H, int D, float eps, cudaStream_t stream) {
  const long rows = tokens * H;
  const bool vec = D % 4 == 0 && z_stride % 4 == 0 && aligned16(o) && aligned16(z) && aligned16(w) && aligned16(out);
  const unsigned blocks = (unsigned)((rows + 7) / 8);
  if (vec)
    gated_head_norm_kernel<T, 4><<<blocks, 256, 0, stream>>>((const T*)o, (const T*)z, z_stride, (const T*)w,
                                                             (T*)out, rows, H, D, eps);
  else
    gated_head_norm_kernel<T, 1><<<blocks, 256, 0, stream>>>((const T*)o, (const T*)z, z_stride, (const T*)w,
                                                             (T*)out, rows, H, D, eps);
  return B200_CHECK_LAUNCH();
}

}  // namespace b200

using namespace b200;

// dtype: 0 bf16, 1 fp32 (y, x, norm weights, table).  Kinds: 0 none, 1 layer norm, 2 RMS norm, 3 plain
// (post: add y as it is; next: round r to the activation type).  emb: 0 none, 1 set, 2 add.
B200_API int b200_stream_norm(void* r, const void* y, long y_stride, int post, const void* post_w, const void* post_b,
                              float post_scale, int emb, const void* ids, const void* table, long table_rows, float emb_scale, int next,
                              const void* next_w, const void* next_b, void* x, long tokens, int W, int post_groups, int next_groups,
                              float eps, int dtype, int* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (post_groups < 1 || next_groups < 1 || W % post_groups || W % next_groups ||
      (post_groups > 1 && post != NORM_RMS && post != NORM_NONE) || (next_groups > 1 && next != NORM_RMS && next != NORM_NONE))
    return 9703;
  if (W < 1 || (post != NORM_NONE && !y) || (next != NORM_NONE && !x) || (emb != EMB_NONE && !table)) return 9700;
  if ((post == NORM_LAYER || post == NORM_RMS) && !post_w) return 9701;
  if ((next == NORM_LAYER || next == NORM_RMS) && !next_w) return 9702;
  StreamParams p{(float*)r, y, y_stride, post, post_w, post_b, post_scale, emb, (const long*)ids, table, table_rows,
                 emb_scale, next, next_w, next_b, x, W, post_groups, next_groups, 0, eps, status};
  return dtype ? stream_norm_t<float>(p, tokens, stream) : stream_norm_t<__nv_bfloat16>(p, tokens, stream);
}

// r [tokens, S, W]; mix [S, S] and out [S] go with y, in [S] (null: ones) with the next norm; emb: 0 none,
// 1 the streams are set to emb_scale * table[ids] + pos_table[positions]
B200_API int b200_stream_mix(void* r, const void* y, long y_stride, int post, const void* post_w, const void* post_b,
                             const void* mix, const void* out, int emb, const void* ids, const void* table,
                             long table_rows, float emb_scale, const void* positions, const void* pos_table,
                             long pos_rows, const void* in, int next, const void* next_w, const void* next_b, void* x,
                             long tokens, int S, int W, int store, float eps, int dtype, int* status,
                             cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (W < 1 || S < 1 || S > 16 || (post != NORM_NONE && (!y || !mix || !out)) || (next != NORM_NONE && !x)) return 9741;
  if ((emb != EMB_NONE && emb != EMB_SET) || (emb == EMB_SET && (!table || post != NORM_NONE))) return 9742;
  if ((post == NORM_LAYER || post == NORM_RMS) && !post_w) return 9743;
  if (((next == NORM_LAYER || next == NORM_RMS) && !next_w) || (pos_table && !positions)) return 9744;
  MixParams p{(float*)r, y, y_stride, post, post_w, post_b, (const float*)mix, (const float*)out, emb, (const long*)ids,
              table, table_rows, emb_scale, (const long*)positions, pos_table, pos_rows, (const float*)in, next, next_w,
              next_b, x, W, S, store, eps, status};
  return dtype ? stream_mix_t<float>(p, tokens, stream) : stream_mix_t<__nv_bfloat16>(p, tokens, stream);
}

B200_API int b200_side_gate(const void* a, long a_stride, const void* ids, const void* table, long table_stride,
                            long table_rows, long offset, void* out, long tokens, int D, int dtype, int* status,
                            cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (D < 1 || offset < 0 || offset + D > table_stride) return 9720;
  return dtype ? side_gate_t<float>(a, a_stride, ids, table, table_stride, table_rows, offset, out, tokens, D, status,
                                    stream)
               : side_gate_t<__nv_bfloat16>(a, a_stride, ids, table, table_stride, table_rows, offset, out, tokens, D,
                                            status, stream);
}

B200_API int b200_gated_head_norm(const void* o, const void* z, long z_stride, const void* w, void* out, long tokens,
                                  int H, int D, float eps, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (H < 1 || D < 1) return 9730;
  return dtype ? gated_head_norm_t<float>(o, z, z_stride, w, out, tokens, H, D, eps, stream)
               : gated_head_norm_t<__nv_bfloat16>(o, z, z_stride, w, out, tokens, H, D, eps, stream);
}
