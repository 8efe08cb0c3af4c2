// MoE routing and token movement kernels.
//   * gating top-k: softmax / sigmoid scores, correction bias, group-limited selection,
//     renormalisation and scaling in one warp-per-token kernel (the reference's
//     moe_gating_top_k op, csrc/moe/moe_gating_top_k; signature torch_binding.cpp:2135-2150)
//   * permute: histogram of tokens per local expert, exclusive offsets, and the gather of
//     token rows into expert-major order (npu_moe_init_routing_v2 / npu_moe_token_permute)
//   * combine: weighted sum (sum, where the inputs were weighted) of the k expert outputs of every token (npu_moe_token_unpermute), where the
//     output of a shared expert joins, scaled by the sigmoid of a dot product with the layer's input
// The grouped GEMMs in between are csrc/gemm_bf16.cu (GROUPED mode) and
// csrc/gemm_fp8_block.cu; moe_linear is the same product on the CUDA cores, for fp32 and for sizes those
// kernels do not take.
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

constexpr int GATE_MAX_PER_LANE = 16;   // experts <= 512

// logits [T, E] fp32 -> weights [T, k] fp32, ids [T, k] int32
// scoring: 0 softmax, 1 sigmoid.  Group-limited: experts are split into n_group groups, the
// topk_group groups with the best group score stay eligible (group score = max, or with top2 the sum
// of the best two).  Selection uses score + bias, the
// returned weight is the unbiased score.
__global__ void moe_gating_topk_kernel(const float* __restrict__ logits, const float* __restrict__ bias,
                                       float* __restrict__ weights, int* __restrict__ ids, int T,
                                       int E, int k, int scoring, int renorm, int n_group,
                                       int topk_group, int top2, float scale) {
  const int warps = blockDim.x >> 5;
  const int t = blockIdx.x * warps + (threadIdx.x >> 5);
  if (t >= T) return;
  const int lane = threadIdx.x & 31;
  const int per = (E + 31) / 32;
  float score[GATE_MAX_PER_LANE], choice[GATE_MAX_PER_LANE];
  const float* row = logits + (size_t)t * E;
  float mx = -INFINITY;
#pragma unroll
  for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
    const int e = lane + 32 * i;
    score[i] = (i < per && e < E) ? row[e] : -INFINITY;
    mx = fmaxf(mx, score[i]);
  }
  if (scoring == 0) {
    mx = warp_reduce_max(mx);
    float sum = 0.f;
#pragma unroll
    for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
      const int e = lane + 32 * i;
      score[i] = (i < per && e < E) ? expf(score[i] - mx) : 0.f;
      sum += score[i];
    }
    sum = warp_reduce_sum(sum);
    const float inv = 1.f / sum;
#pragma unroll
    for (int i = 0; i < GATE_MAX_PER_LANE; i++) score[i] *= inv;
  } else {
#pragma unroll
    for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
      const int e = lane + 32 * i;
      score[i] = (i < per && e < E) ? 1.f / (1.f + expf(-score[i])) : 0.f;
    }
  }
#pragma unroll
  for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
    const int e = lane + 32 * i;
    choice[i] = (i < per && e < E) ? score[i] + (bias ? bias[e] : 0.f) : -INFINITY;
  }
  if (n_group > 1) {
    // group scores; every lane ends up with the eligibility of all groups (n_group <= 32)
    const int gsz = E / n_group;
    float my_gscore = -INFINITY;                 // lane g holds the score of group g
    for (int g = 0; g < n_group; g++) {
      float b1 = -INFINITY, b2 = -INFINITY;      // best two inside the group among my experts
#pragma unroll
      for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
        const int e = lane + 32 * i;
        if (i < per && e < E && e / gsz == g) {
          const float v = choice[i];
          if (v > b1) { b2 = b1; b1 = v; } else if (v > b2) { b2 = v; }
        }
      }
      // merge the per-lane (best, second) pairs across the warp
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float o1 = __shfl_xor_sync(0xffffffffu, b1, o);
        const float o2 = __shfl_xor_sync(0xffffffffu, b2, o);
        const float n1 = fmaxf(b1, o1);
        const float n2 = fmaxf(fminf(b1, o1), fmaxf(b2, o2));
        b1 = n1;
        b2 = n2;
      }
      const float gs = top2 && gsz > 1 ? b1 + b2 : b1;
      if (lane == g) my_gscore = gs;
    }
    // pick topk_group groups
    unsigned keep = 0;
    for (int r = 0; r < topk_group; r++) {
      float v = my_gscore;
      int idx = lane;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, v, o);
        const int oi = __shfl_xor_sync(0xffffffffu, idx, o);
        if (ov > v || (ov == v && oi < idx)) { v = ov; idx = oi; }
      }
      keep |= 1u << idx;
      if (lane == idx) my_gscore = -INFINITY;
    }
#pragma unroll
    for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
      const int e = lane + 32 * i;
      if (i < per && e < E && !((keep >> (e / gsz)) & 1u)) choice[i] = -INFINITY;
    }
  }
  // iterative top-k (lowest index wins ties)
  float wsum = 0.f;
  float my_w = 0.f;
  int my_id = 0;
  for (int r = 0; r < k; r++) {
    float v = -INFINITY;
    int idx = 0x7fffffff;
    float sc = 0.f;
#pragma unroll
    for (int i = 0; i < GATE_MAX_PER_LANE; i++) {
      const int e = lane + 32 * i;
      if (i < per && e < E && (choice[i] > v || (choice[i] == v && e < idx))) {
        v = choice[i]; idx = e; sc = score[i];
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, v, o);
      const int oi = __shfl_xor_sync(0xffffffffu, idx, o);
      const float os = __shfl_xor_sync(0xffffffffu, sc, o);
      if (ov > v || (ov == v && oi < idx)) { v = ov; idx = oi; sc = os; }
    }
    if ((idx & 31) == lane) {
#pragma unroll
      for (int i = 0; i < GATE_MAX_PER_LANE; i++)
        if (lane + 32 * i == idx) choice[i] = -INFINITY;
    }
    wsum += sc;
    if (lane == r) { my_w = sc; my_id = idx; }
  }
  if (lane < k) {
    float w = my_w;
    if (renorm) w /= fmaxf(wsum, 1e-20f);
    weights[(size_t)t * k + lane] = w * scale;
    ids[(size_t)t * k + lane] = my_id;
  }
}

// ---------------------------------------------------------------- permute
// local_ids [T*k] int32 (expert on this rank, or -1).  counts/cursor [E] zeroed by the caller.
__global__ void moe_count_kernel(const int* __restrict__ local_ids, int n, int E, int* counts) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) {
    const int e = local_ids[i];
    if (e >= 0 && e < E) atomicAdd(&counts[e], 1);
  }
}
// offsets[E+1] = exclusive prefix sum of counts (single block)
__global__ void moe_scan_kernel(const int* __restrict__ counts, int E, int* offsets) {
  __shared__ int s[1024];
  const int t = threadIdx.x;
  int v = t < E ? counts[t] : 0;
  s[t] = v;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int add = t >= o ? s[t - o] : 0;
    __syncthreads();
    s[t] += add;
    __syncthreads();
  }
  if (t < E) offsets[t + 1] = s[t];
  if (t == 0) offsets[0] = 0;
}
// pos[i] = destination row of pair i (or -1); src_token[row] = token of that row
__global__ void moe_assign_kernel(const int* __restrict__ local_ids, int n, int k, int E,
                                  const int* __restrict__ offsets, int* cursor, int* pos,
                                  int* src_token) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= n) return;
  const int e = local_ids[i];
  if (e < 0 || e >= E) {
    pos[i] = -1;
    return;
  }
  const int r = offsets[e] + atomicAdd(&cursor[e], 1);
  pos[i] = r;
  src_token[r] = i / k;
}
// weight of every expert-major row: out[pos[i]] = w[i]
__global__ void moe_row_weights_kernel(const float* __restrict__ w, const int* __restrict__ pos, int n,
                                       float* __restrict__ out) {
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n && pos[i] >= 0) out[pos[i]] = w[i];
}
// out[row] = x[src_token[row]] for row < offsets[E]
__global__ void moe_gather_rows_kernel(const __nv_bfloat16* __restrict__ x,
                                       const int* __restrict__ src_token,
                                       const int* __restrict__ offsets, int E, int H,
                                       __nv_bfloat16* __restrict__ out) {
  const int row = blockIdx.x;
  if (row >= offsets[E]) return;
  const uint4* src = reinterpret_cast<const uint4*>(x + (size_t)src_token[row] * H);
  uint4* dst = reinterpret_cast<uint4*>(out + (size_t)row * H);
  for (int v = threadIdx.x; v < (H >> 3); v += blockDim.x) dst[v] = src[v];
}
// out[t] = sum_s w[t,s] * y[pos[t,s]] (+ sigmoid(x[t] . gate) * shared[t])
template <typename T, int VEC>
__global__ void __launch_bounds__(512) moe_combine_kernel(const T* __restrict__ y, const int* __restrict__ pos,
                                                          const float* __restrict__ w, int k, int H, T* __restrict__ out,
                                                          int accumulate, const T* __restrict__ shared,
                                                          const T* __restrict__ x, const T* __restrict__ gate) {
  const long t = blockIdx.x;
  float g = 1.f;
  if (gate) {
    __shared__ float red[16];
    float dot = 0.f;
    for (int c = (int)threadIdx.x * VEC; c < H; c += (int)blockDim.x * VEC) {
      float a[VEC], b[VEC];
      load_vec<T, VEC>(x + t * H + c, a);
      load_vec<T, VEC>(gate + c, b);
#pragma unroll
      for (int e = 0; e < VEC; e++) dot = fmaf(a[e], b[e], dot);
    }
    dot = warp_reduce_sum(dot);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = dot;
    __syncthreads();
    dot = warp_reduce_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f);
    g = 1.f / (1.f + expf(-dot));
  }
  for (int c = (int)threadIdx.x * VEC; c < H; c += (int)blockDim.x * VEC) {
    float acc[VEC], v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) acc[e] = 0.f;
    if (accumulate) load_vec<T, VEC>(out + t * H + c, acc);
#pragma unroll 4
    for (int s = 0; s < k; s++) {
      const int r = pos[t * k + s];
      if (r < 0) continue;
      const float ws = w ? w[t * k + s] : 1.f;
      load_vec<T, VEC>(y + (long)r * H + c, v);
#pragma unroll
      for (int e = 0; e < VEC; e++) acc[e] += ws * v[e];
    }
    if (shared) {
      load_vec<T, VEC>(shared + t * H + c, v);
#pragma unroll
      for (int e = 0; e < VEC; e++) acc[e] = fmaf(g, v[e], acc[e]);
    }
    store_vec<T, VEC>(out + t * H + c, acc);
  }
}

template <typename T>
static int launch_combine(const void* y, const void* pos, const void* w, int tokens, int k, int H, void* out,
                          int accumulate, const void* shared, const void* x, const void* gate, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool vec = H % V == 0 && aligned16(y) && aligned16(out) && aligned16(shared) && aligned16(x) && aligned16(gate);
  int threads = (H / (vec ? V : 1) + 31) / 32 * 32;     // few tokens: a block takes its row at once
  if (threads > (tokens < 2048 ? 512 : 128)) threads = tokens < 2048 ? 512 : 128;
  if (threads < 32) threads = 32;
  if (vec)
    moe_combine_kernel<T, V><<<tokens, threads, 0, stream>>>((const T*)y, (const int*)pos, (const float*)w, k, H, (T*)out,
                                                         accumulate, (const T*)shared, (const T*)x, (const T*)gate);
  else
    moe_combine_kernel<T, 1><<<tokens, threads, 0, stream>>>((const T*)y, (const int*)pos, (const float*)w, k, H, (T*)out,
                                                         accumulate, (const T*)shared, (const T*)x, (const T*)gate);
  return B200_CHECK_LAUNCH();
}

// ---------------------------------------------------------------- grouped product on the CUDA cores
constexpr int ML_TILE = 32;

// Rows [offsets[e], offsets[e + 1]) of a (row r is a[src[r]] with src) meet w[e]: [N, K], or with GLU [2N, K] =
// gate rows | up rows and out = glu(scale a gate^T, scale a up^T) with a factor per row (null: 1).  A block computes
// 32 rows x 32 columns.
template <typename T, bool GLU>
__global__ void __launch_bounds__(256) moe_linear_kernel(const T* __restrict__ a, const int* __restrict__ src,
                                                         const T* __restrict__ w, T* __restrict__ out,
                                                         const int* __restrict__ offsets, int E, int rows, int N, int K,
                                                         const float* __restrict__ scale, float alpha, float limit) {
  __shared__ float sa[ML_TILE][ML_TILE + 1], sw[GLU ? 2 : 1][ML_TILE][ML_TILE + 1];
  const int tile = blockIdx.x;
  int lo = 0, hi = E - 1;
  while (lo < hi) {                                  // group e owns the tiles from offsets[e] / 32 + e on
    const int mid = (lo + hi + 1) >> 1;
    if (offsets[mid] / ML_TILE + mid <= tile) lo = mid; else hi = mid - 1;
  }
  const int r0 = offsets[lo] + (tile - offsets[lo] / ML_TILE - lo) * ML_TILE;
  const int r1 = min(offsets[lo + 1], rows);
  if (r0 < 0 || r0 >= r1) return;
  const int n0 = blockIdx.y * ML_TILE;
  const T* we = w + (long)lo * (GLU ? 2 : 1) * N * K;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[GLU ? 2 : 1][2][2] = {};
  for (int k0 = 0; k0 < K; k0 += ML_TILE) {
    for (int i = threadIdx.x; i < ML_TILE * ML_TILE; i += 256) {
      const int r = i / ML_TILE, k = k0 + i % ML_TILE;
      const int row = r0 + r;
      sa[r][i % ML_TILE] = row < r1 && k < K ? to_f(a[(long)(src ? src[row] : row) * K + k]) : 0.f;
#pragma unroll
      for (int h = 0; h < (GLU ? 2 : 1); h++)
        sw[h][r][i % ML_TILE] = n0 + r < N && k < K ? to_f(we[((long)h * N + n0 + r) * K + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < ML_TILE; k++) {
      const float a0 = sa[ty][k], a1 = sa[ty + 16][k];
#pragma unroll
      for (int h = 0; h < (GLU ? 2 : 1); h++) {
        const float b0 = sw[h][tx][k], b1 = sw[h][tx + 16][k];
        acc[h][0][0] = fmaf(a0, b0, acc[h][0][0]);
        acc[h][0][1] = fmaf(a0, b1, acc[h][0][1]);
        acc[h][1][0] = fmaf(a1, b0, acc[h][1][0]);
        acc[h][1][1] = fmaf(a1, b1, acc[h][1][1]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; i++)
#pragma unroll
    for (int j = 0; j < 2; j++) {
      const int row = r0 + ty + 16 * i, n = n0 + tx + 16 * j;
      if (row >= r1 || n >= N) continue;
      float v = acc[0][i][j];
      if constexpr (GLU) {
        const float f = scale ? scale[row] : 1.f;
        v = glu_f(v * f, acc[1][i][j] * f, alpha, limit);
      }
      out[(long)row * N + n] = from_f<T>(v);
    }
}

template <typename T>
static int launch_moe_linear(const void* a, const void* src, const void* w, void* out, const void* offsets, int E, int rows,
                             int N, int K, int swiglu, const void* scale, float alpha, float limit, cudaStream_t stream) {
  const dim3 grid((unsigned)(rows / ML_TILE + E), (unsigned)((N + ML_TILE - 1) / ML_TILE));
  if (swiglu)
    moe_linear_kernel<T, true><<<grid, 256, 0, stream>>>((const T*)a, (const int*)src, (const T*)w, (T*)out,
                                                         (const int*)offsets, E, rows, N, K, (const float*)scale, alpha,
                                                         limit);
  else
    moe_linear_kernel<T, false><<<grid, 256, 0, stream>>>((const T*)a, (const int*)src, (const T*)w, (T*)out,
                                                          (const int*)offsets, E, rows, N, K, nullptr, 0.f, 0.f);
  return B200_CHECK_LAUNCH();
}

}  // namespace b200

using namespace b200;

B200_API int b200_moe_gating_topk(const void* logits, const void* bias, void* weights, void* ids,
                                  int T, int E, int k, int scoring, int renorm, int n_group,
                                  int topk_group, int top2, float scale, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (E > 32 * GATE_MAX_PER_LANE || k > 32 || k > E) return 9150;
  if (n_group > 1 && (n_group > 32 || E % n_group || topk_group > n_group)) return 9151;
  const int wpb = 4;
  moe_gating_topk_kernel<<<(T + wpb - 1) / wpb, wpb * 32, 0, stream>>>(
      (const float*)logits, (const float*)bias, (float*)weights, (int*)ids, T, E, k, scoring,
      renorm, n_group, topk_group, top2, scale);
  return B200_CHECK_LAUNCH();
}

// Builds expert-major order for the (token, slot) pairs whose expert lives on this rank.
// workspace ints: counts[E] | cursor[E] | offsets[E+1]; all written here.
B200_API int b200_moe_permute(const void* local_ids, int T, int k, int E, void* counts,
                              void* cursor, void* offsets, void* pos, void* src_token,
                              cudaStream_t stream) {
  if (E > 1024) return 9152;
  const int n = T * k;
  cudaMemsetAsync(counts, 0, sizeof(int) * E, stream);
  cudaMemsetAsync(cursor, 0, sizeof(int) * E, stream);
  if (n > 0) {
    moe_count_kernel<<<(n + 255) / 256, 256, 0, stream>>>((const int*)local_ids, n, E, (int*)counts);
  }
  moe_scan_kernel<<<1, 1024, 0, stream>>>((const int*)counts, E, (int*)offsets);
  if (n > 0) {
    moe_assign_kernel<<<(n + 255) / 256, 256, 0, stream>>>((const int*)local_ids, n, k, E,
                                                           (const int*)offsets, (int*)cursor,
                                                           (int*)pos, (int*)src_token);
  }
  return B200_CHECK_LAUNCH();
}

// fp32 out[pos[i]] = w[i] for the n (token, slot) pairs of b200_moe_permute
B200_API int b200_moe_row_weights(const void* w, const void* pos, int n, void* out, cudaStream_t stream) {
  if (n <= 0) return 0;
  moe_row_weights_kernel<<<(n + 255) / 256, 256, 0, stream>>>((const float*)w, (const int*)pos, n, (float*)out);
  return B200_CHECK_LAUNCH();
}

B200_API int b200_moe_gather_rows(const void* x, const void* src_token, const void* offsets, int E,
                                  int H, int max_rows, void* out, cudaStream_t stream) {
  if (max_rows <= 0) return 0;
  if (H & 7) return 9100;
  moe_gather_rows_kernel<<<max_rows, 128, 0, stream>>>((const __nv_bfloat16*)x,
                                                       (const int*)src_token,
                                                       (const int*)offsets, E, H,
                                                       (__nv_bfloat16*)out);
  return B200_CHECK_LAUNCH();
}

// shared [T, H] or null; x [T, H] and gate [H] or null.  dtype: 0 bf16, 1 fp32
B200_API int b200_moe_combine(const void* y, const void* pos, const void* w, int T, int k, int H,
                              void* out, int accumulate, const void* shared, const void* x, const void* gate, int dtype,
                              cudaStream_t stream) {
  if (T <= 0) return 0;
  if (H < 1 || (gate && !x)) return 9100;
  return dtype ? launch_combine<float>(y, pos, w, T, k, H, out, accumulate, shared, x, gate, stream)
               : launch_combine<__nv_bfloat16>(y, pos, w, T, k, H, out, accumulate, shared, x, gate, stream);
}

// a [*, K], src [rows] or null, w [E, N (2N with swiglu), K], out [rows, N], offsets int32 [E + 1].  With swiglu: row_scale
// fp32 [rows] or null, alpha 0 the SiLU gate, else the clamped one.  dtype: 0 bf16, 1 fp32
B200_API int b200_moe_linear(const void* a, const void* src, const void* w, void* out, const void* offsets, int E, int rows,
                             int N, int K, int swiglu, const void* row_scale, float alpha, float limit, int dtype,
                             cudaStream_t stream) {
  if (rows <= 0 || E <= 0) return 0;
  if (N < 1 || K < 1) return 9153;
  return dtype ? launch_moe_linear<float>(a, src, w, out, offsets, E, rows, N, K, swiglu, row_scale, alpha, limit, stream)
               : launch_moe_linear<__nv_bfloat16>(a, src, w, out, offsets, E, rows, N, K, swiglu, row_scale, alpha, limit, stream);
}
