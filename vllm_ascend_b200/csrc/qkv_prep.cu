// From a fused projection row [q | k | v] to attention operands, in one pass over the tokens:
//   short causal convolution over time on every channel (optional, with a per-sequence state of the last
//   taps - 1 inputs), RMS norm over all heads of q (and of k) at once, interleaved rotary positions on the
//   first `rot` dimensions of a head, q to a dense buffer, keys and values to their cache slots.
// The values may be the keys as they were before the norm.  Everything between the projection and the
// stores is fp32; element type bf16 or fp32 (template), all sizes are run-time values.
//
// A block owns up to TILE consecutive tokens of one sequence and either all q channels or all k / v channels;
// a thread owns PER vectors of VEC channels and walks the tokens with the convolution window in registers, the
// next row in flight while the current one is reduced.  Only a sequence's first tile reads the convolution
// state, and the same threads write the new one afterwards, so no two blocks touch a state row.
// The reference fuses split, q / k norm and rotary the same way (vllm_ascend/ops/triton/linearnorm/
// split_qkv_rmsnorm_rope.py).
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

struct QkvPrepArgs {
  const void* qkv;            // [T, qkv_stride]
  const void* conv_w;         // [C, taps] or null
  void* state;                // [state_rows, taps - 1, C], oldest input first
  const int *cu, *slots, *has_init;
  const void *q_norm, *k_norm;
  const long* positions;      // [T]
  const float* cos_sin;       // [cos_rows, rot]: cosines, then sines
  const long* slot_mapping;   // [T]; < 0: not stored
  void* q_out;                // [T, heads * dim]
  void *k_cache, *v_cache;
  float* sums;                // [T, 2] sums of squares of q and k (phases 1 and 2)
  long qkv_stride, state_rows, cache_slots;
  long k_block, k_tok, k_head, v_block, v_tok, v_head;      // cache strides in elements
  long tokens;
  int num_seqs, taps, heads, kv_heads, dim, vdim;
  int q_norm_dims, k_norm_dims;      // widths of the means
  int values_from_keys, rot, cos_rows, block_size;
  int uniform;                // every sequence has exactly one token
  int phase;                  // 0: all; 1: only the sums; 2: with the given sums
  int dtype;
  float eps;
};

struct QkvPrepParams : QkvPrepArgs {
  int tile;                   // tokens of a block
  int* status;
};

constexpr int PREP_THREADS = 512;

// KR: taps held in registers (0: no convolution, 4: up to four taps, -1: any number, read again per token)
template <typename T, int VEC, int PER, int KR>
__global__ void __launch_bounds__(PREP_THREADS) qkv_prep_kernel(const QkvPrepParams p) {
  __shared__ float red[2][32];
  extern __shared__ float row[];                    // VEC == 1: the normalised row, for the rotary partner
  const int part = blockIdx.y;
  const int Nq = p.heads * p.dim, Nk = p.kv_heads * p.dim, Nv = p.values_from_keys ? 0 : p.kv_heads * p.vdim;
  const int C = Nq + Nk + Nv;
  const int width = part == 0 ? Nq : Nk + Nv, col0 = part == 0 ? 0 : Nq;
  const int nvec = width / VEC, normed = part == 0 ? Nq : Nk;
  // ---- tokens [t_seq + i0, t_seq + i1) of sequence b
  int b = 0, i0, i1, n;
  long t_seq;
  if (KR == 0) {                                    // tokens are independent
    t_seq = (long)blockIdx.x * p.tile;
    i0 = 0;
    n = i1 = (int)min((long)p.tile, p.tokens - t_seq);
  } else if (p.uniform) {
    b = blockIdx.x;
    t_seq = b;
    i0 = 0;
    n = i1 = 1;
  } else {
    const int w = blockIdx.x;
    int lo = 0, hi = p.num_seqs - 1;
    while (lo < hi) {                               // sequence b owns the tiles from cu[b] / tile + b on
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu[mid] / p.tile + mid <= w) lo = mid; else hi = mid - 1;
    }
    b = lo;
    t_seq = p.cu[b];
    n = p.cu[b + 1] - (int)t_seq;
    i0 = (w - ((int)t_seq / p.tile + b)) * p.tile;
    i1 = min(i0 + p.tile, n);
  }
  if (i0 >= i1) return;
  const T* x = (const T*)p.qkv + t_seq * p.qkv_stride + col0;
  bool init = false;
  T* st = nullptr;
  if (KR != 0 && p.taps > 1) {
    const int slot = p.slots[b];
    if (slot < 0 || slot >= p.state_rows) {
      if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
      return;
    }
    st = (T*)p.state + (long)slot * (p.taps - 1) * C + col0;
    init = p.has_init[b] != 0;
  }
  auto input = [&](int i, int c, T* v) {            // input of local token i, reaching back into the state
    if (i >= 0) load_raw<T, VEC>(x + (long)i * p.qkv_stride + c, v);
    else if (init && p.taps - 1 + i >= 0) load_raw<T, VEC>(st + (long)(p.taps - 1 + i) * C + c, v);
    else
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] = from_f<T>(0.f);
  };
  constexpr int KW = KR > 0 ? KR : 1;
  T wk[PER][KW][VEC], win[PER][KW][VEC], nxt[PER][VEC];
#pragma unroll
  for (int r = 0; r < PER; r++) {
    const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
    if (v >= nvec) continue;
    if constexpr (KR > 0) {
      const T* w = (const T*)p.conv_w + (long)(col0 + c) * p.taps;
      if (VEC > 1 && p.taps == KR) {                // KR * VEC weights in a row
        constexpr int WV = 16 / (int)sizeof(T);
        T wr[KR * VEC];
#pragma unroll
        for (int k = 0; k < KR * VEC; k += (VEC > 1 ? WV : 1)) load_raw<T, (VEC > 1 ? WV : 1)>(w + k, wr + k);
#pragma unroll
        for (int k = 0; k < KR * VEC; k++) wk[r][k % KR][k / KR] = wr[k];
      } else {
#pragma unroll
        for (int j = 0; j < KR; j++) {
          const int jj = j - (KR - p.taps);         // fewer taps: the oldest places weigh nothing
#pragma unroll
          for (int e = 0; e < VEC; e++) wk[r][j][e] = jj >= 0 ? w[(long)e * p.taps + jj] : from_f<T>(0.f);
        }
      }
#pragma unroll
      for (int j = 0; j < KR - 1; j++) {
        if (j >= KR - p.taps) input(i0 - (KR - 1) + j, c, win[r][j]);
        else
#pragma unroll
          for (int e = 0; e < VEC; e++) win[r][j][e] = from_f<T>(0.f);
      }
    }
    load_raw<T, VEC>(x + (long)i0 * p.qkv_stride + c, nxt[r]);
  }
  const int warps = (blockDim.x + 31) >> 5;
  const T* nw = (const T*)(part == 0 ? p.q_norm : p.k_norm);
  const int half = p.rot >> 1;

  for (int i = i0; i < i1; i++) {
    const long t = t_seq + i;
    float u[PER][VEC];
    float ss = 0.f;
#pragma unroll
    for (int r = 0; r < PER; r++) {
      const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
      if (v >= nvec) continue;
      if constexpr (KR > 0) {
#pragma unroll
        for (int e = 0; e < VEC; e++) {
          win[r][KR - 1][e] = nxt[r][e];
          float a = 0.f;
#pragma unroll
          for (int j = 0; j < KR; j++) a = fmaf(to_f(wk[r][j][e]), to_f(win[r][j][e]), a);
          u[r][e] = a;
        }
#pragma unroll
        for (int j = 0; j + 1 < KR; j++)
#pragma unroll
          for (int e = 0; e < VEC; e++) win[r][j][e] = win[r][j + 1][e];
      } else if constexpr (KR < 0) {
        const T* w = (const T*)p.conv_w + (long)(col0 + c) * p.taps;
#pragma unroll
        for (int e = 0; e < VEC; e++) u[r][e] = 0.f;
        for (int j = 0; j < p.taps; j++) {
          T in[VEC];
          input(i - (p.taps - 1) + j, c, in);
#pragma unroll
          for (int e = 0; e < VEC; e++) u[r][e] = fmaf(to_f(w[(long)e * p.taps + j]), to_f(in[e]), u[r][e]);
        }
      } else {
#pragma unroll
        for (int e = 0; e < VEC; e++) u[r][e] = to_f(nxt[r][e]);
      }
      if (KR >= 0 && i + 1 < i1) load_raw<T, VEC>(x + (long)(i + 1) * p.qkv_stride + c, nxt[r]);
      if (c < normed)
#pragma unroll
        for (int e = 0; e < VEC; e++) ss = fmaf(u[r][e], u[r][e], ss);
    }
    if (p.phase == 2) {
      ss = p.sums[t * 2 + part];
    } else {
      ss = warp_reduce_sum(ss);
      if (warps > 1) {
        float* rd = red[(i - i0) & 1];              // two buffers: one barrier per token
        if ((threadIdx.x & 31) == 0) rd[threadIdx.x >> 5] = ss;
        __syncthreads();
        ss = warp_reduce_sum((threadIdx.x & 31) < warps ? rd[threadIdx.x & 31] : 0.f);
      }
      if (p.phase == 1) {
        if (threadIdx.x == 0) p.sums[t * 2 + part] = ss;
        continue;
      }
    }
    const float inv = 1.f / sqrtf(ss / (float)(part == 0 ? p.q_norm_dims : p.k_norm_dims) + p.eps);
    long slot = -1;
    T *kdst = nullptr, *vdst = nullptr;
    if (part == 1) {
      slot = p.slot_mapping[t];
      if (slot >= p.cache_slots) {
        if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
        slot = -1;
      }
      if (slot >= 0) {
        const long blk = slot / p.block_size, off = slot - blk * p.block_size;
        kdst = (T*)p.k_cache + blk * p.k_block + off * p.k_tok;
        vdst = (T*)p.v_cache + blk * p.v_block + off * p.v_tok;
      }
    }
    const float* cs = nullptr;
    if (p.rot > 0) {
      const long pos = p.positions[t];
      if (pos >= 0 && pos < p.cos_rows) cs = p.cos_sin + pos * p.rot;
      else if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    }
    if constexpr (VEC == 1) {
      if (cs) {
        __syncthreads();                            // the previous token's partners have been read
#pragma unroll
        for (int r = 0; r < PER; r++) {
          const int c = (int)threadIdx.x + r * (int)blockDim.x;
          if (c < normed) row[c] = u[r][0] * inv * to_f(nw[c]);
        }
        __syncthreads();
      }
    }
#pragma unroll
    for (int r = 0; r < PER; r++) {
      const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
      if (v >= nvec) continue;
      if (c >= normed) {                            // values
        const int h = (c - normed) / p.vdim, d = (c - normed) - h * p.vdim;
        if (vdst) store_vec<T, VEC>(vdst + h * p.v_head + d, u[r]);
        continue;
      }
      const int h = c / p.dim, d = c - h * p.dim;
      if (part == 1 && p.values_from_keys && vdst) store_vec<T, VEC>(vdst + h * p.v_head + d, u[r]);
      float wv[VEC], y[VEC];
      load_vec<T, VEC>(nw + c, wv);
#pragma unroll
      for (int e = 0; e < VEC; e++) y[e] = u[r][e] * inv * wv[e];
      if (cs && d < p.rot) {
        if constexpr (VEC == 1) {
          const int k = d >> 1;
          const float other = (d & 1) ? row[c - 1] : row[c + 1];
          y[0] = (d & 1) ? y[0] * cs[k] + other * cs[half + k] : y[0] * cs[k] - other * cs[half + k];
        } else {
#pragma unroll
          for (int e = 0; e + 1 < VEC; e += 2) {
            if (d + e < p.rot) {
              const int k = (d + e) >> 1;
              const float cc = cs[k], sn = cs[half + k], a = y[e], bb = y[e + 1];
              y[e] = a * cc - bb * sn;
              y[e + 1] = bb * cc + a * sn;
            }
          }
        }
      }
      if (part == 0) store_vec<T, VEC>((T*)p.q_out + t * Nq + c, y);
      else if (kdst) store_vec<T, VEC>(kdst + h * p.k_head + d, y);
    }
  }
  // ---- the last taps - 1 inputs of the sequence (its first tile owns the state row)
  if (KR != 0 && p.taps > 1 && i0 == 0 && p.phase != 1) {
#pragma unroll
    for (int r = 0; r < PER; r++) {
      const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
      if (v >= nvec) continue;
      for (int j = 0; j < p.taps - 1; j++) {
        T in[VEC];
        input(n - (p.taps - 1) + j, c, in);         // older rows move towards the front
        float f[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) f[e] = to_f(in[e]);
        store_vec<T, VEC>(st + (long)j * C + c, f);
      }
    }
  }
}

template <typename T, int VEC, int PER>
static int launch_prep(const QkvPrepParams& p, dim3 grid, int threads, size_t smem, cudaStream_t stream) {
  if (smem > 48 * 1024) return 9820;
  if (p.taps == 0) qkv_prep_kernel<T, VEC, PER, 0><<<grid, threads, smem, stream>>>(p);
  else if (p.taps <= 4) qkv_prep_kernel<T, VEC, PER, 4><<<grid, threads, smem, stream>>>(p);
  else qkv_prep_kernel<T, VEC, PER, -1><<<grid, threads, smem, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int prep_t(QkvPrepParams& p, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const int Nq = p.heads * p.dim, Nkv = p.kv_heads * (p.dim + (p.values_from_keys ? 0 : p.vdim));
  const int width = Nq > Nkv ? Nq : Nkv;
  const long s[] = {p.qkv_stride, p.k_block, p.k_tok, p.k_head, p.v_block, p.v_tok, p.v_head, p.dim, p.vdim};
  bool vec = aligned16(p.qkv) && aligned16(p.conv_w) && aligned16(p.state) && aligned16(p.q_norm) &&
             aligned16(p.k_norm) && aligned16(p.q_out) && aligned16(p.k_cache) && aligned16(p.v_cache);
  for (long x : s) vec = vec && x % V == 0;
  const int nvec = width / (vec ? V : 1);
  int per = (nvec + PREP_THREADS - 1) / PREP_THREADS;
  per = vec ? (per <= 1 ? 1 : per <= 2 ? 2 : 4) : (per <= 2 ? 2 : 16);
  if ((long)per * PREP_THREADS < nvec) return 9821;
  const int threads = ((nvec + per - 1) / per + 31) / 32 * 32;
  // tokens of a block: enough to share the convolution's history and weights, few enough to fill the GPU
  p.tile = p.tokens >= 8192 ? 16 : p.tokens >= 2048 ? 8 : p.tokens >= 512 ? 2 : 1;
  if (p.taps > 0 && p.tile < 4) p.tile = 4;
  if (p.tile < p.taps - 1) p.tile = p.taps - 1;     // only a first tile reaches back into the state
  const long tiles = p.taps == 0 ? (p.tokens + p.tile - 1) / p.tile
                                 : p.uniform ? p.num_seqs : p.tokens / p.tile + p.num_seqs;
  const dim3 grid((unsigned)tiles, 2);
  if (vec) {
    if (per == 1) return launch_prep<T, V, 1>(p, grid, threads, 0, stream);
    if (per == 2) return launch_prep<T, V, 2>(p, grid, threads, 0, stream);
    return launch_prep<T, V, 4>(p, grid, threads, 0, stream);
  }
  const size_t smem = p.rot > 0 ? (size_t)width * 4 : 0;
  if (per == 2) return launch_prep<T, 1, 2>(p, grid, threads, smem, stream);
  return launch_prep<T, 1, 16>(p, grid, threads, smem, stream);
}

}  // namespace b200

using namespace b200;

B200_API int b200_qkv_prep(const QkvPrepArgs* a, int* status, cudaStream_t stream) {
  if (a->tokens <= 0) return 0;
  if (a->heads < 1 || a->kv_heads < 1 || a->dim < 1 || a->vdim < 1 || a->block_size < 1 || a->num_seqs < 1) return 9800;
  if (a->rot < 0 || a->rot > a->dim || (a->rot & 1) || (a->rot > 0 && !a->cos_sin)) return 9801;
  if (a->values_from_keys && a->vdim != a->dim) return 9802;
  if (a->taps < 0 || (a->taps > 0 && !a->conv_w)) return 9803;
  if (a->taps > 1 && (!a->state || !a->slots || !a->has_init || !a->cu)) return 9804;
  if (a->phase != 0 && !a->sums) return 9805;
  if (a->taps == 1 && !a->cu) return 9806;
  QkvPrepParams p;
  static_cast<QkvPrepArgs&>(p) = *a;
  p.status = status;
  return a->dtype ? prep_t<float>(p, stream) : prep_t<__nv_bfloat16>(p, stream);
}
