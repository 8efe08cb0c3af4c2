// From a fused projection row [q | k | v] to attention operands, in one pass over the tokens:
//   short causal convolution over time on every channel (optional, with a per-sequence state of the last
//   taps - 1 inputs), RMS norm over all heads of q (and of k) at once, interleaved rotary positions on the
//   first `rot` dimensions of a head, q to a dense buffer, keys and values to their cache slots.
// The norm may also be head by head with one weight for all heads (qkv_head_kernel, no convolution): a group of
// lanes owns one head of one token, so no barrier is needed.  Or absent, with a factor of the queries by position and
// wide queries (qkv_spread_kernel): a cache row holds several projected keys side by side, and part c of an output
// head's query is a weighted sum of the projected queries that go with key part c.
// The values may be the keys as they were before the norm.  Everything between the projection and the
// stores is fp32; element type bf16 or fp32 (template), all sizes are run-time values.
//
// A block owns up to TILE consecutive tokens of one sequence and either all q channels or all k / v channels;
// a thread owns PER vectors of VEC channels and walks the tokens GT at a time with the convolution window in
// registers, the next rows in flight while the current ones are reduced (one barrier per GT tokens).  Only a sequence's first tile reads the convolution
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
  const float* mix;           // [out_heads, heads] or null: identity
  const float* q_scale;       // [q_scale_rows] factor of the queries by position, or null
  long qkv_stride, state_rows, cache_slots;
  long k_block, k_tok, k_head, v_block, v_tok, v_head;      // cache strides in elements
  long tokens;
  int num_seqs, taps, heads, kv_heads, dim, vdim;
  int q_norm_dims, k_norm_dims;      // widths of the means
  int values_from_keys, rot, cos_rows, block_size;
  int uniform;                // every sequence has exactly one token
  int phase;                  // 0: all; 1: only the sums; 2: with the given sums
  int dtype;
  int head_norm;              // every head by itself: q_norm, k_norm [dim]
  int v_heads;
  int key_parts;              // > 0: qkv_spread_kernel, projected keys per cache row
  int part_run;               // projected head g goes with key part (g / part_run) % key_parts
  int out_heads, q_scale_rows;
  float eps;
};

struct QkvPrepParams : QkvPrepArgs {
  int tile;                   // tokens of a block
  int first_part;             // 0: grid.y covers q, then k / v; 1: k / v only
  int* status;
};

constexpr int PREP_THREADS = 512;

// N elements kept packed in registers
template <typename T, int N>
struct Packed {
  union {
    typename RawVec<N * (int)sizeof(T)>::type raw;
    uint32_t word[(N * sizeof(T) + 3) / 4];
  };
  __device__ __forceinline__ void load(const T* p) {
    raw = *reinterpret_cast<const typename RawVec<N * (int)sizeof(T)>::type*>(p);
  }
  __device__ __forceinline__ void zero() {
#pragma unroll
    for (int i = 0; i < (int)(N * sizeof(T) + 3) / 4; i++) word[i] = 0u;
  }
  __device__ __forceinline__ float get(int e) const {
    if constexpr (sizeof(T) == 4) return __uint_as_float(word[e]);
    return __uint_as_float((e & 1) ? word[e >> 1] & 0xffff0000u : word[e >> 1] << 16);
  }
  __device__ __forceinline__ void add(int e, T v) {          // into a zeroed place
    if constexpr (sizeof(T) == 4) word[e] = __float_as_uint(to_f(v));
    else word[e >> 1] |= (e & 1) ? __float_as_uint(to_f(v)) : __float_as_uint(to_f(v)) >> 16;
  }
};

// KR: taps held in registers (0: no convolution, 4: up to four taps, -1: any number, read again per token)
template <typename T, int VEC, int PER, int KR>
__global__ void __launch_bounds__(PREP_THREADS, KR == 0 && PER == 1 && VEC > 1 ? 2 : 1) qkv_prep_kernel(const QkvPrepParams p) {
  // tokens reduced together
  constexpr int GT = KR > 0 && PER == 1 ? 4 : KR == 0 && PER == 1 && VEC > 1 ? 2 : 1;
  __shared__ float red[2][GT][32];
  extern __shared__ float row[];                    // VEC == 1: the normalised row, for the rotary partner
  const int part = p.first_part + blockIdx.y;
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
  using Vec = Packed<T, VEC>;
  auto input = [&](int i, int c, Vec& v) {          // input of local token i, reaching back into the state
    if (i >= 0) v.load(x + (long)i * p.qkv_stride + c);
    else if (init && p.taps - 1 + i >= 0) v.load(st + (long)(p.taps - 1 + i) * C + c);
    else v.zero();
  };
  constexpr int KW = KR > 0 ? KR : 1;
  Vec wk[PER][KW], win[PER][KW], rows[GT][PER], nw[PER];
  int head[PER], dd[PER];                           // head and place in it of the thread's channels
  const T* norm_w = (const T*)(part == 0 ? p.q_norm : p.k_norm);
#pragma unroll
  for (int r = 0; r < PER; r++) {
    const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
    head[r] = dd[r] = 0;
    if (v >= nvec) continue;
    if (c < normed) {
      head[r] = c / p.dim;
      dd[r] = c - head[r] * p.dim;
      nw[r].load(norm_w + c);
    } else {
      head[r] = (c - normed) / p.vdim;
      dd[r] = c - normed - head[r] * p.vdim;
    }
    if constexpr (KR > 0) {
      const T* w = (const T*)p.conv_w + (long)(col0 + c) * p.taps;
      if (VEC > 1 && p.taps == KR) {                // KR * VEC weights in a row
        constexpr int WV = 16 / (int)sizeof(T);
        T wr[KR * VEC];
#pragma unroll
        for (int k = 0; k < KR * VEC; k += (VEC > 1 ? WV : 1)) load_raw<T, (VEC > 1 ? WV : 1)>(w + k, wr + k);
#pragma unroll
        for (int j = 0; j < KR; j++) wk[r][j].zero();
#pragma unroll
        for (int k = 0; k < KR * VEC; k++) wk[r][k % KR].add(k / KR, wr[k]);
      } else {
#pragma unroll
        for (int j = 0; j < KR; j++) {
          const int jj = j - (KR - p.taps);         // fewer taps: the oldest places weigh nothing
          wk[r][j].zero();
          if (jj >= 0)
#pragma unroll
            for (int e = 0; e < VEC; e++) wk[r][j].add(e, w[(long)e * p.taps + jj]);
        }
      }
#pragma unroll
      for (int j = 0; j < KR - 1; j++) {
        if (j >= KR - p.taps) input(i0 - (KR - 1) + j, c, win[r][j]);
        else win[r][j].zero();
      }
    }
    if (KR >= 0)
#pragma unroll
      for (int f = 0; f < GT; f++)
        if (i0 + f < i1) rows[f][r].load(x + (long)(i0 + f) * p.qkv_stride + c);
  }
  const int warps = (blockDim.x + 31) >> 5;
  const int half = p.rot >> 1;

  for (int ib = i0; ib < i1; ib += GT) {
    float u[GT][PER][VEC], ss[GT];
    long pos[GT], slot[GT];
#pragma unroll
    for (int f = 0; f < GT; f++) {
      const bool on = ib + f < i1;
      pos[f] = on && p.rot > 0 ? p.positions[t_seq + ib + f] : 0;
      slot[f] = on && part == 1 ? p.slot_mapping[t_seq + ib + f] : -1;
      ss[f] = 0.f;
      if (!on) continue;
#pragma unroll
      for (int r = 0; r < PER; r++) {
        const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
        if (v >= nvec) continue;
        if constexpr (KR > 0) {
          win[r][KR - 1] = rows[f][r];
#pragma unroll
          for (int e = 0; e < VEC; e++) {
            float a = 0.f;
#pragma unroll
            for (int j = 0; j < KR; j++) a = fmaf(wk[r][j].get(e), win[r][j].get(e), a);
            u[f][r][e] = a;
          }
#pragma unroll
          for (int j = 0; j + 1 < KR; j++) win[r][j] = win[r][j + 1];
        } else if constexpr (KR < 0) {
          const T* w = (const T*)p.conv_w + (long)(col0 + c) * p.taps;
#pragma unroll
          for (int e = 0; e < VEC; e++) u[f][r][e] = 0.f;
          for (int j = 0; j < p.taps; j++) {
            Vec in;
            input(ib + f - (p.taps - 1) + j, c, in);
#pragma unroll
            for (int e = 0; e < VEC; e++) u[f][r][e] = fmaf(to_f(w[(long)e * p.taps + j]), in.get(e), u[f][r][e]);
          }
        } else {
#pragma unroll
          for (int e = 0; e < VEC; e++) u[f][r][e] = rows[f][r].get(e);
        }
        if (KR >= 0 && ib + GT + f < i1) rows[f][r].load(x + (long)(ib + GT + f) * p.qkv_stride + c);
        if (c < normed)
#pragma unroll
          for (int e = 0; e < VEC; e++) ss[f] = fmaf(u[f][r][e], u[f][r][e], ss[f]);
      }
    }
    if (p.phase == 2) {
#pragma unroll
      for (int f = 0; f < GT; f++)
        if (ib + f < i1) ss[f] = p.sums[(t_seq + ib + f) * 2 + part];
    } else {
#pragma unroll
      for (int f = 0; f < GT; f++) ss[f] = warp_reduce_sum(ss[f]);
      if (warps > 1) {
        auto& rd = red[((ib - i0) / GT) & 1];       // two buffers: one barrier per group
        if ((threadIdx.x & 31) == 0)
#pragma unroll
          for (int f = 0; f < GT; f++) rd[f][threadIdx.x >> 5] = ss[f];
        __syncthreads();
#pragma unroll
        for (int f = 0; f < GT; f++) ss[f] = warp_reduce_sum((threadIdx.x & 31) < warps ? rd[f][threadIdx.x & 31] : 0.f);
      }
      if (p.phase == 1) {
        if (threadIdx.x == 0)
#pragma unroll
          for (int f = 0; f < GT; f++)
            if (ib + f < i1) p.sums[(t_seq + ib + f) * 2 + part] = ss[f];
        continue;
      }
    }
#pragma unroll
    for (int f = 0; f < GT; f++) {
      if (ib + f >= i1) break;
      const long t = t_seq + ib + f;
      const float inv = 1.f / sqrtf(ss[f] / (float)(part == 0 ? p.q_norm_dims : p.k_norm_dims) + p.eps);
      T *kdst = nullptr, *vdst = nullptr;
      if (slot[f] >= p.cache_slots) {
        if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
      } else if (slot[f] >= 0) {
        const unsigned blk = (unsigned)slot[f] / (unsigned)p.block_size, off = (unsigned)slot[f] - blk * p.block_size;
        kdst = (T*)p.k_cache + blk * p.k_block + off * p.k_tok;
        vdst = (T*)p.v_cache + blk * p.v_block + off * p.v_tok;
      }
      const float* cs = nullptr;
      if (p.rot > 0) {
        if (pos[f] >= 0 && pos[f] < p.cos_rows) cs = p.cos_sin + pos[f] * p.rot;
        else if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
      }
      if constexpr (VEC == 1) {
        if (cs) {
          __syncthreads();                          // the previous token's partners have been read
#pragma unroll
          for (int r = 0; r < PER; r++) {
            const int c = (int)threadIdx.x + r * (int)blockDim.x;
            if (c < normed) row[c] = u[f][r][0] * inv * nw[r].get(0);
          }
          __syncthreads();
        }
      }
#pragma unroll
      for (int r = 0; r < PER; r++) {
        const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
        if (v >= nvec) continue;
        const int d = dd[r];
        if (c >= normed) {                          // values
          if (vdst) store_vec<T, VEC>(vdst + head[r] * p.v_head + d, u[f][r]);
          continue;
        }
        if (part == 1 && p.values_from_keys && vdst) store_vec<T, VEC>(vdst + head[r] * p.v_head + d, u[f][r]);
        float y[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) y[e] = u[f][r][e] * inv * nw[r].get(e);
        if (cs && d < p.rot) {
          if constexpr (VEC == 1) {
            const int k = d >> 1;
            const float other = (d & 1) ? row[c - 1] : row[c + 1];
            y[0] = (d & 1) ? y[0] * cs[k] + other * cs[half + k] : y[0] * cs[k] - other * cs[half + k];
          } else {
            float cc[VEC / 2], sn[VEC / 2];
            if ((p.rot & (2 * VEC - 1)) == 0) {     // whole aligned vectors of the table
              load_vec<float, VEC / 2>(cs + (d >> 1), cc);
              load_vec<float, VEC / 2>(cs + half + (d >> 1), sn);
            } else {
#pragma unroll
              for (int e = 0; e < VEC / 2; e++) {
                const bool turned = d + 2 * e < p.rot;
                cc[e] = turned ? cs[(d >> 1) + e] : 1.f;
                sn[e] = turned ? cs[half + (d >> 1) + e] : 0.f;
              }
            }
#pragma unroll
            for (int e = 0; e < VEC; e += 2) {
              const float a = y[e], bb = y[e + 1];
              y[e] = a * cc[e / 2] - bb * sn[e / 2];
              y[e + 1] = bb * cc[e / 2] + a * sn[e / 2];
            }
          }
        }
        if (part == 0) store_vec<T, VEC>((T*)p.q_out + t * Nq + c, y);
        else if (kdst) store_vec<T, VEC>(kdst + head[r] * p.k_head + d, y);
      }
    }
  }
  // ---- the last taps - 1 inputs of the sequence (its first tile owns the state row)
  if (KR != 0 && p.taps > 1 && i0 == 0 && p.phase != 1) {
#pragma unroll
    for (int r = 0; r < PER; r++) {
      const int v = (int)threadIdx.x + r * (int)blockDim.x, c = v * VEC;
      if (v >= nvec) continue;
      for (int j = 0; j < p.taps - 1; j++) {
        Vec in;
        input(n - (p.taps - 1) + j, c, in);         // older rows move towards the front
        float f[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) f[e] = in.get(e);
        store_vec<T, VEC>(st + (long)j * C + c, f);
      }
    }
  }
}

// a head [dim] (or value row [vdim]) of one token per LANES lanes
template <typename T, int VEC, int LANES>
__global__ void __launch_bounds__(256) qkv_head_kernel(const QkvPrepParams p) {
  const int units = p.heads + p.kv_heads * (p.values_from_keys ? 1 : 2);
  const long i = ((long)blockIdx.x * 256 + threadIdx.x) / LANES;
  const bool on = i < p.tokens * units;              // lanes beyond the end only take part in the shuffles
  const int lane = threadIdx.x & (LANES - 1);
  const long t = on ? i / units : 0;
  const int u = on ? (int)(i - t * units) : 0;
  const int kind = u < p.heads ? 0 : u < p.heads + p.kv_heads ? 1 : 2;                      // q, k, v
  const int g = kind == 0 ? u : kind == 1 ? u - p.heads : u - p.heads - p.kv_heads;
  const int dim = kind == 2 ? p.vdim : p.dim;
  const T* x = (const T*)p.qkv + t * p.qkv_stride;
  x += kind == 0 ? (long)g * p.dim : kind == 1 ? (long)(p.heads + g) * p.dim : (long)(p.heads + p.kv_heads) * p.dim + (long)g * p.vdim;
  float first[VEC], ss = 0.f;                        // the first chunk stays in registers
#pragma unroll
  for (int e = 0; e < VEC; e++) first[e] = 0.f;
  for (int b = 0; b < dim; b += LANES * VEC) {
    const int c = b + lane * VEC;
    float v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) v[e] = 0.f;
    if (c < dim) load_vec<T, VEC>(x + c, v);
#pragma unroll
    for (int e = 0; e < VEC; e++) {
      ss = fmaf(v[e], v[e], ss);
      if (b == 0) first[e] = v[e];
    }
  }
#pragma unroll
  for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = kind == 2 ? 1.f : 1.f / sqrtf(ss / (float)dim + p.eps);
  const T* w = (const T*)(kind == 0 ? p.q_norm : p.k_norm);
  T *dst = nullptr, *raw = nullptr;
  if (kind == 0) dst = (T*)p.q_out + (t * p.heads + g) * (long)p.dim;
  else {
    const long slot = p.slot_mapping[t];
    if (slot >= p.cache_slots) {
      if (lane == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    } else if (slot >= 0) {
      const unsigned blk = (unsigned)slot / (unsigned)p.block_size, off = (unsigned)slot - blk * p.block_size;
      T* vrow = (T*)p.v_cache + blk * p.v_block + off * p.v_tok + g * p.v_head;
      dst = kind == 1 ? (T*)p.k_cache + blk * p.k_block + off * p.k_tok + g * p.k_head : vrow;
      if (kind == 1 && p.values_from_keys) raw = vrow;
    }
  }
  const float* cs = nullptr;
  if (p.rot > 0 && kind < 2) {
    const long pos = p.positions[t];
    if (pos >= 0 && pos < p.cos_rows) cs = p.cos_sin + pos * p.rot;
    else if (lane == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
  }
  const int half = p.rot >> 1;
  for (int b = 0; b < dim; b += LANES * VEC) {       // same trip count for all lanes of a group
    const int c = b + lane * VEC;
    float v[VEC];
#pragma unroll
    for (int e = 0; e < VEC; e++) v[e] = first[e];
    if (b > 0 && c < dim) load_vec<T, VEC>(x + c, v);
    if (on && raw && c < dim) store_vec<T, VEC>(raw + c, v);
    if (kind < 2 && c < dim) {
      float wv[VEC];
      load_vec<T, VEC>(w + c, wv);
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] *= inv * wv[e];
    }
    if constexpr (VEC == 1) {
      if (p.rot > 0) {                               // the partner of a pair sits in the next lane
        const float other = __shfl_xor_sync(0xffffffffu, v[0], 1);
        if (cs && c < p.rot) {
          const float cc = cs[c >> 1], sn = cs[half + (c >> 1)];
          v[0] = (c & 1) ? v[0] * cc + other * sn : v[0] * cc - other * sn;
        }
      }
    } else if (cs) {
#pragma unroll
      for (int e = 0; e < VEC; e += 2)
        if (c + e < p.rot) {
          const float cc = cs[(c + e) >> 1], sn = cs[half + ((c + e) >> 1)], a = v[e], bb = v[e + 1];
          v[e] = a * cc - bb * sn;
          v[e + 1] = bb * cc + a * sn;
        }
    }
    if (on && dst && c < dim) store_vec<T, VEC>(dst + c, v);
  }
}

template <typename T, int VEC, int LANES>
static int launch_heads(const QkvPrepParams& p, cudaStream_t stream) {
  const long lanes = p.tokens * (p.heads + p.kv_heads * (p.values_from_keys ? 1 : 2)) * LANES;
  qkv_head_kernel<T, VEC, LANES><<<(unsigned)((lanes + 255) / 256), 256, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

// VEC floats of shared memory, 16 bytes at a time
template <int VEC>
__device__ __forceinline__ void smem_get(const float* p, float* v) {
  if constexpr (VEC % 4 == 0)
#pragma unroll
    for (int e = 0; e < VEC; e += 4) load_vec<float, 4>(p + e, v + e);
  else
#pragma unroll
    for (int e = 0; e < VEC; e++) v[e] = p[e];
}
template <int VEC>
__device__ __forceinline__ void smem_put(float* p, const float* v) {
  if constexpr (VEC % 4 == 0)
#pragma unroll
    for (int e = 0; e < VEC; e += 4) store_vec<float, 4>(p + e, v + e);
  else
#pragma unroll
    for (int e = 0; e < VEC; e++) p[e] = v[e];
}

// One block per token.  LANES threads take a head: norm (optional), rotary, factor; keys and values go to their cache
// slots, queries stay in shared memory (fp32) until the wide queries are formed from them: a thread then owns VEC
// dimensions of one key part, keeps what the first CNT projected heads of that part have there, and walks the output heads.
template <typename T, int VEC, int LANES>
__global__ void __launch_bounds__(256) qkv_spread_kernel(const QkvPrepParams p) {
  constexpr int CNT = 4;
  extern __shared__ __align__(16) float sq[];        // [heads, dim], then [out_heads, heads] weights
  float* sm = sq + (p.heads * p.dim + 3) / 4 * 4;
  const long t = blockIdx.x;
  const int lane = threadIdx.x % LANES;
  const int units = p.heads + p.kv_heads + p.v_heads, half = p.rot >> 1;
  const T* x = (const T*)p.qkv + t * p.qkv_stride;
  const long slot = p.slot_mapping[t];
  const bool stored = slot >= 0 && slot < p.cache_slots;
  const unsigned blk = stored ? (unsigned)slot / (unsigned)p.block_size : 0;
  const unsigned off = stored ? (unsigned)slot - blk * p.block_size : 0;
  const long pos = p.rot > 0 || p.q_scale ? p.positions[t] : 0;
  const bool cs_ok = pos >= 0 && pos < p.cos_rows, qs_ok = pos >= 0 && pos < p.q_scale_rows;
  if (threadIdx.x == 0 && p.status &&
      (slot >= p.cache_slots || (p.rot > 0 && !cs_ok) || (p.q_scale && !qs_ok)))
    atomicExch(p.status, B200_BAD_INDEX);
  const float* cs = p.rot > 0 && cs_ok ? p.cos_sin + pos * p.rot : nullptr;
  const float factor = p.q_scale && qs_ok ? p.q_scale[pos] : 1.f;
  if (p.mix)
    for (int i = threadIdx.x; i < p.out_heads * p.heads; i += 256) sm[i] = p.mix[i];
  for (int u0 = 0; u0 < units; u0 += 256 / LANES) {  // same trip count for all threads
    const int u = u0 + (int)threadIdx.x / LANES;
    const bool on = u < units;
    const int kind = !on || u < p.heads ? 0 : u < p.heads + p.kv_heads ? 1 : 2;             // q, k, v
    const int g = kind == 0 ? u : kind == 1 ? u - p.heads : u - p.heads - p.kv_heads;
    const int dim = !on ? 0 : kind == 2 ? p.vdim : p.dim;
    const T* src = x + (kind == 2 ? (long)(p.heads + p.kv_heads) * p.dim + (long)g * p.vdim : (long)u * p.dim);
    float first[VEC];                                // the first vector stays in registers
#pragma unroll
    for (int e = 0; e < VEC; e++) first[e] = 0.f;
    if (lane * VEC < dim) load_vec<T, VEC>(src + lane * VEC, first);
    float inv = 1.f;
    if (p.head_norm) {
      float ss = 0.f;
#pragma unroll
      for (int e = 0; e < VEC; e++) ss = fmaf(first[e], first[e], ss);
      for (int c = (LANES + lane) * VEC; c < dim; c += LANES * VEC) {
        float v[VEC];
        load_vec<T, VEC>(src + c, v);
#pragma unroll
        for (int e = 0; e < VEC; e++) ss = fmaf(v[e], v[e], ss);
      }
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      inv = 1.f / sqrtf(ss / (float)max(dim, 1) + p.eps);
    }
    const T* w = p.head_norm ? (const T*)(kind == 0 ? p.q_norm : p.k_norm) : nullptr;
    T* dst = nullptr;
    if (on && kind == 1 && stored)
      dst = (T*)p.k_cache + blk * p.k_block + off * p.k_tok + g / p.key_parts * p.k_head + (long)(g % p.key_parts) * p.dim;
    else if (on && kind == 2 && stored)
      dst = (T*)p.v_cache + blk * p.v_block + off * p.v_tok + g * p.v_head;
    const int longest = p.dim > p.vdim ? p.dim : p.vdim;
    for (int b = 0; b < longest; b += LANES * VEC) { // same trip count for all lanes
      const int c = b + lane * VEC;
      float v[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] = first[e];
      if (b > 0) {
#pragma unroll
        for (int e = 0; e < VEC; e++) v[e] = 0.f;
        if (c < dim) load_vec<T, VEC>(src + c, v);
      }
      if (w && kind < 2 && c < dim) {
        float wv[VEC];
        load_vec<T, VEC>(w + c, wv);
#pragma unroll
        for (int e = 0; e < VEC; e++) v[e] *= inv * wv[e];
      }
      if constexpr (VEC == 1) {
        if (p.rot > 0) {                             // the partner of a pair sits in the next lane
          const float other = __shfl_xor_sync(0xffffffffu, v[0], 1);
          if (cs && kind < 2 && c < p.rot) {
            const float cc = cs[c >> 1], sn = cs[half + (c >> 1)];
            v[0] = (c & 1) ? v[0] * cc + other * sn : v[0] * cc - other * sn;
          }
        }
      } else if (cs && kind < 2) {
#pragma unroll
        for (int e = 0; e < VEC; e += 2)
          if (c + e < p.rot) {
            const float cc = cs[(c + e) >> 1], sn = cs[half + ((c + e) >> 1)], a = v[e], bb = v[e + 1];
            v[e] = a * cc - bb * sn;
            v[e + 1] = bb * cc + a * sn;
          }
      }
      if (c >= dim) continue;
      if (kind == 0) {
#pragma unroll
        for (int e = 0; e < VEC; e++) v[e] *= factor;
        smem_put<VEC>(sq + (long)g * p.dim + c, v);
      } else if (dst) {
        store_vec<T, VEC>(dst + c, v);
      }
    }
  }
  __syncthreads();
  const int per = p.dim / VEC, row = p.key_parts * per, stride = p.part_run * p.key_parts;
  const int teams = row < 256 ? 256 / row : 1;
  const int team = row < 256 ? (int)threadIdx.x / row : 0;
  if (team >= teams) return;
  T* q = (T*)p.q_out + t * p.out_heads * (long)p.key_parts * p.dim;
  for (int r = (int)threadIdx.x - team * row; r < row; r += 256) {
    const int c = r / per, d = (r - c * per) * VEC;
    if (!p.mix) {
      int left = team % stride;                      // (output head) mod (heads of a round of parts)
      for (int oh = team; oh < p.out_heads; oh += teams) {
        float acc[VEC];
        const bool mine = left >= c * p.part_run && left < (c + 1) * p.part_run;
#pragma unroll
        for (int e = 0; e < VEC; e++) acc[e] = 0.f;
        if (mine) smem_get<VEC>(sq + (long)oh * p.dim + d, acc);
        store_vec<T, VEC>(q + ((long)oh * row + r) * VEC, acc);
        left += teams;
        while (left >= stride) left -= stride;
      }
      continue;
    }
    const int g0 = c * p.part_run, n = p.part_run < CNT ? p.part_run : CNT;
    float kept[CNT][VEC];
#pragma unroll
    for (int j = 0; j < CNT; j++) {
#pragma unroll
      for (int e = 0; e < VEC; e++) kept[j][e] = 0.f;
      if (j < n && g0 + j < p.heads) smem_get<VEC>(sq + (long)(g0 + j) * p.dim + d, kept[j]);
    }
    for (int oh = team; oh < p.out_heads; oh += teams) {
      const float* m = sm + oh * p.heads;
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) acc[e] = 0.f;
#pragma unroll
      for (int j = 0; j < CNT; j++) {
        const float f = j < n && g0 + j < p.heads ? m[g0 + j] : 0.f;
#pragma unroll
        for (int e = 0; e < VEC; e++) acc[e] = fmaf(f, kept[j][e], acc[e]);
      }
      for (int s0 = g0; s0 < p.heads; s0 += stride)  // what does not fit
        for (int g = s0 + (s0 == g0 ? n : 0); g < min(s0 + p.part_run, p.heads); g++) {
          float v[VEC];
          smem_get<VEC>(sq + (long)g * p.dim + d, v);
#pragma unroll
          for (int e = 0; e < VEC; e++) acc[e] = fmaf(m[g], v[e], acc[e]);
        }
      store_vec<T, VEC>(q + ((long)oh * row + r) * VEC, acc);
    }
  }
}

template <typename T, int VEC, int LANES>
static int launch_spread(const QkvPrepParams& p, cudaStream_t stream) {
  const size_t smem = ((size_t)(p.heads * p.dim + 3) / 4 * 4 + (p.mix ? (size_t)p.out_heads * p.heads : 0)) * sizeof(float);
  if (smem > 200 * 1024) return 9822;
  static bool attr_set = false;
  if (smem > 48 * 1024 && !attr_set) {
    const cudaError_t e = cudaFuncSetAttribute(qkv_spread_kernel<T, VEC, LANES>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               200 * 1024);
    if (e != cudaSuccess) return (int)e;
    attr_set = true;
  }
  if (p.tokens > 0x7fffffffL) return 9823;
  qkv_spread_kernel<T, VEC, LANES><<<(unsigned)p.tokens, 256, smem, stream>>>(p);
  return B200_CHECK_LAUNCH();
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
static int launch_parts(const QkvPrepParams& p, unsigned tiles, unsigned parts, int width, bool vec, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const int nvec = width / (vec ? V : 1);
  int per = (nvec + PREP_THREADS - 1) / PREP_THREADS;
  per = vec ? (per <= 1 ? 1 : per <= 2 ? 2 : 4) : (per <= 2 ? 2 : 16);
  if ((long)per * PREP_THREADS < nvec) return 9821;
  const int threads = ((nvec + per - 1) / per + 31) / 32 * 32;
  const dim3 grid(tiles, parts);
  if (vec) {
    if (per == 1) return launch_prep<T, V, 1>(p, grid, threads, 0, stream);
    if (per == 2) return launch_prep<T, V, 2>(p, grid, threads, 0, stream);
    return launch_prep<T, V, 4>(p, grid, threads, 0, stream);
  }
  const size_t smem = p.rot > 0 ? (size_t)width * 4 : 0;
  if (per == 2) return launch_prep<T, 1, 2>(p, grid, threads, smem, stream);
  return launch_prep<T, 1, 16>(p, grid, threads, smem, stream);
}

template <typename T>
static int prep_t(QkvPrepParams& p, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const int Nq = p.heads * p.dim, Nkv = p.kv_heads * (p.dim + (p.values_from_keys ? 0 : p.vdim));
  const long s[] = {p.qkv_stride, p.k_block, p.k_tok, p.k_head, p.v_block, p.v_tok, p.v_head, p.dim, p.vdim};
  bool vec = aligned16(p.cos_sin) && aligned16(p.qkv) && aligned16(p.conv_w) && aligned16(p.state) &&
             aligned16(p.q_norm) && aligned16(p.k_norm) && aligned16(p.q_out) && aligned16(p.k_cache) &&
             aligned16(p.v_cache);
  if (p.key_parts > 0) {
    for (long x : s) vec = vec && x % V == 0;
    if (!vec) return launch_spread<T, 1, 32>(p, stream);
    return p.dim / V <= 8 ? launch_spread<T, V, 8>(p, stream)
                          : p.dim / V <= 16 ? launch_spread<T, V, 16>(p, stream) : launch_spread<T, V, 32>(p, stream);
  }
  for (long x : s) vec = vec && x % V == 0;
  if (p.head_norm) {
    if (!vec) return launch_heads<T, 1, 32>(p, stream);
    const int need = (p.dim > p.vdim ? p.dim : p.vdim) / V;
    return need <= 8 ? launch_heads<T, V, 8>(p, stream)
                     : need <= 16 ? launch_heads<T, V, 16>(p, stream) : launch_heads<T, V, 32>(p, stream);
  }
  // tokens of a block: enough to share the convolution's history and weights, few enough to fill the GPU
  p.tile = p.tokens >= 8192 ? 16 : p.tokens >= 2048 ? 8 : p.tokens >= 512 ? 2 : 1;
  if (p.taps > 0 && p.tile < 4) p.tile = 4;
  if (p.tile < p.taps - 1) p.tile = p.taps - 1;     // only a first tile reaches back into the state
  const long tiles = p.taps == 0 ? (p.tokens + p.tile - 1) / p.tile
                                 : p.uniform ? p.num_seqs : p.tokens / p.tile + p.num_seqs;
  p.first_part = 0;
  // long steps: blocks of their own size for the narrower part
  if (p.tokens >= 2048 && 2 * Nkv <= Nq) {
    const int rc = launch_parts<T>(p, (unsigned)tiles, 1, Nq, vec, stream);
    if (rc) return rc;
    p.first_part = 1;
    return launch_parts<T>(p, (unsigned)tiles, 1, Nkv, vec, stream);
  }
  return launch_parts<T>(p, (unsigned)tiles, 2, Nq > Nkv ? Nq : Nkv, vec, stream);
}

}  // namespace b200

using namespace b200;

B200_API int b200_qkv_prep(const QkvPrepArgs* a, int* status, cudaStream_t stream) {
  if (a->tokens <= 0) return 0;
  if (a->heads < 1 || a->kv_heads < 1 || a->dim < 1 || a->vdim < 1 || a->block_size < 1 || a->num_seqs < 1) return 9800;
  if (a->cache_slots > 0xffffffffL) return 9807;
  if (a->rot < 0 || a->rot > a->dim || (a->rot & 1) || (a->rot > 0 && !a->cos_sin)) return 9801;
  if (a->values_from_keys && a->vdim != a->dim) return 9802;
  if (a->taps < 0 || (a->taps > 0 && !a->conv_w)) return 9803;
  if (a->taps > 1 && (!a->state || !a->slots || !a->has_init || !a->cu)) return 9804;
  if (a->phase != 0 && !a->sums) return 9805;
  if (a->taps == 1 && !a->cu) return 9806;
  if (a->head_norm && (a->taps || a->phase)) return 9808;
  if (a->key_parts > 0) {
    if (a->taps || a->phase || a->values_from_keys || a->v_heads < 1 || a->kv_heads % a->key_parts || a->part_run < 1 ||
        a->out_heads < 1 || (!a->mix && a->out_heads != a->heads) || (a->head_norm && (!a->q_norm || !a->k_norm)))
      return 9809;
  } else if (!a->q_norm || !a->k_norm) {
    return 9810;
  }
  QkvPrepParams p;
  static_cast<QkvPrepArgs&>(p) = *a;
  p.status = status;
  return a->dtype ? prep_t<float>(p, stream) : prep_t<__nv_bfloat16>(p, stream);
}
