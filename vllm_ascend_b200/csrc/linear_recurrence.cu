// Linear recurrences without a correction term, S <- d S + k u^T, o = S^T q, for prefill portions and single-token
// decode, with the state of a head (DK x DV, fp32) read and written once per step:
//   LOG_DECAY    d = exp(g) per token and head, u = v                       (gated linear attention, lightning)
//   STATE_SPACE  d = exp(-exp(A_log) dt), u = dt v, o += D v with dt = clamp(softplus(dt + dt_bias))       (Mamba-2)
//   FORGET       d = f, k = 1 - f per key channel, f = l + (1 - l) sigmoid(f + b), q = silu(q)               (HGRN2)
// In the last form the update is S <- S + (1 - f)(v - S) with 1 - f = (1 - l) sigmoid(-(f + b)), which loses nothing
// where f is close to one.  All of it is fp32; element type of the rows bf16 or fp32 (template), all sizes are run-time
// values.  Counterparts of the reference's Triton kernels (vllm_ascend/ops/triton/mamba/lightning_attn.py,
// vllm_ascend/ops/triton/fla/*).
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

enum : int { REC_LOG_DECAY = 0, REC_STATE_SPACE = 1, REC_FORGET = 2 };

struct RecurrenceArgs {
  const void *q, *k, *v;          // [T, key_heads, dk], [T, heads, dv]: heads dense, token strides given
  const void* f;                  // FORGET: [T, heads * dk] raw gate
  const float* log_decay;         // LOG_DECAY: [T, heads]
  const void* dt;                 // STATE_SPACE: [T, heads] raw step sizes
  const float *dt_bias, *A_log, *D;
  const void *f_bias, *lower;     // FORGET: [heads * dk]
  float* state;                   // [num_slots, heads, dk, dv]
  const int *cu, *slots, *has_init;
  const void* norm_w;             // decode: RMS norm of every head's read-out, [dv]; null: none
  void* out;                      // [T, heads, dv]
  long q_stride, k_stride, v_stride, f_stride, dt_stride, out_stride, num_slots;
  int mode, num_seqs, key_heads, heads, dk, dv, dtype, uniform;
  float dt_lo, dt_hi, eps, out_scale;
};

struct RecParams : RecurrenceArgs {
  int* status;
};

__device__ __forceinline__ float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_f(float x) { return x > 30.f ? x : log1pf(expf(x)); }

// step size of a token and its decay
template <typename T>
__device__ __forceinline__ float2 step_of(const RecParams& p, long t, int h) {
  float dt = softplus_f(to_f(((const T*)p.dt)[t * p.dt_stride + h]) + p.dt_bias[h]);
  dt = fminf(fmaxf(dt, p.dt_lo), p.dt_hi);
  return make_float2(dt, expf(-expf(p.A_log[h]) * dt));
}

// ---------------------------------------------------------------- prefill
// Eight lanes share a column of S, each holding R of its DK rows (row i of a lane: 32 (i / 4) + 4 lane + i % 4, so
// that a staged row is read without bank conflicts); a thread covers CJ adjacent columns, a warp 4 CJ, a block 16 CJ.
// Rows are kept in pairs for the packed fp32 arithmetic.  Inputs are staged in chunks of REC_CHUNK tokens, the next
// chunk's raw elements in flight while one is processed.  The read-outs of eight tokens are reduced together over the
// eight lanes: lane i ends up with token i's.  A token beyond the sequence is staged so that it leaves S as it is.
constexpr int REC_CHUNK = 16;

template <typename T, int MODE, int R, int CJ, bool VEC>
__global__ void __launch_bounds__(128) recurrence_kernel(const RecParams p) {
  constexpr int DKP = 8 * R;                    // rows, padded with zeros
  constexpr int COLS = 16 * CJ;
  constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
  constexpr int PER = DKP / 8;                  // elements of a k (q) row per staging thread
  __shared__ __align__(16) float ks[REC_CHUNK][DKP], qs[REC_CHUNK][DKP], vs[REC_CHUNK][COLS];
  __shared__ float2 sc[REC_CHUNK];              // decay, factor of v
  const int b = blockIdx.x, h = blockIdx.y;
  const int hk = h / (p.heads / p.key_heads);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gl = lane & 7;                                           // row group of the lane
  const int jb = (int)blockIdx.z * COLS, jl = (warp * 4 + (lane >> 3)) * CJ, j0 = jb + jl;
  const int slot = p.slots[b];
  const int t0 = p.cu[b], t1 = p.cu[b + 1];
  const bool init = p.has_init[b] != 0;
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    return;
  }
  if (t0 >= t1) return;
  const int DK = p.dk, DV = p.dv;
  float* sp = p.state + ((long)slot * p.heads + h) * DK * DV;
  auto row_of = [&](int r) { return (r >> 2) * 32 + gl * 4 + (r & 3); };
  f32x2 S[R / 2][CJ];
  float even[CJ];
#pragma unroll
  for (int r = 0; r < R; r++) {
    float row[CJ];
#pragma unroll
    for (int c = 0; c < CJ; c++) row[c] = 0.f;
    if (init && row_of(r) < DK) {
      const float* src = sp + (long)row_of(r) * DV + j0;
      if (VEC) { if (j0 < DV) load_vec<float, CJ>(src, row); }
      else
#pragma unroll
        for (int c = 0; c < CJ; c++) if (j0 + c < DV) row[c] = src[c];
    }
#pragma unroll
    for (int c = 0; c < CJ; c++) {
      if (r & 1) S[r / 2][c] = pack2(even[c], row[c]);
      else even[c] = row[c];
    }
  }
  // staging role: token st of the chunk, part s8 of its rows (V elements at a time, interleaved)
  const int st = threadIdx.x >> 3, s8 = threadIdx.x & 7;
  const T* kp = MODE == REC_FORGET ? (const T*)p.f + (long)h * DK : (const T*)p.k + (long)hk * DK;
  const long k_stride = MODE == REC_FORGET ? p.f_stride : p.k_stride;
  const T* qp = (const T*)p.q + (long)hk * DK;
  const T* vp = (const T*)p.v + (long)h * DV + jb;
  constexpr int VC = VEC ? CJ : 1;              // elements per v access
  constexpr int VPER = COLS / 8;
  T rk[PER], rq[PER], rv[VPER];
  bool here = false;                            // the staged token exists
  auto fetch = [&](int t) {                     // raw elements of token t + st
    t += st;
    here = t < t1;
#pragma unroll
    for (int i = 0; i < PER; i += V) {
      const int e = (i / V * 8 + s8) * V;
      if (here && e < DK) {
        load_raw<T, V>(kp + (long)t * k_stride + e, rk + i);
        load_raw<T, V>(qp + (long)t * p.q_stride + e, rq + i);
      } else {
#pragma unroll
        for (int x = 0; x < V; x++) rk[i + x] = rq[i + x] = from_f<T>(0.f);
      }
    }
#pragma unroll
    for (int i = 0; i < VPER; i += VC) {
      const int e = (i / VC * 8 + s8) * VC;
      if (here && jb + e < DV) load_raw<T, VC>(vp + (long)t * p.v_stride + e, rv + i);
      else
#pragma unroll
        for (int x = 0; x < VC; x++) rv[i + x] = from_f<T>(0.f);
    }
  };
  auto stage = [&](int t) {
    t += st;
    if (s8 == 0) {
      float2 s = make_float2(1.f, 1.f);
      if (MODE == REC_STATE_SPACE) {
        s = make_float2(1.f, 0.f);
        if (here) {
          const float2 d = step_of<T>(p, t, h);
          s = make_float2(d.y, d.x);
        }
      } else if (MODE == REC_LOG_DECAY) {
        if (here) s.x = expf(p.log_decay[(long)t * p.heads + h]);
      }
      sc[st] = s;
    }
#pragma unroll
    for (int i = 0; i < PER; i += V)
#pragma unroll
      for (int x = 0; x < V; x++) {
        const int e = (i / V * 8 + s8) * V + x;
        float k = to_f(rk[i + x]), q = to_f(rq[i + x]);
        if (MODE == REC_FORGET) {
          float keep = 0.f, bias = 0.f;         // 1 - l
          if (here && e < DK) {
            keep = 1.f - to_f(((const T*)p.lower)[(long)h * DK + e]);
            bias = to_f(((const T*)p.f_bias)[(long)h * DK + e]);
          }
          k = keep * sigmoid_exact(-(k + bias));
          q = q * sigmoid_exact(q);
        }
        ks[st][e] = k;
        qs[st][e] = q;
      }
#pragma unroll
    for (int i = 0; i < VPER; i += VC)
#pragma unroll
      for (int x = 0; x < VC; x++) vs[st][(i / VC * 8 + s8) * VC + x] = to_f(rv[i + x]);
  };
  const float skip = MODE == REC_STATE_SPACE ? p.D[h] : 0.f;
  T* op = (T*)p.out + (long)h * DV + j0;
  fetch(t0);
  for (int tc = t0; tc < t1; tc += REC_CHUNK) {
    if (tc > t0) __syncthreads();               // the previous chunk has been read
    stage(tc);
    __syncthreads();
    if (tc + REC_CHUNK < t1) fetch(tc + REC_CHUNK);
    const int n = min(REC_CHUNK, t1 - tc);
    for (int ib = 0; ib < n; ib += 8) {
      float o[8][CJ];
#pragma unroll
      for (int i8 = 0; i8 < 8; i8++) {
        const int i = ib + i8;
        const float2 s2 = sc[i];
        float vt[CJ];
        load_vec<float, CJ>(&vs[i][jl], vt);
        const f32x2 dd = pack2(s2.x, s2.x);
        f32x2 uu[CJ], acc[CJ];
#pragma unroll
        for (int c = 0; c < CJ; c++) {
          const float u = MODE == REC_STATE_SPACE ? vt[c] * s2.y : vt[c];
          uu[c] = pack2(u, u);
          acc[c] = 0;
        }
#pragma unroll
        for (int r = 0; r < R; r += 4) {
          const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(&ks[i][r * 8 + gl * 4]);
          const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(&qs[i][r * 8 + gl * 4]);
#pragma unroll
          for (int c = 0; c < CJ; c++) {
            if (MODE == REC_FORGET) {
              const f32x2 m = pack2(-1.f, -1.f);
              S[r / 2][c] = fma2(k4.x, fma2(S[r / 2][c], m, uu[c]), S[r / 2][c]);
              S[r / 2 + 1][c] = fma2(k4.y, fma2(S[r / 2 + 1][c], m, uu[c]), S[r / 2 + 1][c]);
            } else {
              S[r / 2][c] = fma2(k4.x, uu[c], mul2(S[r / 2][c], dd));
              S[r / 2 + 1][c] = fma2(k4.y, uu[c], mul2(S[r / 2 + 1][c], dd));
            }
            acc[c] = fma2(S[r / 2][c], q4.x, acc[c]);
            acc[c] = fma2(S[r / 2 + 1][c], q4.y, acc[c]);
          }
        }
#pragma unroll
        for (int c = 0; c < CJ; c++) {
          const float2 a = unpack2(acc[c]);
          o[i8][c] = a.x + a.y;
        }
      }
      // lane gl keeps token gl: halve the tokens and double the lanes summed, three times
#pragma unroll
      for (int m = 4; m > 0; m >>= 1) {
        const bool up = gl & m;
#pragma unroll
        for (int i = 0; i < m; i++)
#pragma unroll
          for (int c = 0; c < CJ; c++) {
            const float give = up ? o[i][c] : o[i + m][c];
            o[i][c] = (up ? o[i + m][c] : o[i][c]) + __shfl_xor_sync(0xffffffffu, give, m);
          }
      }
      const int i = ib + gl;
      if (i < n) {
        float res[CJ];
#pragma unroll
        for (int c = 0; c < CJ; c++) res[c] = (MODE == REC_STATE_SPACE ? fmaf(skip, vs[i][jl + c], o[0][c]) : o[0][c]) * p.out_scale;
        T* dst = op + (long)(tc + i) * p.out_stride;
        if (VEC) { if (j0 < DV) store_vec<T, CJ>(dst, res); }
        else
#pragma unroll
          for (int c = 0; c < CJ; c++) if (j0 + c < DV) dst[c] = from_f<T>(res[c]);
      }
    }
  }
#pragma unroll
  for (int r = 0; r < R; r++) {
    if (row_of(r) >= DK) continue;
    float* dst = sp + (long)row_of(r) * DV + j0;
    float row[CJ];
#pragma unroll
    for (int c = 0; c < CJ; c++) {
      const float2 pr = unpack2(S[r / 2][c]);
      row[c] = r & 1 ? pr.y : pr.x;
    }
    if (VEC) { if (j0 < DV) store_vec<float, CJ>(dst, row); }
    else
#pragma unroll
      for (int c = 0; c < CJ; c++) if (j0 + c < DV) dst[c] = row[c];
  }
}

// ---------------------------------------------------------------- decode
// One token per sequence: a block per (sequence, head) streams the head's state once through registers.  Four adjacent
// columns per thread, the threads of a row group cover a row of S, the row groups take every RG-th row (M rows each).
template <typename T, int MODE, int M>
__global__ void __launch_bounds__(256, M > 8 ? 2 : 3) recurrence_decode_kernel(const RecParams p) {
  extern __shared__ float sm[];
  const int DK = p.dk, DV = p.dv, cols = DV >> 2, RG = 256 / cols;
  float* ks = sm;                       // [DK], 1 - f in the FORGET form
  float* qs = ks + DK;                  // [DK]
  float* part = qs + DK;                // [RG][DV]
  __shared__ float red[8];
  const int b = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int hk = h / (p.heads / p.key_heads);
  const int slot = p.slots[b], t = p.cu[b];
  const bool init = p.has_init[b] != 0;
  if (slot < 0 || slot >= p.num_slots) {
    if (tid == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    return;
  }
  const int rg = tid / cols, c4 = (tid - rg * cols) * 4;
  const bool on = rg < RG;
  float* sp = p.state + ((long)slot * p.heads + h) * DK * DV + c4;
  float4 S[M];
#pragma unroll
  for (int m = 0; m < M; m++) {
    const int i = rg + m * RG;
    S[m] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on && init && i < DK) S[m] = *reinterpret_cast<const float4*>(sp + (long)i * DV);
  }
  for (int i = tid; i < DK; i += 256) {
    float q = to_f(((const T*)p.q)[(long)t * p.q_stride + (long)hk * DK + i]), k;
    if (MODE == REC_FORGET) {
      const long c = (long)h * DK + i;
      k = (1.f - to_f(((const T*)p.lower)[c])) *
          sigmoid_exact(-(to_f(((const T*)p.f)[(long)t * p.f_stride + c]) + to_f(((const T*)p.f_bias)[c])));
      q = q * sigmoid_exact(q);
    } else {
      k = to_f(((const T*)p.k)[(long)t * p.k_stride + (long)hk * DK + i]);
    }
    ks[i] = k;
    qs[i] = q;
  }
  float d = 1.f, gain = 1.f;
  if (MODE == REC_STATE_SPACE) {
    const float2 s = step_of<T>(p, t, h);
    gain = s.x;
    d = s.y;
  } else if (MODE == REC_LOG_DECAY) {
    d = expf(p.log_decay[(long)t * p.heads + h]);
  }
  float v[4] = {0.f, 0.f, 0.f, 0.f}, a[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) load_vec<T, 4>((const T*)p.v + (long)t * p.v_stride + (long)h * DV + c4, v);
  __syncthreads();
  if (on) {
    const float u[4] = {v[0] * gain, v[1] * gain, v[2] * gain, v[3] * gain};
#pragma unroll
    for (int m = 0; m < M; m++) {
      const int i = rg + m * RG;
      if (i < DK) {
        const float k = ks[i], q = qs[i];
        float4 s = S[m];
        if (MODE == REC_FORGET) {
          s.x = fmaf(k, u[0] - s.x, s.x); s.y = fmaf(k, u[1] - s.y, s.y);
          s.z = fmaf(k, u[2] - s.z, s.z); s.w = fmaf(k, u[3] - s.w, s.w);
        } else {
          s.x = fmaf(k, u[0], d * s.x); s.y = fmaf(k, u[1], d * s.y);
          s.z = fmaf(k, u[2], d * s.z); s.w = fmaf(k, u[3], d * s.w);
        }
        a[0] = fmaf(s.x, q, a[0]); a[1] = fmaf(s.y, q, a[1]);
        a[2] = fmaf(s.z, q, a[2]); a[3] = fmaf(s.w, q, a[3]);
        *reinterpret_cast<float4*>(sp + (long)i * DV) = s;
      }
    }
    store_vec<float, 4>(part + rg * DV + c4, a);
  }
  __syncthreads();
  float o[4] = {0.f, 0.f, 0.f, 0.f};
  if (rg == 0) {
    for (int w = 0; w < RG; w++) {
      float pa[4];
      load_vec<float, 4>(part + w * DV + c4, pa);
#pragma unroll
      for (int e = 0; e < 4; e++) o[e] += pa[e];
    }
    if (MODE == REC_STATE_SPACE)
#pragma unroll
      for (int e = 0; e < 4; e++) o[e] = fmaf(p.D[h], v[e], o[e]);
  }
  if (p.norm_w) {
    float ss = warp_reduce_sum(o[0] * o[0] + o[1] * o[1] + o[2] * o[2] + o[3] * o[3]);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) ss += red[w];
    const float inv = 1.f / sqrtf(ss / (float)DV + p.eps);
    if (rg == 0) {
      float w4[4];
      load_vec<T, 4>((const T*)p.norm_w + c4, w4);
#pragma unroll
      for (int e = 0; e < 4; e++) o[e] *= inv * w4[e];
    }
  }
  if (rg == 0) {
#pragma unroll
    for (int e = 0; e < 4; e++) o[e] *= p.out_scale;
    store_vec<T, 4>((T*)p.out + (long)t * p.out_stride + (long)h * DV + c4, o);
  }
}

// true (with rc set) when the decode kernel takes these sizes
template <typename T, int MODE>
static bool launch_decode(const RecParams& p, cudaStream_t stream, int* rc) {
  if (p.dv % 4 || p.dv > 1024 || p.v_stride % 4 || p.out_stride % 4 || !aligned16(p.v) || !aligned16(p.out) ||
      !aligned16(p.state) || !aligned16(p.norm_w))
    return false;
  const int RG = 256 / (p.dv / 4), M = (p.dk + RG - 1) / RG;
  const size_t smem = sizeof(float) * (size_t)(2 * p.dk + RG * p.dv);
  if (M > 16 || smem > 40000 || (2 * p.dk) % 4) return false;
  const dim3 grid((unsigned)p.num_seqs, (unsigned)p.heads);
  if (M <= 4) recurrence_decode_kernel<T, MODE, 4><<<grid, 256, smem, stream>>>(p);
  else if (M <= 8) recurrence_decode_kernel<T, MODE, 8><<<grid, 256, smem, stream>>>(p);
  else recurrence_decode_kernel<T, MODE, 16><<<grid, 256, smem, stream>>>(p);
  *rc = B200_CHECK_LAUNCH();
  return true;
}

template <typename T, int MODE, int R, int CJ>
static int launch_prefill(const RecParams& p, cudaStream_t stream) {
  constexpr int V = 16 / (int)sizeof(T);
  const bool vec = R % V == 0 && p.dk % V == 0 && p.q_stride % V == 0 && p.k_stride % V == 0 && p.f_stride % V == 0 &&
                   p.dv % CJ == 0 && p.v_stride % CJ == 0 && p.out_stride % CJ == 0 && aligned16(p.q) && aligned16(p.k) &&
                   aligned16(p.f) && aligned16(p.v) && aligned16(p.out) && aligned16(p.state);
  const dim3 grid((unsigned)p.num_seqs, (unsigned)p.heads, (unsigned)((p.dv + 16 * CJ - 1) / (16 * CJ)));
  if (vec) recurrence_kernel<T, MODE, R, CJ, true><<<grid, 128, 0, stream>>>(p);
  else recurrence_kernel<T, MODE, R, CJ, false><<<grid, 128, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

template <typename T, int MODE>
static int launch_mode(const RecParams& p, cudaStream_t stream) {
  int rc = 0;
  if (p.uniform && launch_decode<T, MODE>(p, stream, &rc)) return rc;
  if (p.norm_w) return -1;
  if (p.dk <= 32) return launch_prefill<T, MODE, 4, 4>(p, stream);
  if (p.dk <= 64) return launch_prefill<T, MODE, 8, 4>(p, stream);
  if (p.dk <= 128) return launch_prefill<T, MODE, 16, 4>(p, stream);
  if (p.dk <= 256) return launch_prefill<T, MODE, 32, 2>(p, stream);
  return 9762;
}

template <typename T>
static int launch_t(const RecParams& p, cudaStream_t stream) {
  if (p.mode == REC_FORGET) return launch_mode<T, REC_FORGET>(p, stream);
  if (p.mode == REC_STATE_SPACE) return launch_mode<T, REC_STATE_SPACE>(p, stream);
  return launch_mode<T, REC_LOG_DECAY>(p, stream);
}

}  // namespace b200

using namespace b200;

// uniform: every sequence has exactly one token.  -1: the norm was asked for and the sizes do not allow the decode
// kernel; nothing was launched
B200_API int b200_linear_recurrence(const RecurrenceArgs* a, int* status, cudaStream_t stream) {
  if (a->num_seqs <= 0) return 0;
  if (a->key_heads < 1 || a->heads < 1 || a->heads % a->key_heads || a->heads > 65535 || a->dk < 1 || a->dv < 1) return 9760;
  if (a->mode == REC_LOG_DECAY ? !a->log_decay || !a->k : a->mode == REC_STATE_SPACE ? !a->dt || !a->k || !a->dt_bias ||
      !a->A_log || !a->D : a->mode != REC_FORGET || !a->f || !a->f_bias || !a->lower || a->key_heads != a->heads)
    return 9761;
  RecParams p;
  static_cast<RecurrenceArgs&>(p) = *a;
  p.status = status;
  return a->dtype ? launch_t<float>(p, stream) : launch_t<__nv_bfloat16>(p, stream);
}
