// Linear-attention building blocks of the delta-rule families (Qwen3-Next style hybrids, Vofelix), for
// prefill portions and single-token decode alike:
//   causal_conv1d     depthwise short convolution over the token axis of variable-length sequences with
//                     a per-sequence state of the last K-1 inputs, + SiLU; optionally in the same launch
//                     the two per-head scalars of the delta rule (write strength, log-decay)
//   gated_delta_rule  S <- S exp(g_t);  u = beta_t (v_t - S^T k_t);  S <- S + k_t u^T;  o_t = S^T q_t
//                     with S in registers
// Element type bf16 or fp32 (template), head sizes and tap counts are run-time values.
// Counterparts of the reference's causal_conv1d and recurrent / chunked gated-delta-rule ops
// (csrc/moe/causal_conv1d*, csrc/attention/recurrent_gated_delta_rule*, ops/triton/fla/*).
#include "common.cuh"
#include "dtypes.cuh"

namespace b200 {

constexpr int CONV_TILE = 16;        // tokens of one sequence per block; K - 1 <= CONV_TILE

struct ConvParams {
  const void* x;
  long x_stride;
  const void* w;          // [C, K]
  const void* bias;       // [C] or null
  void* state;            // [slots, K-1, C], oldest input first
  const int* cu;          // [B + 1]
  const int* slots;
  const int* has_init;
  void* y;
  long y_stride;
  int B, C, K, act, uniform;      // uniform: every sequence has exactly one token
  long num_slots;
  // delta-rule scalars (H == 0: none): ba [T, 2H] = raw write strength, raw decay input
  const void* ba;
  long ba_stride;
  const float* A_log;
  const float* dt_bias;
  int H;
  float* beta;            // [T, H]
  float* log_decay;       // [T, H]
  int* status;
};

// A tile is CONV_TILE consecutive tokens of ONE sequence; sequence b owns the tile slots from
// cu[b] / CONV_TILE + b on (at least as many as it needs).  Only a sequence's first tile reads the
// state, and the same threads write the new state afterwards, so no two blocks touch a state row.
template <typename T, int VEC, int KR>
__global__ void __launch_bounds__(128) causal_conv1d_kernel(const ConvParams p) {
  int b, tile;
  if (p.uniform) {
    b = blockIdx.y;
    tile = 0;
  } else {
    const int w = blockIdx.y;
    int lo = 0, hi = p.B - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (p.cu[mid] / CONV_TILE + mid <= w) lo = mid; else hi = mid - 1;
    }
    b = lo;
    tile = w - (p.cu[b] / CONV_TILE + b);
  }
  const int t0 = p.cu[b], n = p.cu[b + 1] - t0;
  const int i0 = tile * CONV_TILE, i1 = min(i0 + CONV_TILE, n);
  if (i0 >= n) return;
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    return;
  }
  const int conv_blocks = gridDim.x - (p.H > 0 ? 1 : 0);
  if ((int)blockIdx.x >= conv_blocks) {
    for (int e = threadIdx.x; e < (i1 - i0) * p.H; e += blockDim.x) {
      const int i = e / p.H, h = e - i * p.H;
      const long t = t0 + i0 + i;
      const T* row = (const T*)p.ba + t * p.ba_stride;
      const float braw = to_f(row[h]), a = to_f(row[p.H + h]) + p.dt_bias[h];
      const float sp = a > 20.f ? a : log1pf(expf(a));
      p.beta[t * p.H + h] = 1.f / (1.f + expf(-braw));
      p.log_decay[t * p.H + h] = -expf(p.A_log[h]) * sp;
    }
    return;
  }
  const int c = ((int)blockIdx.x * blockDim.x + threadIdx.x) * VEC;
  if (c >= p.C) return;
  const int K = KR ? KR : p.K;
  const T* x = (const T*)p.x + (long)t0 * p.x_stride + c;
  const T* w = (const T*)p.w + (long)c * K;
  T* st = (T*)p.state + (long)slot * (K - 1) * p.C + c;
  T* y = (T*)p.y + (long)t0 * p.y_stride + c;
  const bool init = p.has_init[b] != 0;
  auto input = [&](int i, float* v) {      // input of local token i, reaching back into the state
    if (i >= 0) load_vec<T, VEC>(x + (long)i * p.x_stride, v);
    else if (init) load_vec<T, VEC>(st + (long)(K - 1 + i) * p.C, v);
    else
#pragma unroll
      for (int e = 0; e < VEC; e++) v[e] = 0.f;
  };
  float bs[VEC];
#pragma unroll
  for (int e = 0; e < VEC; e++) bs[e] = p.bias ? to_f(((const T*)p.bias)[c + e]) : 0.f;
  auto finish = [&](int i, float* acc) {
    if (p.act)
#pragma unroll
      for (int e = 0; e < VEC; e++) acc[e] = silu_f<T>(acc[e]);
    store_vec<T, VEC>(y + (long)i * p.y_stride, acc);
  };
  if constexpr (KR > 0) {
    float wk[KR][VEC], win[KR][VEC];
    if constexpr (VEC > 1 && (KR * VEC * sizeof(T)) % 16 == 0) {
      constexpr int WV = 16 / (int)sizeof(T);
      T wr[KR * VEC];
#pragma unroll
      for (int i = 0; i < KR * VEC; i += WV) load_raw<T, WV>(w + i, wr + i);
#pragma unroll
      for (int i = 0; i < KR * VEC; i++) wk[i % KR][i / KR] = to_f(wr[i]);
    } else {
#pragma unroll
      for (int j = 0; j < KR; j++)
#pragma unroll
        for (int e = 0; e < VEC; e++) wk[j][e] = to_f(w[(long)e * KR + j]);
    }
#pragma unroll
    for (int j = 0; j < KR - 1; j++) input(i0 - (KR - 1) + j, win[j]);
    constexpr int FLY = 4;             // rows in flight
    for (int ib = i0; ib < i1; ib += FLY) {
      T row[FLY][VEC];
#pragma unroll
      for (int f = 0; f < FLY; f++)
        if (ib + f < i1) load_raw<T, VEC>(x + (long)(ib + f) * p.x_stride, row[f]);
#pragma unroll
      for (int f = 0; f < FLY; f++) {
        if (ib + f >= i1) break;
        float acc[VEC];
#pragma unroll
        for (int e = 0; e < VEC; e++) {
          win[KR - 1][e] = to_f(row[f][e]);
          acc[e] = bs[e];
        }
#pragma unroll
        for (int j = 0; j < KR; j++)
#pragma unroll
          for (int e = 0; e < VEC; e++) acc[e] = fmaf(wk[j][e], win[j][e], acc[e]);
        finish(ib + f, acc);
#pragma unroll
        for (int j = 0; j < KR - 1; j++)
#pragma unroll
          for (int e = 0; e < VEC; e++) win[j][e] = win[j + 1][e];
      }
    }
  } else {
    for (int i = i0; i < i1; i++) {
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) acc[e] = bs[e];
      for (int j = 0; j < K; j++) {
        float v[VEC];
        input(i - (K - 1) + j, v);
#pragma unroll
        for (int e = 0; e < VEC; e++) acc[e] = fmaf(to_f(w[(long)e * K + j]), v[e], acc[e]);
      }
      finish(i, acc);
    }
  }
  if (tile == 0) {       // the last K - 1 inputs; a short portion keeps the tail of the old state (j < n + j)
    for (int j = 0; j < K - 1; j++) {
      float v[VEC];
      input(n - (K - 1) + j, v);
      store_vec<T, VEC>(st + (long)j * p.C, v);
    }
  }
}

// q, k [T, Hk, DK], v [T, Hv, DV] (token strides given), log-decay and beta [T, Hv] fp32,
// state [slots, Hv, DK, DV] fp32, out [T, Hv, DV].  Hv % Hk == 0 (value heads share keys).
//
// Eight lanes share a column of S, each holding R of its DK rows (row i of a lane: 32 (i / 4) + 4 lane +
// i % 4, so that a staged k or q row is read without bank conflicts); a thread covers CJ adjacent columns,
// a warp 4 CJ, a block 16 CJ.  Rows are kept in pairs for the packed fp32 FMA.  With a = S^T k and
// b = S^T q taken from the state BEFORE the token's write, the token is
//     u = beta (v - d a),   S <- d S + k u^T,   o = d b + (k . q) u        (d = exp(g))
// so both products and their lane reductions run side by side.
//
// Inputs are staged in chunks of tokens: while a chunk is processed, the threads hold the next one's raw
// elements in flight (registers); between two chunks they store it, and eight threads per token turn k and q
// into fp32 unit vectors and form k . q.
struct DeltaParams {
  const void *q, *k, *v;
  long qk_stride, v_stride;
  const float *g, *beta;
  float* state;
  const int *cu, *slots, *has_init;
  void* out;
  long out_stride;
  int Hk, Hv, DK, DV;
  float scale;
  int l2norm;
  long num_slots;
  int* status;
};

constexpr int DELTA_CHUNK = 16;      // tokens per stage: eight of the 128 threads work on each

template <typename T, int R, int CJ, bool VEC>
__global__ void __launch_bounds__(128) gated_delta_rule_kernel(const DeltaParams p) {
  constexpr int DKP = 8 * R;                    // rows, padded with zeros
  constexpr int COLS = 16 * CJ;
  constexpr int V = VEC ? 16 / (int)sizeof(T) : 1;
  constexpr int PER = DKP / 8;                  // elements of a k (q) row per staging thread
  __shared__ __align__(16) float ks[DELTA_CHUNK][DKP], qs[DELTA_CHUNK][DKP], vs[DELTA_CHUNK][COLS];
  __shared__ __align__(16) float4 sc[DELTA_CHUNK];            // d, beta, k . q
  const int b = blockIdx.x, hv = blockIdx.y;
  const int hk = hv / (p.Hv / p.Hk);
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
  const int DK = p.DK, DV = p.DV;
  float* sp = p.state + ((long)slot * p.Hv + hv) * DK * DV;
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
  const T* kp = (const T*)p.k + (long)hk * DK;
  const T* qp = (const T*)p.q + (long)hk * DK;
  const T* vp = (const T*)p.v + (long)hv * DV + jb;
  constexpr int VC = VEC ? CJ : 1;              // elements per v access
  constexpr int VPER = COLS / 8;
  T rk[PER], rq[PER], rv[VPER];
  float rg = 0.f, rb = 0.f;
  auto fetch = [&](int t) {                     // raw elements of token t + st
    t += st;
    const bool on = t < t1;
#pragma unroll
    for (int i = 0; i < PER; i += V) {
      const int e = (i / V * 8 + s8) * V;
      if (on && e < DK) {
        load_raw<T, V>(kp + (long)t * p.qk_stride + e, rk + i);
        load_raw<T, V>(qp + (long)t * p.qk_stride + e, rq + i);
      } else {
#pragma unroll
        for (int x = 0; x < V; x++) rk[i + x] = rq[i + x] = from_f<T>(0.f);
      }
    }
#pragma unroll
    for (int i = 0; i < VPER; i += VC) {
      const int e = (i / VC * 8 + s8) * VC;
      if (on && jb + e < DV) load_raw<T, VC>(vp + (long)t * p.v_stride + e, rv + i);
      else
#pragma unroll
        for (int x = 0; x < VC; x++) rv[i + x] = from_f<T>(0.f);
    }
    rg = on ? p.g[(long)t * p.Hv + hv] : 0.f;
    rb = on ? p.beta[(long)t * p.Hv + hv] : 0.f;
  };
  auto stage = [&]() {
    float kk = 0.f, qq = 0.f, kq = 0.f;
#pragma unroll
    for (int i = 0; i < PER; i++) {
      const float a = to_f(rk[i]), c = to_f(rq[i]);
      kk = fmaf(a, a, kk);
      qq = fmaf(c, c, qq);
      kq = fmaf(a, c, kq);
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) {
      kk += __shfl_xor_sync(0xffffffffu, kk, o);
      qq += __shfl_xor_sync(0xffffffffu, qq, o);
      kq += __shfl_xor_sync(0xffffffffu, kq, o);
    }
    const float ik = p.l2norm ? rsqrtf(kk + 1e-6f) : 1.f;
    const float iq = (p.l2norm ? rsqrtf(qq + 1e-6f) : 1.f) * p.scale;
#pragma unroll
    for (int i = 0; i < PER; i += V)
#pragma unroll
      for (int x = 0; x < V; x++) {
        const int e = (i / V * 8 + s8) * V + x;
        ks[st][e] = to_f(rk[i + x]) * ik;
        qs[st][e] = to_f(rq[i + x]) * iq;
      }
#pragma unroll
    for (int i = 0; i < VPER; i += VC)
#pragma unroll
      for (int x = 0; x < VC; x++) vs[st][(i / VC * 8 + s8) * VC + x] = to_f(rv[i + x]);
    if (s8 == 0) sc[st] = make_float4(expf(rg), rb, kq * ik * iq, 0.f);
  };
  T* op = (T*)p.out + (long)hv * DV + j0;
  fetch(t0);
  for (int tc = t0; tc < t1; tc += DELTA_CHUNK) {
    if (tc > t0) __syncthreads();               // the previous chunk has been read
    stage();
    __syncthreads();
    if (tc + DELTA_CHUNK < t1) fetch(tc + DELTA_CHUNK);
    const int n = min(DELTA_CHUNK, t1 - tc);
    for (int i = 0; i < n; i++) {
      const float4 s4 = sc[i];
      float vt[CJ];
      load_vec<float, CJ>(&vs[i][jl], vt);
      f32x2 a2[CJ], b2[CJ];
#pragma unroll
      for (int c = 0; c < CJ; c++) a2[c] = b2[c] = 0;
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(&ks[i][r * 8 + gl * 4]);
        const ulonglong2 q4 = *reinterpret_cast<const ulonglong2*>(&qs[i][r * 8 + gl * 4]);
#pragma unroll
        for (int c = 0; c < CJ; c++) {
          a2[c] = fma2(S[r / 2][c], k4.x, a2[c]);
          b2[c] = fma2(S[r / 2][c], q4.x, b2[c]);
          a2[c] = fma2(S[r / 2 + 1][c], k4.y, a2[c]);
          b2[c] = fma2(S[r / 2 + 1][c], q4.y, b2[c]);
        }
      }
      float red[2 * CJ];
#pragma unroll
      for (int c = 0; c < CJ; c++) {
        const float2 av = unpack2(a2[c]), bv = unpack2(b2[c]);
        red[c] = av.x + av.y;
        red[CJ + c] = bv.x + bv.y;
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1)
#pragma unroll
        for (int x = 0; x < 2 * CJ; x++) red[x] += __shfl_xor_sync(0xffffffffu, red[x], o);
      const float d = s4.x;
      float u[CJ], o[CJ];
#pragma unroll
      for (int c = 0; c < CJ; c++) {
        u[c] = s4.y * (vt[c] - d * red[c]);
        o[c] = d * red[CJ + c] + s4.z * u[c];
      }
      const f32x2 dd = pack2(d, d);
      f32x2 uu[CJ];
#pragma unroll
      for (int c = 0; c < CJ; c++) uu[c] = pack2(u[c], u[c]);
#pragma unroll
      for (int r = 0; r < R; r += 4) {
        const ulonglong2 k4 = *reinterpret_cast<const ulonglong2*>(&ks[i][r * 8 + gl * 4]);
#pragma unroll
        for (int c = 0; c < CJ; c++) {
          S[r / 2][c] = fma2(k4.x, uu[c], mul2(S[r / 2][c], dd));
          S[r / 2 + 1][c] = fma2(k4.y, uu[c], mul2(S[r / 2 + 1][c], dd));
        }
      }
      if (gl == 0) {
        T* dst = op + (long)(tc + i) * p.out_stride;
        if (VEC) { if (j0 < DV) store_vec<T, CJ>(dst, o); }
        else
#pragma unroll
          for (int c = 0; c < CJ; c++) if (j0 + c < DV) dst[c] = from_f<T>(o[c]);
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

// One token per sequence (decode): a block per (sequence, value head) streams the head's state once through
// registers.  Four adjacent columns per thread, the threads of a row group cover a row of S, the row groups
// take every RG-th row (M rows each).  With z the gated RMS norm of the read-out,
// out = rms_norm(o) * w * silu(z), is part of the same pass.
struct DeltaDecodeExtra {
  const void* z;          // null: the bare read-out
  long z_stride;
  const void* norm_w;     // [DV]
  float eps;
};

template <typename T, int M>
__global__ void __launch_bounds__(256, M > 8 ? 2 : 3) delta_decode_kernel(const DeltaParams p, const DeltaDecodeExtra x) {
  extern __shared__ float sm[];
  const int DK = p.DK, DV = p.DV, cols = DV >> 2, RG = 256 / cols;
  float* ks = sm;                       // [DK]
  float* qs = ks + DK;                  // [DK]
  float* part = qs + DK;                // [2][RG][DV]
  __shared__ float red[8][3];
  const int b = blockIdx.x, hv = blockIdx.y, tid = threadIdx.x;
  const int hk = hv / (p.Hv / p.Hk);
  const int slot = p.slots[b], t = p.cu[b];
  const bool init = p.has_init[b] != 0;
  if (slot < 0 || slot >= p.num_slots) {
    if (tid == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    return;
  }
  const int rg = tid / cols, c4 = (tid - rg * cols) * 4;
  const bool on = rg < RG;
  float* sp = p.state + ((long)slot * p.Hv + hv) * DK * DV + c4;
  float4 S[M];
#pragma unroll
  for (int m = 0; m < M; m++) {
    const int i = rg + m * RG;
    S[m] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (on && init && i < DK) S[m] = *reinterpret_cast<const float4*>(sp + (long)i * DV);
  }
  float kk = 0.f, qq = 0.f, kq = 0.f;
  for (int i = tid; i < DK; i += 256) {
    const float k = to_f(((const T*)p.k)[(long)t * p.qk_stride + (long)hk * DK + i]);
    const float q = to_f(((const T*)p.q)[(long)t * p.qk_stride + (long)hk * DK + i]);
    ks[i] = k;
    qs[i] = q;
    kk += k * k;
    qq += q * q;
    kq += k * q;
  }
  const float d = expf(p.g[(long)t * p.Hv + hv]), bt = p.beta[(long)t * p.Hv + hv];
  float v[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) load_vec<T, 4>((const T*)p.v + (long)t * p.v_stride + (long)hv * DV + c4, v);
  kk = warp_reduce_sum(kk);
  qq = warp_reduce_sum(qq);
  kq = warp_reduce_sum(kq);
  if ((tid & 31) == 0) {
    red[tid >> 5][0] = kk;
    red[tid >> 5][1] = qq;
    red[tid >> 5][2] = kq;
  }
  __syncthreads();
  kk = qq = kq = 0.f;
#pragma unroll
  for (int w = 0; w < 8; w++) {
    kk += red[w][0];
    qq += red[w][1];
    kq += red[w][2];
  }
  const float ik = p.l2norm ? rsqrtf(kk + 1e-6f) : 1.f;
  const float iq = (p.l2norm ? rsqrtf(qq + 1e-6f) : 1.f) * p.scale;
  float a[4] = {0.f, 0.f, 0.f, 0.f}, bq[4] = {0.f, 0.f, 0.f, 0.f};
  if (on) {
#pragma unroll
    for (int m = 0; m < M; m++) {
      const int i = rg + m * RG;
      if (i < DK) {
        const float k = ks[i], q = qs[i];
        a[0] = fmaf(S[m].x, k, a[0]); bq[0] = fmaf(S[m].x, q, bq[0]);
        a[1] = fmaf(S[m].y, k, a[1]); bq[1] = fmaf(S[m].y, q, bq[1]);
        a[2] = fmaf(S[m].z, k, a[2]); bq[2] = fmaf(S[m].z, q, bq[2]);
        a[3] = fmaf(S[m].w, k, a[3]); bq[3] = fmaf(S[m].w, q, bq[3]);
      }
    }
    store_vec<float, 4>(part + rg * DV + c4, a);
    store_vec<float, 4>(part + (RG + rg) * DV + c4, bq);
  }
  __syncthreads();
#pragma unroll
  for (int e = 0; e < 4; e++) a[e] = bq[e] = 0.f;
  if (on)
    for (int w = 0; w < RG; w++) {
      float pa[4], pb[4];
      load_vec<float, 4>(part + w * DV + c4, pa);
      load_vec<float, 4>(part + (RG + w) * DV + c4, pb);
#pragma unroll
      for (int e = 0; e < 4; e++) { a[e] += pa[e]; bq[e] += pb[e]; }
    }
  float u[4], o[4];
#pragma unroll
  for (int e = 0; e < 4; e++) {
    u[e] = bt * (v[e] - d * ik * a[e]);
    o[e] = d * iq * bq[e] + kq * ik * iq * u[e];
    u[e] *= ik;
  }
  if (on)
#pragma unroll
    for (int m = 0; m < M; m++) {
      const int i = rg + m * RG;
      if (i < DK) {
        const float k = ks[i];
        *reinterpret_cast<float4*>(sp + (long)i * DV) = make_float4(
            fmaf(k, u[0], d * S[m].x), fmaf(k, u[1], d * S[m].y), fmaf(k, u[2], d * S[m].z), fmaf(k, u[3], d * S[m].w));
      }
    }
  if (x.z != nullptr) {                  // every row group holds the whole read-out; the first one counts
    float ss = rg == 0 ? o[0] * o[0] + o[1] * o[1] + o[2] * o[2] + o[3] * o[3] : 0.f;
    ss = warp_reduce_sum(ss);
    if ((tid & 31) == 0) red[tid >> 5][0] = ss;      // the sums of k and q were read before the last barrier
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; w++) ss += red[w][0];
    const float inv = 1.f / sqrtf(ss / (float)DV + x.eps);
    if (rg == 0) {
      float z[4], w4[4];
      load_vec<T, 4>((const T*)x.z + (long)t * x.z_stride + (long)hv * DV + c4, z);
      load_vec<T, 4>((const T*)x.norm_w + c4, w4);
#pragma unroll
      for (int e = 0; e < 4; e++) o[e] = o[e] * inv * w4[e] * silu_f<T>(z[e]);
    }
  }
  if (rg == 0) store_vec<T, 4>((T*)p.out + (long)t * p.out_stride + (long)hv * DV + c4, o);
}

// true (with rc set) when the decode kernel takes these sizes
template <typename T>
static bool launch_delta_decode(const DeltaParams& p, const DeltaDecodeExtra& x, int B, cudaStream_t stream, int* rc) {
  if (p.DV % 4 || p.DV > 1024 || p.v_stride % 4 || p.out_stride % 4 || !aligned16(p.v) || !aligned16(p.out) ||
      !aligned16(p.state) || (x.z && (x.z_stride % 4 || !aligned16(x.z) || !aligned16(x.norm_w))))
    return false;
  const int RG = 256 / (p.DV / 4), M = (p.DK + RG - 1) / RG;
  const size_t smem = sizeof(float) * (size_t)(2 * p.DK + 2 * RG * p.DV);
  if (M > 16 || smem > 40000 || (2 * p.DK) % 4) return false;
  const dim3 grid((unsigned)B, (unsigned)p.Hv);
  if (M <= 4) delta_decode_kernel<T, 4><<<grid, 256, smem, stream>>>(p, x);
  else if (M <= 8) delta_decode_kernel<T, 8><<<grid, 256, smem, stream>>>(p, x);
  else delta_decode_kernel<T, 16><<<grid, 256, smem, stream>>>(p, x);
  *rc = B200_CHECK_LAUNCH();
  return true;
}

template <typename T>
static int launch_conv(const ConvParams& p, long T_tokens, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = p.C % V == 0 && p.x_stride % V == 0 && p.y_stride % V == 0 && aligned16(p.x) && aligned16(p.y) &&
                   aligned16(p.w) && aligned16(p.state);
  const int per = 128 * (vec ? V : 1);
  const long tiles = p.uniform ? p.B : T_tokens / CONV_TILE + p.B;
  if (tiles > 65535) return 9805;
  dim3 grid((unsigned)((p.C + per - 1) / per + (p.H > 0 ? 1 : 0)), (unsigned)tiles);
#define LAUNCH_CONV(KK)                                                        \
  if (vec) causal_conv1d_kernel<T, V, KK><<<grid, 128, 0, stream>>>(p);        \
  else causal_conv1d_kernel<T, 1, KK><<<grid, 128, 0, stream>>>(p)
  if (p.K == 4) { LAUNCH_CONV(4); }
  else if (p.K == 3) { LAUNCH_CONV(3); }
  else if (p.K == 2) { LAUNCH_CONV(2); }
  else { LAUNCH_CONV(0); }
#undef LAUNCH_CONV
  return B200_CHECK_LAUNCH();
}

template <typename T, int R, int CJ>
static int launch_delta_r(const DeltaParams& p, int B, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = R % V == 0 && p.DK % V == 0 && p.qk_stride % V == 0 && p.DV % CJ == 0 && p.v_stride % CJ == 0 &&
                   p.out_stride % CJ == 0 && aligned16(p.q) && aligned16(p.k) && aligned16(p.v) && aligned16(p.out) &&
                   aligned16(p.state);
  dim3 grid((unsigned)B, (unsigned)p.Hv, (unsigned)((p.DV + 16 * CJ - 1) / (16 * CJ)));
  if (vec) gated_delta_rule_kernel<T, R, CJ, true><<<grid, 128, 0, stream>>>(p);
  else gated_delta_rule_kernel<T, R, CJ, false><<<grid, 128, 0, stream>>>(p);
  return B200_CHECK_LAUNCH();
}

template <typename T>
static int launch_delta(const DeltaParams& p, int B, cudaStream_t stream) {
  if (p.DK <= 32) return launch_delta_r<T, 4, 4>(p, B, stream);
  if (p.DK <= 64) return launch_delta_r<T, 8, 4>(p, B, stream);
  if (p.DK <= 128) return launch_delta_r<T, 16, 4>(p, B, stream);
  if (p.DK <= 256) return launch_delta_r<T, 32, 2>(p, B, stream);
  return 9802;
}

}  // namespace b200

using namespace b200;

// cu: int32 [B + 1] token offsets, slots: int32 [B] state rows, has_init: int32 [B].  T: tokens of the
// step (cu[B]).  dtype: 0 bf16, 1 fp32 (x, w, bias, state, y, ba).  H > 0 adds the delta-rule scalars.
B200_API int b200_causal_conv1d(const void* x, long x_stride, const void* w, const void* bias, void* state,
                                const void* cu, const void* slots, const void* has_init, void* y,
                                long y_stride, long T, int B, int C, int K, int act, int uniform, long num_slots,
                                int dtype, const void* ba, long ba_stride, const void* A_log, const void* dt_bias,
                                int H, void* beta, void* log_decay, int* status, cudaStream_t stream) {
  if (B <= 0 || C <= 0 || T <= 0) return 0;
  if (K < 1 || K - 1 > CONV_TILE) return 9800;
  ConvParams p{x, x_stride, w, bias, state, (const int*)cu, (const int*)slots, (const int*)has_init, y, y_stride,
               B, C, K, act, uniform, num_slots, ba, ba_stride, (const float*)A_log, (const float*)dt_bias, H,
               (float*)beta, (float*)log_decay, status};
  return dtype ? launch_conv<float>(p, T, stream) : launch_conv<__nv_bfloat16>(p, T, stream);
}

// uniform: every sequence of the step has exactly one token.  z (optional, with norm_w [DV] and eps, uniform
// steps only): the output is the gated RMS norm of the read-out; returns -1 when the sizes do not allow that.
B200_API int b200_gated_delta_rule(const void* q, const void* k, const void* v, long qk_stride,
                                   long v_stride, const void* g, const void* beta, void* state,
                                   const void* cu, const void* slots, const void* has_init, void* out,
                                   long out_stride, int B, int Hk, int Hv, int DK, int DV, float scale,
                                   int l2norm, long num_slots, int dtype, int uniform, const void* z, long z_stride,
                                   const void* norm_w, float eps, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (Hk <= 0 || Hv % Hk || Hv > 65535) return 9801;
  DeltaParams p{q, k, v, qk_stride, v_stride, (const float*)g, (const float*)beta, (float*)state, (const int*)cu,
                (const int*)slots, (const int*)has_init, out, out_stride, Hk, Hv, DK, DV, scale, l2norm, num_slots,
                status};
  if (uniform) {
    DeltaDecodeExtra x{z, z_stride, norm_w, eps};
    int rc = 0;
    if (dtype ? launch_delta_decode<float>(p, x, B, stream, &rc)
              : launch_delta_decode<__nv_bfloat16>(p, x, B, stream, &rc))
      return rc;
  }
  if (z) return -1;
  return dtype ? launch_delta<float>(p, B, stream) : launch_delta<__nv_bfloat16>(p, B, stream);
}
