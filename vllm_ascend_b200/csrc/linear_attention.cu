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
#pragma unroll
    for (int j = 0; j < KR; j++)
#pragma unroll
      for (int e = 0; e < VEC; e++) wk[j][e] = to_f(w[(long)e * KR + j]);
#pragma unroll
    for (int j = 0; j < KR - 1; j++) input(i0 - (KR - 1) + j, win[j]);
    for (int i = i0; i < i1; i++) {
      load_vec<T, VEC>(x + (long)i * p.x_stride, win[KR - 1]);
      float acc[VEC];
#pragma unroll
      for (int e = 0; e < VEC; e++) acc[e] = bs[e];
#pragma unroll
      for (int j = 0; j < KR; j++)
#pragma unroll
        for (int e = 0; e < VEC; e++) acc[e] = fmaf(wk[j][e], win[j][e], acc[e]);
      finish(i, acc);
#pragma unroll
      for (int j = 0; j < KR - 1; j++)
#pragma unroll
        for (int e = 0; e < VEC; e++) win[j][e] = win[j + 1][e];
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
// Eight lanes share a column of S, each holding R of its DK rows; a thread covers CJ adjacent columns, a
// warp 4 CJ, a block 16 CJ.  Rows are kept in pairs for the packed fp32 FMA.  With a = S^T k and
// b = S^T q taken from the state BEFORE the token's write, the token is
//     u = beta (v - d a),   S <- d S + k u^T,   o = d b + (k . q) u        (d = exp(g))
// so both products and their lane reductions run side by side.  The unit norms of k and q are applied
// as scalars.  The next token's inputs are fetched while this one is processed.
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

template <typename T, int R, int CJ, bool VEC>
__global__ void __launch_bounds__(128) gated_delta_rule_kernel(const DeltaParams p) {
  const int b = blockIdx.x, hv = blockIdx.y;
  const int hk = hv / (p.Hv / p.Hk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gl = lane & 7;                                           // row group of the lane
  const int j0 = (((int)blockIdx.z * 4 + warp) * 4 + (lane >> 3)) * CJ;    // first column
  const int slot = p.slots[b];
  if (slot < 0 || slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicExch(p.status, B200_BAD_INDEX);
    return;
  }
  const int t0 = p.cu[b], t1 = p.cu[b + 1];
  if (t0 >= t1) return;
  const int DK = p.DK, DV = p.DV;
  const int r0 = gl * R;
  float2 S[R / 2][CJ];
  float* sp = p.state + ((long)slot * p.Hv + hv) * DK * DV;
  const bool init = p.has_init[b] != 0;
#pragma unroll
  for (int r = 0; r < R; r++) {
    float row[CJ];
#pragma unroll
    for (int c = 0; c < CJ; c++) row[c] = 0.f;
    if (init && r0 + r < DK) {
      const float* src = sp + (long)(r0 + r) * DV + j0;
      if (VEC) { if (j0 < DV) load_vec<float, CJ>(src, row); }
      else
#pragma unroll
        for (int c = 0; c < CJ; c++) if (j0 + c < DV) row[c] = src[c];
    }
#pragma unroll
    for (int c = 0; c < CJ; c++) (r & 1 ? S[r / 2][c].y : S[r / 2][c].x) = row[c];
  }
  const T* qp = (const T*)p.q + (long)hk * DK + r0;
  const T* kp = (const T*)p.k + (long)hk * DK + r0;
  const T* vp = (const T*)p.v + (long)hv * DV + j0;
  T* op = (T*)p.out + (long)hv * DV + j0;
  RawSlice<T, R> nk, nq;
  T nv[CJ];
  float ng = 0.f, nb = 0.f;
  auto fetch = [&](int t) {
    nk.template load<VEC>(kp + (long)t * p.qk_stride, DK - r0);
    nq.template load<VEC>(qp + (long)t * p.qk_stride, DK - r0);
    const T* vr = vp + (long)t * p.v_stride;
    if (VEC) { if (j0 < DV) load_raw<T, CJ>(vr, nv); }
    else
#pragma unroll
      for (int c = 0; c < CJ; c++) if (j0 + c < DV) nv[c] = vr[c];
    ng = p.g[(long)t * p.Hv + hv];
    nb = p.beta[(long)t * p.Hv + hv];
  };
#pragma unroll
  for (int c = 0; c < CJ; c++) nv[c] = from_f<T>(0.f);
  fetch(t0);
  for (int t = t0; t < t1; t++) {
    float2 k2[R / 2], q2[R / 2];
    float vt[CJ];
    nk.unpack(k2);
    nq.unpack(q2);
#pragma unroll
    for (int c = 0; c < CJ; c++) vt[c] = to_f(nv[c]);
    const float d = expf(ng), bt = nb;
    if (t + 1 < t1) fetch(t + 1);
    float2 kk = {0.f, 0.f}, qq = {0.f, 0.f}, kq = {0.f, 0.f}, a2[CJ], b2[CJ];
#pragma unroll
    for (int c = 0; c < CJ; c++) a2[c] = b2[c] = make_float2(0.f, 0.f);
#pragma unroll
    for (int r = 0; r < R / 2; r++) {
      kk = fma2(k2[r], k2[r], kk);
      qq = fma2(q2[r], q2[r], qq);
      kq = fma2(k2[r], q2[r], kq);
#pragma unroll
      for (int c = 0; c < CJ; c++) {
        a2[c] = fma2(S[r][c], k2[r], a2[c]);
        b2[c] = fma2(S[r][c], q2[r], b2[c]);
      }
    }
    float red[3 + 2 * CJ];
    red[0] = kk.x + kk.y;
    red[1] = qq.x + qq.y;
    red[2] = kq.x + kq.y;
#pragma unroll
    for (int c = 0; c < CJ; c++) {
      red[3 + c] = a2[c].x + a2[c].y;
      red[3 + CJ + c] = b2[c].x + b2[c].y;
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1)
#pragma unroll
      for (int i = 0; i < 3 + 2 * CJ; i++) red[i] += __shfl_xor_sync(0xffffffffu, red[i], o);
    const float ik = p.l2norm ? rsqrtf(red[0] + 1e-6f) : 1.f;
    const float iq = (p.l2norm ? rsqrtf(red[1] + 1e-6f) : 1.f) * p.scale;
    const float kqn = red[2] * ik * iq;
    float u[CJ], o[CJ];
#pragma unroll
    for (int c = 0; c < CJ; c++) {
      u[c] = bt * (vt[c] - d * ik * red[3 + c]);
      o[c] = d * iq * red[3 + CJ + c] + kqn * u[c];
      u[c] *= ik;
    }
    const float2 dd = {d, d};
#pragma unroll
    for (int c = 0; c < CJ; c++) {
      const float2 uu = {u[c], u[c]};
#pragma unroll
      for (int r = 0; r < R / 2; r++) S[r][c] = fma2(k2[r], uu, mul2(S[r][c], dd));
    }
    if (gl == 0) {
      T* dst = op + (long)t * p.out_stride;
      if (VEC) { if (j0 < DV) store_vec<T, CJ>(dst, o); }
      else
#pragma unroll
        for (int c = 0; c < CJ; c++) if (j0 + c < DV) dst[c] = from_f<T>(o[c]);
    }
  }
#pragma unroll
  for (int r = 0; r < R; r++) {
    if (r0 + r >= DK) continue;
    float* dst = sp + (long)(r0 + r) * DV + j0;
    float row[CJ];
#pragma unroll
    for (int c = 0; c < CJ; c++) row[c] = r & 1 ? S[r / 2][c].y : S[r / 2][c].x;
    if (VEC) { if (j0 < DV) store_vec<float, CJ>(dst, row); }
    else
#pragma unroll
      for (int c = 0; c < CJ; c++) if (j0 + c < DV) dst[c] = row[c];
  }
}

template <typename T>
static int launch_conv(const ConvParams& p, long T_tokens, cudaStream_t stream) {
  constexpr int V = 16 / sizeof(T);
  const bool vec = p.C % V == 0 && p.x_stride % V == 0 && p.y_stride % V == 0 && aligned16(p.x) && aligned16(p.y) &&
                   aligned16(p.state);
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

B200_API int b200_gated_delta_rule(const void* q, const void* k, const void* v, long qk_stride,
                                   long v_stride, const void* g, const void* beta, void* state,
                                   const void* cu, const void* slots, const void* has_init, void* out,
                                   long out_stride, int B, int Hk, int Hv, int DK, int DV, float scale,
                                   int l2norm, long num_slots, int dtype, int* status, cudaStream_t stream) {
  if (B <= 0) return 0;
  if (Hk <= 0 || Hv % Hk || Hv > 65535) return 9801;
  DeltaParams p{q, k, v, qk_stride, v_stride, (const float*)g, (const float*)beta, (float*)state, (const int*)cu,
                (const int*)slots, (const int*)has_init, out, out_stride, Hk, Hv, DK, DV, scale, l2norm, num_slots,
                status};
  return dtype ? launch_delta<float>(p, B, stream) : launch_delta<__nv_bfloat16>(p, B, stream);
}
