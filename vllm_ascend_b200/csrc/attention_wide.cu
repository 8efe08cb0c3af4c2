// Paged attention on tcgen05 tensor cores for keys wider than one operand tile (several projected keys side by side in
// a cache row), where several value heads may share a key row: scores mixed over the heads, two softmax maps per head.
// Options of AttnVariantArgs: window, output scale, fp32 output; bf16 caches.  Key row of value head g: g * key_heads / Hkv.
//
// attn_wide_kernel: tiles of 128 query rows (token, head of one value head) x 128 keys, any number of rows per sequence.
//   The queries' chunks of 64 dimensions stay in shared memory, the keys' chunks stream through a ring and accumulate
//   S in TMEM (double-buffered); the probabilities go back to TMEM as the A operand of P V, which leaves the shared
//   memory to the rings.
// attn_wide_decode_kernel: one query row per sequence.  A work item is (sequence, key head, KV split): all heads of the
//   key head are the columns of S^T = K Q^T, so every key and value is read once; the output has one accumulator per
//   value head.  Persistent, the K / V rings run across items.
// Roles: warp 0 TMA producer, warp 1 MMA issuer, warps 2-5 softmax and epilogue.  All waits are bounded; on timeout the
// CTA aborts cleanly and reports a status.  Behavioural parity with the reference's paged attention as in attention_tc.cu.
#include "attention.h"
#include "attention_score.cuh"
#include "common.cuh"

#include <mutex>
#include <string.h>
#include <string>
#include <unordered_map>

namespace b200 {

constexpr int WIDE_THREADS = 192;
constexpr int WIDE_CHUNK = 128 * 128;          // 128 rows x 64 bf16
constexpr int WIDE_RING = 16;                  // most stages of a ring
constexpr int WIDE_SMEM = 232448;
constexpr float kWideRescale = 8.f;

struct WideParams {
  const int *cu, *seq_lens, *block_table;
  int max_blocks, block_size, rows_per_load;
  int G, Hkv, Hq, key_heads, Dv, tok_per_tile;
  int num_seqs, window, num_splits, num_items;
  int chunks, k_stages, v_stages;              // chunks of 64 key dimensions; ring sizes
  float scale_log2, out_scale;
  int out_f32;
  void* out;
  long out_stride, num_blocks_total;
  float *partial_o, *partial_lse;
  int* status;
};

__device__ __forceinline__ void store_out(const WideParams& p, long at, float v) {
  if (p.out_f32) ((float*)p.out)[at] = v;
  else ((__nv_bfloat16*)p.out)[at] = __float2bfloat16(v);
}

// common end of both kernels: report, free the tensor memory
__device__ __forceinline__ void wide_finish(volatile int* abort_word, int* status, uint32_t tmem_base, int warp) {
  tc_fence_before();
  __syncthreads();
  if (*abort_word != 0) {
    // let copies still in flight land before the CTA's shared memory is released
    const uint64_t t_start = globaltimer_ns();
    while (globaltimer_ns() - t_start < 50000ull) __nanosleep(1000);
    if (threadIdx.x == 0 && status) atomicExch(status, *abort_word);
    __syncthreads();
  }
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

// Place in a ring of stages and the parity of its round.  Counted instead of divided: the producer and the MMA issuer
// are single warps whose instructions wait for one another.
struct Ring {
  int st = 0;
  uint32_t ph = 0;
  __device__ __forceinline__ void next(int stages) {
    if (++st == stages) {
      st = 0;
      ph ^= 1u;
    }
  }
};

// A matrix descriptor moves by adding bytes / 16; built once, since the issuer would wait for every step of building one
__device__ __forceinline__ uint64_t desc_at(uint64_t base, int bytes) { return base + (uint64_t)(uint32_t)(bytes >> 4); }

// one 64-dimension chunk of 128 keys from the pages of a sequence (lane i holds the block of part i), ``off`` rows into
// a page that is longer than 128; whole warp
__device__ __forceinline__ void load_chunk(uint8_t* dst, const CUtensorMap* tm, uint64_t* bar, int x, int head, int off,
                                           int blk_lane, int parts, int rpl, int lane) {
  for (int part = 0; part < parts; part++) {
    const int blk = __shfl_sync(0xffffffffu, blk_lane, part);
    if (lane == 0) tma_load_4d(dst + part * rpl * 128, tm, bar, x, off, head, blk);
  }
}

template <int NV>            // value size in units of 64
__global__ void __launch_bounds__(WIDE_THREADS, 1)
attn_wide_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                 const __grid_constant__ CUtensorMap tmap_v, const WideParams p) {
  // TMEM columns: two S of 128, O, two P of 64 (two bf16 keys per column)
  constexpr int V_BYTES = NV * WIDE_CHUNK, O_COL = 256, P_COL = 384;
  // ---------------- work decode (uniform over the CTA): sequence b owns the tiles from (cu[b] - cu[0]) / tok + b on
  const int h = blockIdx.x, wi = gridDim.y - 1 - blockIdx.y, base = p.cu[0];
  int seq, lo_ = 0, hi_ = p.num_seqs - 1;
  while (lo_ < hi_) {
    const int mid = (lo_ + hi_ + 1) >> 1;
    if ((p.cu[mid] - base) / p.tok_per_tile + mid <= wi) lo_ = mid; else hi_ = mid - 1;
  }
  seq = lo_;
  const int tok0 = (wi - ((p.cu[seq] - base) / p.tok_per_tile + seq)) * p.tok_per_tile;
  const int q_start = p.cu[seq], q_len = p.cu[seq + 1] - q_start, seq_len = p.seq_lens[seq];
  const int ctx = seq_len - q_len, G = p.G, ntok = min(p.tok_per_tile, q_len - tok0);
  if (ntok <= 0) return;
  const int kv_end = min(seq_len, ctx + tok0 + ntok);
  const int kv_lo = p.window > 0 ? max(0, ctx + tok0 - p.window + 1) : 0;
  const int t0 = kv_lo >> 7, n = ((kv_end + 127) >> 7) - t0;
  if (n <= 0) return;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int NC = p.chunks, KST = p.k_stages, VST = p.v_stages;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* Qs = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* Ks = Qs + NC * WIDE_CHUNK;
  uint8_t* Vs = Ks + KST * WIDE_CHUNK;
  uint64_t* q_full = (uint64_t*)(Vs + VST * V_BYTES);
  uint64_t* k_full = q_full + 1;             // WIDE_RING each
  uint64_t* k_empty = k_full + WIDE_RING;
  uint64_t* v_full = k_empty + WIDE_RING;    // 2 each
  uint64_t* v_empty = v_full + 2;
  uint64_t* s_ready = v_empty + 2;
  uint64_t* s_free = s_ready + 2;
  uint64_t* p_ready = s_free + 2;
  uint64_t* pv_done = p_ready + 2;
  uint32_t* tmem_ptr = (uint32_t*)(pv_done + 2);
  volatile int* abort_word = (volatile int*)(tmem_ptr + 1);
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < KST; s++) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
    }
    for (int b = 0; b < 2; b++) {
      mbar_init(&v_full[b], 1);
      mbar_init(&v_empty[b], 1);
      mbar_init(&s_ready[b], 1);
      mbar_init(&s_free[b], 4);
      mbar_init(&p_ready[b], 4);
      mbar_init(&pv_done[b], 1);
    }
    *abort_word = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, 512);
    tmem_relinquish();
  }
  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;

  if (warp == 0) {
    // ------------------------------------------------------------ producer, in the order of consumption
    const int* bt = p.block_table + (long)seq * p.max_blocks;
    const int rpl = p.rows_per_load, parts = 128 / rpl, hk = h * p.key_heads / p.Hkv;
    Ring kr, vr;
    if (lane == 0) {
      mbar_expect_tx(q_full, NC * 128 * G * p.tok_per_tile);
      for (int c = 0; c < NC; c++) tma_load_4d(Qs + c * WIDE_CHUNK, &tmap_q, q_full, c * 64, 0, h, q_start + tok0);
    }
    __syncwarp();
    auto block_of = [&](int j) -> int {
      if (j >= n || lane >= parts) return 0;
      return bt[min(((t0 + j) << 7) + lane * rpl, seq_len - 1) / p.block_size];
    };
    auto page_row = [&](int j) { return p.block_size > 128 ? ((t0 + j) << 7) % p.block_size : 0; };
    auto load_k = [&](int j, int blk) -> bool {
      if (__any_sync(0xffffffffu, (blk < 0 || blk >= p.num_blocks_total) && lane < parts)) {
        *abort_word = B200_BAD_INDEX;
        return false;
      }
      const int off = page_row(j);
      for (int c = 0; c < NC; c++, kr.next(KST)) {
        if (!mbar_wait(&k_empty[kr.st], kr.ph ^ 1u, abort_word)) return false;
        if (lane == 0) mbar_expect_tx(&k_full[kr.st], WIDE_CHUNK);
        __syncwarp();
        load_chunk(Ks + kr.st * WIDE_CHUNK, &tmap_k, &k_full[kr.st], c * 64, hk, off, blk, parts, rpl, lane);
      }
      return true;
    };
    int blk = block_of(0), blk_next = block_of(1);
    if (!load_k(0, blk)) goto done;
    for (int j = 0; j < n; j++) {
      const int blk_after = block_of(j + 2);
      if (j + 1 < n && !load_k(j + 1, blk_next)) goto done;
      if (!mbar_wait(&v_empty[vr.st], vr.ph ^ 1u, abort_word)) goto done;
      if (lane == 0) mbar_expect_tx(&v_full[vr.st], V_BYTES);
      __syncwarp();
      const int off = page_row(j);
#pragma unroll
      for (int hf = 0; hf < NV; hf++)
        load_chunk(Vs + vr.st * V_BYTES + hf * WIDE_CHUNK, &tmap_v, &v_full[vr.st], hf * 64, h, off, blk, parts, rpl, lane);
      vr.next(VST);
      blk = blk_next;
      blk_next = blk_after;
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_s = make_idesc_f16(128, 128, true, false, false);
    constexpr uint32_t idesc_o = make_idesc_f16(128, NV * 64, true, false, true);
    const uint64_t q_desc = make_smem_desc(smem_u32(Qs), 16, 1024, kLayoutSw128);
    const uint64_t k_desc = make_smem_desc(smem_u32(Ks), 16, 1024, kLayoutSw128);
    const uint64_t v_desc = make_smem_desc(smem_u32(Vs), WIDE_CHUNK, 1024, kLayoutSw128);
    if (!mbar_wait(q_full, 0, abort_word)) goto done;
    Ring kr, vr;
    auto issue_s = [&](int j) -> bool {
      const int b = j & 1;
      if (!mbar_wait(&s_free[b], (((uint32_t)j >> 1) & 1u) ^ 1u, abort_word)) return false;
      for (int c = 0; c < NC; c++, kr.next(KST)) {
        const int st = kr.st;
        if (!mbar_wait(&k_full[st], kr.ph, abort_word)) return false;
        tc_fence_after();
        if (lane == 0) {
          const uint64_t da = desc_at(q_desc, c * WIDE_CHUNK), db = desc_at(k_desc, st * WIDE_CHUNK);
#pragma unroll
          for (int kk = 0; kk < 4; kk++)
            umma_f16_ss(tmem_base + b * 128, da + 2 * kk, db + 2 * kk, idesc_s, c > 0 || kk > 0 ? 1u : 0u);
          umma_commit(&k_empty[st]);
          if (c == NC - 1) umma_commit(&s_ready[b]);
        }
        __syncwarp();
      }
      return true;
    };
    if (!issue_s(0)) goto done;
    for (int j = 0; j < n; j++) {
      if (j + 1 < n && !issue_s(j + 1)) goto done;
      const int st = vr.st, pb = j & 1;
      if (!mbar_wait(&v_full[st], vr.ph, abort_word)) goto done;
      vr.next(VST);
      if (!mbar_wait(&p_ready[pb], ((uint32_t)j >> 1) & 1u, abort_word)) goto done;
      tc_fence_after();
      if (lane == 0) {
        const uint64_t db = desc_at(v_desc, st * V_BYTES);
#pragma unroll
        for (int kk = 0; kk < 8; kk++)
          umma_f16_ts(tmem_base + O_COL, tmem_base + P_COL + pb * 64 + kk * 8, db + 128 * kk, idesc_o,
                      j > 0 || kk > 0 ? 1u : 0u);
        umma_commit(&v_empty[st]);
        umma_commit(&pv_done[pb]);
      }
      __syncwarp();
    }
  } else {
    // ------------------------------------------------------------ softmax / epilogue
    const int qd = warp & 3, row = qd * 32 + lane, tok = row / G, g = row % G;
    const bool row_valid = tok < ntok;
    const int q_pos = ctx + tok0 + tok, hi = min(seq_len, q_pos + 1);           // keys [lo, hi) are visible to this row
    const int lo = p.window > 0 ? max(0, q_pos - p.window + 1) : 0;
    const uint32_t t_lane = tmem_base + ((uint32_t)(qd * 32) << 16);
    const float sl2 = p.scale_log2;
    // a negative scale turns the order of the products around
    const float sign = sl2 < 0.f ? -1.f : 1.f, asl2 = fabsf(sl2);
    float m = -INFINITY, l = 0.f;
    for (int j = 0; j < n; j++) {
      const int b = j & 1;
      if (!mbar_wait(&s_ready[b], ((uint32_t)j >> 1) & 1u, abort_word)) goto done;
      tc_fence_after();
      const int tile_base = (t0 + j) << 7;
      const bool need_mask = tile_base + 128 > min(seq_len, ctx + tok0 + 1) ||
                             (p.window > 0 && tile_base <= ctx + tok0 + ntok - 1 - p.window);
      uint32_t sreg[128];
      tmem_ld_32x32b_x32(t_lane + b * 128, sreg);
      tmem_ld_32x32b_x32(t_lane + b * 128 + 32, sreg + 32);
      tmem_ld_32x32b_x32(t_lane + b * 128 + 64, sreg + 64);
      tmem_ld_32x32b_x32(t_lane + b * 128 + 96, sreg + 96);
      tmem_ld_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_free[b]);
      if (sl2 < 0.f) {
#pragma unroll
        for (int i = 0; i < 128; i++) sreg[i] = __float_as_uint(sign * __uint_as_float(sreg[i]));
      }
      if (need_mask) {
#pragma unroll
        for (int i = 0; i < 128; i++)
          if (tile_base + i < lo || tile_base + i >= hi) sreg[i] = 0xff800000u;   // -inf
      }
      float mx0 = -INFINITY, mx1 = -INFINITY, mx2 = -INFINITY, mx3 = -INFINITY;
#pragma unroll
      for (int i = 0; i < 128; i += 4) {
        mx0 = fmaxf(mx0, __uint_as_float(sreg[i]));
        mx1 = fmaxf(mx1, __uint_as_float(sreg[i + 1]));
        mx2 = fmaxf(mx2, __uint_as_float(sreg[i + 2]));
        mx3 = fmaxf(mx3, __uint_as_float(sreg[i + 3]));
      }
      const float mx = fmaxf(fmaxf(mx0, mx1), fmaxf(mx2, mx3));
      float alpha = 1.f;
      bool need = false;
      if (mx > m && (m == -INFINITY || (mx - m) * asl2 > kWideRescale)) {
        alpha = m == -INFINITY ? 0.f : score_exp2((m - mx) * asl2);
        need = j > 0 && m != -INFINITY;         // an all-masked row has accumulated zeros only
        m = mx;
      }
      l *= alpha;
      const bool warp_need = __any_sync(0xffffffffu, need && row_valid);
      // the P buffer was last read by PV(j - 2); O must be quiescent only for a rescale
      if (j >= 2 && !mbar_wait(&pv_done[j & 1], (((uint32_t)j - 2) >> 1) & 1u, abort_word)) goto done;
      if (warp_need) {
        if (!mbar_wait(&pv_done[(j - 1) & 1], (((uint32_t)j - 1) >> 1) & 1u, abort_word)) goto done;
        tc_fence_after();
        const float a = need ? alpha : 1.f;
#pragma unroll 1
        for (int c = 0; c < NV * 2; c++) {
          uint32_t r[32];
          tmem_ld_32x32b_x32(t_lane + O_COL + c * 32, r);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 32; i++) r[i] = __float_as_uint(__uint_as_float(r[i]) * a);
          tmem_st_32x32b_x32(t_lane + O_COL + c * 32, r);
        }
        tmem_st_wait();
      }
      // ---- probabilities, two keys to a column -> TMEM (A operand of P V)
      tc_fence_after();
      const float nmb = m == -INFINITY ? 0.f : -m * asl2;
      float rs0 = 0.f, rs1 = 0.f;
#pragma unroll
      for (int hf = 0; hf < 2; hf++) {
        uint32_t pk[32];
#pragma unroll
        for (int i = 0; i < 32; i++) {
          const float p0 = score_exp2(fmaf(__uint_as_float(sreg[hf * 64 + 2 * i]), asl2, nmb));
          const float p1 = score_exp2(fmaf(__uint_as_float(sreg[hf * 64 + 2 * i + 1]), asl2, nmb));
          rs0 += p0;
          rs1 += p1;
          pk[i] = pack_bf16x2(p0, p1);
        }
        tmem_st_32x32b_x32(t_lane + P_COL + b * 64 + hf * 32, pk);
      }
      l += rs0 + rs1;
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_ready[b]);
    }
    if (!mbar_wait(&pv_done[(n - 1) & 1], (((uint32_t)n - 1) >> 1) & 1u, abort_word)) goto done;
    tc_fence_after();
    const long at = ((long)q_start + tok0 + tok) * p.out_stride + (long)(h * G + g) * p.Dv;
    const float inv = l > 0.f ? p.out_scale / l : 0.f;
#pragma unroll 1
    for (int c = 0; c < NV * 2; c++) {
      uint32_t r[32];
      tmem_ld_32x32b_x32(t_lane + O_COL + c * 32, r);
      tmem_ld_wait();
      if (!row_valid) continue;
#pragma unroll
      for (int q4 = 0; q4 < 4; q4++) {             // Dv is a multiple of 8
        if (c * 32 + q4 * 8 >= p.Dv) break;
        float v[8];
#pragma unroll
        for (int e = 0; e < 8; e++) v[e] = __uint_as_float(r[q4 * 8 + e]) * inv;
        if (p.out_f32) {
          float4* dst = reinterpret_cast<float4*>((float*)p.out + at + c * 32 + q4 * 8);
          dst[0] = make_float4(v[0], v[1], v[2], v[3]);
          dst[1] = make_float4(v[4], v[5], v[6], v[7]);
        } else {
          *reinterpret_cast<uint4*>((__nv_bfloat16*)p.out + at + c * 32 + q4 * 8) =
              make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
        }
      }
    }
  }
done:
  wide_finish(abort_word, p.status, tmem_base, warp);
}

// ---------------------------------------------------------------- decode
struct WideItem {
  int kh, seq, split, row, seq_len, t0, n, lo;         // visible keys [lo, seq_len), tiles t0 .. t0 + n - 1
};

__device__ __forceinline__ WideItem wide_item(const WideParams& p, int item) {
  WideItem w;
  w.kh = item % p.key_heads;
  const int q = item / p.key_heads;
  w.seq = q % p.num_seqs;
  w.split = q / p.num_seqs;
  w.row = p.cu[w.seq];
  const int q_len = p.cu[w.seq + 1] - w.row;
  w.seq_len = p.seq_lens[w.seq];
  w.lo = p.window > 0 ? max(0, w.seq_len - p.window) : 0;
  const int first = w.lo >> 7, n_all = ((w.seq_len + 127) >> 7) - first;
  const int per = (n_all + p.num_splits - 1) / p.num_splits;
  w.t0 = first + w.split * per;
  w.n = q_len > 0 ? max(0, min(n_all, (w.split + 1) * per) - w.split * per) : 0;
  return w;
}

__device__ __forceinline__ void wide_softmax_bar() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// NQ: columns of S^T (heads of a key head, padded), 16 or 32
template <int NQ>
__global__ void __launch_bounds__(WIDE_THREADS, 1)
attn_wide_decode_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                        const __grid_constant__ CUtensorMap tmap_v, const WideParams p) {
  constexpr int QC = NQ * 128;                  // a chunk of the queries: NQ rows x 64 bf16
  constexpr int P_BYTES = 2 * QC;               // two 64-key halves
  constexpr int V_BYTES = 2 * WIDE_CHUNK;       // 128 keys x one value head, padded to 128 dimensions
  constexpr int O_COL = 2 * NQ;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int NC = p.chunks, KST = p.k_stages, VST = p.v_stages;
  const int VH = p.Hkv / p.key_heads, C = p.Hq / p.key_heads, GV = C / VH;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* Ks = (uint8_t*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
  uint8_t* Vs = Ks + KST * WIDE_CHUNK;
  uint8_t* Qs = Vs + VST * V_BYTES;
  uint8_t* Ps = Qs + NC * QC;
  uint64_t* k_full = (uint64_t*)(Ps + 2 * P_BYTES);
  uint64_t* k_empty = k_full + WIDE_RING;
  uint64_t* v_full = k_empty + WIDE_RING;       // 2 each from here on
  uint64_t* v_empty = v_full + 2;
  uint64_t* s_ready = v_empty + 2;
  uint64_t* s_free = s_ready + 2;
  uint64_t* p_ready = s_free + 2;
  uint64_t* pv_done = p_ready + 2;
  uint64_t* q_full = pv_done + 2;               // 1 each
  uint64_t* q_empty = q_full + 1;
  uint64_t* o_free = q_empty + 1;
  uint32_t* tmem_ptr = (uint32_t*)(o_free + 1);
  volatile int* abort_word = (volatile int*)(tmem_ptr + 1);
  int* redi = (int*)(tmem_ptr + 2);             // [2 tiles][4 warps][NQ] maxima
  float* red_sum = (float*)(redi + 8 * NQ);     // [4 warps][NQ]
  // rows of the queries beyond the heads, and dimensions of a value beyond its size, must be finite
  for (int i = threadIdx.x; i < (NC * QC) / 16; i += WIDE_THREADS)
    reinterpret_cast<uint4*>(Qs)[i] = make_uint4(0u, 0u, 0u, 0u);
  fence_proxy_async_smem();
  if (threadIdx.x == 0) {
    for (int s = 0; s < KST; s++) {
      mbar_init(&k_full[s], 1);
      mbar_init(&k_empty[s], 1);
    }
    for (int b = 0; b < 2; b++) {
      mbar_init(&v_full[b], 1);
      mbar_init(&v_empty[b], 1);
      mbar_init(&s_ready[b], 1);
      mbar_init(&s_free[b], 4);
      mbar_init(&p_ready[b], 4);
      mbar_init(&pv_done[b], 1);
    }
    mbar_init(q_full, 1);
    mbar_init(q_empty, 1);
    mbar_init(o_free, 4);
    *abort_word = 0;
    mbar_fence_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_ptr, 512);
    tmem_relinquish();
  }
  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_k);
    tma_prefetch_desc(&tmap_v);
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_ptr;
  uint32_t it = 0, gt = 0;                      // non-empty items and tiles of this CTA so far
  Ring kr, vr;

  if (warp == 0) {
    // ------------------------------------------------------------ producer, in the order of consumption
    const int rpl = p.rows_per_load, parts = 128 / rpl;
    for (int item = blockIdx.x; item < p.num_items; item += gridDim.x) {
      const WideItem w = wide_item(p, item);
      if (w.n <= 0) continue;
      const int* bt = p.block_table + (long)w.seq * p.max_blocks;
      auto block_of = [&](int j) -> int {
        if (j >= w.n || lane >= parts) return 0;
        return bt[min(((w.t0 + j) << 7) + lane * rpl, w.seq_len - 1) / p.block_size];
      };
      auto page_row = [&](int j) { return p.block_size > 128 ? ((w.t0 + j) << 7) % p.block_size : 0; };
      auto load_k = [&](int j, int blk) -> bool {
        if (__any_sync(0xffffffffu, (blk < 0 || blk >= p.num_blocks_total) && lane < parts)) {
          *abort_word = B200_BAD_INDEX;
          return false;
        }
        const int off = page_row(j);
        for (int c = 0; c < NC; c++, kr.next(KST)) {
          if (!mbar_wait(&k_empty[kr.st], kr.ph ^ 1u, abort_word)) return false;
          if (lane == 0) mbar_expect_tx(&k_full[kr.st], WIDE_CHUNK);
          __syncwarp();
          load_chunk(Ks + kr.st * WIDE_CHUNK, &tmap_k, &k_full[kr.st], c * 64, w.kh, off, blk, parts, rpl, lane);
        }
        return true;
      };
      int blk = block_of(0), blk_next = block_of(1);
      if (!mbar_wait(q_empty, (it & 1u) ^ 1u, abort_word)) goto done;
      if (lane == 0) {
        mbar_expect_tx(q_full, NC * 128 * C);
        for (int c = 0; c < NC; c++) tma_load_4d(Qs + c * QC, &tmap_q, q_full, c * 64, 0, w.kh, w.row);
      }
      __syncwarp();
      if (!load_k(0, blk)) goto done;
      for (int j = 0; j < w.n; j++) {
        const int blk_after = block_of(j + 2);
        if (j + 1 < w.n && !load_k(j + 1, blk_next)) goto done;
        const int off = page_row(j);
        for (int v = 0; v < VH; v++, vr.next(VST)) {
          if (!mbar_wait(&v_empty[vr.st], vr.ph ^ 1u, abort_word)) goto done;
          if (lane == 0) mbar_expect_tx(&v_full[vr.st], V_BYTES);
          __syncwarp();
          for (int hf = 0; hf < 2; hf++)
            load_chunk(Vs + vr.st * V_BYTES + hf * WIDE_CHUNK, &tmap_v, &v_full[vr.st], hf * 64, w.kh * VH + v, off, blk, parts,
                       rpl, lane);
        }
        blk = blk_next;
        blk_next = blk_after;
      }
      it++;
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    constexpr uint32_t idesc_s = make_idesc_f16(128, NQ, true, false, false);
    constexpr uint32_t idesc_o = make_idesc_f16(128, NQ, true, true, false);      // A = V, MN-major
    const uint64_t q_desc = make_smem_desc(smem_u32(Qs), 16, 1024, kLayoutSw128);
    const uint64_t k_desc = make_smem_desc(smem_u32(Ks), 16, 1024, kLayoutSw128);
    const uint64_t v_desc = make_smem_desc(smem_u32(Vs), WIDE_CHUNK, 1024, kLayoutSw128);
    const uint64_t p_desc = make_smem_desc(smem_u32(Ps), 16, 1024, kLayoutSw128);
    for (int item = blockIdx.x; item < p.num_items; item += gridDim.x) {
      const WideItem w = wide_item(p, item);
      if (w.n <= 0) continue;
      if (!mbar_wait(q_full, it & 1u, abort_word)) goto done;
      if (!mbar_wait(o_free, (it & 1u) ^ 1u, abort_word)) goto done;      // read out by the previous item's epilogue
      auto issue_s = [&](int j) -> bool {
        const uint32_t g = gt + (uint32_t)j;
        const int b = g & 1;
        if (!mbar_wait(&s_free[b], ((g >> 1) & 1u) ^ 1u, abort_word)) return false;
        for (int c = 0; c < NC; c++, kr.next(KST)) {
          const int st = kr.st;
          if (!mbar_wait(&k_full[st], kr.ph, abort_word)) return false;
          tc_fence_after();
          if (lane == 0) {
            const uint64_t da = desc_at(k_desc, st * WIDE_CHUNK), db = desc_at(q_desc, c * QC);
#pragma unroll
            for (int kk = 0; kk < 4; kk++)
              umma_f16_ss(tmem_base + b * NQ, da + 2 * kk, db + 2 * kk, idesc_s, c > 0 || kk > 0 ? 1u : 0u);
            umma_commit(&k_empty[st]);
            if (c == NC - 1) {
              umma_commit(&s_ready[b]);
              if (j == w.n - 1) umma_commit(q_empty);          // last read of this item's Q
            }
          }
          __syncwarp();
        }
        return true;
      };
      if (!issue_s(0)) goto done;
      for (int j = 0; j < w.n; j++) {
        if (j + 1 < w.n && !issue_s(j + 1)) goto done;
        const uint32_t g = gt + (uint32_t)j;
        const int pb = g & 1;
        if (!mbar_wait(&p_ready[pb], (g >> 1) & 1u, abort_word)) goto done;
        for (int v = 0; v < VH; v++, vr.next(VST)) {
          const int st = vr.st;
          if (!mbar_wait(&v_full[st], vr.ph, abort_word)) goto done;
          tc_fence_after();
          if (lane == 0) {
            // A: 16 keys of V^T (two 64-wide d atoms a chunk apart, 8-key groups 1024 B apart)
            const uint64_t da = desc_at(v_desc, st * V_BYTES), db = desc_at(p_desc, pb * P_BYTES);
#pragma unroll
            for (int kk = 0; kk < 8; kk++)
              umma_f16_ss(tmem_base + O_COL + v * NQ, da + 128 * kk, db + (kk >> 2) * (QC >> 4) + 2 * (kk & 3), idesc_o,
                          j > 0 || kk > 0 ? 1u : 0u);
            umma_commit(&v_empty[st]);
            if (v == VH - 1) umma_commit(&pv_done[pb]);
          }
          __syncwarp();
        }
      }
      gt += (uint32_t)w.n;
      it++;
    }
  } else {
    // ------------------------------------------------------------ softmax / epilogue
    const int qd = warp & 3, tid = qd * 32 + lane;         // key inside the tile; dimension of a value
    const uint32_t t_lane = tmem_base + ((uint32_t)(qd * 32) << 16);
    const float sign = p.scale_log2 < 0.f ? -1.f : 1.f, sl2 = fabsf(p.scale_log2);
    for (int item = blockIdx.x; item < p.num_items; item += gridDim.x) {
      const WideItem w = wide_item(p, item);
      if (w.n <= 0) {
        if (p.num_splits > 1) {                            // an empty split still owns its partial slots
          for (int c = 0; c < C; c++) {
            const long pidx = ((long)w.seq * p.Hq + w.kh * C + c) * p.num_splits + w.split;
            if (tid == 0) p.partial_lse[pidx] = -INFINITY;
            if (tid < p.Dv) p.partial_o[pidx * p.Dv + tid] = 0.f;
          }
        }
        continue;
      }
      float m[NQ], lsum[NQ];
#pragma unroll
      for (int c = 0; c < NQ; c++) {
        m[c] = -INFINITY;
        lsum[c] = 0.f;
      }
      for (int j = 0; j < w.n; j++) {
        const uint32_t g = gt + (uint32_t)j;
        const int b = g & 1, key = ((w.t0 + j) << 7) + tid;
        if (!mbar_wait(&s_ready[b], (g >> 1) & 1u, abort_word)) goto done;
        tc_fence_after();
        uint32_t r[NQ];
#pragma unroll
        for (int c = 0; c < NQ; c += 16) tmem_ld_32x32b_x16(t_lane + b * NQ + c, r + c);
        tmem_ld_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&s_free[b]);
        const bool seen = key >= w.lo && key < w.seq_len;
        float s[NQ];
        int* rj = redi + b * 4 * NQ + qd * NQ;
#pragma unroll
        for (int c = 0; c < NQ; c++) {
          s[c] = seen ? sign * __uint_as_float(r[c]) : -INFINITY;
          if (c < C) {
            int ob = __float_as_int(s[c]);
            ob ^= (ob >> 31) & 0x7fffffff;                 // order-preserving float -> int
            const int wm = __reduce_max_sync(0xffffffffu, ob);
            if (lane == 0) rj[c] = wm;
          }
        }
        wide_softmax_bar();
        const int* ra = redi + b * 4 * NQ;
        bool any_change = false;
        float alpha[NQ];
#pragma unroll
        for (int c = 0; c < NQ; c++) {
          alpha[c] = 1.f;
          if (c >= C) continue;
          int t = max(max(ra[c], ra[NQ + c]), max(ra[2 * NQ + c], ra[3 * NQ + c]));
          t ^= (t >> 31) & 0x7fffffff;
          const float mn = fmaxf(m[c], __int_as_float(t));
          if (mn > m[c] && (m[c] == -INFINITY || (mn - m[c]) * sl2 > kWideRescale)) {
            alpha[c] = m[c] == -INFINITY ? 0.f : score_exp2((m[c] - mn) * sl2);
            any_change = any_change || m[c] != -INFINITY;
            m[c] = mn;
          }
          lsum[c] *= alpha[c];
        }
        // the P buffer was last read by the products of two tiles ago (possibly of the previous item)
        if (g >= 2 && !mbar_wait(&pv_done[b], ((g - 2) >> 1) & 1u, abort_word)) goto done;
        if (j > 0 && any_change) {                         // uniform over the 128 threads: O^T must be quiescent
          if (!mbar_wait(&pv_done[(g - 1) & 1], ((g - 1) >> 1) & 1u, abort_word)) goto done;
          tc_fence_after();
          for (int v = 0; v < VH; v++) {
            uint32_t o[NQ];
#pragma unroll
            for (int c = 0; c < NQ; c += 16) tmem_ld_32x32b_x16(t_lane + O_COL + v * NQ + c, o + c);
            tmem_ld_wait();
#pragma unroll
            for (int c = 0; c < NQ; c++) o[c] = __float_as_uint(__uint_as_float(o[c]) * alpha[c]);
#pragma unroll
            for (int c = 0; c < NQ; c += 16) tmem_st_32x32b_x16(t_lane + O_COL + v * NQ + c, o + c);
            tmem_st_wait();
          }
        }
        // probabilities of this key for every column -> P[c][key] (K-major, swizzled)
        uint8_t* pbase = Ps + b * P_BYTES + (tid >> 6) * QC;
        const int kin = tid & 63;
#pragma unroll
        for (int c = 0; c < NQ; c++) {
          const float pv = c < C && seen ? score_exp2((s[c] - m[c]) * sl2) : 0.f;
          lsum[c] += pv;
          *reinterpret_cast<__nv_bfloat16*>(pbase + c * 128 + (((kin >> 3) ^ (c & 7)) << 4) + (kin & 7) * 2) =
              __float2bfloat16(pv);
        }
        tc_fence_before();
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_ready[b]);
      }
      gt += (uint32_t)w.n;
      {
        const uint32_t gl = gt - 1;
        if (!mbar_wait(&pv_done[gl & 1], (gl >> 1) & 1u, abort_word)) goto done;
      }
      tc_fence_after();
#pragma unroll
      for (int c = 0; c < NQ; c++) {
        const float ws = warp_reduce_sum(lsum[c]);
        if (lane == 0) red_sum[qd * NQ + c] = ws;
      }
      wide_softmax_bar();
#pragma unroll
      for (int c = 0; c < NQ; c++) lsum[c] = red_sum[c] + red_sum[NQ + c] + red_sum[2 * NQ + c] + red_sum[3 * NQ + c];
      for (int v = 0; v < VH; v++) {
        uint32_t o[NQ];
#pragma unroll
        for (int c = 0; c < NQ; c += 16) tmem_ld_32x32b_x16(t_lane + O_COL + v * NQ + c, o + c);
        tmem_ld_wait();
        if (tid >= p.Dv) continue;
#pragma unroll
        for (int c = 0; c < NQ; c++) {
          if (c / GV != v) continue;                       // columns of this value head (none beyond the heads)
          const float l = lsum[c], inv = l > 0.f ? 1.f / l : 0.f, val = __uint_as_float(o[c]) * inv;
          const int hq = w.kh * C + c;
          if (p.num_splits == 1) {
            store_out(p, (long)w.row * p.out_stride + (long)hq * p.Dv + tid, val * p.out_scale);
          } else {
            const long pidx = ((long)w.seq * p.Hq + hq) * p.num_splits + w.split;
            p.partial_o[pidx * p.Dv + tid] = val;
            if (tid == 0) p.partial_lse[pidx] = l > 0.f ? m[c] * sl2 * 0.6931471805599453f + logf(l) : -INFINITY;
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(o_free);
      // the next item's epilogue overwrites red_sum only after a softmax_bar of its tile loop
    }
  }
done:
  wide_finish(abort_word, p.status, tmem_base, warp);
}

// ---------------------------------------------------------------- host
static std::unordered_map<std::string, CUtensorMap> g_wide_maps;
static std::mutex g_wide_mu;

static int wide_map(CUtensorMap* out, const void* base, const uint64_t* dims, const uint64_t* strides, const uint32_t* box) {
  char key[80];
  memcpy(key, &base, 8);
  memcpy(key + 8, dims, 32);
  memcpy(key + 40, strides, 24);
  memcpy(key + 64, box, 16);
  const std::string k(key, 80);
  std::lock_guard<std::mutex> g(g_wide_mu);
  auto it = g_wide_maps.find(k);
  if (it == g_wide_maps.end()) {
    CUtensorMap m;
    const int rc = make_tmap(&m, base, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, dims, strides, box, CU_TENSOR_MAP_SWIZZLE_128B);
    if (rc) return rc;
    if (g_wide_maps.size() > 4096) g_wide_maps.clear();
    it = g_wide_maps.emplace(k, m).first;
  }
  *out = it->second;
  return 0;
}

// the rows of a box are consecutive in the map's second dimension
static int cache_map(CUtensorMap* out, const AttnVariantArgs* a, bool values, int rows) {
  uint64_t dims[4] = {(uint64_t)(values ? a->Dv : a->D), (uint64_t)a->block_size, (uint64_t)(values ? a->Hkv : a->key_heads),
                      (uint64_t)a->num_blocks};
  uint64_t str[3] = {(uint64_t)(values ? a->v_tok : a->k_tok) * 2, (uint64_t)(values ? a->v_head : a->k_head) * 2,
                     (uint64_t)(values ? a->v_block : a->k_block) * 2};
  uint32_t box[4] = {64, (uint32_t)rows, 1, 1};
  return wide_map(out, values ? a->v_cache : a->k_cache, dims, str, box);
}

static int wide_params(const AttnVariantArgs* a, int* status, WideParams& p) {
  if (a->Hkv < 1 || a->Hq % a->Hkv || a->key_heads < 1 || a->Hkv % a->key_heads || a->dtype != 0) return 9880;
  if (a->D < 8 || a->D % 8 || a->D > 64 * WIDE_RING || a->Dv < 8 || a->Dv > 128 || a->Dv % 8) return 9881;
  const int bs = a->block_size;
  if (bs < 8 || (bs < 128 && 128 % bs) || (bs > 128 && bs % 128)) return 9882;
  if ((a->q_stride & 7) || (a->out_stride & 7) || a->bias || a->sink || a->gate || a->softcap > 0.f) return 9883;
  if (a->window > 0 && a->keep_first > 0) return 9884;
  p = {};
  p.cu = a->cu; p.seq_lens = a->seq_lens; p.block_table = a->block_table;
  p.max_blocks = a->max_blocks; p.block_size = bs; p.rows_per_load = bs < 128 ? bs : 128;
  p.G = a->Hq / a->Hkv; p.Hkv = a->Hkv; p.Hq = a->Hq; p.key_heads = a->key_heads; p.Dv = a->Dv;
  p.num_seqs = a->num_seqs; p.window = a->window; p.num_splits = 1;
  p.chunks = (a->D + 63) / 64;
  p.scale_log2 = a->scale * kLog2e; p.out_scale = a->out_scale;
  p.out_f32 = a->out_f32; p.out = a->out; p.out_stride = a->out_stride;
  p.num_blocks_total = a->num_blocks;
  p.status = status;
  return 0;
}

template <typename K>
static int allow_smem(K kernel, bool* done) {
  if (*done) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, WIDE_SMEM);
  if (e != cudaSuccess) return (int)e;
  *done = true;
  return 0;
}

template <int NV>
static int launch_wide(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const WideParams& p, int tiles,
                       cudaStream_t stream) {
  static bool set = false;
  const int rc = allow_smem(attn_wide_kernel<NV>, &set);
  if (rc) return rc;
  const int bytes = (p.chunks + p.k_stages + NV * p.v_stages) * WIDE_CHUNK + 1024 + 512;
  if (bytes > WIDE_SMEM) return 9886;
  attn_wide_kernel<NV><<<dim3((unsigned)p.Hkv, (unsigned)tiles), WIDE_THREADS, bytes, stream>>>(tq, tk, tv, p);
  return B200_CHECK_LAUNCH();
}

template <int NQ>
static int launch_wide_decode(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, WideParams& p,
                              cudaStream_t stream) {
  static bool set = false;
  const int rc = allow_smem(attn_wide_decode_kernel<NQ>, &set);
  if (rc) return rc;
  const int fixed = p.chunks * NQ * 128 + 2 * NQ * 256 + 1024 + 1024 + 12 * NQ * 4;
  p.v_stages = 2;
  p.k_stages = (WIDE_SMEM - fixed - 4 * WIDE_CHUNK) / WIDE_CHUNK;
  if (p.k_stages > WIDE_RING) p.k_stages = WIDE_RING;
  if (p.k_stages < 2) return 9887;
  const int bytes = fixed + (4 + p.k_stages) * WIDE_CHUNK;
  const int grid = p.num_items < num_sms() ? p.num_items : num_sms();
  attn_wide_decode_kernel<NQ><<<grid, WIDE_THREADS, bytes, stream>>>(tq, tk, tv, p);
  return B200_CHECK_LAUNCH();
}

}  // namespace b200

// rows of several tokens per sequence; at most 128 query heads on one value head, keys of up to 512 dimensions
B200_API int b200_attention_wide_prefill(const b200::AttnVariantArgs* a, int* status, cudaStream_t stream) {
  using namespace b200;
  if (a->tokens <= 0 || a->num_seqs <= 0) return 0;
  WideParams p;
  int rc = wide_params(a, status, p);
  if (rc) return rc;
  if (p.G > 128 || p.chunks > 8) return 9885;
  p.tok_per_tile = 128 / p.G;
  const int NV = a->Dv > 64 ? 2 : 1, left = 14 - p.chunks;      // chunks of shared memory beside the queries
  p.v_stages = left >= 2 * NV + 6 ? 2 : 1;
  p.k_stages = left - NV * p.v_stages;
  CUtensorMap tq, tk, tv;
  {
    uint64_t dims[4] = {(uint64_t)a->D, (uint64_t)p.G, (uint64_t)p.Hkv, (uint64_t)a->tokens};
    uint64_t str[3] = {(uint64_t)a->D * 2, (uint64_t)p.G * a->D * 2, (uint64_t)a->q_stride * 2};
    uint32_t box[4] = {64, (uint32_t)p.G, 1, (uint32_t)p.tok_per_tile};
    rc = wide_map(&tq, a->q, dims, str, box);
  }
  if (!rc) rc = cache_map(&tk, a, false, p.rows_per_load);
  if (!rc) rc = cache_map(&tv, a, true, p.rows_per_load);
  if (rc) return rc;
  const long tiles = a->tokens / p.tok_per_tile + a->num_seqs;
  if (tiles > 65535) return 9888;
  return NV == 2 ? launch_wide<2>(tq, tk, tv, p, (int)tiles, stream) : launch_wide<1>(tq, tk, tv, p, (int)tiles, stream);
}

// one query row per sequence (row b of q belongs to sequence b); at most 32 query heads on one key head
B200_API int b200_attention_wide_decode(const b200::AttnVariantArgs* a, int* status, cudaStream_t stream) {
  using namespace b200;
  if (a->tokens <= 0 || a->num_seqs <= 0) return 0;
  WideParams p;
  int rc = wide_params(a, status, p);
  if (rc) return rc;
  const int C = p.Hq / p.key_heads, VH = p.Hkv / p.key_heads, NQ = C <= 16 ? 16 : 32;
  if (C > 32 || (2 + VH) * NQ > 512 || a->tokens < a->num_seqs) return 9890;
  if (a->num_splits < 1 || (a->num_splits > 1 && !a->scratch)) return 9891;
  p.num_splits = a->num_splits;
  p.partial_o = a->scratch;
  p.partial_lse = a->scratch ? a->scratch + (long)a->num_seqs * a->Hq * (long)a->num_splits * a->Dv : nullptr;
  const long items = (long)p.key_heads * p.num_seqs * p.num_splits;
  if (items > 0x7fffffffL) return 9892;
  p.num_items = (int)items;
  CUtensorMap tq, tk, tv;
  {
    uint64_t dims[4] = {(uint64_t)a->D, (uint64_t)C, (uint64_t)p.key_heads, (uint64_t)a->tokens};
    uint64_t str[3] = {(uint64_t)a->D * 2, (uint64_t)C * a->D * 2, (uint64_t)a->q_stride * 2};
    uint32_t box[4] = {64, (uint32_t)C, 1, 1};
    rc = wide_map(&tq, a->q, dims, str, box);
  }
  if (!rc) rc = cache_map(&tk, a, false, p.rows_per_load);
  if (!rc) rc = cache_map(&tv, a, true, p.rows_per_load);
  if (rc) return rc;
  rc = NQ == 16 ? launch_wide_decode<16>(tq, tk, tv, p, stream) : launch_wide_decode<32>(tq, tk, tv, p, stream);
  if (rc || p.num_splits == 1) return rc;
  return launch_merge_splits(p.partial_o, p.partial_lse, a->num_seqs, a->Hq, p.num_splits, a->Dv, a->out, a->out_stride,
                             stream, nullptr, 0, nullptr, nullptr, 0, a->out_f32, a->out_scale);
}
