// Internal launchers shared between the attention translation units.
#pragma once
#include <cuda_runtime.h>

namespace b200 {

// lse_out (optional, [T, Hq]): log-sum-exp of the merged result; out_head: elements between the heads of
// a row of out (0: dense, D); sink (optional, [Hq]): one more term exp(sink) of the denominator; gate
// (optional, bf16 [T, Hq]): the result is scaled by its sigmoid; out_f32: out is fp32
int launch_merge_splits(const float* partial_o, const float* partial_lse, long T, int Hq,
                        int num_splits, int D, void* out, long out_stride, cudaStream_t stream,
                        float* lse_out = nullptr, long out_head = 0, const float* sink = nullptr,
                        const void* gate = nullptr, long gate_stride = 0, bool out_f32 = false, float out_scale = 1.f);

// Paged grouped-query attention with options, one launch (attention_variant.cu, attention_tc.cu,
// attention_decode_tc.cu).  Scores s = scale q.k; with softcap s = cap tanh(s / cap); with a bias table
// s += bias[h][min(distance, bias_len - 1)].  A row at position i sees j <= i with i - j < window (0: all) or
// j < keep_first.  With a sink the denominator also holds exp(sink[h]).  With a gate the output of head h is
// scaled by sigmoid(gate[t][h]).  The output is scaled by out_scale and may be fp32.  Value head g belongs to key head
// g * key_heads / Hkv.
struct AttnVariantArgs {
  const void* q;              // [T, Hq, D], heads dense
  const void *k_cache, *v_cache;
  void* out;                  // [T, Hq, Dv], heads dense
  const int *cu, *seq_lens;   // [num_seqs + 1], [num_seqs]
  const int* block_table;     // [num_seqs, max_blocks]
  const int *row_seq, *row_kv_len;     // per query row (CUDA-core kernel)
  const float* bias;          // [Hq, bias_len]
  const float* sink;          // [Hq]
  const void* gate;           // [T, Hq], row stride gate_stride
  float* scratch;             // split partials: rows * Hq * num_splits * (Dv + 1) floats
  long q_stride, out_stride, gate_stride, num_blocks, tokens;
  long k_block, k_tok, k_head, v_block, v_tok, v_head;      // cache strides in elements
  int num_seqs, max_blocks, block_size, Hq, Hkv, D, Dv;
  int window, keep_first, bias_len, num_splits, dtype, key_heads, out_f32;
  float scale, softcap, out_scale;
};

int launch_paged_decode(const void* q, long q_stride, const void* k_cache, const void* v_cache,
                        const int* block_table, int max_blocks, const int* seq_lens, int B,
                        int Hq, int Hkv, int D, int block_size, float scale, int window,
                        int num_splits, void* out, long out_stride, float* partial_o,
                        float* partial_lse, long num_blocks_total, int* status,
                        cudaStream_t stream);

}  // namespace b200
