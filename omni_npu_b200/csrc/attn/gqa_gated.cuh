// Grouped-query attention over the paged cache with a sliding window, a softmax sink without a value
// and an element-wise output gate: the arguments its kernels share.
//
//   s_j = scale * (q . k_j)                    keys 0 <= pos - j < window (window 0: all earlier keys)
//   p_j = exp(s_j) / (exp(sink) + sum exp(s))  (has_sink; without it the plain softmax)
//   out = (sum_j p_j v_j) * sigmoid(gate)      (gate null: no gate)
//
// Query and value head sizes are run-time values.  The cache rows are padded to DP / DVP elements (a
// multiple of 16); the padding holds zeros and is never written.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

namespace b200 {

struct GatedAttnParams {
  const void* q;               // [T, Hq * D] rotated queries, row pitch q_stride
  const void* gate;            // [T, Hq * DV] before the sigmoid, row pitch g_stride, or null
  const void* k_cache;         // [blocks, Hk, block_size, DP]
  const void* v_cache;         // [blocks, Hk, block_size, DVP]
  void* out;                   // [T, Hq * DV], row pitch out_stride
  const int* block_tables;     // [B, max_blocks]; with contiguous set: [B], the first row of a sequence
  int contiguous;              // keys lie in rows one after another, [keys, Hk, DP]: no blocks
  const int* cu_q;             // [B + 1]; null: every sequence has q_len rows
  const int* seq_lens;         // [B] keys including this step's
  int B, max_blocks, block_size, num_cache_blocks;
  int bs_shift;                // log2(block_size), -1 when it is not a power of two
  int Hq, Hk, D, DV, DP, DVP;
  long long q_stride, g_stride, out_stride;
  float scale_log2;            // scale * log2(e)
  int window;
  int has_sink;
  float sink_log2;             // sink score * log2(e)
  int q_len;                   // decode: rows per sequence
  int splits;                  // decode: CTAs (of one cluster) that share a sequence's keys
};

__device__ __forceinline__ float gate_sigmoid(float g) { return 1.f / (1.f + __expf(-g)); }

}  // namespace b200
