// Attention over the paged cache whose heads mix their scores before the softmax: the arguments its kernels share.
//
//   a_g  = scale * (q_g . k)                         of score head g and a key `dist` tokens back
//   a_g <- softcap * tanh(a_g / softcap)             (softcap 0: none)
//   a_g <- a_g - r1_g * ln(1 + r2_g * dist)          (r1 null: none)
//   s_h  = sum_g talk[h, g] a_g                      for every output head h
//   p_h  = exp(s_h) / (exp(sink_h) + sum exp(s_h))   over the keys at or before the query (sink null: plain softmax)
//   out  = sum p_h v
//
// Score head g reads key head g / (Hs / Hk), output head h value head h / (Ho / Hv).  All of it is fp32 but the
// products, whose operands may be bf16.  The cache rows are padded to DP / DVP elements; the padding holds zeros.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

namespace b200 {

struct MixedAttnParams {
  const void* q;               // [T, Hs * D], row pitch q_stride
  const void* k_cache;         // [blocks, Hk, block_size, DP]
  const void* v_cache;         // [blocks, Hv, block_size, DVP]
  void* out;                   // [T, >= Ho * DV], row pitch out_stride
  const int* block_tables;     // [B, max_blocks]
  const int* cu_q;             // [B + 1]; null: every sequence has q_len rows
  const int* seq_lens;         // [B] keys including this step's
  const float* r1;             // [Hs] or null
  const float* r2;
  const float* talk;           // [Ho, Hs]
  const float* sink;           // [Ho] or null
  int B, rows, q_len, max_blocks, block_size;
  int bs_shift;                // log2(block_size), -1 when it is not a power of two
  int Hs, Hk, Ho, Hv, D, DV, DP, DVP;
  long long q_stride, out_stride;
  float scale, softcap;
  int splits;                  // decode: CTAs that share a row's keys
  float* scratch;              // decode: [rows, splits, Ho, DVP], then [rows, splits, Ho, 2]; prompts: see pitch
  // prompts: portions are cut into tiles of 16 queries, numbered through all sequences; this call makes tiles
  // tile0 .. tile0 + tiles - 1, whose mixed scores (times log2 e) are [tiles, 16, Ho, pitch]
  int tile0, tiles, max_q_len, max_keys;
  int range;                   // keys of a score CTA
  int talk_terms;              // 1: bf16 holds every element of talk exactly, 3: it does not
  long long pitch;
};

// Index of the key's row in a cache with `heads` heads.
__device__ __forceinline__ long long cache_row(const MixedAttnParams& p, const int* bt, int key, int head, int heads) {
  const int blk = p.bs_shift >= 0 ? key >> p.bs_shift : key / p.block_size;
  const int off = p.bs_shift >= 0 ? key & (p.block_size - 1) : key - blk * p.block_size;
  return (static_cast<long long>(bt[blk]) * heads + head) * p.block_size + off;
}

// The score of one head before the mixture, from the raw product; hardware exponentials and logarithms (absolute
// errors of a few 1e-7 times softcap and r1).  tanh(z) = 1 - 2 / (exp(2 z) + 1).
struct ScoreConst {
  float in;                    // capped: 2 scale / softcap * log2 e, else the scale
  float cap;                   // softcap
};
__device__ __forceinline__ ScoreConst score_const(const MixedAttnParams& p) {
  return {p.softcap > 0.f ? 2.f * 1.4426950408889634f * p.scale / p.softcap : p.scale, p.softcap};
}
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lg2_approx(float x) {
  float y;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_approx(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <bool CAP>
__device__ __forceinline__ float capped_score(const ScoreConst& c, float x) {
  if constexpr (CAP) return fmaf(-2.f * c.cap, rcp_approx(ex2_approx(x * c.in) + 1.f), c.cap);
  else return x * c.in;
}
// the same less a bias, from `start` = cap - bias (without a cap: -bias)
template <bool CAP>
__device__ __forceinline__ float biased_score(const ScoreConst& c, float x, float start) {
  if constexpr (CAP) return fmaf(-2.f * c.cap, rcp_approx(ex2_approx(x * c.in) + 1.f), start);
  else return fmaf(x, c.in, start);
}
// r1 ln(1 + r2 dist), with r1 already times ln 2
__device__ __forceinline__ float distance_bias(float r1_ln2, float r2, float dist) {
  return r1_ln2 * lg2_approx(fmaf(r2, dist, 1.f));
}
constexpr float kLn2 = 0.6931471805599453f;

}  // namespace b200
