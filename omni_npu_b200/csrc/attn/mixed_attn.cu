// Attention with mixed heads (mixed_attn.cuh): the kernel for models run in 32-bit and for sizes beyond the tensor-core
// kernels, the join of split decode rows, and the entry points.  Compiled without the fast-math flag.

#include <cuda_runtime.h>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "../common/rows.cuh"
#include "attn_params.cuh"
#include "mixed_attn.cuh"

namespace b200 {

bool mixed_decode_fits(int Hs, int Hk, int Ho, int Hv, int DP, int DVP);
bool mixed_prefill_fits(int Hs, int Hk, int Ho, int Hv, int DP, int DVP);
int mixed_decode(const MixedAttnParams& p, cudaStream_t stream);
int mixed_prefill(const MixedAttnParams& p, cudaStream_t stream);

// ------------------------------------------------------------- one CTA per query row, all heads
static constexpr int kMixThreads = 256, kMixKeys = 32;

static size_t plain_smem(int Hs, int Ho, int D, int DV) {
  return static_cast<size_t>(Hs * D + Ho * DV + (Hs + Ho) * kMixKeys + 3 * Ho + kMixKeys) * 4;
}

template <typename T>
__global__ void __launch_bounds__(kMixThreads) mixed_plain_kernel(const MixedAttnParams p) {
  extern __shared__ float sm[];
  float* sq = sm;                                      // [Hs][D]
  float* so = sq + p.Hs * p.D;                         // [Ho][DV]
  float* sa = so + p.Ho * p.DV;                        // [Hs][keys] scores before the mixture
  float* sp = sa + p.Hs * kMixKeys;                    // [Ho][keys] mixed scores, then weights
  float* s_max = sp + p.Ho * kMixKeys;                 // [Ho]
  float* s_sum = s_max + p.Ho;
  float* s_cor = s_sum + p.Ho;
  int* s_key = reinterpret_cast<int*>(s_cor + p.Ho);   // [keys] first cache row of a key's block and place in it
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int b, q_begin, q_len;
  if (p.cu_q) {
    int x = 0, y = p.B;                                // last b with cu_q[b] <= t
    while (y - x > 1) {
      const int m = (x + y) >> 1;
      if (p.cu_q[m] <= t) x = m; else y = m;
    }
    b = x;
    q_begin = p.cu_q[b];
    q_len = p.cu_q[b + 1] - q_begin;
    if (t < q_begin || t >= q_begin + q_len) return;
  } else {
    b = t / p.q_len;
    q_begin = b * p.q_len;
    q_len = p.q_len;
  }
  const int pos = p.seq_lens[b] - q_len + (t - q_begin), hi = pos + 1;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const T* q = static_cast<const T*>(p.q) + t * p.q_stride;
  const T* kc = static_cast<const T*>(p.k_cache);
  const T* vc = static_cast<const T*>(p.v_cache);
  for (int i = tid; i < p.Hs * p.D; i += kMixThreads) sq[i] = as_float(q[i]);
  for (int i = tid; i < p.Ho * p.DV; i += kMixThreads) so[i] = 0.f;
  for (int h = tid; h < p.Ho; h += kMixThreads) {
    s_max[h] = p.sink ? p.sink[h] : -INFINITY;         // the sink is a key seen from the start
    s_sum[h] = p.sink ? 1.f : 0.f;
  }
  const int per_k = p.Hs / p.Hk, per_v = p.Ho / p.Hv;
  for (int n0 = 0; n0 < hi; n0 += kMixKeys) {
    const int n = min(kMixKeys, hi - n0);
    __syncthreads();
    if (tid < n) s_key[tid] = bt[(n0 + tid) / p.block_size];
    __syncthreads();
    for (int i = tid; i < p.Hs * kMixKeys; i += kMixThreads) {
      const int g = i / kMixKeys, j = i % kMixKeys;
      if (j >= n) continue;
      const long long row =
          (static_cast<long long>(s_key[j]) * p.Hk + g / per_k) * p.block_size + (n0 + j) % p.block_size;
      const T* k = kc + row * p.DP;
      const float* qg = sq + g * p.D;
      float x = 0.f;
      for (int d = 0; d < p.D; ++d) x = fmaf(qg[d], as_float(k[d]), x);
      x *= p.scale;
      if (p.softcap > 0.f) x = p.softcap * tanhf(x / p.softcap);
      if (p.r1) x -= p.r1[g] * log1pf(p.r2[g] * static_cast<float>(pos - n0 - j));
      sa[i] = x;
    }
    __syncthreads();
    for (int h = warp; h < p.Ho; h += kMixThreads / 32) {
      float s = -INFINITY;
      if (lane < n) {
        s = 0.f;
        for (int g = 0; g < p.Hs; ++g) s = fmaf(p.talk[h * p.Hs + g], sa[g * kMixKeys + lane], s);
      }
      float mx = s;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float old = s_max[h];
      mx = fmaxf(mx, old);
      const float e = lane < n ? expf(s - mx) : 0.f;
      sp[h * kMixKeys + lane] = e;
      float sum = e;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      __syncwarp();
      if (lane == 0) {
        const float c = old == -INFINITY ? 0.f : expf(old - mx);
        s_max[h] = mx;
        s_sum[h] = s_sum[h] * c + sum;
        s_cor[h] = c;
      }
    }
    __syncthreads();
    for (int i = tid; i < p.Ho * p.DV; i += kMixThreads) {
      const int h = i / p.DV, d = i - h * p.DV, vh = h / per_v;
      float acc = so[i] * s_cor[h];
      for (int j = 0; j < n; ++j) {
        const long long row = (static_cast<long long>(s_key[j]) * p.Hv + vh) * p.block_size + (n0 + j) % p.block_size;
        acc = fmaf(sp[h * kMixKeys + j], as_float(vc[row * p.DVP + d]), acc);
      }
      so[i] = acc;
    }
  }
  __syncthreads();
  T* out = static_cast<T*>(p.out) + t * p.out_stride;
  for (int i = tid; i < p.Ho * p.DV; i += kMixThreads) {
    const float l = s_sum[i / p.DV];
    out[i] = from_float<T>(l > 0.f ? so[i] / l : 0.f);
  }
}

template <typename T>
static int launch_mixed_plain(const MixedAttnParams& p, cudaStream_t stream) {
  const size_t smem = plain_smem(p.Hs, p.Ho, p.D, p.DV);
  if (smem > 227 * 1024) return -2;
  auto kern = mixed_plain_kernel<T>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -20;
    once.mark(dev);
  }
  return launch_pdl(kern, dim3(p.rows), dim3(kMixThreads), smem, stream, 1, p) == cudaSuccess ? 0 : -21;
}

}  // namespace b200

using namespace b200;

// 0: the plain kernel, 1: the tensor-core kernels
extern "C" int b200_mixed_attention_kind(int Hs, int Hk, int Ho, int Hv, int DP, int DVP, int prompt, int is_fp32) {
  if (is_fp32 || (DP & 15) || (DVP & 15)) return 0;
  return (prompt ? mixed_prefill_fits(Hs, Hk, Ho, Hv, DP, DVP) : mixed_decode_fits(Hs, Hk, Ho, Hv, DP, DVP)) ? 1 : 0;
}

// kind: as above.  cu_q null: every sequence has q_len rows; else prompt portions.  scratch: see MixedAttnParams.
extern "C" int b200_mixed_attention(const void* q, const void* k_cache, const void* v_cache, void* out,
                                    const int* block_tables, const int* cu_q, const int* seq_lens, const float* r1,
                                    const float* r2, const float* talk, const float* sink, int B, int rows, int q_len,
                                    int max_keys, int max_blocks, int block_size, int Hs, int Hk, int Ho, int Hv, int D,
                                    int DV, int DP, int DVP, long long q_stride, long long out_stride, float scale,
                                    float softcap, int kind, int talk_terms, int splits, float* scratch, int tile0,
                                    int tiles, long long pitch, int is_fp32, cudaStream_t stream) {
  if (B <= 0 || rows <= 0) return 0;
  if (Hk <= 0 || Hv <= 0 || Hs % Hk || Ho % Hv || DP < D || DVP < DV || block_size <= 0) return -1;
  MixedAttnParams p{};
  p.q = q;
  p.k_cache = k_cache;
  p.v_cache = v_cache;
  p.out = out;
  p.block_tables = block_tables;
  p.cu_q = cu_q;
  p.seq_lens = seq_lens;
  p.r1 = r1;
  p.r2 = r2;
  p.talk = talk;
  p.sink = sink;
  p.B = B;
  p.rows = rows;
  p.q_len = q_len;
  p.max_q_len = q_len;
  p.max_keys = max_keys;
  p.max_blocks = max_blocks;
  p.block_size = block_size;
  p.bs_shift = -1;
  for (int i = 0; i < 30; ++i)
    if ((1 << i) == block_size) p.bs_shift = i;
  p.Hs = Hs;
  p.Hk = Hk;
  p.Ho = Ho;
  p.Hv = Hv;
  p.D = D;
  p.DV = DV;
  p.DP = DP;
  p.DVP = DVP;
  p.q_stride = q_stride;
  p.out_stride = out_stride;
  p.scale = scale;
  p.softcap = softcap;
  p.splits = splits < 1 ? 1 : splits;
  p.scratch = scratch;
  p.talk_terms = talk_terms;
  p.tile0 = tile0;
  p.tiles = tiles;
  p.pitch = pitch;
  if (kind == 0) return is_fp32 ? launch_mixed_plain<float>(p, stream) : launch_mixed_plain<__nv_bfloat16>(p, stream);
  if (is_fp32 || !b200_mixed_attention_kind(Hs, Hk, Ho, Hv, DP, DVP, cu_q != nullptr, 0)) return -2;
  if (cu_q == nullptr) return p.splits > 1 && scratch == nullptr ? -1 : mixed_decode(p, stream);
  if (scratch == nullptr || tiles <= 0 || pitch % 64 || pitch < max_keys) return -1;
  return mixed_prefill(p, stream);
}
