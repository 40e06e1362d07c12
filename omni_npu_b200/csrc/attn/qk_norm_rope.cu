// From the q / k / v projections of a step to rotated queries and cache rows, in one pass per token:
//
//   norm over the projection:  x <- x / sqrt(mean(x^2) + eps) * w over all rows of q (and of k) at once, then rotation
//   norm per head:             rotation, then every head of q and k / sqrt(mean over the head + eps)
//   weighted norm per head:    every head / sqrt(mean over the head + eps) * w, w shared by the heads, then rotation
//   rotation:                  of the first `rot` dimensions of a head, i paired with i + rot / 2
//   query temperature:         q at position p times 1 + c ln(floor((p + 1) / n) + 1)
//   values:                    v, or (1 - lambda) v + lambda v_first with v_first those of another layer
//
// q goes to rows of its own, k and v into the paged cache (rows padded to DP / DVP, the padding is never
// written).  All arithmetic is fp32; compiled without the fast-math flag.

#include <cuda_runtime.h>

#include "../common/pdl.cuh"
#include "../common/rows.cuh"

namespace b200 {

enum : int { kNormNone = 0, kNormProjection = 1, kNormHead = 2, kNormHeadWeight = 3 };

struct QkNormParams {
  const void* q;
  const void* k;
  const void* v;
  const void* v_first;         // or null
  void* q_out;                 // [T, Hq * D]
  void* k_cache;               // [blocks, Hk, block_size, DP]
  void* v_cache;               // [blocks, Hv, block_size, DVP]
  const int* positions;
  const int* slots;            // < 0: nothing is stored
  const float* cos_sin;        // [max_pos, rot]: cosines then sines
  const void* q_w;             // norm weights of the whole projections, or of a head
  const void* k_w;
  const float* sums;           // [T, 2] sums of squares of q and k over all ranks, or null: computed here
  int n_q, n_k;                // elements they stand for
  int Hq, Hk, Hv, D, DV, DP, DVP, rot, block_size, max_pos;
  int lanes;                   // of a warp that share a head: a power of two
  long long q_stride, k_stride, v_stride, f_stride;
  float eps, lambda;
  float temp;                  // c of the query temperature
  int temp_every;              // n, 0: none
};

static constexpr int kQkThreads = 256, kQkWarps = kQkThreads / 32;

// W elements from p + d; with W = 1 any address will do
template <typename T, int W>
__device__ __forceinline__ void load_w(const T* p, int d, float (&x)[W]) {
  if constexpr (W == 4) Row4<T>::load(p + d, 0, x);
  else x[0] = as_float(p[d]);
}
template <typename T, int W>
__device__ __forceinline__ void store_w(T* p, int d, const float (&x)[W]) {
  if constexpr (W == 4) Row4<T>::store(p + d, 0, x);
  else p[d] = from_float<T>(x[0]);
}

template <typename T, int W>
__device__ __forceinline__ float row_sum_squares(const T* row, int n) {
  float s = 0.f;
  for (int d = threadIdx.x * W; d < n; d += kQkThreads * W) {
    float x[W];
    load_w<T, W>(row, d, x);
#pragma unroll
    for (int j = 0; j < W; ++j) s = fmaf(x[j], x[j], s);
  }
  return s;
}

template <typename T, int W, int NORM>
__global__ void __launch_bounds__(kQkThreads) qk_norm_rope_kernel(const QkNormParams p) {
  __shared__ float red[2][kQkWarps];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const T* q = static_cast<const T*>(p.q) + t * p.q_stride;
  const T* k = static_cast<const T*>(p.k) + t * p.k_stride;
  const T* v = static_cast<const T*>(p.v) + t * p.v_stride;
  const int slot = p.slots[t];
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  const float* cs = p.cos_sin + static_cast<long long>(pos) * p.rot;
  constexpr bool WEIGHTS = NORM == kNormProjection || NORM == kNormHeadWeight;
  const float heat =
      p.temp_every > 0 ? 1.f + p.temp * logf(static_cast<float>((p.positions[t] + 1) / p.temp_every) + 1.f) : 1.f;
  float inv_q = 1.f, inv_k = 1.f;
  if constexpr (NORM == kNormProjection) {
    float sq, sk;
    if (p.sums) {
      sq = p.sums[2 * t];
      sk = p.sums[2 * t + 1];
    } else {
      sq = row_sum_squares<T, W>(q, p.Hq * p.D);
      sk = row_sum_squares<T, W>(k, p.Hk * p.D);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        sq += __shfl_xor_sync(0xffffffffu, sq, o);
        sk += __shfl_xor_sync(0xffffffffu, sk, o);
      }
      if (lane == 0) {
        red[0][warp] = sq;
        red[1][warp] = sk;
      }
      __syncthreads();
      sq = sk = 0.f;
#pragma unroll
      for (int w = 0; w < kQkWarps; ++w) {
        sq += red[0][w];
        sk += red[1][w];
      }
    }
    inv_q = 1.f / sqrtf(sq / static_cast<float>(p.n_q) + p.eps);
    inv_k = 1.f / sqrtf(sk / static_cast<float>(p.n_k) + p.eps);
  }
  const long long blk = slot < 0 ? 0 : slot / p.block_size, off = slot < 0 ? 0 : slot % p.block_size;
  const int half = p.rot >> 1, per_warp = 32 / p.lanes, li = lane & (p.lanes - 1);
  const int units = slot < 0 ? p.Hq : p.Hq + p.Hk + p.Hv;
  const int step = gridDim.y * kQkWarps * per_warp;
  const int base = (blockIdx.y * kQkWarps + warp) * per_warp;
  for (int u0 = base; u0 < units; u0 += step) {            // (warp-uniform)
    const int unit = u0 + lane / p.lanes;
    const bool live = unit < units;
    if (live && unit >= p.Hq + p.Hk) {                     // a value head
      const int h = unit - p.Hq - p.Hk;
      T* dst = static_cast<T*>(p.v_cache) + ((blk * p.Hv + h) * p.block_size + off) * p.DVP;
      const T* src = v + h * p.DV;
      const T* first = p.v_first ? static_cast<const T*>(p.v_first) + t * p.f_stride + h * p.DV : nullptr;
      for (int d = li * W; d < p.DV; d += p.lanes * W) {
        float x[W];
        load_w<T, W>(src, d, x);
        if (first) {
          float f[W];
          load_w<T, W>(first, d, f);
#pragma unroll
          for (int j = 0; j < W; ++j) x[j] = (1.f - p.lambda) * x[j] + p.lambda * f[j];
        }
        store_w<T, W>(dst, d, x);
      }
    }
    const bool is_q = unit < p.Hq;
    const bool head = live && unit < p.Hq + p.Hk;
    const int h = is_q ? unit : unit - p.Hq;
    const T* src = (is_q ? q : k) + (head ? h * p.D : 0);
    T* dst = is_q ? static_cast<T*>(p.q_out) + (t * p.Hq + h) * p.D
                  : static_cast<T*>(p.k_cache) + ((blk * p.Hk + h) * p.block_size + off) * p.DP;
    float inv = is_q ? inv_q : inv_k;
    const T* w = static_cast<const T*>(is_q ? p.q_w : p.k_w);
    if (NORM == kNormProjection && head) w += h * p.D;
    if constexpr (NORM == kNormHead || NORM == kNormHeadWeight) {    // (a rotation leaves the sum of squares as it is)
      float ss = 0.f;
      if (head)
        for (int d = li * W; d < p.D; d += p.lanes * W) {
          float x[W];
          load_w<T, W>(src, d, x);
#pragma unroll
          for (int j = 0; j < W; ++j) ss = fmaf(x[j], x[j], ss);
        }
      for (int o = p.lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      inv = 1.f / sqrtf(ss / static_cast<float>(p.D) + p.eps);
    }
    if (!head) continue;
    if (is_q) inv *= heat;
    for (int d = li * W; d < p.D; d += p.lanes * W) {
      float x[W];
      load_w<T, W>(src, d, x);
      if constexpr (WEIGHTS) {
        float g[W];
        load_w<T, W>(w, d, g);
#pragma unroll
        for (int j = 0; j < W; ++j) x[j] *= g[j];
      }
      if (d < p.rot) {
        const bool lo = d < half;
        const int a = lo ? d : d - half;
        float y[W], c[W], s[W];
        load_w<T, W>(src, lo ? d + half : a, y);
        load_w<float, W>(cs, a, c);
        load_w<float, W>(cs + half, a, s);
        if constexpr (WEIGHTS) {
          float g[W];
          load_w<T, W>(w, lo ? d + half : a, g);
#pragma unroll
          for (int j = 0; j < W; ++j) y[j] *= g[j];
        }
#pragma unroll
        for (int j = 0; j < W; ++j) x[j] = x[j] * c[j] + (lo ? -y[j] : y[j]) * s[j];
      }
#pragma unroll
      for (int j = 0; j < W; ++j) x[j] *= inv;
      store_w<T, W>(dst, d, x);
    }
  }
}

template <typename T, int W>
static cudaError_t launch_qk(const QkNormParams& p, int norm, dim3 grid, cudaStream_t stream) {
  const dim3 block(kQkThreads);
  if (norm == kNormProjection) return launch_pdl(qk_norm_rope_kernel<T, W, kNormProjection>, grid, block, 0, stream, 1, p);
  if (norm == kNormHead) return launch_pdl(qk_norm_rope_kernel<T, W, kNormHead>, grid, block, 0, stream, 1, p);
  if (norm == kNormHeadWeight) return launch_pdl(qk_norm_rope_kernel<T, W, kNormHeadWeight>, grid, block, 0, stream, 1, p);
  return launch_pdl(qk_norm_rope_kernel<T, W, kNormNone>, grid, block, 0, stream, 1, p);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_qk_norm_rope(const void* q, const void* k, const void* v, const void* v_first, void* q_out,
                                 void* k_cache, void* v_cache, const int* positions, const int* slots,
                                 const float* cos_sin, int max_pos, int norm, const void* q_w, const void* k_w,
                                 const float* sums, int n_q, int n_k, float eps, float lambda, int T, int Hq, int Hk, int Hv,
                                 int D, int DV, int DP, int DVP, int rot, long long q_stride, long long k_stride,
                                 long long v_stride, long long f_stride, int block_size, float temp, int temp_every,
                                 int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot < 0 || rot > D || (rot & 1) || DP < D || DVP < DV || norm < 0 || norm > 3 || temp_every < 0) return -1;
  if (rot > 0 && cos_sin == nullptr) return -1;
  const uintptr_t align = is_fp32 ? 15 : 7;
  const auto ok = [&](const void* ptr, long long stride) {
    return (reinterpret_cast<uintptr_t>(ptr) & align) == 0 && stride % 4 == 0;
  };
  const bool vec = D % 4 == 0 && DV % 4 == 0 && rot % 8 == 0 && ok(q, q_stride) && ok(k, k_stride) && ok(v, v_stride) &&
                   ok(v_first, f_stride) && ok(k_cache, DP) && ok(v_cache, DVP) && ok(q_out, 0) && ok(q_w, 0) &&
                   ok(k_w, 0) && (reinterpret_cast<uintptr_t>(cos_sin) & 15) == 0;
  int lanes = 1;
  while (lanes < 32 && lanes * (vec ? 4 : 1) < D) lanes <<= 1;
  QkNormParams p{q, k, v, v_first, q_out, k_cache, v_cache, positions, slots, cos_sin, q_w, k_w, sums, n_q, n_k, Hq, Hk, Hv,
                 D, DV, DP, DVP, rot, block_size, max_pos, lanes, q_stride, k_stride, v_stride, f_stride, eps, lambda, temp, temp_every};
  const int per_cta = kQkWarps * (32 / lanes);
  int ny = (Hq + Hk + Hv + per_cta - 1) / per_cta;
  if (T >= 256) ny = 1;                                   // enough tokens: longer CTAs
  const dim3 grid(T, ny);
  cudaError_t e;
  if (is_fp32) e = vec ? launch_qk<float, 4>(p, norm, grid, stream) : launch_qk<float, 1>(p, norm, grid, stream);
  else e = vec ? launch_qk<__nv_bfloat16, 4>(p, norm, grid, stream) : launch_qk<__nv_bfloat16, 1>(p, norm, grid, stream);
  return e == cudaSuccess ? 0 : -3;
}
