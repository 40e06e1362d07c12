// The end of one layer and the start of the next on a 32-bit residual stream, in one pass per token:
//
//   residual  = scale * table[id]                       (start of the model), or
//   residual += mult * (a + b + sum_j w_j * y[slot_j])  (end of a sublayer)
//   out       = residual / sqrt(mean(residual^2) + eps) * (w_offset + norm_w)
//
// a, b: dense sublayer outputs (either may be absent); y, slots, w: the rows that a mixture of
// experts left in expert order, brought back to their token and weighted here, so that neither the
// combined expert output nor the sum of the sublayers is ever written.  The residual is fp32; the
// sublayer outputs, the norm's weight and its result are bf16 or fp32 (one type per call).
// w_offset: 0 for weights stored as they multiply, 1 for weights stored around zero.
// Without out the stream is only advanced (hand-over to another pipeline stage).

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/pdl.cuh"
#include "../common/rows.cuh"

namespace b200 {

static constexpr int kResThreads = 256;

struct ResidualNormParams {
  float* residual;
  long long res_vecs;          // pitches in vectors of eight elements
  const int* ids;              // embedding: row of the table per token, or null
  const void* table;
  int table_rows;
  float table_scale;
  const void* a;
  long long a_vecs;
  const void* b;
  long long b_vecs;
  const void* y;               // [rows, H] expert outputs, or null
  const int* slots;            // [T, k] row of y per chosen expert (< 0: none)
  const float* w;              // [T, k]
  int k;
  float mult;                  // of everything that is added
  const void* norm_w;
  float eps;
  float w_offset;
  void* out;                   // or null
  long long out_vecs;
  int nvec;                    // H / 8
  int n_true;                  // columns that count in the mean (the rest are zero padding)
};

template <typename T, int VPT>
__global__ void __launch_bounds__(kResThreads) residual_norm_kernel(const ResidualNormParams p) {
  __shared__ float red[kResThreads / 32];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  float* res = p.residual + t * p.res_vecs * 8;
  float x[VPT][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= p.nvec) continue;
    if (p.ids) {
      int id = p.ids[t];
      id = id < 0 ? 0 : (id >= p.table_rows ? p.table_rows - 1 : id);
      Row8<T>::load(p.table, static_cast<long long>(id) * p.nvec + v, x[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[i][j] *= p.table_scale;
    } else {
      float add[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      float in[8];
      if (p.y) {
        for (int j0 = 0; j0 < p.k; j0 += 4) {
          // the rows of four experts are requested before the first is used
          float row[4][8];
          float wt[4];
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            wt[u] = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j) row[u][j] = 0.f;
            if (j0 + u < p.k) {
              const int slot = p.slots[t * p.k + j0 + u];
              if (slot >= 0) {
                wt[u] = p.w[t * p.k + j0 + u];
                Row8<T>::load(p.y, static_cast<long long>(slot) * p.nvec + v, row[u]);
              }
            }
          }
#pragma unroll
          for (int u = 0; u < 4; ++u)
#pragma unroll
            for (int j = 0; j < 8; ++j) add[j] += wt[u] * row[u][j];
        }
      }
      if (p.b) {
        Row8<T>::load(p.b, t * p.b_vecs + v, in);
#pragma unroll
        for (int j = 0; j < 8; ++j) add[j] += in[j];
      }
      if (p.a) {
        Row8<T>::load(p.a, t * p.a_vecs + v, in);
#pragma unroll
        for (int j = 0; j < 8; ++j) add[j] += in[j];
      }
      Row8<float>::load(res, v, x[i]);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[i][j] = fmaf(p.mult, add[j], x[i][j]);
    }
    Row8<float>::store(res, v, x[i]);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss += x[i][j] * x[i][j];
  }
  if (p.out == nullptr) return;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) tot += red[w];
  const float inv = rsqrtf(tot / static_cast<float>(p.n_true) + p.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= p.nvec) continue;
    float g[8];
    Row8<T>::load(p.norm_w, v, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) x[i][j] = x[i][j] * inv * (p.w_offset + g[j]);
    Row8<T>::store(p.out, t * p.out_vecs + v, x[i]);
  }
}

template <typename T>
static int launch_residual_norm(const ResidualNormParams& p, long long rows, cudaStream_t stream) {
  int threads = (p.nvec + 31) / 32 * 32;
  if (threads > kResThreads) threads = kResThreads;
  const int vpt = (p.nvec + threads - 1) / threads;
  cudaError_t e;
  const dim3 grid(static_cast<unsigned>(rows));
  if (vpt <= 1) e = launch_pdl(residual_norm_kernel<T, 1>, grid, dim3(threads), 0, stream, 1, p);
  else if (vpt <= 2) e = launch_pdl(residual_norm_kernel<T, 2>, grid, dim3(threads), 0, stream, 1, p);
  else if (vpt <= 4) e = launch_pdl(residual_norm_kernel<T, 4>, grid, dim3(threads), 0, stream, 1, p);
  else if (vpt <= 8) e = launch_pdl(residual_norm_kernel<T, 8>, grid, dim3(threads), 0, stream, 1, p);
  else return -2;
  return e == cudaSuccess ? 0 : -3;
}

}  // namespace b200

using namespace b200;

// H: row width in elements, a multiple of 8 (all pitches too), at most 16384.
extern "C" int b200_residual_norm(float* residual, long long res_stride, const int* ids, const void* table,
                                  int table_rows, float table_scale, const void* a, long long a_stride,
                                  const void* b, long long b_stride, const void* y, const int* slots,
                                  const float* w, int k, float mult, const void* norm_w, float eps, float w_offset, void* out,
                                  long long out_stride, long long rows, int H, int n_true, int is_fp32,
                                  cudaStream_t stream) {
  if (rows <= 0) return 0;
  if ((H & 7) || (res_stride & 7) || (a_stride & 7) || (b_stride & 7) || (out_stride & 7) || n_true <= 0) return -1;
  ResidualNormParams p{};
  p.residual = residual;
  p.res_vecs = res_stride >> 3;
  p.ids = ids;
  p.table = table;
  p.table_rows = table_rows;
  p.table_scale = table_scale;
  p.a = a;
  p.a_vecs = a_stride >> 3;
  p.b = b;
  p.b_vecs = b_stride >> 3;
  p.y = y;
  p.slots = slots;
  p.w = w;
  p.k = k;
  p.mult = mult;
  p.norm_w = norm_w;
  p.eps = eps;
  p.w_offset = w_offset;
  p.out = out;
  p.out_vecs = out_stride >> 3;
  p.nvec = H >> 3;
  p.n_true = n_true;
  return is_fp32 ? launch_residual_norm<float>(p, rows, stream)
                 : launch_residual_norm<__nv_bfloat16>(p, rows, stream);
}
