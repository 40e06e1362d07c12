// Layers that norm what a sublayer gives, not what it reads, on a 32-bit residual stream:
//
//   post_norm_residual   x += norm(y) * w  (or x = table[id], the start of the model), and the row the next product
//                        reads: x itself rounded, or norm(x) * w_out at the end of the model.  One pass per token.
//   gelu_rows            gelu(z) * table[id, offset ..]: the gated row of a per-layer token input
//
// The norm treats `groups` equal parts of a row one by one: part / sqrt(mean(part^2) + eps).  The residual is fp32, the
// rest bf16 or fp32 (one type per call).  Compiled without the fast-math flag.

#include <cuda_runtime.h>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "../common/rows.cuh"
#include "../gemm/gated_act.cuh"

namespace b200 {

static constexpr int kPostThreads = 256;

struct PostNormParams {
  float* residual;
  long long res_vecs;          // pitches in vectors of eight elements
  const int* ids;              // the residual starts as rows of the table, or null
  const void* table;
  int table_rows;
  const void* y;
  long long y_vecs;
  const void* w;
  int groups;
  const void* out_w;           // or null: the residual itself
  int out_groups;
  void* out;
  long long out_vecs;
  float eps;
  int nvec;                    // padded width / 8
  int n_true;                  // columns of the groups (the rest are zero padding)
};

// The reciprocal root mean square of every group, in `inv` of shared memory.  `part` holds one number per vector, or
// per element when a vector may belong to two groups.
template <int VPT>
__device__ __forceinline__ void group_scales(const float (&x)[VPT][8], int nvec, int n_true, int groups, float eps,
                                             float* part, float* inv) {
  const int size = n_true / groups, tid = threadIdx.x, lane = tid & 31, warps = blockDim.x >> 5;
  const bool whole = groups == 1 || (size & 7) == 0;
  __syncthreads();                                     // (the arrays may still be read from an earlier use)
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = tid + i * blockDim.x;
    if (v >= nvec) continue;
    if (whole) {
      float s = 0.f;
#pragma unroll
      for (int j = 0; j < 8; ++j) s = fmaf(x[i][j], x[i][j], s);
      part[v] = s;
    } else {
#pragma unroll
      for (int j = 0; j < 8; ++j) part[v * 8 + j] = x[i][j] * x[i][j];
    }
  }
  __syncthreads();
  const int step = whole ? (groups == 1 ? nvec : size >> 3) : size;
  if (groups == 1) {
    // every warp sums the whole row: no further exchange
    float s = 0.f;
    for (int e = lane; e < step; e += 32) s += part[e];
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (tid == 0) inv[0] = 1.f / sqrtf(s / static_cast<float>(size) + eps);
  } else {
    for (int g = tid >> 5; g < groups; g += warps) {
      float s = 0.f;
      for (int e = lane; e < step; e += 32) s += part[g * step + e];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (lane == 0) inv[g] = 1.f / sqrtf(s / static_cast<float>(size) + eps);
    }
  }
  __syncthreads();
}

// x <- x * inv[group] * w; columns beyond the groups become zero
template <typename T>
__device__ __forceinline__ void scale_groups(float (&x)[8], int v, const void* w, int n_true, int groups,
                                             const float* inv) {
  float g[8];
  Row8<T>::load(w, v, g);
  const int size = n_true / groups;
  if (groups == 1 || (size & 7) == 0) {
    const float f = v * 8 < n_true ? inv[groups == 1 ? 0 : v * 8 / size] : 0.f;
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] = x[j] * f * g[j];
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) x[j] = v * 8 + j < n_true ? x[j] * inv[(v * 8 + j) / size] * g[j] : 0.f;
  }
}

template <typename T, int VPT>
__global__ void __launch_bounds__(kPostThreads) post_norm_kernel(const PostNormParams p) {
  extern __shared__ float sm[];
  const int big = p.groups > p.out_groups ? p.groups : p.out_groups;
  float* inv = sm;                                     // [groups]
  float* part = sm + big;
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  float* res = p.residual + t * p.res_vecs * 8;
  float x[VPT][8];
  if (p.ids) {
    int id = p.ids[t];
    id = id < 0 ? 0 : (id >= p.table_rows ? p.table_rows - 1 : id);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < p.nvec) Row8<T>::load(p.table, static_cast<long long>(id) * p.nvec + v, x[i]);
    }
  } else {
    float y[VPT][8];
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v >= p.nvec) continue;
      Row8<T>::load(p.y, t * p.y_vecs + v, y[i]);
      Row8<float>::load(res, v, x[i]);
    }
    group_scales<VPT>(y, p.nvec, p.n_true, p.groups, p.eps, part, inv);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v >= p.nvec) continue;
      scale_groups<T>(y[i], v, p.w, p.n_true, p.groups, inv);
#pragma unroll
      for (int j = 0; j < 8; ++j) x[i][j] += y[i][j];
    }
  }
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < p.nvec) Row8<float>::store(res, v, x[i]);
  }
  if (p.out_w) group_scales<VPT>(x, p.nvec, p.n_true, p.out_groups, p.eps, part, inv);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= p.nvec) continue;
    if (p.out_w) scale_groups<T>(x[i], v, p.out_w, p.n_true, p.out_groups, inv);
    Row8<T>::store(p.out, t * p.out_vecs + v, x[i]);
  }
}

template <typename T, int VPT>
static int launch_post_norm_vpt(const PostNormParams& p, long long rows, int threads, size_t smem, cudaStream_t stream) {
  auto kern = post_norm_kernel<T, VPT>;
  static DeviceOnce once;
  int dev = 0;
  if (smem > 48 * 1024 && once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess) return -20;
    once.mark(dev);
  }
  return launch_pdl(kern, dim3(static_cast<unsigned>(rows)), dim3(threads), smem, stream, 1, p) == cudaSuccess ? 0 : -3;
}

template <typename T>
static int launch_post_norm(const PostNormParams& p, long long rows, cudaStream_t stream) {
  int threads = (p.nvec + 31) / 32 * 32;
  if (threads > kPostThreads) threads = kPostThreads;
  const int vpt = (p.nvec + threads - 1) / threads;
  const auto elementwise = [&](int groups) { return groups > 1 && (p.n_true / groups) % 8 != 0; };
  const int big = p.groups > p.out_groups ? p.groups : p.out_groups;
  const size_t smem = (big + p.nvec * (elementwise(p.groups) || elementwise(p.out_groups) ? 8 : 1)) * sizeof(float);
  if (smem > 200 * 1024) return -2;
  if (vpt <= 1) return launch_post_norm_vpt<T, 1>(p, rows, threads, smem, stream);
  if (vpt <= 2) return launch_post_norm_vpt<T, 2>(p, rows, threads, smem, stream);
  if (vpt <= 4) return launch_post_norm_vpt<T, 4>(p, rows, threads, smem, stream);
  if (vpt <= 8) return launch_post_norm_vpt<T, 8>(p, rows, threads, smem, stream);
  return -2;
}

// ------------------------------------------------------------- gated rows of a token table
struct GeluRowsParams {
  const void* z;
  void* out;                   // [T, width]
  long long z_stride;
  const int* ids;
  const void* table;
  long long table_stride;      // in elements
  int table_rows, offset, dim, width, T, vec;
};

template <typename T>
__global__ void __launch_bounds__(256) gelu_rows_kernel(const GeluRowsParams p) {
  pdl_trigger();
  pdl_wait();
  const int per = p.width >> 3;
  const long long i = blockIdx.x * 256ll + threadIdx.x;
  if (i >= static_cast<long long>(p.T) * per) return;
  const long long t = i / per;
  const int v = static_cast<int>(i - t * per), d = v * 8;
  int id = p.ids[t];
  id = id < 0 ? 0 : (id >= p.table_rows ? p.table_rows - 1 : id);
  const T* row = static_cast<const T*>(p.table) + id * p.table_stride + p.offset;
  float x[8], e[8];
  Row8<T>::load(static_cast<const T*>(p.z) + t * p.z_stride, v, x);
  if (p.vec) {
    Row8<T>::load(row, v, e);
  } else {
#pragma unroll
    for (int j = 0; j < 8; ++j) e[j] = d + j < p.dim ? as_float(row[d + j]) : 0.f;
  }
#pragma unroll
  for (int j = 0; j < 8; ++j) x[j] = d + j < p.dim ? gated_act_exact(kActGeluTanh, x[j], e[j], 0.f, 0.f) : 0.f;
  Row8<T>::store(static_cast<T*>(p.out) + t * p.width, v, x);
}

}  // namespace b200

using namespace b200;

// W: padded row width, a multiple of 8 (all pitches too), at most 16384.
extern "C" int b200_post_norm_residual(float* residual, long long res_stride, const int* ids, const void* table,
                                       int table_rows, const void* y, long long y_stride, const void* w, int groups,
                                       const void* out_w, int out_groups, void* out, long long out_stride, float eps,
                                       long long rows, int W, int n_true, int is_fp32, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if ((W & 7) || (res_stride & 7) || (y_stride & 7) || (out_stride & 7) || n_true <= 0 || n_true > W) return -1;
  if (groups < 1 || out_groups < 1 || n_true % groups || n_true % out_groups || (ids == nullptr) == (y == nullptr)) return -1;
  PostNormParams p{residual, res_stride >> 3, ids, table, table_rows, y, y_stride >> 3, w, groups, out_w, out_groups,
                   out, out_stride >> 3, eps, W >> 3, n_true};
  return is_fp32 ? launch_post_norm<float>(p, rows, stream) : launch_post_norm<__nv_bfloat16>(p, rows, stream);
}

// width: a multiple of 8, at least dim; z's rows are as wide.
extern "C" int b200_gelu_rows(const void* z, long long z_stride, const int* ids, const void* table, int table_rows,
                              long long table_stride, int offset, int dim, int width, void* out, int T, int is_fp32,
                              cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((width & 7) || (z_stride & 7) || dim > width || offset + dim > table_stride) return -1;
  GeluRowsParams p{z, out, z_stride, ids, table, table_stride, table_rows, offset, dim, width, T,
                   (dim % 8 == 0 && offset % 8 == 0 && table_stride % 8 == 0) ? 1 : 0};
  const long long items = static_cast<long long>(T) * (width >> 3);
  const dim3 grid(static_cast<unsigned>((items + 255) / 256));
  const cudaError_t e = is_fp32 ? launch_pdl(gelu_rows_kernel<float>, grid, dim3(256), 0, stream, 1, p)
                                : launch_pdl(gelu_rows_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, 1, p);
  return e == cudaSuccess ? 0 : -3;
}
