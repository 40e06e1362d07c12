// Latent attention with run-time sizes: what stands around its attention kernels.
//
//   latent_prep     RMS norm of the latent, rotation of the shared key part and of the queries, cache row; RMS norm
//                   of the queries' own latent
//   head_gemm       out[t, h] = W[h] a[t, h] for few tokens (folding queries into the latent space and back)
//   latent_gather   cached rows of all sequences of a step, one after another

#include <cuda_runtime.h>

#include "../common/pdl.cuh"
#include "../common/rows.cuh"
#include "attn_common.cuh"

namespace b200 {

// ------------------------------------------------------------- norm, rotation, cache row
struct LatentPrepParams {
  void* q;                     // [T, H * (dim + rot)], rotated in place from row num_latent on; or null
  long long q_stride;
  const void* kv;              // [T, rank + rot], or null
  long long kv_stride;
  const void* norm_w;          // [rank]
  float eps;
  void* cache;                 // rows of `row` elements
  const int* positions;
  const int* slots;
  const float* cos_sin;        // [max_pos, rot]: cosines then sines
  int max_pos, H, dim, rot, rank, row, neox, num_latent;
  void* q_latent;              // [num_latent, H, row]: columns rank .. of a row take the rotated part
  const void* low;             // [T, low_rank], normed into low_out [T, low_width] (zeros behind), or null
  long long low_stride;
  const void* low_w;
  void* low_out;
  int low_rank, low_width;
};

static constexpr int kLatentThreads = 256;

template <typename T>
__device__ __forceinline__ void rotate_pair(const T* src, T* dst, int i, int half, int neox, const float* cs) {
  const int a = neox ? i : 2 * i, b = neox ? i + half : 2 * i + 1;
  const float u = as_float(src[a]), v = as_float(src[b]), c = cs[i], s = cs[half + i];
  dst[a] = from_float<T>(u * c - v * s);
  dst[b] = from_float<T>(v * c + u * s);
}

// 1 / root mean square of a row, the same in every thread
template <typename T>
__device__ __forceinline__ float row_inv_rms(const T* x, int n, float eps, float* red) {
  float ss = 0.f;
  for (int d = threadIdx.x; d < n; d += kLatentThreads) {
    const float v = as_float(x[d]);
    ss = fmaf(v, v, ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int w = 0; w < kLatentThreads / 32; ++w) tot += red[w];
  return 1.f / sqrtf(tot / static_cast<float>(n) + eps);
}

template <typename T>
__global__ void __launch_bounds__(kLatentThreads) latent_prep_kernel(const LatentPrepParams p) {
  __shared__ float red[2][kLatentThreads / 32];
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  const float* cs = p.cos_sin + static_cast<long long>(pos) * p.rot;
  const int half = p.rot >> 1, tid = threadIdx.x;
  const int slot = p.slots[t];
  if (p.kv && blockIdx.y == 0 && slot >= 0) {
    const T* kv = static_cast<const T*>(p.kv) + t * p.kv_stride;
    const float inv = row_inv_rms(kv, p.rank, p.eps, red[0]);
    T* dst = static_cast<T*>(p.cache) + static_cast<long long>(slot) * p.row;
    const T* w = static_cast<const T*>(p.norm_w);
    for (int d = tid; d < p.rank; d += kLatentThreads) dst[d] = from_float<T>(as_float(kv[d]) * inv * as_float(w[d]));
    for (int i = tid; i < half; i += kLatentThreads) rotate_pair<T>(kv + p.rank, dst + p.rank, i, half, p.neox, cs);
    for (int d = p.rank + p.rot + tid; d < p.row; d += kLatentThreads) dst[d] = from_float<T>(0.f);
  }
  if (p.low && blockIdx.y == gridDim.y - 1) {
    const T* z = static_cast<const T*>(p.low) + t * p.low_stride;
    const float inv = row_inv_rms(z, p.low_rank, p.eps, red[1]);
    T* dst = static_cast<T*>(p.low_out) + t * p.low_width;
    const T* w = static_cast<const T*>(p.low_w);
    for (int d = tid; d < p.low_width; d += kLatentThreads)
      dst[d] = from_float<T>(d < p.low_rank ? as_float(z[d]) * inv * as_float(w[d]) : 0.f);
  }
  if (p.q == nullptr) return;
  const bool fold = t < p.num_latent;
  const int total = p.H * half;
  for (int i = blockIdx.y * kLatentThreads + tid; i < total; i += gridDim.y * kLatentThreads) {
    const int h = i / half, j = i - h * half;
    T* q = static_cast<T*>(p.q) + t * p.q_stride + static_cast<long long>(h) * (p.dim + p.rot) + p.dim;
    T* dst = fold ? static_cast<T*>(p.q_latent) + (t * p.H + h) * p.row + p.rank : q;
    rotate_pair<T>(q, dst, j, half, p.neox, cs);
  }
  if (fold) {
    const int pad = p.row - p.rank - p.rot;
    for (int i = blockIdx.y * kLatentThreads + tid; i < p.H * pad; i += gridDim.y * kLatentThreads) {
      const int h = i / pad;
      static_cast<T*>(p.q_latent)[(t * p.H + h) * p.row + p.rank + p.rot + i - h * pad] = from_float<T>(0.f);
    }
  }
}

// The norms alone (no queries to rotate), rows of whole 16-byte pieces: one warp per (token, part), part 0 the cache row,
// the last part the queries' latent.
static constexpr int kNormVecs = 8;                      // vectors of eight elements per lane at most

template <typename T>
__device__ __forceinline__ void warp_norm_row(const T* src, const T* w, T* dst, int n, float eps, int lane) {
  float x[kNormVecs][8];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < kNormVecs; ++i) {
    const int v = lane + i * 32;
    if (v * 8 >= n) continue;
    Row8<T>::load(src, v, x[i]);
#pragma unroll
    for (int j = 0; j < 8; ++j) ss = fmaf(x[i][j], x[i][j], ss);
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(n) + eps);
#pragma unroll
  for (int i = 0; i < kNormVecs; ++i) {
    const int v = lane + i * 32;
    if (v * 8 >= n) continue;
    float g[8];
    Row8<T>::load(w, v, g);
#pragma unroll
    for (int j = 0; j < 8; ++j) x[i][j] = x[i][j] * inv * g[j];
    Row8<T>::store(dst, v, x[i]);
  }
}

template <typename T>
__global__ void __launch_bounds__(kLatentThreads) latent_norm_kernel(const LatentPrepParams p, const int T_rows) {
  pdl_trigger();
  pdl_wait();
  const int parts = (p.kv ? 1 : 0) + (p.low ? 1 : 0), lane = threadIdx.x & 31;
  const int item = blockIdx.x * (kLatentThreads / 32) + (threadIdx.x >> 5);
  if (item >= T_rows * parts) return;
  const int part = item / T_rows;
  const long long t = item - part * T_rows;
  if (p.low && part == parts - 1) {
    warp_norm_row<T>(static_cast<const T*>(p.low) + t * p.low_stride, static_cast<const T*>(p.low_w),
                     static_cast<T*>(p.low_out) + t * p.low_width, p.low_rank, p.eps, lane);
    return;
  }
  const int slot = p.slots[t];
  if (slot < 0) return;
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  const T* kv = static_cast<const T*>(p.kv) + t * p.kv_stride;
  T* dst = static_cast<T*>(p.cache) + static_cast<long long>(slot) * p.row;
  const int half = p.rot >> 1;
  const float* cs = p.cos_sin + static_cast<long long>(pos) * p.rot;
  for (int i = lane; i < half; i += 32) rotate_pair<T>(kv + p.rank, dst + p.rank, i, half, p.neox, cs);
  for (int d = p.rank + p.rot + lane; d < p.row; d += 32) dst[d] = from_float<T>(0.f);
  warp_norm_row<T>(kv, static_cast<const T*>(p.norm_w), dst, p.rank, p.eps, lane);
}

// ------------------------------------------------------------- per-head products
struct HeadGemmParams {
  const void* a;               // [T, H, K]
  const void* w;               // [H, N, K] contiguous
  void* out;                   // [T, H, N]
  long long a_t, a_h, o_t, o_h;
  int T, H, N, K, vec;         // vec: rows of a and w are whole 16-byte pieces
};

namespace hg {
constexpr int BM = 64, BN = 64, BK = 64, THREADS = 128;
}

// One CTA = 64 tokens x 64 outputs of a head; four warps with 16 outputs each; K in steps of 64, the next
// step on its way while one is worked off.
__global__ void __launch_bounds__(hg::THREADS) head_gemm_kernel(const HeadGemmParams p) {
  using namespace hg;
  __shared__ __align__(128) uint8_t sA[2][BM * BK * 2];
  __shared__ __align__(128) uint8_t sW[2][BN * BK * 2];
  pdl_trigger();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int n0 = blockIdx.x * BN, h = blockIdx.y, t0 = blockIdx.z * BM;
  const __nv_bfloat16* a = static_cast<const __nv_bfloat16*>(p.a) + h * p.a_h;
  const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(p.w) + static_cast<long long>(h) * p.N * p.K;
  const int rows = min(BM, p.T - t0), m_tiles = (rows + 15) >> 4;
  const int steps = (p.K + BK - 1) / BK;

  auto load = [&](const __nv_bfloat16* base, long long pitch, int r0, int r_max, int k0, uint8_t* dst, int n_rows) {
    for (int i = tid; i < n_rows * (BK / 8); i += THREADS) {
      const int r = i >> 3, c = i & 7;
      const int row = r0 + r, k = k0 + c * 8;
      uint8_t* d = dst + tile_offset<BK>(r, c);
      const __nv_bfloat16* src = base + static_cast<long long>(row) * pitch + k;
      if (p.vec) {
        const bool ok = row < r_max && k < p.K;
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(d)), "l"(ok ? src : base),
                     "r"(ok ? 16 : 0) : "memory");
      } else {
#pragma unroll
        for (int j = 0; j < 8; ++j)
          reinterpret_cast<__nv_bfloat16*>(d)[j] = row < r_max && k + j < p.K ? src[j] : __float2bfloat16(0.f);
      }
    }
  };
  // (the weights are no earlier kernel's result)
  load(w, p.K, n0, p.N, 0, sW[0], BN);
  pdl_wait();
  load(a, p.a_t, t0, p.T, 0, sA[0], m_tiles * 16);
  asm volatile("cp.async.commit_group;" ::: "memory");

  float acc[BM / 16][2][4];
#pragma unroll
  for (int i = 0; i < BM / 16; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;

  for (int s = 0; s < steps; ++s) {
    if (s + 1 < steps) {
      load(w, p.K, n0, p.N, (s + 1) * BK, sW[(s + 1) & 1], BN);
      load(a, p.a_t, t0, p.T, (s + 1) * BK, sA[(s + 1) & 1], m_tiles * 16);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const uint32_t at = smem_u32(sA[s & 1]), wt = smem_u32(sW[s & 1]);
#pragma unroll
    for (int ks = 0; ks < BK / 16; ++ks) {
      uint32_t wf[4];
      ldmatrix_x4(wf, wt + tile_offset<BK>(warp * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
#pragma unroll
      for (int m = 0; m < BM / 16; ++m) {
        if (m < m_tiles) {
          uint32_t af[4];
          ldmatrix_x4(af, at + tile_offset<BK>(m * 16 + (lane & 15), ks * 2 + (lane >> 4)));
          mma_bf16_16816(acc[m][0], af, wf[0], wf[1]);
          mma_bf16_16816(acc[m][1], af, wf[2], wf[3]);
        }
      }
    }
    __syncthreads();
  }
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + h * p.o_h;
#pragma unroll
  for (int m = 0; m < BM / 16; ++m)
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = t0 + m * 16 + (lane >> 2) + r * 8;
        const int n = n0 + warp * 16 + j * 8 + (lane & 3) * 2;
        if (m >= m_tiles || t >= p.T) continue;
        __nv_bfloat16* dst = out + t * p.o_t + n;
        const float x0 = acc[m][j][2 * r], x1 = acc[m][j][2 * r + 1];
        if (n + 1 < p.N && (reinterpret_cast<uintptr_t>(dst) & 3) == 0) {
          *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(x0, x1);
        } else {
          if (n < p.N) dst[0] = __float2bfloat16(x0);
          if (n + 1 < p.N) dst[1] = __float2bfloat16(x1);
        }
      }
}

// The same in fp32: one warp per output.
__global__ void __launch_bounds__(128) head_gemm_f32_kernel(const HeadGemmParams p) {
  pdl_trigger();
  pdl_wait();
  const int h = blockIdx.y, lane = threadIdx.x & 31;
  const long long t = blockIdx.x;
  const float* a = static_cast<const float*>(p.a) + t * p.a_t + h * p.a_h;
  const float* w = static_cast<const float*>(p.w) + static_cast<long long>(h) * p.N * p.K;
  float* out = static_cast<float*>(p.out) + t * p.o_t + h * p.o_h;
  for (int n = threadIdx.x >> 5; n < p.N; n += 4) {
    float acc = 0.f;
    for (int k = lane; k < p.K; k += 32) acc = fmaf(a[k], w[static_cast<long long>(n) * p.K + k], acc);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (lane == 0) out[n] = acc;
  }
}

// ------------------------------------------------------------- cached rows, one sequence after another
struct LatentGatherParams {
  const uint4* cache;
  uint4* out;
  const int* block_tables;
  const int* seq_lens;
  const int* start;
  int max_blocks, block_size, vecs, total;
};

static constexpr int kGatherRows = 8;

__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentGatherParams p) {
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.y;
  const int n = p.seq_lens[b], j0 = blockIdx.x * kGatherRows;
  if (j0 >= n) return;
  const long long dst0 = p.start[b];
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const int rows = min(kGatherRows, n - j0);
  for (int i = threadIdx.x; i < rows * p.vecs; i += blockDim.x) {
    const int r = i / p.vecs, v = i - r * p.vecs;
    const int key = j0 + r;
    const long long row = static_cast<long long>(bt[key / p.block_size]) * p.block_size + key % p.block_size;
    if (dst0 + key < p.total) p.out[(dst0 + key) * p.vecs + v] = p.cache[row * p.vecs + v];
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_latent_prep(void* q, long long q_stride, const void* kv, long long kv_stride, const void* norm_w,
                                float eps, void* cache, const int* positions, const int* slots, const float* cos_sin,
                                int max_pos, int T, int H, int dim, int rot, int rank, int row, int neox,
                                void* q_latent, int num_latent, const void* low, long long low_stride,
                                const void* low_w, void* low_out, int low_rank, int low_width, int is_fp32,
                                cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((rot & 1) || row < rank + rot || (num_latent > 0 && q_latent == nullptr)) return -1;
  if (low != nullptr && (low_rank <= 0 || low_width < low_rank)) return -1;
  LatentPrepParams p{q, q_stride, kv, kv_stride, norm_w, eps, cache, positions, slots, cos_sin, max_pos,
                     H, dim, rot, rank, row, neox, num_latent, q_latent, low, low_stride, low_w, low_out, low_rank,
                     low_width};
  int ny = q ? (H * rot / 2 + 4 * kLatentThreads - 1) / (4 * kLatentThreads) : (kv && low ? 2 : 1);
  if (T >= 1024 || ny < 1) ny = 1;
  const auto whole = [&](const void* ptr, long long stride, int n) {
    return ptr == nullptr || ((reinterpret_cast<uintptr_t>(ptr) & (is_fp32 ? 31 : 15)) == 0 && stride % 8 == 0 && n % 8 == 0 &&
                              n <= kNormVecs * 256);
  };
  if (q == nullptr && whole(kv, kv_stride, rank) && whole(norm_w, 0, rank) && whole(low, low_stride, low_rank) &&
      whole(low_w, 0, low_rank) && whole(low_out, low_width, low_rank) && whole(kv ? cache : nullptr, row, rank) &&
      (low == nullptr || low_rank == low_width)) {
    const int items = T * ((kv ? 1 : 0) + (low ? 1 : 0)), per = kLatentThreads / 32;
    const dim3 grid((items + per - 1) / per), block(kLatentThreads);
    const cudaError_t e = is_fp32 ? launch_pdl(latent_norm_kernel<float>, grid, block, 0, stream, 1, p, T)
                                  : launch_pdl(latent_norm_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, p, T);
    return e == cudaSuccess ? 0 : -3;
  }
  const dim3 grid(T, ny), block(kLatentThreads);
  const cudaError_t e = is_fp32 ? launch_pdl(latent_prep_kernel<float>, grid, block, 0, stream, 1, p)
                                : launch_pdl(latent_prep_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, p);
  return e == cudaSuccess ? 0 : -3;
}

extern "C" int b200_head_gemm(const void* a, long long a_t, long long a_h, const void* w, void* out, long long o_t,
                              long long o_h, int T, int H, int N, int K, int is_fp32, cudaStream_t stream) {
  if (T <= 0 || N <= 0) return 0;
  const bool vec = K % 8 == 0 && a_t % 8 == 0 && a_h % 8 == 0 && (reinterpret_cast<uintptr_t>(a) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  HeadGemmParams p{a, w, out, a_t, a_h, o_t, o_h, T, H, N, K, vec ? 1 : 0};
  if (is_fp32)
    return launch_pdl(head_gemm_f32_kernel, dim3(T, H), dim3(128), 0, stream, 1, p) == cudaSuccess ? 0 : -3;
  const dim3 grid((N + hg::BN - 1) / hg::BN, H, (T + hg::BM - 1) / hg::BM);
  return launch_pdl(head_gemm_kernel, grid, dim3(hg::THREADS), 0, stream, 1, p) == cudaSuccess ? 0 : -3;
}

// row_bytes: a multiple of 16
extern "C" int b200_latent_gather(const void* cache, void* out, const int* block_tables, const int* seq_lens,
                                  const int* start, int B, int max_len, int max_blocks, int block_size, int row_bytes,
                                  int total, cudaStream_t stream) {
  if (B <= 0 || max_len <= 0) return 0;
  if (row_bytes & 15) return -1;
  LatentGatherParams p{static_cast<const uint4*>(cache), static_cast<uint4*>(out), block_tables, seq_lens, start,
                       max_blocks, block_size, row_bytes / 16, total};
  const dim3 grid((max_len + kGatherRows - 1) / kGatherRows, B);
  return launch_pdl(latent_gather_kernel, grid, dim3(256), 0, stream, 1, p) == cudaSuccess ? 0 : -3;
}
