// fp32 products on the CUDA cores: C[M,N] = A[M,K] * W[N,K]^T, dense or grouped by expert, with the
// activations of the tensor-core kernels.  It serves models that are run entirely in 32-bit
// (no reduced-precision tensor-core mode); any M, N, K.
//
// One CTA = a 64 x 64 tile, 256 threads x (4 x 4) outputs, K in steps of 16 through shared memory.

#include <cuda_runtime.h>
#include <stdint.h>

#include "../common/pdl.cuh"
#include "gated_act.cuh"

namespace b200 {

namespace simt {
constexpr int BM = 64, BN = 64, BK = 16, THREADS = 256;
}

struct SimtGemmParams {
  const float* A;
  const float* W;
  float* C;
  int M, N, K;
  long long lda, ldw, ldc;
  const int* expert_offsets;   // grouped: [E + 1] row offsets into A / C, W is [E, N, K]; null = dense
  int num_experts;
  const float* bias;           // [N] or null: added before a gated activation, after a unary one
  int act;                     // activation (gated: gate / up columns interleaved in groups of eight)
  float act_alpha, act_limit;
};

__global__ void __launch_bounds__(simt::THREADS) gemm_simt_kernel(const SimtGemmParams p) {
  using namespace simt;
  __shared__ float sA[BK][BM + 4];
  __shared__ float sW[BK][BN + 4];
  __shared__ float sC[BM][BN + 1];
  __shared__ int s_tile[3];    // first row, one past the last row, expert
  pdl_trigger();
  pdl_wait();
  const int tid = threadIdx.x;
  if (tid == 0) {
    int m0 = blockIdx.y * BM, m1 = p.M, e = 0;
    if (p.expert_offsets) {
      int tile = blockIdx.y;
      m0 = m1 = 0;
      for (; e < p.num_experts; ++e) {
        const int lo = p.expert_offsets[e], hi = p.expert_offsets[e + 1];
        const int tiles = (hi - lo + BM - 1) / BM;
        if (tile < tiles) {
          m0 = lo + tile * BM;
          m1 = hi;
          break;
        }
        tile -= tiles;
      }
    }
    s_tile[0] = m0;
    s_tile[1] = m1;
    s_tile[2] = e;
  }
  __syncthreads();
  const int m0 = s_tile[0], m1 = s_tile[1];
  if (m0 >= m1) return;                     // past the last expert's rows
  const float* W = p.W + (p.expert_offsets ? static_cast<long long>(s_tile[2]) * p.N * p.K : 0);
  const int n0 = blockIdx.x * BN;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += BK) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int r = (tid >> 4) + i * 16, c = tid & 15;
      const int row = m0 + r, col = n0 + r, k = k0 + c;
      sA[c][r] = (row < m1 && k < p.K) ? p.A[row * p.lda + k] : 0.f;
      sW[c][r] = (col < p.N && k < p.K) ? W[col * p.ldw + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < BK; ++k) {
      const float4 a = *reinterpret_cast<const float4*>(&sA[k][ty * 4]);
      const float4 b = *reinterpret_cast<const float4*>(&sW[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (!act_is_gated(p.act)) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int row = m0 + ty * 4 + i;
      if (row >= m1) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = n0 + tx * 4 + j;
        if (col >= p.N) continue;
        float x = acc[i][j];
        if (act_is_unary(p.act)) x = unary_act_exact(p.act, x, p.act_alpha, p.act_limit);
        p.C[row * p.ldc + col] = p.bias ? x + p.bias[col] : x;
      }
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) sC[ty * 4 + i][tx * 4 + j] = acc[i][j];
  __syncthreads();
  for (int idx = tid; idx < BM * BN / 2; idx += THREADS) {
    const int r = idx / (BN / 2), o = idx % (BN / 2);
    const int c = (o >> 3) * 16 + (o & 7);              // gate column of output column o
    if (m0 + r < m1 && n0 + c + 8 < p.N) {
      float g = sC[r][c], u = sC[r][c + 8];
      if (p.bias) {
        g += p.bias[n0 + c];
        u += p.bias[n0 + c + 8];
      }
      p.C[(m0 + r) * p.ldc + n0 / 2 + o] = gated_act_exact(p.act, g, u, p.act_alpha, p.act_limit);
    }
  }
}

}  // namespace b200

using namespace b200;

extern "C" int b200_gemm_simt(const float* A, const float* W, float* C, const float* bias, int M, int N, int K, long long lda,
                              long long ldw, long long ldc, const int* expert_offsets, int num_experts, int act,
                              float act_alpha, float act_limit, cudaStream_t stream) {
  if (M <= 0 || N <= 0) return 0;
  if (act_is_gated(act) && (N % 16) != 0) return -11;
  SimtGemmParams p{A, W, C, M, N, K, lda, ldw, ldc, expert_offsets, num_experts, bias, act, act_alpha, act_limit};
  // grouped: every expert may end in a partly filled tile
  const long long tiles = (M + simt::BM - 1) / simt::BM + (expert_offsets ? num_experts : 0);
  if (tiles > 65535) return -12;
  const dim3 grid((N + simt::BN - 1) / simt::BN, static_cast<unsigned>(tiles));
  return launch_pdl(gemm_simt_kernel, grid, dim3(simt::THREADS), 0, stream, 1, p) == cudaSuccess ? 0 : -3;
}
