// Several residual streams x_0 .. x_(N-1) per token: the join of one sublayer and the reading of the next,
// in one pass.
//
//   x_r  = table[id]                                     (start of the model; every stream), or
//   x_r <- sum_s mix[s, r] x_s + out_r * (scale * y)     (end of a sublayer, all r from the old streams)
//   u    = sum_s in_s x_s
//   h    = ((u - mean(u)) / sqrt(var(u) + eps) * w + b) * out_scale
//   out  = h + (h_before - h) * mu                       (token shift; h_before of the previous token)
//
// Streams, h and the shift's state are fp32; y, the vectors and out are bf16 or fp32.
//
// A CTA takes a run of consecutive tokens.  The token shift needs h of the token before the run: it is
// computed again from the old streams, which is why the new ones go to another buffer.  At the first token
// of a sequence's portion h_before comes from the sequence's state; the same CTA then stores the h of the
// portion's LAST token there (computing it again when it lies elsewhere), so that no other CTA touches the
// state.

#include <cuda_runtime.h>

#include "../common/pdl.cuh"
#include "../common/rows.cuh"

namespace b200 {

struct HyperNormParams {
  const float* streams;        // [T, N, W], or null with ids
  float* streams_out;          // [T, N, W], or null
  const int* ids;              // row of the table per token
  const void* table;           // [table_rows, W]
  int table_rows;
  const void* y;               // [T, W], pitch y_vecs
  long long y_vecs;
  const void* ls;              // [W]
  const float* mix;            // [N, N], [from, to]
  const float* w_out;          // [N]
  const float* w_in;           // [N]
  const void* norm_w;          // [W]
  const void* norm_b;          // [W]
  float eps, out_scale;
  const void* mu;              // [W], or null: no token shift
  float* state;                // [slots, W]
  const int* seq_idx;          // [T]
  const int* state_slots;      // [B], -1 = none
  const int* cu_q;             // [B + 1]
  const int* seq_lens;         // [B]
  void* out;                   // [T, W]
  int T, N, nvec, n_true, run;
};

// sum over the block, the same in every thread
__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  __syncthreads();                              // the previous sum has been read
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < static_cast<int>(blockDim.x >> 5); ++w) tot += red[w];
  return tot;
}

// h of token t in registers, four columns per vector; the new streams are written when asked for
template <typename T, int NMAX, int VPT>
__device__ __forceinline__ void hyper_row(const HyperNormParams& p, long long t, bool write, float (&h)[VPT][4],
                                          const float* s_mix, const float* s_out, const float* s_in, float* red) {
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
    for (int j = 0; j < 4; ++j) h[i][j] = 0.f;
    if (v >= p.nvec) continue;
    if (p.ids) {
      int id = p.ids[t];
      id = id < 0 ? 0 : (id >= p.table_rows ? p.table_rows - 1 : id);
      float x[4];
      Row4<T>::load(p.table, static_cast<long long>(id) * p.nvec + v, x);
      float w = 0.f;
#pragma unroll
      for (int s = 0; s < NMAX; ++s) {
        if (s < p.N) {
          w += s_in[s];
          if (write) Row4<float>::store(p.streams_out, (t * p.N + s) * p.nvec + v, x);
        }
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) h[i][j] = w * x[j];
    } else {
      float x[NMAX][4], y[4], ls[4];
#pragma unroll
      for (int s = 0; s < NMAX; ++s)
        if (s < p.N) Row4<float>::load(p.streams, (t * p.N + s) * p.nvec + v, x[s]);
      Row4<T>::load(p.y, t * p.y_vecs + v, y);
      Row4<T>::load(p.ls, v, ls);
#pragma unroll
      for (int j = 0; j < 4; ++j) y[j] *= ls[j];
#pragma unroll
      for (int r = 0; r < NMAX; ++r) {
        if (r < p.N) {
          float n[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) n[j] = s_out[r] * y[j];
#pragma unroll
          for (int s = 0; s < NMAX; ++s)
            if (s < p.N) {
              const float m = s_mix[s * p.N + r];
#pragma unroll
              for (int j = 0; j < 4; ++j) n[j] = fmaf(m, x[s][j], n[j]);
            }
          if (write) Row4<float>::store(p.streams_out, (t * p.N + r) * p.nvec + v, n);
#pragma unroll
          for (int j = 0; j < 4; ++j) h[i][j] = fmaf(s_in[r], n[j], h[i][j]);
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (v * 4 + j < p.n_true) sum += h[i][j];
  }
  const float mean = block_sum(sum, red) / static_cast<float>(p.n_true);
  float sq = 0.f;
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      h[i][j] -= mean;
      if (v * 4 + j < p.n_true) sq = fmaf(h[i][j], h[i][j], sq);
    }
  }
  const float inv = 1.f / sqrtf(block_sum(sq, red) / static_cast<float>(p.n_true) + p.eps);
#pragma unroll
  for (int i = 0; i < VPT; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v >= p.nvec) continue;
    float w[4], b[4];
    Row4<T>::load(p.norm_w, v, w);
    Row4<T>::load(p.norm_b, v, b);
#pragma unroll
    for (int j = 0; j < 4; ++j)
      h[i][j] = v * 4 + j < p.n_true ? fmaf(h[i][j] * inv, w[j], b[j]) * p.out_scale : 0.f;
  }
}

template <typename T, int NMAX, int VPT>
__global__ void __launch_bounds__(512) hyper_norm_kernel(const HyperNormParams p) {
  __shared__ float red[16];
  __shared__ float s_mix[NMAX * NMAX], s_out[NMAX], s_in[NMAX];
  pdl_trigger();
  // (parameters: no earlier kernel writes them)
  if (threadIdx.x < p.N * p.N && p.mix) s_mix[threadIdx.x] = p.mix[threadIdx.x];
  if (threadIdx.x < p.N) {
    s_in[threadIdx.x] = p.w_in[threadIdx.x];
    s_out[threadIdx.x] = p.w_out ? p.w_out[threadIdx.x] : 0.f;
  }
  __syncthreads();
  pdl_wait();
  const long long t0 = static_cast<long long>(blockIdx.x) * p.run;
  const long long t1 = min(t0 + p.run, static_cast<long long>(p.T));
  const bool write = p.streams_out != nullptr;
  float prev[VPT][4], h[VPT][4];
#pragma unroll
  for (int i = 0; i < VPT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) prev[i][j] = 0.f;

  // rows are computed in one place: the token before the run, the run's tokens, and behind the first token
  // of a portion the portion's last one
  enum { kBefore, kOwn, kLast };
  long long t = t0, last = -1;
  int slot = -1, what = kOwn;
  auto enter = [&]() {                                     // looks up where token t lies
    slot = -1;
    what = kOwn;
    if (!p.mu) return;
    const int b = p.seq_idx[t];
    if (p.cu_q[b] == t) {
      slot = p.state_slots[b];
      last = p.cu_q[b + 1] - 1;
      const bool from_state = slot >= 0 && p.seq_lens[b] > static_cast<int>(last - t) + 1;
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
#pragma unroll
        for (int j = 0; j < 4; ++j) prev[i][j] = 0.f;
        if (from_state && v < p.nvec) Row4<float>::load(p.state, static_cast<long long>(slot) * p.nvec + v, prev[i]);
      }
    } else if (t == t0) {
      what = kBefore;
    }
  };
  enter();
  while (true) {
    hyper_row<T, NMAX, VPT>(p, what == kBefore ? t - 1 : what == kOwn ? t : last, write && what == kOwn, h, s_mix, s_out,
                            s_in, red);
    if (what == kBefore) {
#pragma unroll
      for (int i = 0; i < VPT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) prev[i][j] = h[i][j];
      what = kOwn;
      continue;
    }
    if (what == kOwn) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v >= p.nvec) continue;
        float o[4] = {h[i][0], h[i][1], h[i][2], h[i][3]};
        if (p.mu) {
          float mu[4];
          Row4<T>::load(p.mu, v, mu);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            o[j] = fmaf(prev[i][j] - h[i][j], mu[j], h[i][j]);
            prev[i][j] = h[i][j];
          }
        }
        Row4<T>::store(p.out, t * p.nvec + v, o);
      }
      if (slot >= 0 && last != t) {
        what = kLast;
        continue;
      }
    }
    if (slot >= 0) {
#pragma unroll
      for (int i = 0; i < VPT; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < p.nvec) Row4<float>::store(p.state, static_cast<long long>(slot) * p.nvec + v, h[i]);
      }
    }
    if (++t >= t1) break;
    enter();
  }
}

template <typename T, int NMAX>
static cudaError_t launch_hyper_norm(const HyperNormParams& p, int threads, int vpt, int blocks, cudaStream_t stream) {
  if (vpt <= 1) return launch_pdl(hyper_norm_kernel<T, NMAX, 1>, dim3(blocks), dim3(threads), 0, stream, 1, p);
  if (vpt <= 2) return launch_pdl(hyper_norm_kernel<T, NMAX, 2>, dim3(blocks), dim3(threads), 0, stream, 1, p);
  if (vpt <= 4) return launch_pdl(hyper_norm_kernel<T, NMAX, 4>, dim3(blocks), dim3(threads), 0, stream, 1, p);
  return launch_pdl(hyper_norm_kernel<T, NMAX, 8>, dim3(blocks), dim3(threads), 0, stream, 1, p);
}

template <typename T>
static cudaError_t pick_hyper_norm(const HyperNormParams& p, int threads, int vpt, int blocks, cudaStream_t stream) {
  if (p.N <= 2) return launch_hyper_norm<T, 2>(p, threads, vpt, blocks, stream);
  if (p.N <= 4) return launch_hyper_norm<T, 4>(p, threads, vpt, blocks, stream);
  return launch_hyper_norm<T, 8>(p, threads, vpt, blocks, stream);
}

}  // namespace b200

using namespace b200;

// W: row width in elements, a multiple of 8, at most 16384; N: 1 to 8 streams.
extern "C" int b200_hyper_norm(const float* streams, float* streams_out, const int* ids, const void* table,
                               int table_rows, const void* y, long long y_stride, const void* ls, const float* mix,
                               const float* w_out, const float* w_in, const void* norm_w, const void* norm_b, float eps,
                               float out_scale, const void* mu, float* state, const int* seq_idx,
                               const int* state_slots, const int* cu_q, const int* seq_lens, void* out, int T, int N,
                               int W, int n_true, int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if ((W & 7) || (y_stride & 7) || W > 16384 || N < 1 || N > 8 || n_true <= 0 || n_true > W) return -1;
  HyperNormParams p{streams, streams_out, ids, table, table_rows, y, y_stride >> 2, ls, mix, w_out, w_in, norm_w, norm_b,
                    eps, out_scale, mu, state, seq_idx, state_slots, cu_q, seq_lens, out, T, N, W >> 2, n_true, 1};
  int threads = (p.nvec + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  if (threads < 64) threads = 64;                       // the streams' small matrices are loaded by one thread each
  const int vpt = (p.nvec + threads - 1) / threads;
  // the token before a run is computed twice: longer runs when there are tokens enough for every SM
  if (mu) p.run = T >= 148 * 16 ? 8 : T >= 148 * 4 ? 4 : 1;
  const int blocks = (T + p.run - 1) / p.run;
  const cudaError_t e = is_fp32 ? pick_hyper_norm<float>(p, threads, vpt, blocks, stream)
                                : pick_hyper_norm<__nv_bfloat16>(p, threads, vpt, blocks, stream);
  return e == cudaSuccess ? 0 : -3;
}
