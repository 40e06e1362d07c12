// Preparation of the recurrent layers with a free decay (recurrent.cu: S <- diag(g) S + k v^T):
//
//   token_mix         rows h_t + (h_(t-1) - h_t) mu_s for several s at once; h_(t-1) of a portion's first
//                     token is kept per sequence
//   time_mix_prep     r, k, g = exp(-exp(z + w0)) and the weight sum_d r u k of the current token
//   decay_prep        q * scale, k, g = sigmoid(z + bias)^(1 / tau)
//
// Arrays with a "d" axis are padded to a multiple of four (DP); the padding holds zeros.  Compiled without
// the fast-math flag, like recurrent.cu.

#include <cuda_runtime.h>

#include "../common/pdl.cuh"
#include "../common/rows.cuh"
#include "recurrent_common.cuh"

namespace b200 {

// ------------------------------------------------------------- blends with the previous token
static constexpr int kMixThreads = 128;
static constexpr int kMaxMixes = 6;

struct TokenMixParams {
  const void* h;               // [T, W], W a multiple of 8
  long long h_vecs;            // pitch in vectors of eight elements
  const void* mu;              // [n, W]
  float* state;                // [slots, W]: h of a sequence's newest token
  const int* seq_idx;
  const int* state_slots;
  const int* cu_q;
  const int* seq_lens;
  void* out;                   // [n, T, W]
  int* offsets;                // [n + 1] first row of each blend in out
  int T, nvec, run;
};

// One thread = eight columns over a run of tokens.  The thread with a portion's first token reads the
// sequence's state and then replaces it by the portion's last row, so no other one touches it.
template <typename T, int N>
__global__ void __launch_bounds__(kMixThreads) token_mix_kernel(const TokenMixParams p) {
  pdl_trigger();
  const int v = blockIdx.y * kMixThreads + threadIdx.x;
  pdl_wait();
  if (blockIdx.x == 0 && v <= N) p.offsets[v] = v * p.T;
  if (v >= p.nvec) return;
  float mu[N][8];
#pragma unroll
  for (int s = 0; s < N; ++s) Row8<T>::load(p.mu, static_cast<long long>(s) * p.nvec + v, mu[s]);
  const long long t0 = static_cast<long long>(blockIdx.x) * p.run;
  const long long t1 = min(t0 + p.run, static_cast<long long>(p.T));
  long long end = -1;
  float before[8], x[8], y[8];
  for (long long t = t0; t < t1; ++t) {
    Row8<T>::load(p.h, t * p.h_vecs + v, x);
    if (t >= end) {                                       // first token of the run or of a portion
      const int b = p.seq_idx[t];
      const long long begin = p.cu_q[b];
      end = p.cu_q[b + 1];
      if (t > begin) {
        Row8<T>::load(p.h, (t - 1) * p.h_vecs + v, before);
      } else {
        const int slot = p.state_slots[b];
#pragma unroll
        for (int j = 0; j < 8; ++j) before[j] = 0.f;
        if (slot >= 0) {
          const long long row = static_cast<long long>(slot) * p.nvec + v;
          if (p.seq_lens[b] > static_cast<int>(end - begin)) Row8<float>::load(p.state, row, before);
          Row8<T>::load(p.h, (end - 1) * p.h_vecs + v, y);
          Row8<float>::store(p.state, row, y);
        }
      }
    }
#pragma unroll
    for (int s = 0; s < N; ++s) {
#pragma unroll
      for (int j = 0; j < 8; ++j) y[j] = fmaf(before[j] - x[j], mu[s][j], x[j]);
      Row8<T>::store(p.out, (static_cast<long long>(s) * p.T + t) * p.nvec + v, y);
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) before[j] = x[j];
  }
}

// ------------------------------------------------------------- decays
struct DecayPrepParams {
  const void* q;               // [T, heads * dim] each
  const void* k;
  long long q_stride, k_stride;
  const float* z;              // [T, heads * dim]
  long long z_stride;
  const float* bias;           // [heads * dim]
  const float* u;              // [heads, dim], time mixing only
  float* q_out;                // [T, heads, DP] each
  float* k_out;
  float* g_out;
  float* bonus;                // [T, heads], time mixing only
  long long units;             // T * heads
  int heads, dim, DP;
  int lanes;                   // of a warp that share a head: a power of two
  float q_scale, inv_tau;
  int vec;                     // heads are whole four-element pieces everywhere
};

static constexpr int kDecayWarps = 8;

template <typename T, bool TIME_MIX>
__global__ void __launch_bounds__(kDecayWarps * 32) decay_prep_kernel(const DecayPrepParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, per_warp = 32 / p.lanes;
  const long long unit = (static_cast<long long>(blockIdx.x) * kDecayWarps + (threadIdx.x >> 5)) * per_warp + lane / p.lanes;
  const bool live = unit < p.units;
  const long long t = live ? unit / p.heads : 0;
  const int h = live ? static_cast<int>(unit - t * p.heads) : 0;
  const int c0 = h * p.dim, quads = live ? p.DP >> 2 : 0;
  const T* qs = static_cast<const T*>(p.q) + t * p.q_stride + c0;
  const T* ks = static_cast<const T*>(p.k) + t * p.k_stride + c0;
  const float* zs = p.z + t * p.z_stride + c0;
  float sum = 0.f;
  for (int i = lane & (p.lanes - 1); i < quads; i += p.lanes) {
    float q[4], k[4], g[4], b[4], u[4];
    if (p.vec) {
      Row4<T>::load(qs, i, q);
      Row4<T>::load(ks, i, k);
      Row4<float>::load(zs, i, g);
      Row4<float>::load(p.bias + c0, i, b);
      if (TIME_MIX) Row4<float>::load(p.u + c0, i, u);
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int d = i * 4 + j;
        q[j] = k[j] = g[j] = b[j] = u[j] = 0.f;
        if (d < p.dim) {
          q[j] = as_float(qs[d]);
          k[j] = as_float(ks[d]);
          g[j] = zs[d];
          b[j] = p.bias[c0 + d];
          if (TIME_MIX) u[j] = p.u[c0 + d];
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float z = g[j] + b[j];
      if (TIME_MIX) {
        sum = fmaf(q[j] * u[j], k[j], sum);
        g[j] = expf(-expf(z));
      } else {
        q[j] *= p.q_scale;
        g[j] = expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau);       // log sigmoid(z) / tau
      }
      if (!p.vec && i * 4 + j >= p.dim) g[j] = 0.f;
    }
    const long long o = unit * (p.DP >> 2) + i;
    Row4<float>::store(p.q_out, o, q);
    Row4<float>::store(p.k_out, o, k);
    Row4<float>::store(p.g_out, o, g);
  }
  if (TIME_MIX) {
    for (int o = p.lanes >> 1; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (live && (lane & (p.lanes - 1)) == 0) p.bonus[unit] = sum;
  }
}

template <typename T>
static cudaError_t launch_decay_prep(const DecayPrepParams& p, bool time_mix, cudaStream_t stream) {
  const long long per_cta = static_cast<long long>(kDecayWarps) * (32 / p.lanes);
  const dim3 grid(static_cast<unsigned>((p.units + per_cta - 1) / per_cta)), block(kDecayWarps * 32);
  return time_mix ? launch_pdl(decay_prep_kernel<T, true>, grid, block, 0, stream, 1, p)
                  : launch_pdl(decay_prep_kernel<T, false>, grid, block, 0, stream, 1, p);
}

template <typename T>
static cudaError_t launch_token_mix(const TokenMixParams& p, int n, cudaStream_t stream) {
  const dim3 grid(static_cast<unsigned>((p.T + p.run - 1) / p.run), (p.nvec + kMixThreads - 1) / kMixThreads);
  const dim3 block(kMixThreads);
  switch (n) {
    case 1: return launch_pdl(token_mix_kernel<T, 1>, grid, block, 0, stream, 1, p);
    case 2: return launch_pdl(token_mix_kernel<T, 2>, grid, block, 0, stream, 1, p);
    case 3: return launch_pdl(token_mix_kernel<T, 3>, grid, block, 0, stream, 1, p);
    case 4: return launch_pdl(token_mix_kernel<T, 4>, grid, block, 0, stream, 1, p);
    case 5: return launch_pdl(token_mix_kernel<T, 5>, grid, block, 0, stream, 1, p);
    default: return launch_pdl(token_mix_kernel<T, 6>, grid, block, 0, stream, 1, p);
  }
}

}  // namespace b200

using namespace b200;

// W and the pitch: multiples of 8; n: 1 to 6 blends.
extern "C" int b200_token_mix(const void* h, long long h_stride, const void* mu, int n, float* state,
                              const int* seq_idx, const int* state_slots, const int* cu_q, const int* seq_lens,
                              void* out, int* offsets, int T, int W, int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (n < 1 || n > kMaxMixes || (W & 7) || (h_stride & 7) || (reinterpret_cast<uintptr_t>(h) & 15)) return -1;
  const int run = T >= 4096 ? 8 : T >= 1024 ? 4 : 1;
  TokenMixParams p{h, h_stride >> 3, mu, state, seq_idx, state_slots, cu_q, seq_lens, out, offsets, T, W >> 3, run};
  const cudaError_t e = is_fp32 ? launch_token_mix<float>(p, n, stream) : launch_token_mix<__nv_bfloat16>(p, n, stream);
  return e == cudaSuccess ? 0 : -3;
}

// u null: decay sigmoid(z + bias)^inv_tau, q times q_scale; else the time mixing's decay and bonus.
extern "C" int b200_decay_prep(const void* q, long long q_stride, const void* k, long long k_stride, const float* z,
                               long long z_stride, const float* bias, const float* u, float* q_out, float* k_out,
                               float* g_out, float* bonus, int T, int heads, int dim, float q_scale, float inv_tau,
                               int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const int DP = (dim + 3) / 4 * 4;
  int lanes = 1;
  while (lanes < 32 && lanes < DP / 4) lanes <<= 1;
  const uintptr_t align = is_fp32 ? 15 : 7;
  const bool vec = dim % 4 == 0 && q_stride % 4 == 0 && k_stride % 4 == 0 && z_stride % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(q) & align) == 0 && (reinterpret_cast<uintptr_t>(k) & align) == 0 &&
                   (reinterpret_cast<uintptr_t>(z) & 15) == 0 && (reinterpret_cast<uintptr_t>(bias) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(u) & 15) == 0;
  DecayPrepParams p{q, k, q_stride, k_stride, z, z_stride, bias, u, q_out, k_out, g_out, bonus,
                    static_cast<long long>(T) * heads, heads, dim, DP, lanes, q_scale, inv_tau, vec ? 1 : 0};
  const cudaError_t e = is_fp32 ? launch_decay_prep<float>(p, u != nullptr, stream)
                                : launch_decay_prep<__nv_bfloat16>(p, u != nullptr, stream);
  return e == cudaSuccess ? 0 : -3;
}
