// Recurrent layers: a matrix S per sequence and head, fp32, carried from token to token.
//
//   S <- diag(g) S;  S <- S + k u^T;  o = S^T q
//   gated linear attention:  u = v,                   k = 1 - g
//   delta rule:              u = beta (v - S^T k)     (after the decay)
//
// One elementwise kernel per kind prepares q, k, g and beta in fp32 from the projections, the scan runs
// the recurrence over a step's tokens (any mixture of prompt portions and single tokens), a last kernel
// norms each head's result and applies the output gate.  This file is compiled without the fast-math
// flag: what enters a recurrence keeps the accuracy of the fp32 functions.
//
// Arrays with a "d" axis are padded to a multiple of four (DP); the padding holds zeros.

#include <cuda_runtime.h>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "../common/rows.cuh"

namespace b200 {

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

// ------------------------------------------------------------- gated linear attention: q and keys
struct GatedPrepParams {
  const void* proj;
  long long stride;
  int q_off, f_off, heads, dim, DP;
  const float* f_bias;         // [heads * dim]
  const float* lower;          // [heads * dim]
  float* q;                    // [T, heads, DP]
  float* k;
};

template <typename T>
__global__ void __launch_bounds__(256) gated_prep_kernel(const GatedPrepParams p) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const T* row = static_cast<const T*>(p.proj) + t * p.stride;
  const int quads = p.DP >> 2, total = p.heads * quads;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < total; i += gridDim.y * blockDim.x) {
    const int h = i / quads, d0 = (i - h * quads) * 4;
    float q[4], k[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = d0 + j, c = h * p.dim + d;
      q[j] = k[j] = 0.f;
      if (d < p.dim) {
        q[j] = silu_f(as_float(row[p.q_off + c]));
        k[j] = (1.f - p.lower[c]) * sigmoid_f(-(as_float(row[p.f_off + c]) + p.f_bias[c]));
      }
    }
    const long long o = (t * total + i) * 4;
    *reinterpret_cast<float4*>(p.q + o) = make_float4(q[0], q[1], q[2], q[3]);
    *reinterpret_cast<float4*>(p.k + o) = make_float4(k[0], k[1], k[2], k[3]);
  }
}

// ------------------------------------------------------------- delta rule: convolutions, norms, decays
struct DeltaPrepParams {
  const void* proj;            // [T, ..]: q, k, v (the convolved columns) first, then the step sizes
  long long stride;
  const void* low;             // [T, heads * dim] decay before its bias
  long long low_stride;
  int q_off, k_off, v_off, b_off;
  int heads, groups, dim, vdim, DP, taps, channels;
  const void* conv_w;          // [channels, taps]
  const void* conv_state;      // [slots, taps - 1, channels]
  const float* dt_bias;        // [heads * dim]
  const float* a_log;          // [heads]
  float unit_eps, q_scale;
  const int* seq_idx;
  const int* state_slots;
  const int* cu_q;
  const int* seq_lens;
  float* q;                    // [T, groups, DP]
  float* k;                    // [T, groups, DP]
  float* g;                    // [T, heads, DP]
  void* v;                     // [T, heads * vdim]
  float* beta;                 // [T, heads]
  int T, run, v_parts;         // v_parts: warps that share a value head
};

static constexpr int kPrepWarps = 8;

// One warp = one unit (a head of q, k, v, or a head's decays) over a run of tokens; lane l has the
// channels l + 32 i.  The convolution's window slides in registers.
template <typename T, int CPL, int TAPS>
__global__ void __launch_bounds__(kPrepWarps * 32) delta_prep_kernel(const DeltaPrepParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  int unit = blockIdx.y * kPrepWarps + (threadIdx.x >> 5);
  const long long t0 = static_cast<long long>(blockIdx.x) * p.run;
  const long long t1 = min(t0 + p.run, static_cast<long long>(p.T));
  const int n_qk = 2 * p.groups, n_v = p.heads * p.v_parts;
  if (unit >= n_qk + n_v + p.heads) return;

  if (unit >= n_qk + n_v) {                               // decays and step size of a head
    const int h = unit - n_qk - n_v;
    const float a = expf(p.a_log[h]);
    for (long long t = t0; t < t1; ++t) {
      const T* low = static_cast<const T*>(p.low) + t * p.low_stride + static_cast<long long>(h) * p.dim;
      float* g = p.g + (t * p.heads + h) * p.DP;
      for (int d = lane; d < p.DP; d += 32)
        g[d] = d < p.dim ? expf(-a * softplus_f(as_float(low[d]) + p.dt_bias[h * p.dim + d])) : 0.f;
      if (lane == 0)
        p.beta[t * p.heads + h] = sigmoid_f(as_float(static_cast<const T*>(p.proj)[t * p.stride + p.b_off + h]));
    }
    return;
  }
  const bool is_v = unit >= n_qk;
  int col0, width, head, part = 0;
  if (is_v) {
    unit -= n_qk;
    head = unit / p.v_parts;
    part = unit - head * p.v_parts;
    col0 = p.v_off + head * p.vdim + part * 32 * CPL;
    width = min(p.vdim - part * 32 * CPL, 32 * CPL);
  } else {
    head = unit % p.groups;
    col0 = (unit < p.groups ? p.q_off : p.k_off) + head * p.dim;
    width = p.dim;
  }
  float w[CPL][TAPS], win[CPL][TAPS];
#pragma unroll
  for (int i = 0; i < CPL; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      // the last register is the current token's; shorter convolutions leave the first ones idle
      const int tap = j - (TAPS - p.taps);
      const int c = lane + 32 * i;
      w[i][j] = tap >= 0 && c < width
                    ? as_float(static_cast<const T*>(p.conv_w)[static_cast<long long>(col0 + c) * p.taps + tap]) : 0.f;
      win[i][j] = 0.f;
    }
  const T* proj = static_cast<const T*>(p.proj);
  long long begin = -1, end = -1;
  for (long long t = t0; t < t1; ++t) {
    if (t >= end) {                                       // first token of the run or of a portion
      const int b = p.seq_idx[t];
      begin = p.cu_q[b];
      end = p.cu_q[b + 1];
      const int slot = p.seq_lens[b] > static_cast<int>(end - begin) ? p.state_slots[b] : -1;
      // (the loop below shifts the window before it adds the current token)
#pragma unroll
      for (int j = 1; j < TAPS; ++j) {
        const long long rel = t - begin - (TAPS - j);
        const int row = static_cast<int>(rel) + p.taps - 1;         // of the stored inputs, when rel < 0
#pragma unroll
        for (int i = 0; i < CPL; ++i) {
          const int c = lane + 32 * i;
          float x = 0.f;
          if (c < width) {
            if (rel >= 0) x = as_float(proj[(begin + rel) * p.stride + col0 + c]);
            else if (row >= 0 && slot >= 0)
              x = as_float(static_cast<const T*>(p.conv_state)[(static_cast<long long>(slot) * (p.taps - 1) + row) *
                                                                   p.channels + col0 + c]);
          }
          win[i][j] = x;
        }
      }
    }
    float y[CPL], ss = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      const int c = lane + 32 * i;
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) win[i][j] = win[i][j + 1];
      win[i][TAPS - 1] = c < width ? as_float(proj[t * p.stride + col0 + c]) : 0.f;
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(w[i][j], win[i][j], acc);
      y[i] = silu_f(acc);
      ss = fmaf(y[i], y[i], ss);
    }
    if (is_v) {
      T* v = static_cast<T*>(p.v) + (t * p.heads + head) * p.vdim + part * 32 * CPL;
#pragma unroll
      for (int i = 0; i < CPL; ++i)
        if (lane + 32 * i < width) v[lane + 32 * i] = from_float<T>(y[i]);
      continue;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = (unit < p.groups ? p.q_scale : 1.f) / sqrtf(ss + p.unit_eps);
    float* dst = (unit < p.groups ? p.q : p.k) + (t * p.groups + head) * p.DP;
#pragma unroll
    for (int i = 0; i < CPL; ++i)
      if (lane + 32 * i < p.DP) dst[lane + 32 * i] = lane + 32 * i < width ? y[i] * inv : 0.f;
  }
}

// ------------------------------------------------------------- the scan
// One CTA = 32 columns (of the value axis) of one (sequence, head); a warp has 8 of them and all rows:
// lane = 16 * (column half) + row group, a thread 4 columns x RPT rows.  The column sums (S^T k, S^T q) are
// folded inside the warp, so that no block barrier stands between tokens.  q, k, g are staged CH tokens
// at a time through shared memory, the next ones on their way while these are worked off.
struct ScanParams {
  const float* q;              // [T, G, DP]
  const float* k;              // [T, G, DP]
  const float* g;              // [T, H, DP] (delta rule)
  const void* v;               // [T, H * E], row pitch v_stride
  long long v_stride;
  const float* beta;           // [T, H] (delta rule)
  float* state;                // [slots, H, E, DP]
  float* o;                    // [T, H, E]
  const int* state_slots;
  const int* cu_q;
  const int* seq_lens;
  int H, G, E, DP;
  const void* proj;            // newest convolution inputs to be kept, or null
  long long proj_stride;
  void* conv_state;            // [slots, keep, channels]
  int keep, channels;
};

namespace scan {
constexpr int WARPS = 4, THREADS = WARPS * 32, COLS = 32;
template <int RPT, bool DELTA>
struct Cfg {
  static constexpr int ROWS = 16 * RPT;
  static constexpr int CH = RPT <= 8 ? 16 : RPT <= 16 ? 8 : 4;
  static constexpr int ARR = DELTA ? 3 : 2;
  static constexpr int STAGE = ARR * CH * ROWS;                     // floats
  static constexpr int SMEM = (2 * STAGE + 2 * CH * (COLS + 1)) * 4;
};
}  // namespace scan

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src) : "memory");
}

// Sums of four columns over the 16 row groups; every lane ends with the one of column
// 2 * (bit 3 of the lane) + (bit 2).
__device__ __forceinline__ float fold_columns(const float (&a)[4], int lane) {
  const bool hi = lane & 8, odd = lane & 4;
  float k0 = hi ? a[2] : a[0], k1 = hi ? a[3] : a[1];
  k0 += __shfl_xor_sync(0xffffffffu, hi ? a[0] : a[2], 8);
  k1 += __shfl_xor_sync(0xffffffffu, hi ? a[1] : a[3], 8);
  float c = (odd ? k1 : k0) + __shfl_xor_sync(0xffffffffu, odd ? k0 : k1, 4);
  c += __shfl_xor_sync(0xffffffffu, c, 2);
  c += __shfl_xor_sync(0xffffffffu, c, 1);
  return c;
}

template <typename T, int RPT, bool DELTA>
__global__ void __launch_bounds__(scan::THREADS) recurrent_scan_kernel(const ScanParams p) {
  using namespace scan;
  using C = Cfg<RPT, DELTA>;
  constexpr int CH = C::CH, ROWS = C::ROWS, Q4 = RPT / 4;
  extern __shared__ __align__(16) float smem[];
  float* s_v = smem + 2 * C::STAGE;                       // [2][CH][COLS]
  float* s_b = s_v + 2 * CH * COLS;                       // [2][CH]

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int rg = lane & 15;
  const int b = blockIdx.z, h = blockIdx.y, c_base = blockIdx.x * COLS;
  const int grp = h / (p.H / p.G);
  const int col0 = warp * 8 + (lane >> 4) * 4;            // first of this thread's columns, within the CTA

  if (p.DP < ROWS) {                                      // rows beyond the head's size stay zero
    for (int i = tid; i < 2 * C::STAGE; i += THREADS) smem[i] = 0.f;
  }
  __syncthreads();
  pdl_trigger();
  pdl_wait();

  const long long begin = p.cu_q[b];
  const int n = static_cast<int>(p.cu_q[b + 1] - begin);
  if (n <= 0) return;
  const int slot = p.state_slots[b];
  const bool fresh = p.seq_lens[b] <= n || slot < 0;

  const int quads = p.DP >> 2;
  auto stage = [&](int c) {                               // start copying chunk c
    const int t0 = c * CH, m = min(CH, n - t0);
    float* dst = smem + (c & 1) * C::STAGE;
    for (int i = tid; i < C::ARR * m * quads; i += THREADS) {
      const int quad = i % quads, r = i / quads;
      const int arr = r / m, j = r - arr * m;
      const long long t = begin + t0 + j;
      const float* src = arr == 0 ? p.q + (t * p.G + grp) * p.DP
                                  : arr == 1 ? p.k + (t * p.G + grp) * p.DP : p.g + (t * p.H + h) * p.DP;
      cp_async16(dst + (arr * CH + j) * ROWS + quad * 4, src + quad * 4);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
    for (int i = tid; i < m * COLS; i += THREADS) {
      const int j = i / COLS, col = i % COLS;
      const long long t = begin + t0 + j;
      s_v[((c & 1) * CH + j) * COLS + col] =
          c_base + col < p.E ? as_float(static_cast<const T*>(p.v)[t * p.v_stride + static_cast<long long>(h) * p.E +
                                                                   c_base + col]) : 0.f;
    }
    if (DELTA && tid < m) s_b[(c & 1) * CH + tid] = p.beta[(begin + t0 + tid) * p.H + h];
  };
  stage(0);

  float s[4][RPT];
  float* st = p.state + ((static_cast<long long>(slot < 0 ? 0 : slot) * p.H + h) * p.E + c_base + col0) * p.DP;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int i = 0; i < Q4; ++i) {
      const int r = i * 64 + rg * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && r < p.DP && c_base + col0 + c < p.E)
        x = *reinterpret_cast<const float4*>(st + static_cast<long long>(c) * p.DP + r);
      s[c][4 * i] = x.x;
      s[c][4 * i + 1] = x.y;
      s[c][4 * i + 2] = x.z;
      s[c][4 * i + 3] = x.w;
    }

  const int my_col = col0 + ((lane >> 3) & 1) * 2 + ((lane >> 2) & 1);     // the column this lane has after a fold
  const bool writes = (lane & 3) == 0 && c_base + my_col < p.E;
  float* o = p.o + (begin * p.H + h) * p.E + c_base + my_col;
  const long long o_step = static_cast<long long>(p.H) * p.E;

  const int chunks = (n + CH - 1) / CH;
  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                      // chunk c is there; the buffer of c + 1 is free
    if (c + 1 < chunks) stage(c + 1);
    const float* sq = smem + (c & 1) * C::STAGE;
    const float* sk = sq + CH * ROWS;
    const float* sg = sk + CH * ROWS;
    const float* vv = s_v + (c & 1) * CH * COLS;
    const float* bb = s_b + (c & 1) * CH;
    const int m = min(CH, n - c * CH);
    for (int j = 0; j < m; ++j) {
      float k[RPT];
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(sk + j * ROWS + i * 64 + rg * 4);
        k[4 * i] = x.x; k[4 * i + 1] = x.y; k[4 * i + 2] = x.z; k[4 * i + 3] = x.w;
      }
      if (DELTA) {
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int i = 0; i < Q4; ++i) {
          const float4 x = *reinterpret_cast<const float4*>(sg + j * ROWS + i * 64 + rg * 4);
          const float g[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
          for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int cc = 0; cc < 4; ++cc) {
              s[cc][4 * i + e] *= g[e];
              acc[cc] = fmaf(s[cc][4 * i + e], k[4 * i + e], acc[cc]);
            }
        }
        const float u = bb[j] * (vv[j * COLS + my_col] - fold_columns(acc, lane));
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) {
          const float uc = __shfl_sync(0xffffffffu, u, (lane & 16) | (cc << 2));
#pragma unroll
          for (int r = 0; r < RPT; ++r) s[cc][r] = fmaf(k[r], uc, s[cc][r]);
        }
      } else {
        const float4 x = *reinterpret_cast<const float4*>(vv + j * COLS + col0);
        const float u[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int r = 0; r < RPT; ++r) {
          const float g = 1.f - k[r];
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) s[cc][r] = fmaf(s[cc][r], g, k[r] * u[cc]);
        }
      }
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < Q4; ++i) {
        const float4 x = *reinterpret_cast<const float4*>(sq + j * ROWS + i * 64 + rg * 4);
        const float q[4] = {x.x, x.y, x.z, x.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) acc[cc] = fmaf(s[cc][4 * i + e], q[e], acc[cc]);
      }
      const float r = fold_columns(acc, lane);
      if (writes) *o = r;
      o += o_step;
    }
  }
  if (slot < 0) return;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int i = 0; i < Q4; ++i) {
      const int r = i * 64 + rg * 4;
      if (r < p.DP && c_base + col0 + c < p.E)
        *reinterpret_cast<float4*>(st + static_cast<long long>(c) * p.DP + r) =
            make_float4(s[c][4 * i], s[c][4 * i + 1], s[c][4 * i + 2], s[c][4 * i + 3]);
    }
  if (p.proj && p.keep > 0) {
    // the newest `keep` inputs of the convolution, channels dealt out over this sequence's CTAs; a channel
    // is one thread's, oldest first, so that a row is read before it is overwritten
    T* cs = static_cast<T*>(p.conv_state) + static_cast<long long>(slot) * p.keep * p.channels;
    const T* src = static_cast<const T*>(p.proj);
    const int cta = h * gridDim.x + blockIdx.x, ctas = p.H * gridDim.x;
    for (int ch = cta * THREADS + tid; ch < p.channels; ch += ctas * THREADS)
      for (int j = 0; j < p.keep; ++j) {
        const int idx = n - p.keep + j;                   // token of the portion
        T x = from_float<T>(0.f);
        if (idx >= 0) x = src[(begin + idx) * p.proj_stride + ch];
        else if (!fresh) x = cs[static_cast<long long>(n + j) * p.channels + ch];
        cs[static_cast<long long>(j) * p.channels + ch] = x;
      }
  }
}

template <typename T, int RPT, bool DELTA>
static int launch_scan(const ScanParams& p, int B, cudaStream_t stream) {
  auto kern = recurrent_scan_kernel<T, RPT, DELTA>;
  constexpr int smem = scan::Cfg<RPT, DELTA>::SMEM;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -20;
    once.mark(dev);
  }
  const dim3 grid((p.E + scan::COLS - 1) / scan::COLS, p.H, B);
  return launch_pdl(kern, grid, dim3(scan::THREADS), smem, stream, 1, p) == cudaSuccess ? 0 : -21;
}

template <typename T, bool DELTA>
static int pick_scan(const ScanParams& p, int B, cudaStream_t stream) {
  if (p.DP <= 64) return launch_scan<T, 4, DELTA>(p, B, stream);
  if (p.DP <= 128) return launch_scan<T, 8, DELTA>(p, B, stream);
  if (p.DP <= 256) return launch_scan<T, 16, DELTA>(p, B, stream);
  if (p.DP <= 512) return launch_scan<T, 32, DELTA>(p, B, stream);
  return -2;
}

// ------------------------------------------------------------- norm and gate of a head's result
struct HeadNormParams {
  const float* o;              // [T, H, E]
  const void* w;               // [E]
  const void* gate;            // [T, H * E] before the sigmoid, or null
  long long gate_stride;
  void* out;                   // [T, out_width]
  int out_width, T, H, E;
  float eps;
};

static constexpr int kHeadNormWarps = 8;

template <typename T>
__global__ void __launch_bounds__(kHeadNormWarps * 32) head_norm_kernel(const HeadNormParams p) {
  pdl_trigger();
  pdl_wait();
  const long long unit = static_cast<long long>(blockIdx.x) * kHeadNormWarps + (threadIdx.x >> 5);
  if (unit >= static_cast<long long>(p.T) * p.H) return;
  const int lane = threadIdx.x & 31;
  const long long t = unit / p.H;
  const int h = static_cast<int>(unit - t * p.H);
  const float* o = p.o + unit * p.E;
  float ss = 0.f;
  for (int d = lane; d < p.E; d += 32) ss = fmaf(o[d], o[d], ss);
#pragma unroll
  for (int i = 16; i > 0; i >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, i);
  const float inv = 1.f / sqrtf(ss / static_cast<float>(p.E) + p.eps);
  const T* w = static_cast<const T*>(p.w);
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + t * p.gate_stride + static_cast<long long>(h) * p.E : nullptr;
  T* dst = static_cast<T*>(p.out) + t * p.out_width;
  for (int d = lane; d < p.E; d += 32) {
    float y = o[d] * inv * as_float(w[d]);
    if (gate) y *= sigmoid_f(as_float(gate[d]));
    dst[h * p.E + d] = from_float<T>(y);
  }
  if (h == p.H - 1)
    for (int d = p.H * p.E + lane; d < p.out_width; d += 32) dst[d] = from_float<T>(0.f);
}

template <typename T, int CPL>
static cudaError_t launch_delta_prep(const DeltaPrepParams& p, dim3 grid, cudaStream_t stream) {
  const dim3 block(kPrepWarps * 32);
  if (p.taps <= 4) return launch_pdl(delta_prep_kernel<T, CPL, 4>, grid, block, 0, stream, 1, p);
  return launch_pdl(delta_prep_kernel<T, CPL, 8>, grid, block, 0, stream, 1, p);
}

template <typename T>
static cudaError_t pick_delta_prep(const DeltaPrepParams& p, int cpl, dim3 grid, cudaStream_t stream) {
  if (cpl <= 4) return launch_delta_prep<T, 4>(p, grid, stream);
  if (cpl <= 8) return launch_delta_prep<T, 8>(p, grid, stream);
  return launch_delta_prep<T, 16>(p, grid, stream);
}

}  // namespace b200

using namespace b200;

extern "C" int b200_gated_linear_prep(const void* proj, long long stride, int q_off, int f_off, int heads, int dim,
                                      const float* f_bias, const float* lower, float* q, float* k, int T, int is_fp32,
                                      cudaStream_t stream) {
  if (T <= 0) return 0;
  const int DP = (dim + 3) / 4 * 4;
  GatedPrepParams p{proj, stride, q_off, f_off, heads, dim, DP, f_bias, lower, q, k};
  int ny = (heads * DP / 4 + 255) / 256;
  if (T >= 1024) ny = 1;
  const dim3 grid(T, ny);
  const cudaError_t e = is_fp32 ? launch_pdl(gated_prep_kernel<float>, grid, dim3(256), 0, stream, 1, p)
                                : launch_pdl(gated_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, 1, p);
  return e == cudaSuccess ? 0 : -3;
}

// dim up to 512, taps up to 8
extern "C" int b200_delta_prep(const void* proj, long long stride, const void* low, long long low_stride, int q_off,
                               int k_off, int v_off, int b_off, int heads, int groups, int dim, int vdim, int taps,
                               int channels, const void* conv_w, const void* conv_state, const float* dt_bias,
                               const float* a_log, float unit_eps, float q_scale, const int* seq_idx,
                               const int* state_slots, const int* cu_q, const int* seq_lens, float* q, float* k,
                               float* g, void* v, float* beta, int T, int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (dim > 512 || taps < 1 || taps > 8) return -1;
  int cpl = (dim + 31) / 32;
  cpl = cpl <= 4 ? 4 : cpl <= 8 ? 8 : 16;
  const int v_parts = (vdim + 32 * cpl - 1) / (32 * cpl);
  const int run = T >= 4096 ? 16 : T >= 1024 ? 4 : 1;
  DeltaPrepParams p{proj, stride, low, low_stride, q_off, k_off, v_off, b_off, heads, groups, dim, vdim,
                    (dim + 3) / 4 * 4, taps, channels, conv_w, conv_state, dt_bias, a_log, unit_eps, q_scale, seq_idx,
                    state_slots, cu_q, seq_lens, q, k, g, v, beta, T, run, v_parts};
  const int units = 2 * groups + heads * (v_parts + 1);
  const dim3 grid((T + run - 1) / run, (units + kPrepWarps - 1) / kPrepWarps);
  const cudaError_t e = is_fp32 ? pick_delta_prep<float>(p, cpl, grid, stream)
                                : pick_delta_prep<__nv_bfloat16>(p, cpl, grid, stream);
  return e == cudaSuccess ? 0 : -3;
}

// g and beta null: gated linear attention.  Head sizes (rows) up to 512.
extern "C" int b200_recurrent_scan(const float* q, const float* k, const float* g, const void* v, long long v_stride,
                                   const float* beta, float* state, float* o, const int* state_slots, const int* cu_q,
                                   const int* seq_lens, int B, int H, int G, int E, int DP, const void* proj,
                                   long long proj_stride, void* conv_state, int keep, int channels, int is_fp32,
                                   cudaStream_t stream) {
  if (B <= 0) return 0;
  if ((DP & 3) || G <= 0 || H % G) return -1;
  ScanParams p{q, k, g, v, v_stride, beta, state, o, state_slots, cu_q, seq_lens, H, G, E, DP, proj, proj_stride,
               conv_state, keep, channels};
  if (g) return is_fp32 ? pick_scan<float, true>(p, B, stream) : pick_scan<__nv_bfloat16, true>(p, B, stream);
  return is_fp32 ? pick_scan<float, false>(p, B, stream) : pick_scan<__nv_bfloat16, false>(p, B, stream);
}

extern "C" int b200_head_norm_gate(const float* o, const void* w, const void* gate, long long gate_stride, void* out,
                                   int out_width, int T, int H, int E, float eps, int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  HeadNormParams p{o, w, gate, gate_stride, out, out_width, T, H, E, eps};
  const long long units = static_cast<long long>(T) * H;
  const dim3 grid(static_cast<unsigned>((units + kHeadNormWarps - 1) / kHeadNormWarps)), block(kHeadNormWarps * 32);
  const cudaError_t e = is_fp32 ? launch_pdl(head_norm_kernel<float>, grid, block, 0, stream, 1, p)
                                : launch_pdl(head_norm_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, p);
  return e == cudaSuccess ? 0 : -3;
}
