// Recurrent layers: a matrix S per sequence and head, fp32, carried from token to token.
//
//   S <- diag(g) S;  S <- S + k u^T;  o = S^T q
//   tied:    u = v,                   k = 1 - g
//   delta:   u = beta (v - S^T k)     (after the decay)
//   decay:   u = v,                   g free
//   bonus:   as decay, but o = S^T q + beta v of the S before this token (beta: the current token's weight)
//
// One elementwise kernel per kind prepares q, k, g and beta in fp32 from the projections (here and in
// decay_prep.cu), the scan runs
// the recurrence over a step's tokens (any mixture of prompt portions and single tokens), a last kernel
// norms each head's result and applies the output gate.  This file is compiled without the fast-math
// flag: what enters a recurrence keeps the accuracy of the fp32 functions.
//
// Arrays with a "d" axis are padded to a multiple of four (DP); the padding holds zeros.

#include <cuda_runtime.h>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "../common/rows.cuh"
#include "recurrent_common.cuh"

namespace b200 {

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

// One warp = one unit (a head of q, k, v, or a head's decays) over a run of tokens.  PAIR: a lane has the
// channels 2 lane + 64 i and the one after it, else lane + 32 i.  The convolution's window slides in
// registers; the next token's inputs are requested before the current ones are worked off.
template <typename T>
__device__ __forceinline__ void load_pair(const T* p, float& a, float& b);
template <>
__device__ __forceinline__ void load_pair(const float* p, float& a, float& b) {
  const float2 x = *reinterpret_cast<const float2*>(p);
  a = x.x;
  b = x.y;
}
template <>
__device__ __forceinline__ void load_pair(const __nv_bfloat16* p, float& a, float& b) {
  const uint32_t x = *reinterpret_cast<const uint32_t*>(p);
  a = __uint_as_float(x << 16);
  b = __uint_as_float(x & 0xffff0000u);
}

__device__ __forceinline__ void store_pair(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store_pair(__nv_bfloat16* p, float a, float b) {
  *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// CPL channels of a lane from a row; those at or beyond `width` are zero
template <typename T, int CPL, bool PAIR>
__device__ __forceinline__ void load_channels(const T* row, int lane, int width, float (&x)[CPL]) {
  if constexpr (PAIR) {
#pragma unroll
    for (int i = 0; i < CPL; i += 2) {
      const int c = lane * 2 + 32 * i;
      x[i] = x[i + 1] = 0.f;
      if (c < width) load_pair<T>(row + c, x[i], x[i + 1]);
    }
  } else {
#pragma unroll
    for (int i = 0; i < CPL; ++i) x[i] = lane + 32 * i < width ? as_float(row[lane + 32 * i]) : 0.f;
  }
}

__device__ __forceinline__ float quick_sigmoid(float z) { return __fdividef(1.f, 1.f + expf(-z)); }

template <typename T, int CPL, int TAPS, bool PAIR>
__global__ void __launch_bounds__(kPrepWarps * 32) delta_prep_kernel(const DeltaPrepParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  int unit = blockIdx.y * kPrepWarps + (threadIdx.x >> 5);
  const long long t0 = static_cast<long long>(blockIdx.x) * p.run;
  const long long t1 = min(t0 + p.run, static_cast<long long>(p.T));
  const int n_qk = 2 * p.groups, n_v = p.heads * p.v_parts;
  if (unit >= n_qk + n_v + p.heads) return;
  auto channel = [&](int i) { return PAIR ? lane * 2 + 32 * (i & ~1) + (i & 1) : lane + 32 * i; };

  if (unit >= n_qk + n_v) {                               // decays and step size of a head
    const int h = unit - n_qk - n_v;
    const float a = expf(p.a_log[h]);
    float bias[CPL], x[CPL], nx[CPL];
    load_channels<float, CPL, PAIR>(p.dt_bias + h * p.dim, lane, p.dim, bias);
    const T* low = static_cast<const T*>(p.low) + static_cast<long long>(h) * p.dim;
    load_channels<T, CPL, PAIR>(low + t0 * p.low_stride, lane, p.dim, nx);
    for (long long t = t0; t < t1; ++t) {
#pragma unroll
      for (int i = 0; i < CPL; ++i) x[i] = nx[i];
      if (t + 1 < t1) load_channels<T, CPL, PAIR>(low + (t + 1) * p.low_stride, lane, p.dim, nx);
      float* g = p.g + (t * p.heads + h) * p.DP;
#pragma unroll
      for (int i = 0; i < CPL; ++i) x[i] = channel(i) < p.dim ? expf(-a * softplus_f(x[i] + bias[i])) : 0.f;
#pragma unroll
      for (int i = 0; i < CPL; i += 2) {
        if constexpr (PAIR) {
          if (channel(i) < p.DP) *reinterpret_cast<float2*>(g + channel(i)) = make_float2(x[i], x[i + 1]);
        } else {
          if (channel(i) < p.DP) g[channel(i)] = x[i];
          if (channel(i + 1) < p.DP) g[channel(i + 1)] = x[i + 1];
        }
      }
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
  float w[CPL][TAPS], win[CPL][TAPS], next[CPL];
#pragma unroll
  for (int i = 0; i < CPL; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      // the last register is the current token's; shorter convolutions leave the first ones idle
      const int tap = j - (TAPS - p.taps);
      const int c = channel(i);
      w[i][j] = tap >= 0 && c < width
                    ? as_float(static_cast<const T*>(p.conv_w)[static_cast<long long>(col0 + c) * p.taps + tap]) : 0.f;
      win[i][j] = 0.f;
    }
  const T* proj = static_cast<const T*>(p.proj) + col0;
  load_channels<T, CPL, PAIR>(proj + t0 * p.stride, lane, width, next);
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
        float x[CPL];
#pragma unroll
        for (int i = 0; i < CPL; ++i) x[i] = 0.f;
        if (rel >= 0)
          load_channels<T, CPL, PAIR>(proj + (begin + rel) * p.stride, lane, width, x);
        else if (row >= 0 && slot >= 0)
          load_channels<T, CPL, PAIR>(static_cast<const T*>(p.conv_state) +
                                          (static_cast<long long>(slot) * (p.taps - 1) + row) * p.channels + col0,
                                      lane, width, x);
#pragma unroll
        for (int i = 0; i < CPL; ++i) win[i][j] = x[i];
      }
    }
    float y[CPL], ss = 0.f;
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
#pragma unroll
      for (int j = 0; j + 1 < TAPS; ++j) win[i][j] = win[i][j + 1];
      win[i][TAPS - 1] = next[i];
    }
    if (t + 1 < t1) load_channels<T, CPL, PAIR>(proj + (t + 1) * p.stride, lane, width, next);
#pragma unroll
    for (int i = 0; i < CPL; ++i) {
      float acc = 0.f;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) acc = fmaf(w[i][j], win[i][j], acc);
      y[i] = acc * quick_sigmoid(acc);
      ss = fmaf(y[i], y[i], ss);
    }
    if (is_v) {
      T* v = static_cast<T*>(p.v) + (t * p.heads + head) * p.vdim + part * 32 * CPL;
#pragma unroll
      for (int i = 0; i < CPL; i += 2) {
        if constexpr (PAIR) {
          if (channel(i) < width) store_pair(v + channel(i), y[i], y[i + 1]);
        } else {
          if (channel(i) < width) v[channel(i)] = from_float<T>(y[i]);
          if (channel(i + 1) < width) v[channel(i + 1)] = from_float<T>(y[i + 1]);
        }
      }
      continue;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float inv = (unit < p.groups ? p.q_scale : 1.f) / sqrtf(ss + p.unit_eps);
    float* dst = (unit < p.groups ? p.q : p.k) + (t * p.groups + head) * p.DP;
#pragma unroll
    for (int i = 0; i < CPL; i += 2) {
      // (channels beyond the head have no weights and are zero)
      if constexpr (PAIR) {
        if (channel(i) < p.DP) *reinterpret_cast<float2*>(dst + channel(i)) = make_float2(y[i] * inv, y[i + 1] * inv);
      } else {
        if (channel(i) < p.DP) dst[channel(i)] = y[i] * inv;
        if (channel(i + 1) < p.DP) dst[channel(i + 1)] = y[i + 1] * inv;
      }
    }
  }
}

// ------------------------------------------------------------- the scan
// One CTA = 32 columns (of the value axis) of one (sequence, head); a warp has 8 of them and all rows:
// lane = 16 * (column half) + row group, a thread four columns x RPT rows, rows in pairs for the packed fp32
// instructions.  (Every thread reads RPT elements of q, k and g per token: with more rows and fewer columns
// per thread shared memory, 128 bytes per clock and SM, would have as much to do as the arithmetic.)  The
// column sums (S^T k, and S^T q of four tokens at a time) are folded inside the warp, so that no block
// barrier stands between tokens.  q, k, g and v are staged CH tokens at a time through shared memory, the
// next ones on their way while these are worked off.
struct ScanParams {
  const float* q;              // [T, G, DP]
  const float* k;              // [T, G, DP]
  const float* g;              // [T, H, DP] (not tied)
  const void* v;               // [T, H * E], row pitch v_stride
  long long v_stride;
  const float* beta;           // [T, H] (delta, bonus)
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
constexpr int WARPS = 4, THREADS = WARPS * 32, COLS = 32, GROUP = 4;
enum : int { TIED = 0, DELTA = 1, DECAY = 2, BONUS = 3 };
template <int RPT, int MODE>
struct Cfg {
  static constexpr int ROWS = 16 * RPT;
  static constexpr int CH = RPT <= 8 ? 16 : RPT <= 16 ? 8 : 4;
  static constexpr int ARR = MODE == TIED ? 2 : 3;
  static constexpr int STAGE = ARR * CH * ROWS;                     // floats
  static constexpr int SMEM = (2 * STAGE + 2 * CH * (COLS + 1)) * 4;
};
}  // namespace scan

__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(static_cast<uint32_t>(__cvta_generic_to_shared(dst))),
               "l"(src) : "memory");
}

// two fp32 numbers in a 64-bit register
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ float sum2(f32x2 x) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(x));
  return lo + hi;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

template <typename T, int RPT, int MODE>
__global__ void __launch_bounds__(scan::THREADS) recurrent_scan_kernel(const ScanParams p) {
  using namespace scan;
  using C = Cfg<RPT, MODE>;
  constexpr int CH = C::CH, ROWS = C::ROWS, Q4 = RPT / 4;
  constexpr bool KEEP_K = RPT <= 16;                      // k of a token in registers between its two uses
  extern __shared__ __align__(16) float smem[];
  T* s_v = reinterpret_cast<T*>(smem + 2 * C::STAGE);     // [2][CH][COLS]
  float* s_b = smem + 2 * C::STAGE + 2 * CH * COLS;       // [2][CH]

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
  const T* v_src = static_cast<const T*>(p.v) + begin * p.v_stride + static_cast<long long>(h) * p.E + c_base;
  constexpr int VPIECES = COLS * static_cast<int>(sizeof(T)) / 16;          // 16-byte pieces of a token's columns
  const bool v_vec = c_base + COLS <= p.E && (reinterpret_cast<uintptr_t>(v_src) & 15) == 0 &&
                     (p.v_stride * sizeof(T)) % 16 == 0;
  auto stage = [&](int c) {                               // start copying chunk c
    const int t0 = c * CH, m = min(CH, n - t0);
    float* dst = smem + (c & 1) * C::STAGE;
#pragma unroll
    for (int arr = 0; arr < C::ARR; ++arr) {
      const float* src = (arr == 0 ? p.q : arr == 1 ? p.k : p.g) +
                         ((begin + t0) * (arr == 2 ? p.H : p.G) + (arr == 2 ? h : grp)) * p.DP;
      const long long pitch = static_cast<long long>(arr == 2 ? p.H : p.G) * p.DP;
      for (int j = warp; j < m; j += WARPS)
        for (int quad = lane; quad < quads; quad += 32)
          cp_async16(dst + (arr * CH + j) * ROWS + quad * 4, src + j * pitch + quad * 4);
    }
    T* dv = s_v + (c & 1) * CH * COLS;
    if (v_vec) {
      for (int i = tid; i < m * VPIECES; i += THREADS) {
        const int j = i / VPIECES, piece = i % VPIECES;
        cp_async16(reinterpret_cast<char*>(dv + j * COLS) + piece * 16,
                   reinterpret_cast<const char*>(v_src + (t0 + j) * p.v_stride) + piece * 16);
      }
    } else {
      for (int i = tid; i < m * COLS; i += THREADS) {
        const int j = i / COLS, col = i % COLS;
        dv[i] = c_base + col < p.E ? v_src[(t0 + j) * p.v_stride + col] : from_float<T>(0.f);
      }
    }
    if ((MODE == DELTA || MODE == BONUS) && tid < m) cp_async4(s_b + (c & 1) * CH + tid, p.beta + (begin + t0 + tid) * p.H + h);
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(0);

  f32x2 s[4][RPT / 2];
  float* st = p.state + ((static_cast<long long>(slot < 0 ? 0 : slot) * p.H + h) * p.E + c_base + col0) * p.DP;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int i = 0; i < Q4; ++i) {
      const int r = i * 64 + rg * 4;
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && r < p.DP && c_base + col0 + c < p.E)
        x = *reinterpret_cast<const float4*>(st + static_cast<long long>(c) * p.DP + r);
      s[c][2 * i] = pack2(x.x, x.y);
      s[c][2 * i + 1] = pack2(x.z, x.w);
    }

  const int my_col = col0 + (lane & 3);                   // the column this lane has after a fold
  const bool writes = c_base + my_col < p.E;
  float* o = p.o + (begin * p.H + h) * p.E + c_base + my_col;
  const long long o_step = static_cast<long long>(p.H) * p.E;
  const f32x2 one = pack2(1.f, 1.f), minus = pack2(-1.f, -1.f), zero = pack2(0.f, 0.f);

  const int chunks = (n + CH - 1) / CH;
  for (int c = 0; c < chunks; ++c) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                      // chunk c is there; the buffer of c + 1 is free
    if (c + 1 < chunks) stage(c + 1);
    const float* sq = smem + (c & 1) * C::STAGE + rg * 4;
    const float* sk = sq + CH * ROWS;
    const float* sg = sk + CH * ROWS;
    const T* vv = s_v + (c & 1) * CH * COLS;
    const float* bb = s_b + (c & 1) * CH;
    const int m = min(CH, n - c * CH);
    for (int j0 = 0; j0 < m; j0 += GROUP) {
      const float *qj = sq + j0 * ROWS, *kj = sk + j0 * ROWS, *gj = sg + j0 * ROWS, *bj = bb + j0;
      const T* vj = vv + j0 * COLS;
      float acc_o[GROUP][4];
      auto token = [&](int jj) {
        auto load = [&](const float* base, int i) {
          return *reinterpret_cast<const ulonglong2*>(base + jj * ROWS + i * 64);
        };
        f32x2 k[KEEP_K ? RPT / 2 : 1];
        if constexpr (KEEP_K) {
#pragma unroll
          for (int i = 0; i < Q4; ++i) {
            const ulonglong2 x = load(kj, i);
            k[2 * i] = x.x;
            k[2 * i + 1] = x.y;
          }
        }
        auto k_pair = [&](int i) {                        // rows 4 i .. 4 i + 3 of this thread
          if constexpr (KEEP_K) return make_ulonglong2(k[2 * i], k[2 * i + 1]);
          else return load(kj, i);
        };
        f32x2 u[4];                                       // of the four columns, in both halves
        if constexpr (MODE == DELTA) {
          f32x2 acc[4] = {zero, zero, zero, zero};
#pragma unroll
          for (int i = 0; i < Q4; ++i) {
            const ulonglong2 g = load(gj, i), kk = k_pair(i);
#pragma unroll
            for (int cc = 0; cc < 4; ++cc) {
              s[cc][2 * i] = mul2(s[cc][2 * i], g.x);
              s[cc][2 * i + 1] = mul2(s[cc][2 * i + 1], g.y);
              acc[cc] = fma2(s[cc][2 * i], kk.x, acc[cc]);
              acc[cc] = fma2(s[cc][2 * i + 1], kk.y, acc[cc]);
            }
          }
          // four sums over sixteen lanes: lane bits 1, 0 end up choosing the column
          float f[4];
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) f[cc] = sum2(acc[cc]);
          const bool hi = lane & 2, odd = lane & 1;
          const float f0 = (hi ? f[2] : f[0]) + __shfl_xor_sync(0xffffffffu, hi ? f[0] : f[2], 2);
          const float f1 = (hi ? f[3] : f[1]) + __shfl_xor_sync(0xffffffffu, hi ? f[1] : f[3], 2);
          float fc = (odd ? f1 : f0) + __shfl_xor_sync(0xffffffffu, odd ? f0 : f1, 1);
          fc += __shfl_xor_sync(0xffffffffu, fc, 4);
          fc += __shfl_xor_sync(0xffffffffu, fc, 8);
          const float mine = bj[jj] * (as_float(vj[jj * COLS + my_col]) - fc);
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) {
            const float x = __shfl_sync(0xffffffffu, mine, (lane & 16) | cc);
            u[cc] = pack2(x, x);
          }
        } else {
          float x[4];
          Row4<T>::load(vj + jj * COLS + col0, 0, x);
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) u[cc] = pack2(x[cc], x[cc]);
        }
        f32x2 oo[4] = {zero, zero, zero, zero};
#pragma unroll
        for (int i = 0; i < Q4; ++i) {
          const ulonglong2 q = load(qj, i), kk = k_pair(i);
          f32x2 gx = zero, gy = zero;
          if constexpr (MODE == TIED) {
            gx = fma2(kk.x, minus, one);
            gy = fma2(kk.y, minus, one);
          } else if constexpr (MODE != DELTA) {
            const ulonglong2 g = load(gj, i);
            gx = g.x;
            gy = g.y;
          }
#pragma unroll
          for (int cc = 0; cc < 4; ++cc) {
            if constexpr (MODE == BONUS) {                // the state before this token is read
              oo[cc] = fma2(s[cc][2 * i], q.x, oo[cc]);
              oo[cc] = fma2(s[cc][2 * i + 1], q.y, oo[cc]);
            }
            if constexpr (MODE == DELTA) {
              s[cc][2 * i] = fma2(kk.x, u[cc], s[cc][2 * i]);
              s[cc][2 * i + 1] = fma2(kk.y, u[cc], s[cc][2 * i + 1]);
            } else {
              s[cc][2 * i] = fma2(s[cc][2 * i], gx, mul2(kk.x, u[cc]));
              s[cc][2 * i + 1] = fma2(s[cc][2 * i + 1], gy, mul2(kk.y, u[cc]));
            }
            if constexpr (MODE != BONUS) {
              oo[cc] = fma2(s[cc][2 * i], q.x, oo[cc]);
              oo[cc] = fma2(s[cc][2 * i + 1], q.y, oo[cc]);
            }
          }
        }
#pragma unroll
        for (int cc = 0; cc < 4; ++cc) acc_o[jj][cc] = sum2(oo[cc]);
      };
      if (j0 + GROUP <= m) {
#pragma unroll
        for (int jj = 0; jj < GROUP; ++jj) token(jj);
      } else {
#pragma unroll
        for (int jj = 0; jj < GROUP; ++jj) {
          acc_o[jj][0] = acc_o[jj][1] = acc_o[jj][2] = acc_o[jj][3] = 0.f;
          if (j0 + jj < m) token(jj);
        }
      }
      // sixteen sums over sixteen lanes: lane bits 3, 2 end up choosing the token, bits 1, 0 the column
      float x[2][4], y[4], z[2];
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int cc = 0; cc < 4; ++cc)
          x[e][cc] = (lane & 8 ? acc_o[2 + e][cc] : acc_o[e][cc]) +
                     __shfl_xor_sync(0xffffffffu, lane & 8 ? acc_o[e][cc] : acc_o[2 + e][cc], 8);
#pragma unroll
      for (int cc = 0; cc < 4; ++cc)
        y[cc] = (lane & 4 ? x[1][cc] : x[0][cc]) + __shfl_xor_sync(0xffffffffu, lane & 4 ? x[0][cc] : x[1][cc], 4);
#pragma unroll
      for (int e = 0; e < 2; ++e)
        z[e] = (lane & 2 ? y[2 + e] : y[e]) + __shfl_xor_sync(0xffffffffu, lane & 2 ? y[e] : y[2 + e], 2);
      float r = (lane & 1 ? z[1] : z[0]) + __shfl_xor_sync(0xffffffffu, lane & 1 ? z[0] : z[1], 1);
      const int jt = (lane >> 2) & 3;
      if constexpr (MODE == BONUS) r = fmaf(bj[jt], as_float(vj[jt * COLS + my_col]), r);
      if (writes && j0 + jt < m) o[(c * CH + j0 + jt) * o_step] = r;
    }
  }
  if (slot < 0) return;
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int i = 0; i < Q4; ++i) {
      const int r = i * 64 + rg * 4;
      if (r < p.DP && c_base + col0 + c < p.E)
        *reinterpret_cast<ulonglong2*>(st + static_cast<long long>(c) * p.DP + r) =
            make_ulonglong2(s[c][2 * i], s[c][2 * i + 1]);
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

template <typename T, int RPT, int MODE>
static int launch_scan(const ScanParams& p, int B, cudaStream_t stream) {
  auto kern = recurrent_scan_kernel<T, RPT, MODE>;
  constexpr int smem = scan::Cfg<RPT, MODE>::SMEM;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem) != cudaSuccess) return -20;
    once.mark(dev);
  }
  const dim3 grid((p.E + scan::COLS - 1) / scan::COLS, p.H, B);
  return launch_pdl(kern, grid, dim3(scan::THREADS), smem, stream, 1, p) == cudaSuccess ? 0 : -21;
}

template <typename T, int MODE>
static int pick_scan(const ScanParams& p, int B, cudaStream_t stream) {
  if (p.DP <= 64) return launch_scan<T, 4, MODE>(p, B, stream);
  if (p.DP <= 128) return launch_scan<T, 8, MODE>(p, B, stream);
  if (p.DP <= 256) return launch_scan<T, 16, MODE>(p, B, stream);
  if (p.DP <= 512) return launch_scan<T, 32, MODE>(p, B, stream);
  return -2;
}

template <typename T>
static int scan_mode(const ScanParams& p, int mode, int B, cudaStream_t stream) {
  switch (mode) {
    case scan::TIED: return pick_scan<T, scan::TIED>(p, B, stream);
    case scan::DELTA: return pick_scan<T, scan::DELTA>(p, B, stream);
    case scan::DECAY: return pick_scan<T, scan::DECAY>(p, B, stream);
    case scan::BONUS: return pick_scan<T, scan::BONUS>(p, B, stream);
  }
  return -2;
}

// ------------------------------------------------------------- norm and gate of a head's result
struct HeadNormParams {
  const float* o;              // [T, H, E]
  const void* w;               // [E], or [H, E] (w_step = E)
  int w_step;
  const void* gate;            // [T, H * E] before its activation, or null
  long long gate_stride;
  int gate_silu;               // silu instead of sigmoid
  void* out;                   // [T, out_width], row pitch out_stride
  long long out_stride;
  int out_width, T, H, E;
  float eps, scale;
  int vec;                     // rows are whole eight-element pieces
  int lanes;                   // of a warp that share a head
};

static constexpr int kHeadNormWarps = 8;

// `lanes` (a power of two) of a warp share a head; rows of whole eight-element pieces, up to 512 columns, stay in
// registers.
template <typename T>
__global__ void __launch_bounds__(kHeadNormWarps * 32) head_norm_kernel(const HeadNormParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, per_warp = 32 / p.lanes, li = lane & (p.lanes - 1);
  const long long unit =
      (static_cast<long long>(blockIdx.x) * kHeadNormWarps + (threadIdx.x >> 5)) * per_warp + lane / p.lanes;
  const bool live = unit < static_cast<long long>(p.T) * p.H;
  const long long t = live ? unit / p.H : 0;
  const int h = live ? static_cast<int>(unit - t * p.H) : 0;
  const int E = live ? p.E : 0;
  const float* o = p.o + (live ? unit * p.E : 0);
  const T* w = static_cast<const T*>(p.w) + h * p.w_step;
  const T* gate = p.gate ? static_cast<const T*>(p.gate) + t * p.gate_stride + static_cast<long long>(h) * p.E : nullptr;
  T* dst = static_cast<T*>(p.out) + t * p.out_stride + static_cast<long long>(h) * p.E;
  const bool silu = p.gate_silu != 0;
  float ss = 0.f, x[2][8], g[2][8];
  if (p.vec) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int v = li + p.lanes * i;
      if (v * 8 < E) {
        Row8<float>::load(o, v, x[i]);
        if (gate) Row8<T>::load(gate, v, g[i]);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss = fmaf(x[i][j], x[i][j], ss);
      }
    }
  } else {
    for (int d = li; d < E; d += p.lanes) ss = fmaf(o[d], o[d], ss);
  }
  for (int i = p.lanes >> 1; i > 0; i >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, i);
  if (!live) return;
  const float inv = p.scale / sqrtf(ss / static_cast<float>(p.E) + p.eps);
  if (p.vec) {
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int v = li + p.lanes * i;
      if (v * 8 < E) {
        float ww[8];
        Row8<T>::load(w, v, ww);
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          x[i][j] *= inv * ww[j];
          if (gate) x[i][j] *= quick_sigmoid(g[i][j]) * (silu ? g[i][j] : 1.f);
        }
        Row8<T>::store(dst, v, x[i]);
      }
    }
  } else {
    for (int d = li; d < E; d += p.lanes) {
      float y = o[d] * inv * as_float(w[d]);
      if (gate) y *= quick_sigmoid(as_float(gate[d])) * (silu ? as_float(gate[d]) : 1.f);
      dst[d] = from_float<T>(y);
    }
  }
  if (h == p.H - 1)
    for (int d = p.E + li; d < p.out_width - h * p.E; d += p.lanes) dst[d] = from_float<T>(0.f);
}

template <typename T, int CPL>
static cudaError_t launch_delta_prep(const DeltaPrepParams& p, dim3 grid, cudaStream_t stream) {
  const dim3 block(kPrepWarps * 32);
  const int W = 2;                                       // pairs: everything a pair touches starts at an even channel
  const bool pair = p.dim % W == 0 && p.vdim % W == 0 && p.stride % W == 0 && p.low_stride % W == 0 &&
                    p.channels % W == 0 && p.q_off % W == 0 && p.k_off % W == 0 && p.v_off % W == 0 &&
                    (reinterpret_cast<uintptr_t>(p.proj) & 7) == 0 && (reinterpret_cast<uintptr_t>(p.low) & 7) == 0;
  if (pair) {
    if (p.taps <= 4) return launch_pdl(delta_prep_kernel<T, CPL, 4, true>, grid, block, 0, stream, 1, p);
    return launch_pdl(delta_prep_kernel<T, CPL, 8, true>, grid, block, 0, stream, 1, p);
  }
  if (p.taps <= 4) return launch_pdl(delta_prep_kernel<T, CPL, 4, false>, grid, block, 0, stream, 1, p);
  return launch_pdl(delta_prep_kernel<T, CPL, 8, false>, grid, block, 0, stream, 1, p);
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

// mode: 0 tied (g and beta null), 1 delta, 2 decay (beta null), 3 bonus.  Head sizes (rows) up to 512.
extern "C" int b200_recurrent_scan(const float* q, const float* k, const float* g, const void* v, long long v_stride,
                                   const float* beta, float* state, float* o, const int* state_slots, const int* cu_q,
                                   const int* seq_lens, int B, int H, int G, int E, int DP, const void* proj,
                                   long long proj_stride, void* conv_state, int keep, int channels, int mode,
                                   int is_fp32, cudaStream_t stream) {
  if (B <= 0) return 0;
  if ((DP & 3) || G <= 0 || H % G) return -1;
  ScanParams p{q, k, g, v, v_stride, beta, state, o, state_slots, cu_q, seq_lens, H, G, E, DP, proj, proj_stride,
               conv_state, keep, channels};
  if ((mode != scan::TIED && !g) || ((mode == scan::DELTA || mode == scan::BONUS) && !beta)) return -1;
  return is_fp32 ? scan_mode<float>(p, mode, B, stream) : scan_mode<__nv_bfloat16>(p, mode, B, stream);
}

extern "C" int b200_head_norm_gate(const float* o, const void* w, int w_step, const void* gate, long long gate_stride,
                                   int gate_silu, void* out, long long out_stride, int out_width, int T, int H, int E,
                                   float eps, float scale, int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  const bool vec = E % 8 == 0 && E <= 512 && out_stride % 8 == 0 && gate_stride % 8 == 0 &&
                   (reinterpret_cast<uintptr_t>(gate) & 15) == 0 && (reinterpret_cast<uintptr_t>(out) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(w) & 15) == 0;
  int lanes = 1;
  while (lanes < 32 && lanes * (vec ? 8 : 1) < E) lanes <<= 1;
  HeadNormParams p{o, w, w_step, gate, gate_stride, gate_silu, out, out_stride, out_width, T, H, E, eps, scale, vec ? 1 : 0, lanes};
  const long long units = static_cast<long long>(T) * H, per_cta = static_cast<long long>(kHeadNormWarps) * (32 / lanes);
  const dim3 grid(static_cast<unsigned>((units + per_cta - 1) / per_cta)), block(kHeadNormWarps * 32);
  const cudaError_t e = is_fp32 ? launch_pdl(head_norm_kernel<float>, grid, block, 0, stream, 1, p)
                                : launch_pdl(head_norm_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, p);
  return e == cudaSuccess ? 0 : -3;
}
