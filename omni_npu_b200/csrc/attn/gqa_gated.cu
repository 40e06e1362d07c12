// Gated, windowed grouped-query attention (gqa_gated.cuh): rotation + cache write, the kernel for
// models run in 32-bit and for head sizes beyond the tensor-core kernels, and the entry points.

#include <cuda_runtime.h>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "attn_params.cuh"
#include "gqa_gated.cuh"

namespace b200 {

int gated_decode(const GatedAttnParams& p, cudaStream_t stream);
int gated_prefill(const GatedAttnParams& p, int max_q_len, cudaStream_t stream);
int gated_prefill_tc(const GatedAttnParams& p, int max_q_len, long long total_q_rows, int* status,
                     cudaStream_t stream);

__device__ __forceinline__ float to_f(float x) { return x; }
__device__ __forceinline__ float to_f(__nv_bfloat16 x) { return __bfloat162float(x); }
template <typename T>
__device__ __forceinline__ T from_f(float x);
template <>
__device__ __forceinline__ float from_f<float>(float x) { return x; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float x) { return __float2bfloat16(x); }

// ------------------------------------------------------------- rotation + cache write
// q is rotated in place, k is rotated into the cache, v is copied into the cache.  Aligned rows with
// interleaved pairs go 16 bytes at a time, a token per CTA row (split over gridDim.y CTAs when there are
// few tokens); anything else takes one warp per (token, head).
struct RopeCacheParams {
  void* q;
  const void* k;
  const void* v;
  void* k_cache;
  void* v_cache;
  const int* positions;
  const int* slots;
  const float* cos_sin;        // [max_pos, rot]: cosines then sines
  int Hq, Hk, D, DV, DP, DVP, rot, neox, block_size, max_pos;
  long long q_stride, k_stride, v_stride;
};

// 16 bytes of a row as floats
template <typename T>
struct Chunk;
template <>
struct Chunk<float> {
  static constexpr int W = 4;
  static __device__ __forceinline__ void load(const float* p, float (&x)[4]) {
    const float4 v = *reinterpret_cast<const float4*>(p);
    x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w;
  }
  static __device__ __forceinline__ void store(float* p, const float (&x)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(x[0], x[1], x[2], x[3]);
  }
};
template <>
struct Chunk<__nv_bfloat16> {
  static constexpr int W = 8;
  static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&x)[8]) {
    const uint4 u = *reinterpret_cast<const uint4*>(p);
    const uint32_t r[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x[2 * i] = __uint_as_float(r[i] << 16);
      x[2 * i + 1] = __uint_as_float(r[i] & 0xffff0000u);
    }
  }
  static __device__ __forceinline__ void store(__nv_bfloat16* p, const float (&x)[8]) {
    uint4 u;
    uint32_t* r = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 v = __floats2bfloat162_rn(x[2 * i], x[2 * i + 1]);
      r[i] = *reinterpret_cast<const uint32_t*>(&v);
    }
    *reinterpret_cast<uint4*>(p) = u;
  }
};

static constexpr int kRopeThreads = 256;

template <typename T>
__global__ void __launch_bounds__(kRopeThreads) gated_rope_cache_vec_kernel(const RopeCacheParams p) {
  constexpr int W = Chunk<T>::W;
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int slot = p.slots[t];
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  const float* cs = p.cos_sin + static_cast<long long>(pos) * p.rot;
  const int half = p.rot >> 1;
  const int qc = p.rot / W, kc = p.D / W, vc = p.DV / W;         // chunks per head (q: rotated part only)
  const int nq = p.Hq * qc, nk = p.Hk * kc, nv = p.Hk * vc;
  const int total = slot < 0 ? nq : nq + nk + nv;
  const long long blk = slot < 0 ? 0 : slot / p.block_size;
  const int off = slot < 0 ? 0 : slot % p.block_size;
  for (int i = blockIdx.y * kRopeThreads + threadIdx.x; i < total; i += gridDim.y * kRopeThreads) {
    const T* src;
    T* dst;
    int d;
    bool turn = true;
    if (i < nq) {
      const int h = i / qc;
      d = (i - h * qc) * W;
      dst = static_cast<T*>(p.q) + t * p.q_stride + static_cast<long long>(h) * p.D + d;
      src = dst;
    } else if (i < nq + nk) {
      const int h = (i - nq) / kc;
      d = (i - nq - h * kc) * W;
      src = static_cast<const T*>(p.k) + t * p.k_stride + static_cast<long long>(h) * p.D + d;
      dst = static_cast<T*>(p.k_cache) + ((blk * p.Hk + h) * p.block_size + off) * p.DP + d;
      turn = d < p.rot;
    } else {
      const int h = (i - nq - nk) / vc;
      d = (i - nq - nk - h * vc) * W;
      src = static_cast<const T*>(p.v) + t * p.v_stride + static_cast<long long>(h) * p.DV + d;
      dst = static_cast<T*>(p.v_cache) + ((blk * p.Hk + h) * p.block_size + off) * p.DVP + d;
      turn = false;
    }
    float x[W];
    Chunk<T>::load(src, x);
    if (turn) {
      const float2* c2 = reinterpret_cast<const float2*>(cs + (d >> 1));
      const float2* s2 = reinterpret_cast<const float2*>(cs + half + (d >> 1));
#pragma unroll
      for (int j = 0; j < W / 4; ++j) {
        const float2 c = c2[j], s = s2[j];
        const float u0 = x[4 * j], w0 = x[4 * j + 1], u1 = x[4 * j + 2], w1 = x[4 * j + 3];
        x[4 * j] = u0 * c.x - w0 * s.x;
        x[4 * j + 1] = w0 * c.x + u0 * s.x;
        x[4 * j + 2] = u1 * c.y - w1 * s.y;
        x[4 * j + 3] = w1 * c.y + u1 * s.y;
      }
    }
    Chunk<T>::store(dst, x);
  }
}

static constexpr int kRopeWarps = 4;

template <typename T>
__global__ void __launch_bounds__(kRopeWarps * 32) gated_rope_cache_kernel(const RopeCacheParams p) {
  pdl_trigger();
  pdl_wait();
  const long long t = blockIdx.x;
  const int lane = threadIdx.x & 31;
  int h = blockIdx.y * kRopeWarps + (threadIdx.x >> 5);
  if (h >= p.Hq + 2 * p.Hk) return;
  const bool is_q = h < p.Hq;
  const bool is_v = h >= p.Hq + p.Hk;
  const int slot = is_q ? 0 : p.slots[t];
  if (slot < 0) return;
  const T* src;
  T* dst;
  int dim = p.D;
  if (is_q) {
    dst = static_cast<T*>(p.q) + t * p.q_stride + static_cast<long long>(h) * p.D;
    src = dst;
  } else {
    const long long blk = slot / p.block_size, off = slot % p.block_size;
    h -= is_v ? p.Hq + p.Hk : p.Hq;
    const long long row = (blk * p.Hk + h) * p.block_size + off;
    if (is_v) {
      dim = p.DV;
      src = static_cast<const T*>(p.v) + t * p.v_stride + static_cast<long long>(h) * p.DV;
      dst = static_cast<T*>(p.v_cache) + row * p.DVP;
    } else {
      src = static_cast<const T*>(p.k) + t * p.k_stride + static_cast<long long>(h) * p.D;
      dst = static_cast<T*>(p.k_cache) + row * p.DP;
    }
  }
  const int rot = is_v ? 0 : p.rot, half = p.rot >> 1;
  int pos = p.positions[t];
  pos = pos < 0 ? 0 : (pos >= p.max_pos ? p.max_pos - 1 : pos);
  const float* cs = p.cos_sin + static_cast<long long>(pos) * p.rot;
  for (int j = lane; j < (rot >> 1); j += 32) {
    const int a = p.neox ? j : 2 * j, b = a + (p.neox ? half : 1);
    const float c = cs[j], s = cs[half + j], u = to_f(src[a]), w = to_f(src[b]);
    dst[a] = from_f<T>(u * c - w * s);
    dst[b] = from_f<T>(w * c + u * s);
  }
  if (!is_q)
    for (int d = rot + lane; d < dim; d += 32) dst[d] = src[d];
}

// ------------------------------------------------------------- one CTA per (token, head), fp32 math
static constexpr int kPlainThreads = 128;

template <typename T>
__global__ void __launch_bounds__(kPlainThreads) gated_plain_kernel(const GatedAttnParams p, const int total_rows) {
  extern __shared__ float sm[];
  float* sq = sm;                          // [D]
  float* so = sq + p.D;                    // [DV]
  float* sp = so + p.DV;                   // [kPlainThreads] weights of the chunk
  long long* srow = reinterpret_cast<long long*>(sp + kPlainThreads + ((p.D + p.DV) & 1));
  __shared__ float red[kPlainThreads / 32];
  pdl_trigger();
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  // the sequence this row belongs to
  int b, q_begin, q_len;
  if (p.cu_q) {
    int x = 0, y = p.B;                    // last b with cu_q[b] <= t
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
  const int kv_len = p.seq_lens[b];
  const int pos = kv_len - q_len + (t - q_begin);
  const int kvh = h / (p.Hq / p.Hk);
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const T* q = static_cast<const T*>(p.q) + t * p.q_stride + static_cast<long long>(h) * p.D;
  const T* kc = static_cast<const T*>(p.k_cache);
  const T* vc = static_cast<const T*>(p.v_cache);
  for (int d = tid; d < p.D; d += kPlainThreads) sq[d] = to_f(q[d]);
  for (int d = tid; d < p.DV; d += kPlainThreads) so[d] = 0.f;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int hi = min(kv_len, pos + 1);
  float m = p.has_sink ? p.sink_log2 : -INFINITY, l = p.has_sink ? 1.f : 0.f;
  __syncthreads();
  for (int n0 = lo; n0 < hi; n0 += kPlainThreads) {
    const int key = n0 + tid;
    float s = -INFINITY;
    long long row = 0;
    if (key < hi) {
      row = p.contiguous ? static_cast<long long>(bt[0] + key) * p.Hk + kvh
                         : (static_cast<long long>(bt[key / p.block_size]) * p.Hk + kvh) * p.block_size + key % p.block_size;
      const T* k = kc + row * p.DP;
      float acc = 0.f;
      for (int d = 0; d < p.D; ++d) acc = fmaf(sq[d], to_f(k[d]), acc);
      s = acc * p.scale_log2;
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    if (lane == 0) red[warp] = mx;
    __syncthreads();
    float nm = m;
#pragma unroll
    for (int w = 0; w < kPlainThreads / 32; ++w) nm = fmaxf(nm, red[w]);
    const float corr = m == -INFINITY ? 0.f : exp2f(m - nm);
    const float e = key < hi ? exp2f(s - nm) : 0.f;
    m = nm;
    sp[tid] = e;
    srow[tid] = row;
    float sum = e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    __syncthreads();
    if (lane == 0) red[warp] = sum;
    __syncthreads();
    l *= corr;
#pragma unroll
    for (int w = 0; w < kPlainThreads / 32; ++w) l += red[w];
    const int n = min(kPlainThreads, hi - n0);
    for (int d = tid; d < p.DV; d += kPlainThreads) {
      float acc = so[d] * corr;
      for (int j = 0; j < n; ++j) acc = fmaf(sp[j], to_f(vc[srow[j] * p.DVP + d]), acc);
      so[d] = acc;
    }
    __syncthreads();
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  const long long col = static_cast<long long>(h) * p.DV;
  for (int d = tid; d < p.DV; d += kPlainThreads) {
    float o = so[d] * inv;
    if (p.gate) o *= gate_sigmoid(to_f(static_cast<const T*>(p.gate)[t * p.g_stride + col + d]));
    static_cast<T*>(p.out)[t * p.out_stride + col + d] = from_f<T>(o);
  }
}

template <typename T>
static int launch_plain(const GatedAttnParams& p, int rows, cudaStream_t stream) {
  const size_t smem = (p.D + p.DV + kPlainThreads + 2) * sizeof(float) + kPlainThreads * sizeof(long long);
  if (smem > 48 * 1024) return -2;
  return launch_pdl(gated_plain_kernel<T>, dim3(rows, p.Hq), dim3(kPlainThreads), smem, stream, 1, p, rows) ==
                 cudaSuccess ? 0 : -21;
}

}  // namespace b200

using namespace b200;

extern "C" int b200_gated_rope_cache(void* q, const void* k, const void* v, void* k_cache, void* v_cache,
                                     const int* positions, const int* slots, const float* cos_sin, int max_pos, int T,
                                     int Hq, int Hk, int D, int DV, int DP, int DVP, int rot, int neox,
                                     long long q_stride, long long k_stride, long long v_stride, int block_size,
                                     int is_fp32, cudaStream_t stream) {
  if (T <= 0) return 0;
  if (rot < 0 || rot > D || (rot & 1) || DP < D || DVP < DV) return -1;
  RopeCacheParams p{q, k, v, k_cache, v_cache, positions, slots, cos_sin, Hq, Hk, D, DV, DP, DVP, rot, neox,
                    block_size, max_pos, q_stride, k_stride, v_stride};
  const int W = is_fp32 ? 4 : 8;
  const auto ok = [&](const void* ptr, long long stride) {
    return (reinterpret_cast<uintptr_t>(ptr) & 15) == 0 && stride % W == 0;
  };
  cudaError_t e;
  if (!neox && D % W == 0 && DV % W == 0 && rot % W == 0 && ok(q, q_stride) && ok(k, k_stride) && ok(v, v_stride) &&
      ok(k_cache, DP) && ok(v_cache, DVP)) {
    const int chunks = (Hq * rot + Hk * (D + DV)) / W;
    int ny = (chunks + kRopeThreads - 1) / kRopeThreads;
    if (T >= 512) ny = 1;                              // enough tokens: fewer, longer CTAs
    const dim3 grid(T, ny), block(kRopeThreads);
    e = is_fp32 ? launch_pdl(gated_rope_cache_vec_kernel<float>, grid, block, 0, stream, 1, p)
                : launch_pdl(gated_rope_cache_vec_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, p);
  } else {
    const dim3 grid(T, (Hq + 2 * Hk + kRopeWarps - 1) / kRopeWarps), block(kRopeWarps * 32);
    e = is_fp32 ? launch_pdl(gated_rope_cache_kernel<float>, grid, block, 0, stream, 1, p)
                : launch_pdl(gated_rope_cache_kernel<__nv_bfloat16>, grid, block, 0, stream, 1, p);
  }
  return e == cudaSuccess ? 0 : -3;
}

// cu_q null: every sequence has q_len rows (decode step); else prompt portions, at most max_q_len rows each.
// variant: 0 = by shape, 1 = mma.sync kernels, 2 = the plain kernel.
extern "C" int b200_gated_attention(const void* q, const void* gate, const void* k_cache, const void* v_cache,
                                    void* out, const int* block_tables, const int* cu_q, const int* seq_lens,
                                    int total_rows, int B, int q_len, int max_q_len, int max_blocks, int block_size,
                                    int num_cache_blocks, int Hq, int Hk, int D, int DV, int DP, int DVP,
                                    long long q_stride, long long g_stride, long long out_stride, float scale,
                                    int window, int has_sink, float sink, int splits, int is_fp32, int variant,
                                    int* status, int contiguous, cudaStream_t stream) {
  if (B <= 0 || total_rows <= 0) return 0;
  if (Hk <= 0 || Hq % Hk != 0) return -1;
  GatedAttnParams p{};
  p.q = q;
  p.gate = gate;
  p.k_cache = k_cache;
  p.v_cache = v_cache;
  p.out = out;
  p.block_tables = block_tables;
  p.contiguous = contiguous;
  p.cu_q = cu_q;
  p.seq_lens = seq_lens;
  p.B = B;
  p.max_blocks = max_blocks;
  p.block_size = block_size;
  p.num_cache_blocks = num_cache_blocks;
  p.bs_shift = -1;
  for (int i = 0; i < 30; ++i)
    if ((1 << i) == block_size) p.bs_shift = i;
  p.Hq = Hq;
  p.Hk = Hk;
  p.D = D;
  p.DV = DV;
  p.DP = DP;
  p.DVP = DVP;
  p.q_stride = q_stride;
  p.g_stride = g_stride;
  p.out_stride = out_stride;
  p.scale_log2 = scale * kLog2e;
  p.window = window;
  p.has_sink = has_sink;
  p.sink_log2 = sink * kLog2e;
  p.q_len = q_len;
  p.splits = splits < 1 ? 1 : splits;
  const bool tensor = !is_fp32 && variant != 2 && (DP & 15) == 0 && (DVP & 15) == 0 && DP <= 256 && DVP <= 256;
  if (!tensor) return is_fp32 ? launch_plain<float>(p, total_rows, stream)
                              : launch_plain<__nv_bfloat16>(p, total_rows, stream);
  if (cu_q == nullptr) return contiguous ? -3 : gated_decode(p, stream);
  if (variant == 0 && !contiguous) {
    const int rc = gated_prefill_tc(p, max_q_len, total_rows, status, stream);
    if (rc <= 0) return rc;
  }
  return gated_prefill(p, max_q_len, stream);
}
