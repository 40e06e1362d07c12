// Decode step of the attention with mixed heads (mixed_attn.cuh), bf16.
//
// One CTA = one query row, a share of its keys, ALL heads (the mixture needs every head's score of a key).  Tiles of 16
// or 32 keys of all key and value heads come in with cp.async, one tile ahead.  Per tile:
//
//   S^T = K Q^T       on mma.sync, 16 keys x 8 heads of a group per product; capped, lowered, to shared memory (fp32)
//   mixture, softmax  a lane holds one key of a head: the sum over score heads, running maximum and sum, weights (bf16)
//   O^T += V^T P^T    on mma.sync, accumulators stay with the warp that owns (8 heads, 16 columns)
//
// With one share the row is normalised here; otherwise the shares meet in a small second kernel.

#include <algorithm>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "attn_common.cuh"
#include "attn_params.cuh"
#include "mixed_attn.cuh"

namespace b200 {

namespace mdec {

// 16-byte piece `chunk` of row `row` of a tile whose rows hold `width` elements (a multiple of 64)
__device__ __forceinline__ uint32_t piece(int row, int chunk, int width) {
  return static_cast<uint32_t>(row * width * 2 + ((chunk ^ (row & 7)) << 4));
}

struct Layout {
  int dk, dv;                  // row widths in shared memory
  int hs4;                     // score heads rounded up to 4
  int s_pitch, p_pitch;        // floats per score head, bf16 per weight row
  int k_bytes, v_bytes, stages;
  int q_off, ring_off, s_off, p_off, t_off, r_off, m_off, bytes;
};

__host__ __device__ inline Layout layout(int Hs, int Hk, int Ho, int Hv, int DP, int DVP, int kt, int stages) {
  Layout l;
  l.dk = (DP + 63) / 64 * 64;
  l.dv = (DVP + 63) / 64 * 64;
  l.hs4 = (Hs + 3) / 4 * 4;
  l.s_pitch = kt + 4;
  l.p_pitch = kt + 8;
  l.k_bytes = Hk * kt * l.dk * 2;
  l.v_bytes = Hv * kt * l.dv * 2;
  l.stages = stages;
  int at = 0;
  const auto take = [&](int bytes) {
    const int r = at;
    at += (bytes + 127) / 128 * 128;
    return r;
  };
  l.q_off = take(Hs * l.dk * 2);
  l.ring_off = take(stages * (l.k_bytes + l.v_bytes));
  l.s_off = take(l.hs4 * l.s_pitch * 4);
  l.p_off = take(Ho * l.p_pitch * 2);
  l.t_off = take(Ho * l.hs4 * 4);
  l.r_off = take(2 * Hs * 4);
  l.m_off = take(3 * Ho * 4);
  l.bytes = at;
  return l;
}

struct Plan {
  int kt, stages, warps, units;
};

// The first of the layouts, from fast to small, that fits; kt 0: none.
inline Plan plan(int Hs, int Hk, int Ho, int Hv, int DP, int DVP) {
  if (DP > 512 || DVP > 512) return {0, 0, 0, 0};
  const int units = Hv * ((Ho / Hv + 7) / 8) * (DVP / 16);
  const int warps = units <= 16 * 8 ? 8 : 16;
  const int each = (units + warps - 1) / warps;
  if (each > 16) return {0, 0, 0, 0};
  const int order[5][3] = {{32, 2, 112}, {16, 2, 112}, {32, 2, 226}, {16, 2, 226}, {16, 1, 226}};
  for (const auto& o : order)
    if (layout(Hs, Hk, Ho, Hv, DP, DVP, o[0], o[1]).bytes <= o[2] * 1024) return {o[0], o[1], warps, each};
  return {0, 0, 0, 0};
}

}  // namespace mdec

bool mixed_decode_fits(int Hs, int Hk, int Ho, int Hv, int DP, int DVP) {
  return mdec::plan(Hs, Hk, Ho, Hv, DP, DVP).kt > 0;
}

// UNITS: accumulator tiles (8 heads x 16 columns) per warp
template <int UNITS, int WARPS, int KT>
__global__ void __launch_bounds__(WARPS * 32) mixed_decode_kernel(const MixedAttnParams p, const int stages) {
  using namespace mdec;
  constexpr int THREADS = WARPS * 32, SUB = 32 / KT;
  extern __shared__ __align__(128) uint8_t smem[];
  const Layout L = layout(p.Hs, p.Hk, p.Ho, p.Hv, p.DP, p.DVP, KT, stages);
  uint8_t* sQ = smem + L.q_off;
  float* sS = reinterpret_cast<float*>(smem + L.s_off);                       // [hs4][s_pitch]
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(smem + L.p_off);       // [Ho][p_pitch]
  float* sT = reinterpret_cast<float*>(smem + L.t_off);                       // [Ho][hs4], times log2 e
  float* sR = reinterpret_cast<float*>(smem + L.r_off);                       // r1, r2
  float* sMax = reinterpret_cast<float*>(smem + L.m_off);
  float* sSum = sMax + p.Ho;
  float* sCor = sSum + p.Ho;
  const uint32_t ring = smem_u32(smem + L.ring_off);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = blockIdx.x / p.splits, split = blockIdx.x % p.splits;
  const int per_k = p.Hs / p.Hk, per_v = p.Ho / p.Hv;
  const int kchunks8 = (per_k + 7) >> 3, vchunks8 = (per_v + 7) >> 3;

  // constants of the layer are no earlier kernel's result
  for (int i = tid; i < p.Ho * L.hs4; i += THREADS) {
    const int h = i / L.hs4, g = i - h * L.hs4;
    sT[i] = g < p.Hs ? p.talk[h * p.Hs + g] * kLog2e : 0.f;
  }
  for (int i = tid; i < p.Hs; i += THREADS) {
    sR[i] = p.r1 ? p.r1[i] : 0.f;
    sR[p.Hs + i] = p.r1 ? p.r2[i] : 0.f;
  }
  for (int i = tid; i < L.hs4 * L.s_pitch; i += THREADS) sS[i] = 0.f;
  for (int h = tid; h < p.Ho; h += THREADS) {
    sMax[h] = -INFINITY;
    sSum[h] = 0.f;
  }
  pdl_trigger();
  pdl_wait();

  const int b = row / p.q_len;
  const int pos = p.seq_lens[b] - p.q_len + row % p.q_len;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q) + row * p.q_stride;
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(p.k_cache);
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(p.v_cache);
  const int all = (pos + KT) / KT;                                            // tiles with a visible key
  const int share = (all + p.splits - 1) / p.splits;
  const int t_begin = min(all, split * share), t_end = min(all, t_begin + share);

  // one tile of rows (all heads); lanes_log2: lanes that share a row
  auto load = [&](const __nv_bfloat16* cache, int heads, int width, int smem_width, uint32_t dst, int n0) {
    const int chunks = width >> 3;
    int ll = 0;
    while (ll < 5 && (1 << ll) < chunks) ++ll;
    const int li = lane & ((1 << ll) - 1), rows_per = 32 >> ll;
    for (int r = warp * rows_per + (lane >> ll); r < heads * KT; r += WARPS * rows_per) {
      const int g = r / KT, key = n0 + r % KT;
      const bool ok = key <= pos;
      const __nv_bfloat16* src = ok ? cache + cache_row(p, bt, key, g, heads) * width : cache;
      const int sz = ok ? 16 : 0;
      for (int c = li; c < chunks; c += 1 << ll)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + piece(r, c, smem_width)),
                     "l"(ok ? src + c * 8 : src), "r"(sz) : "memory");
    }
  };
  auto issue = [&](int tile) {
    if (tile < t_end) {
      const uint32_t dst = ring + (stages == 2 ? (tile - t_begin) & 1 : 0) * (L.k_bytes + L.v_bytes);
      load(kc, p.Hk, p.DP, L.dk, dst, tile * KT);
      load(vc, p.Hv, p.DVP, L.dv, dst + L.k_bytes, tile * KT);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (stages == 2) issue(t_begin);

  // query heads -> shared, zero beyond the head size
  for (int i = tid; i < p.Hs * (p.DP >> 3); i += THREADS) {
    const int g = i / (p.DP >> 3), c = i - g * (p.DP >> 3);
    const __nv_bfloat16* src = q + g * p.D + c * 8;
    __nv_bfloat16 h[8];
#pragma unroll
    for (int j = 0; j < 8; ++j) h[j] = c * 8 + j < p.D ? src[j] : __float2bfloat16(0.f);
    uint4 u;
    uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
    for (int j = 0; j < 4; ++j)
      w[j] = static_cast<uint32_t>(__bfloat16_as_ushort(h[2 * j])) |
             (static_cast<uint32_t>(__bfloat16_as_ushort(h[2 * j + 1])) << 16);
    *reinterpret_cast<uint4*>(sQ + piece(g, c, L.dk)) = u;
  }

  float acc[UNITS][4];
#pragma unroll
  for (int i = 0; i < UNITS; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  const int vtiles = p.DVP >> 4, units = p.Hv * vchunks8 * vtiles;
  const int k_units = p.Hk * kchunks8 * (KT / 16);

  for (int tile = t_begin; tile < t_end; ++tile) {
    if (stages == 1) {
      __syncthreads();                                     // the tile before is used up
      issue(tile);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (stages == 2) issue(tile + 1);
    const uint32_t kt = ring + (stages == 2 ? (tile - t_begin) & 1 : 0) * (L.k_bytes + L.v_bytes), vt = kt + L.k_bytes;
    const int n0 = tile * KT;

    // ---- scores of 16 keys x 8 heads of a key head
    for (int u = warp; u < k_units; u += WARPS) {
      const int sub = u % (KT / 16), gc = u / (KT / 16), g = gc / kchunks8, ch = gc - g * kchunks8;
      const int krow = g * KT + sub * 16 + (lane & 15);
      const int head0 = g * per_k + ch * 8;
      const int qrow = min(head0 + (lane & 7), p.Hs - 1);
      float s[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
      for (int ks = 0; ks < (p.DP >> 4); ++ks) {
        uint32_t kf[4], qf[4];
        ldmatrix_x4(kf, kt + piece(krow, ks * 2 + (lane >> 4), L.dk));
        ldmatrix_x4(qf, smem_u32(sQ) + piece(qrow, ks * 2 + ((lane >> 3) & 1), L.dk));
        mma_bf16_16816(s, kf, qf[0], qf[1]);
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int hl = ch * 8 + (lane & 3) * 2 + (j & 1), key = sub * 16 + (lane >> 2) + (j >> 1) * 8;
        if (hl < per_k) {
          const int h = g * per_k + hl;
          const float dist = static_cast<float>(max(0, pos - n0 - key));
          sS[h * L.s_pitch + key] = head_score(p, s[j], dist, sR[h], sR[p.Hs + h]);
        }
      }
    }
    __syncthreads();

    // ---- mixture and softmax: a lane = one key, KT lanes = a head, four heads at a time
    {
      const int key = lane % KT, sub = lane / KT;
      const bool seen = n0 + key <= pos;
      for (int h0 = (warp * SUB + sub) * 4; h0 - sub * 4 < p.Ho; h0 += WARPS * SUB * 4) {      // (warp-uniform)
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        const float* t[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) t[i] = sT + min(h0 + i, p.Ho - 1) * L.hs4;
        for (int g = 0; g < L.hs4; g += 4) {
          float a[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) a[e] = sS[(g + e) * L.s_pitch + key];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const float4 w = *reinterpret_cast<const float4*>(t[i] + g);
            s[i] = fmaf(w.x, a[0], fmaf(w.y, a[1], fmaf(w.z, a[2], fmaf(w.w, a[3], s[i]))));
          }
        }
        float mx[4], e[4], sum[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) mx[i] = seen ? s[i] : -INFINITY;
#pragma unroll
        for (int o = KT / 2; o > 0; o >>= 1)
#pragma unroll
          for (int i = 0; i < 4; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], o));
        float old[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          old[i] = sMax[min(h0 + i, p.Ho - 1)];
          mx[i] = fmaxf(mx[i], old[i]);                    // (a tile holds a visible key: finite)
          e[i] = seen ? exp2f(s[i] - mx[i]) : 0.f;
          sum[i] = e[i];
        }
#pragma unroll
        for (int o = KT / 2; o > 0; o >>= 1)
#pragma unroll
          for (int i = 0; i < 4; ++i) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], o);
        __syncwarp();
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const int h = h0 + i;
          if (h >= p.Ho) continue;
          sP[h * L.p_pitch + key] = __float2bfloat16(e[i]);
          if (key == 0) {
            const float c = exp2f(old[i] - mx[i]);         // (the first tile: 0)
            sMax[h] = mx[i];
            sSum[h] = sSum[h] * c + sum[i];
            sCor[h] = c;
          }
        }
      }
    }
    __syncthreads();

    // ---- values: (8 heads of a value head) x 16 columns
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
      const int u = warp + i * WARPS;
      if (u >= units) continue;
      const int vtile = u % vtiles, gc = u / vtiles, g = gc / vchunks8, ch = gc - g * vchunks8;
      const int head0 = g * per_v + ch * 8;
      const float c0 = sCor[min(head0 + (lane & 3) * 2, p.Ho - 1)], c1 = sCor[min(head0 + (lane & 3) * 2 + 1, p.Ho - 1)];
      acc[i][0] *= c0;
      acc[i][1] *= c1;
      acc[i][2] *= c0;
      acc[i][3] *= c1;
      const __nv_bfloat16* pr = sP + min(head0 + (lane >> 2), p.Ho - 1) * L.p_pitch + (lane & 3) * 2;
#pragma unroll
      for (int ks = 0; ks < KT / 16; ++ks) {
        uint32_t vf[4];
        ldmatrix_x4_trans(vf, vt + piece(g * KT + ks * 16 + ((lane >> 4) << 3) + (lane & 7),
                                         vtile * 2 + ((lane >> 3) & 1), L.dv));
        mma_bf16_16816(acc[i], vf, *reinterpret_cast<const uint32_t*>(pr + ks * 16),
                       *reinterpret_cast<const uint32_t*>(pr + ks * 16 + 8));
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");

  // ---- the row, or this share of it
  if (p.splits == 1) {
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
      const int u = warp + i * WARPS;
      if (u >= units) continue;
      const int vtile = u % vtiles, gc = u / vtiles, g = gc / vchunks8, ch = gc - g * vchunks8;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int hl = ch * 8 + (lane & 3) * 2 + (j & 1), d = vtile * 16 + (lane >> 2) + (j >> 1) * 8;
        if (hl >= per_v || d >= p.DV) continue;
        const int h = g * per_v + hl;
        float m = sMax[h], f = 1.f, l = sSum[h];
        if (p.sink) {
          const float z = p.sink[h] * kLog2e, top = fmaxf(m, z);
          f = exp2f(m - top);
          l = l * f + exp2f(z - top);
        }
        static_cast<__nv_bfloat16*>(p.out)[row * p.out_stride + static_cast<long long>(h) * p.DV + d] =
            __float2bfloat16(l > 0.f ? acc[i][j] * f / l : 0.f);
      }
    }
    return;
  }
  float* part = p.scratch + (static_cast<long long>(row) * p.splits + split) * p.Ho * (p.DVP + 2);
#pragma unroll
  for (int i = 0; i < UNITS; ++i) {
    const int u = warp + i * WARPS;
    if (u >= units) continue;
    const int vtile = u % vtiles, gc = u / vtiles, g = gc / vchunks8, ch = gc - g * vchunks8;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int hl = ch * 8 + (lane & 3) * 2 + (j & 1), d = vtile * 16 + (lane >> 2) + (j >> 1) * 8;
      if (hl < per_v) part[(g * per_v + hl) * (p.DVP + 2) + d] = acc[i][j];
    }
  }
  __syncthreads();                                         // (a row without a tile: the initial values are written here)
  for (int h = tid; h < p.Ho; h += THREADS) {
    part[h * (p.DVP + 2) + p.DVP] = sMax[h];
    part[h * (p.DVP + 2) + p.DVP + 1] = sSum[h];
  }
}

// One warp per (row, head): the shares' maxima and sums, the sink, then the columns.
__global__ void __launch_bounds__(128) mixed_merge_kernel(const MixedAttnParams p) {
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const long long item = blockIdx.x * 4ll + (threadIdx.x >> 5);
  if (item >= static_cast<long long>(p.rows) * p.Ho) return;
  const long long row = item / p.Ho;
  const int h = static_cast<int>(item - row * p.Ho), pitch = p.DVP + 2;
  const float* part = p.scratch + row * p.splits * p.Ho * pitch + static_cast<long long>(h) * pitch;
  const long long step = static_cast<long long>(p.Ho) * pitch;
  // lane s looks after share s (at most 32)
  const float m = lane < p.splits ? part[lane * step + p.DVP] : -INFINITY;
  const float z = p.sink ? p.sink[h] * kLog2e : -INFINITY;
  float top = m;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
  top = fmaxf(top, z);
  const float f = m == -INFINITY ? 0.f : exp2f(m - top);
  float l = f > 0.f ? f * part[lane * step + p.DVP + 1] : 0.f;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (p.sink) l += exp2f(z - top);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + row * p.out_stride + static_cast<long long>(h) * p.DV;
  for (int d0 = 0; d0 < p.DV; d0 += 32) {
    const int d = d0 + lane;
    float o = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float w = __shfl_sync(0xffffffffu, f, s);
      if (w > 0.f && d < p.DV) o = fmaf(w, part[s * step + d], o);
    }
    if (d < p.DV) out[d] = __float2bfloat16(o * inv);
  }
}

template <int UNITS, int WARPS, int KT>
static int launch_mixed_decode(const MixedAttnParams& p, int stages, int bytes, cudaStream_t stream) {
  auto kern = mixed_decode_kernel<UNITS, WARPS, KT>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -20;
    once.mark(dev);
  }
  return launch_pdl(kern, dim3(p.rows * p.splits), dim3(WARPS * 32), bytes, stream, 1, p, stages) == cudaSuccess ? 0 : -21;
}

template <int KT>
static int launch_mixed_decode_kt(const MixedAttnParams& p, const mdec::Plan& c, int bytes, cudaStream_t stream) {
  if (c.warps == 16) return launch_mixed_decode<16, 16, KT>(p, c.stages, bytes, stream);
  if (c.units <= 4) return launch_mixed_decode<4, 8, KT>(p, c.stages, bytes, stream);
  if (c.units <= 8) return launch_mixed_decode<8, 8, KT>(p, c.stages, bytes, stream);
  return launch_mixed_decode<16, 8, KT>(p, c.stages, bytes, stream);
}

int mixed_decode(const MixedAttnParams& p, cudaStream_t stream) {
  const mdec::Plan c = mdec::plan(p.Hs, p.Hk, p.Ho, p.Hv, p.DP, p.DVP);
  if (c.kt == 0 || p.splits > 32 || p.rows != p.B * p.q_len) return -2;
  const int bytes = mdec::layout(p.Hs, p.Hk, p.Ho, p.Hv, p.DP, p.DVP, c.kt, c.stages).bytes;
  const int rc = c.kt == 32 ? launch_mixed_decode_kt<32>(p, c, bytes, stream) : launch_mixed_decode_kt<16>(p, c, bytes, stream);
  if (rc != 0 || p.splits == 1) return rc;
  const long long items = static_cast<long long>(p.rows) * p.Ho;
  return launch_pdl(mixed_merge_kernel, dim3(static_cast<unsigned>((items + 3) / 4)), dim3(128), 0, stream, 1, p) ==
                 cudaSuccess ? 0 : -22;
}

}  // namespace b200
