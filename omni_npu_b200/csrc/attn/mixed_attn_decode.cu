// Decode step of the attention with mixed heads (mixed_attn.cuh), bf16.
//
// One CTA = one query row, a share of its keys, ALL heads (the mixture needs every head's score of a key).  Tiles of 16
// or 32 keys of all key and value heads come in with cp.async: a tile's values while its scores are made, the next
// tile's keys while the values are worked off, so that one buffer of each is enough and several CTAs share an SM.  Per
// tile:
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
  int q_off, k_off, v_off, s_off, p_off, t_off, r_off, m_off, bytes;
  int per_k, per_v;            // heads of a key head, of a value head
};

inline Layout layout(int Hs, int Hk, int Ho, int Hv, int DP, int DVP, int kt) {
  Layout l{};
  l.per_k = Hs / Hk;
  l.per_v = Ho / Hv;
  l.dk = (DP + 63) / 64 * 64;
  l.dv = (DVP + 63) / 64 * 64;
  l.hs4 = (Hs + 3) / 4 * 4;
  l.s_pitch = kt + 4;
  l.p_pitch = kt + 8;
  int at = 0;
  const auto take = [&](int bytes) {
    const int r = at;
    at += (bytes + 127) / 128 * 128;
    return r;
  };
  l.q_off = take(Hs * l.dk * 2);
  l.k_off = take(Hk * kt * l.dk * 2);
  l.v_off = take(Hv * kt * l.dv * 2);
  l.s_off = take(l.hs4 * l.s_pitch * 4);
  l.p_off = take(Ho * l.p_pitch * 2);
  l.t_off = take(Ho * l.hs4 * 4);
  l.r_off = take(2 * Hs * 4);
  l.m_off = take(3 * Ho * 4);
  l.bytes = at;
  return l;
}

struct Plan {
  int kt, warps, units;
};

// The first of the layouts, from fast to small, that fits; kt 0: none.
inline Plan plan(int Hs, int Hk, int Ho, int Hv, int DP, int DVP) {
  if (DP > 512 || DVP > 512) return {0, 0, 0};
  const int units = Hv * ((Ho / Hv + 7) / 8) * (DVP / 16);
  const int warps = units <= 16 * 8 ? 8 : 16;
  const int each = (units + warps - 1) / warps;
  if (each > 16) return {0, 0, 0};
  const int order[4][2] = {{32, 90}, {16, 112}, {32, 112}, {16, 226}};
  for (const auto& o : order)
    if (layout(Hs, Hk, Ho, Hv, DP, DVP, o[0]).bytes <= o[1] * 1024) return {o[0], warps, each};
  return {0, 0, 0};
}

}  // namespace mdec

bool mixed_decode_fits(int Hs, int Hk, int Ho, int Hv, int DP, int DVP) {
  return mdec::plan(Hs, Hk, Ho, Hv, DP, DVP).kt > 0;
}

// UNITS: accumulator tiles (8 heads x 16 columns) per warp.  HB: output heads that a lane mixes at a time
template <int UNITS, int WARPS, int KT, int HB>
__global__ void __launch_bounds__(WARPS * 32, WARPS == 8 && UNITS <= 8 ? 2 : 1)
mixed_decode_kernel(const MixedAttnParams p, const mdec::Layout L) {
  using namespace mdec;
  constexpr int THREADS = WARPS * 32, SUB = 32 / KT;
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t* sQ = smem + L.q_off;
  float* sS = reinterpret_cast<float*>(smem + L.s_off);                       // [hs4][s_pitch]
  __nv_bfloat16* sP = reinterpret_cast<__nv_bfloat16*>(smem + L.p_off);       // [Ho][p_pitch]
  float* sT = reinterpret_cast<float*>(smem + L.t_off);                       // [Ho][hs4], times log2 e
  float* sR = reinterpret_cast<float*>(smem + L.r_off);                       // r1, r2
  float* sMax = reinterpret_cast<float*>(smem + L.m_off);
  float* sSum = sMax + p.Ho;
  float* sCor = sSum + p.Ho;
  const uint32_t kt = smem_u32(smem + L.k_off), vt = smem_u32(smem + L.v_off);

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int row = blockIdx.x / p.splits, split = blockIdx.x % p.splits;
  const int per_k = L.per_k, per_v = L.per_v;
  const int kchunks8 = (per_k + 7) >> 3, vchunks8 = (per_v + 7) >> 3;

  pdl_trigger();
  // constants of the layer are no earlier kernel's result
  for (int i = tid; i < p.Ho * L.hs4; i += THREADS) {
    const int h = i / L.hs4, g = i - h * L.hs4;
    sT[i] = g < p.Hs ? p.talk[h * p.Hs + g] * kLog2e : 0.f;
  }
  for (int i = tid; i < p.Hs; i += THREADS) {
    sR[i] = p.r1 ? p.r1[i] * kLn2 : 0.f;
    sR[p.Hs + i] = p.r1 ? p.r2[i] : 0.f;
  }
  for (int i = tid; i < L.hs4 * L.s_pitch; i += THREADS) sS[i] = 0.f;
  for (int h = tid; h < p.Ho; h += THREADS) {
    sMax[h] = -INFINITY;
    sSum[h] = 0.f;
  }
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

  // Rows of a tile: `1 << ll` threads share a row, a thread has the same keys of every tile and walks over the heads.
  constexpr int MAX_KEYS = 4;                                                 // (ll is at most 5)
  auto lanes_log2 = [](int chunks) {
    int ll = 0;
    while (ll < 5 && (1 << ll) < chunks) ++ll;
    return ll;
  };
  const int kll = lanes_log2(p.DP >> 3), vll = lanes_log2(p.DVP >> 3);
  // the places of this thread's keys of a tile, looked up ahead of the copies
  auto look_up = [&](int tile, int ll, int (&place)[MAX_KEYS]) {
    const int slots = THREADS >> ll, kstep = min(slots, KT);
#pragma unroll
    for (int i = 0; i < MAX_KEYS; ++i) {
      const int j = ((tid >> ll) & (kstep - 1)) + i * kstep, key = tile * KT + j;
      place[i] = -1;
      if (j < KT && tile < t_end && key <= pos) {
        const int blk = p.bs_shift >= 0 ? key >> p.bs_shift : key / p.block_size;
        place[i] = bt[blk];
      }
    }
  };
  auto issue = [&](const __nv_bfloat16* cache, int heads, int width, int smem_width, int ll, uint32_t dst, int tile,
                   const int (&place)[MAX_KEYS]) {
    if (tile < t_end) {
      const int slots = THREADS >> ll, kstep = min(slots, KT), slot = tid >> ll, li = tid & ((1 << ll) - 1);
      const int g0 = slots > KT ? slot / KT : 0, gstep = slots > KT ? slots / KT : 1, chunks = width >> 3;
#pragma unroll
      for (int i = 0; i < MAX_KEYS; ++i) {
        const int j = (slot & (kstep - 1)) + i * kstep;
        if (j >= KT) continue;
        const int key = tile * KT + j;
        const int off = p.bs_shift >= 0 ? key & (p.block_size - 1) : key % p.block_size;
        const bool ok = place[i] >= 0;
        const __nv_bfloat16* row0 =
            ok ? cache + ((static_cast<long long>(place[i]) * heads + g0) * p.block_size + off) * width : cache;
        const long long step = ok ? static_cast<long long>(gstep) * p.block_size * width : 0;
        const uint32_t dst_step = gstep * KT * smem_width * 2;
        const int sz = ok ? 16 : 0;
        for (int c = li; c < chunks; c += 1 << ll) {
          const __nv_bfloat16* src = ok ? row0 + c * 8 : row0;
          uint32_t to = dst + piece(g0 * KT + j, c, smem_width);
#pragma unroll 4
          for (int g = g0; g < heads; g += gstep, src += step, to += dst_step)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to), "l"(src), "r"(sz) : "memory");
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  int place[MAX_KEYS], place_v[MAX_KEYS];
  look_up(t_begin, kll, place);
  look_up(t_begin, vll, place_v);
  issue(kc, p.Hk, p.DP, L.dk, kll, kt, t_begin, place);

  // query heads -> shared, zero beyond the head size
  const bool vec_q = (p.D & 7) == 0 && (p.q_stride & 7) == 0 && (reinterpret_cast<uintptr_t>(p.q) & 15) == 0;
  for (int i = tid; i < p.Hs * (p.DP >> 3); i += THREADS) {
    const int g = i / (p.DP >> 3), c = i - g * (p.DP >> 3);
    const __nv_bfloat16* src = q + g * p.D + c * 8;
    uint4 u = make_uint4(0u, 0u, 0u, 0u);
    if (vec_q) {
      if (c * 8 < p.D) u = *reinterpret_cast<const uint4*>(src);
    } else {
      __nv_bfloat16 h[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) h[j] = c * 8 + j < p.D ? src[j] : __float2bfloat16(0.f);
      uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
      for (int j = 0; j < 4; ++j)
        w[j] = static_cast<uint32_t>(__bfloat16_as_ushort(h[2 * j])) |
               (static_cast<uint32_t>(__bfloat16_as_ushort(h[2 * j + 1])) << 16);
    }
    *reinterpret_cast<uint4*>(sQ + piece(g, c, L.dk)) = u;
  }

  const ScoreConst c = score_const(p);
  float acc[UNITS][4];
#pragma unroll
  for (int i = 0; i < UNITS; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  // units: (key head, 8 of its heads, 16 keys), dealt out in turn; (value head, 8 of its heads, 16 columns), in runs of
  // neighbours.  A unit is taken apart with divisions only here.
  const int vtiles = p.DVP >> 4, units = p.Hv * vchunks8 * vtiles, run = (units + WARPS - 1) / WARPS;
  const int k_units = p.Hk * kchunks8 * (KT / 16);
  const int u_begin = min(units, warp * run), u_count = min(units, u_begin + run) - u_begin;
  const int gc_begin = u_begin / vtiles, vt_begin = u_begin - gc_begin * vtiles;
  const int g_begin = gc_begin / vchunks8, ch_begin = gc_begin - g_begin * vchunks8;
  const int k_sub = warp % (KT / 16), k_gc = warp / (KT / 16), k_g = k_gc / kchunks8, k_ch = k_gc - k_g * kchunks8;
  const int steps = p.DP >> 4;

  for (int tile = t_begin; tile < t_end; ++tile) {
    const int n0 = tile * KT;
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // keys are there; the values before are used up
    issue(vc, p.Hv, p.DVP, L.dv, vll, vt, tile, place_v);
    look_up(tile + 1, kll, place);
    look_up(tile + 1, vll, place_v);

    // ---- scores of 16 keys x 8 heads of a key head
    int sub = k_sub, g = k_g, ch = k_ch;
    for (int u = warp; u < k_units; u += WARPS) {
      if (u != warp) {
        const int gc = u / (KT / 16);
        sub = u % (KT / 16);
        g = gc / kchunks8;
        ch = gc - g * kchunks8;
      }
      const int krow = g * KT + sub * 16 + (lane & 15);
      const int head0 = g * per_k + ch * 8;
      const int qrow = min(head0 + (lane & 7), p.Hs - 1);
      float s[4] = {0.f, 0.f, 0.f, 0.f}, s2[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t k_at = kt + krow * L.dk * 2, q_at = smem_u32(sQ) + qrow * L.dk * 2;
      const uint32_t kx = ((lane >> 4) ^ (krow & 7)) << 4, qx = ((lane >> 3) ^ (qrow & 7)) << 4;
#pragma unroll 4
      for (int ks = 0; ks + 1 < steps; ks += 2) {          // two chains (chunks 2 ks .. 2 ks + 3)
        uint32_t ka[4], kb[4], qf[4];
        ldmatrix_x4(ka, k_at + ((ks << 5) ^ kx));
        ldmatrix_x4(kb, k_at + (((ks + 1) << 5) ^ kx));
        ldmatrix_x4(qf, q_at + ((ks << 5) ^ qx));
        mma_bf16_16816(s, ka, qf[0], qf[1]);
        mma_bf16_16816(s2, kb, qf[2], qf[3]);
      }
      if (steps & 1) {
        uint32_t ka[4], qf[4];
        ldmatrix_x4(ka, kt + piece(krow, steps * 2 - 2 + (lane >> 4), L.dk));
        ldmatrix_x4(qf, smem_u32(sQ) + piece(qrow, steps * 2 - 2 + ((lane >> 3) & 1), L.dk));
        mma_bf16_16816(s, ka, qf[0], qf[1]);
      }
      const float d0 = static_cast<float>(pos - n0 - sub * 16 - (lane >> 2));
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int hl = ch * 8 + (lane & 3) * 2 + (j & 1), key = sub * 16 + (lane >> 2) + (j >> 1) * 8;
        if (hl < per_k) {
          const int h = g * per_k + hl;
          const float x = s[j] + s2[j], dist = fmaxf(j < 2 ? d0 : d0 - 8.f, 0.f);
          sS[h * L.s_pitch + key] = (c.cap > 0.f ? capped_score<true>(c, x) : capped_score<false>(c, x)) -
                                    distance_bias(sR[h], sR[p.Hs + h], dist);
        }
      }
    }
    __syncthreads();                                       // scores are there; the keys are used up
    issue(kc, p.Hk, p.DP, L.dk, kll, kt, tile + 1, place);

    // ---- mixture and softmax: a lane = one key, KT lanes = a head, HB heads at a time
    {
      const int key = lane % KT, sub = lane / KT;
      const bool seen = n0 + key <= pos;
      for (int h0 = (warp * SUB + sub) * HB; h0 - sub * HB < p.Ho; h0 += WARPS * SUB * HB) {      // (warp-uniform)
        float s[HB], mx[HB], e[HB], sum[HB], old[HB];
        const float* t[HB];
#pragma unroll
        for (int i = 0; i < HB; ++i) {
          s[i] = 0.f;
          t[i] = sT + min(h0 + i, p.Ho - 1) * L.hs4;
          old[i] = sMax[min(h0 + i, p.Ho - 1)];
        }
#pragma unroll 4
        for (int g = 0; g < L.hs4; g += 4) {
          float a[4];
#pragma unroll
          for (int k = 0; k < 4; ++k) a[k] = sS[(g + k) * L.s_pitch + key];
#pragma unroll
          for (int i = 0; i < HB; ++i) {
            const float4 w = *reinterpret_cast<const float4*>(t[i] + g);
            s[i] = fmaf(w.x, a[0], fmaf(w.y, a[1], fmaf(w.z, a[2], fmaf(w.w, a[3], s[i]))));
          }
        }
#pragma unroll
        for (int i = 0; i < HB; ++i) mx[i] = seen ? s[i] : -INFINITY;
#pragma unroll
        for (int o = KT / 2; o > 0; o >>= 1)
#pragma unroll
          for (int i = 0; i < HB; ++i) mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], o));
#pragma unroll
        for (int i = 0; i < HB; ++i) {
          mx[i] = fmaxf(mx[i], old[i]);                    // (a tile holds a visible key: finite)
          e[i] = seen ? exp2f(s[i] - mx[i]) : 0.f;
          sum[i] = e[i];
          if (h0 + i < p.Ho) sP[(h0 + i) * L.p_pitch + key] = __float2bfloat16(e[i]);
        }
#pragma unroll
        for (int o = KT / 2; o > 0; o >>= 1)
#pragma unroll
          for (int i = 0; i < HB; ++i) sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], o);
        if (key == 0) {
#pragma unroll
          for (int i = 0; i < HB; ++i) {
            const int h = h0 + i;
            if (h >= p.Ho) continue;
            const float f = exp2f(old[i] - mx[i]);         // (the first tile: 0)
            sMax[h] = mx[i];
            sSum[h] = sSum[h] * f + sum[i];
            sCor[h] = f;
          }
        }
      }
    }
    asm volatile("cp.async.wait_group 1;" ::: "memory");   // this tile's values; the next keys may be on their way
    __syncthreads();

    // ---- values: (8 heads of a value head) x 16 columns
    {
      int vtile = vt_begin, vg = g_begin, vch = ch_begin;
      float c0 = 0.f, c1 = 0.f;
      uint32_t pf[KT / 16][2], v_at = 0;
      const int vr = ((lane >> 4) << 3) + (lane & 7);      // (rows of a tile start at multiples of 8)
      const uint32_t vx = (((lane >> 3) & 1) ^ (lane & 7)) << 4;
#pragma unroll
      for (int i = 0; i < UNITS; ++i) {
        if (i >= u_count) continue;
        if (i == 0 || vtile == vtiles) {                   // the next 8 heads
          if (i != 0) {
            vtile = 0;
            if (++vch == vchunks8) {
              vch = 0;
              ++vg;
            }
          }
          const int head0 = vg * per_v + vch * 8, hc = head0 + (lane & 3) * 2;
          c0 = sCor[min(hc, p.Ho - 1)];
          c1 = sCor[min(hc + 1, p.Ho - 1)];
          const __nv_bfloat16* pr = sP + min(head0 + (lane >> 2), p.Ho - 1) * L.p_pitch + (lane & 3) * 2;
#pragma unroll
          for (int ks = 0; ks < KT / 16; ++ks) {
            pf[ks][0] = *reinterpret_cast<const uint32_t*>(pr + ks * 16);
            pf[ks][1] = *reinterpret_cast<const uint32_t*>(pr + ks * 16 + 8);
          }
          v_at = vt + (vg * KT + vr) * L.dv * 2;
        }
        acc[i][0] *= c0;
        acc[i][1] *= c1;
        acc[i][2] *= c0;
        acc[i][3] *= c1;
#pragma unroll
        for (int ks = 0; ks < KT / 16; ++ks) {
          uint32_t vf[4];
          ldmatrix_x4_trans(vf, v_at + ks * 16 * L.dv * 2 + ((vtile << 5) ^ vx));
          mma_bf16_16816(acc[i], vf, pf[ks][0], pf[ks][1]);
        }
        ++vtile;
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");

  // ---- the row, or this share of it
  if (p.splits == 1) {
#pragma unroll
    for (int i = 0; i < UNITS; ++i) {
      if (i >= u_count) continue;
      const int u = u_begin + i, vtile = u % vtiles, gc = u / vtiles, g = gc / vchunks8, ch = gc - g * vchunks8;
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
  const long long share_row = static_cast<long long>(row) * p.splits + split;
  float* part = p.scratch + share_row * p.Ho * p.DVP;
  float2* stat = reinterpret_cast<float2*>(p.scratch + static_cast<long long>(p.rows) * p.splits * p.Ho * p.DVP) +
                 share_row * p.Ho;
#pragma unroll
  for (int i = 0; i < UNITS; ++i) {
    if (i >= u_count) continue;
    const int u = u_begin + i, vtile = u % vtiles, gc = u / vtiles, g = gc / vchunks8, ch = gc - g * vchunks8;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int hl = ch * 8 + (lane & 3) * 2 + (j & 1), d = vtile * 16 + (lane >> 2) + (j >> 1) * 8;
      if (hl < per_v) part[(g * per_v + hl) * p.DVP + d] = acc[i][j];
    }
  }
  __syncthreads();                                         // (a row without a tile: the initial values are written here)
  for (int h = tid; h < p.Ho; h += THREADS) stat[h] = make_float2(sMax[h], sSum[h]);
}

// One CTA per (row, head): every warp works out the shares' factors, with the sink, and adds up a quarter of the shares.
static constexpr int kMergeWarps = 4;

__global__ void __launch_bounds__(kMergeWarps * 32) mixed_merge_kernel(const MixedAttnParams p) {
  extern __shared__ float sm[];                            // [kMergeWarps][DVP]
  pdl_trigger();
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, h = blockIdx.x;
  const long long row = blockIdx.y;
  const long long step = static_cast<long long>(p.Ho) * p.DVP;
  const float* part = p.scratch + row * p.splits * step + static_cast<long long>(h) * p.DVP;
  const float2* stat = reinterpret_cast<const float2*>(p.scratch + static_cast<long long>(p.rows) * p.splits * step) +
                       row * p.splits * p.Ho + h;
  // lane s looks after shares s and s + 32
  const float2 none = make_float2(-INFINITY, 0.f);
  const float2 a = lane < p.splits ? stat[static_cast<long long>(lane) * p.Ho] : none;
  const float2 b = lane + 32 < p.splits ? stat[static_cast<long long>(lane + 32) * p.Ho] : none;
  const float z = p.sink ? p.sink[h] * kLog2e : -INFINITY;
  float top = fmaxf(a.x, b.x);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
  top = fmaxf(top, z);
  const float fa = a.x == -INFINITY ? 0.f : exp2f(a.x - top), fb = b.x == -INFINITY ? 0.f : exp2f(b.x - top);
  float l = fa * a.y + fb * b.y;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
  if (p.sink) l += exp2f(z - top);
  for (int d = lane * 4; d - lane * 4 < p.DVP; d += 128) { // (a share without keys holds zeros)
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = warp; s < p.splits; s += kMergeWarps) {
      const float w = __shfl_sync(0xffffffffu, s < 32 ? fa : fb, s & 31);
      if (d < p.DVP) {
        const float4 x = *reinterpret_cast<const float4*>(part + s * step + d);
        o.x = fmaf(w, x.x, o.x);
        o.y = fmaf(w, x.y, o.y);
        o.z = fmaf(w, x.z, o.z);
        o.w = fmaf(w, x.w, o.w);
      }
    }
    if (d < p.DVP) *reinterpret_cast<float4*>(sm + warp * p.DVP + d) = o;
  }
  __syncthreads();
  const float inv = l > 0.f ? 1.f / l : 0.f;
  __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out) + row * p.out_stride + static_cast<long long>(h) * p.DV;
  for (int d = threadIdx.x; d < p.DV; d += kMergeWarps * 32) {
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kMergeWarps; ++w) o += sm[w * p.DVP + d];
    out[d] = __float2bfloat16(o * inv);
  }
}

template <int UNITS, int WARPS, int KT, int HB>
static int launch_mixed_decode(const MixedAttnParams& p, const mdec::Layout& l, cudaStream_t stream) {
  auto kern = mixed_decode_kernel<UNITS, WARPS, KT, HB>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -20;
    once.mark(dev);
  }
  return launch_pdl(kern, dim3(p.rows * p.splits), dim3(WARPS * 32), l.bytes, stream, 1, p, l) == cudaSuccess ? 0 : -21;
}

template <int KT>
static int launch_mixed_decode_kt(const MixedAttnParams& p, const mdec::Plan& c, cudaStream_t stream) {
  const mdec::Layout l = mdec::layout(p.Hs, p.Hk, p.Ho, p.Hv, p.DP, p.DVP, KT);
  const int groups = c.warps * (32 / KT);                // lanes' groups that mix a head each
  if (c.warps == 16) return launch_mixed_decode<16, 16, KT, 2>(p, l, stream);
  if (c.units <= 4) {
    if (p.Ho <= groups) return launch_mixed_decode<4, 8, KT, 1>(p, l, stream);
    return p.Ho <= 2 * groups ? launch_mixed_decode<4, 8, KT, 2>(p, l, stream)
                              : launch_mixed_decode<4, 8, KT, 4>(p, l, stream);
  }
  if (c.units <= 8) return p.Ho <= 2 * groups ? launch_mixed_decode<8, 8, KT, 2>(p, l, stream)
                                              : launch_mixed_decode<8, 8, KT, 4>(p, l, stream);
  return launch_mixed_decode<16, 8, KT, 4>(p, l, stream);
}

int mixed_decode(const MixedAttnParams& p, cudaStream_t stream) {
  const mdec::Plan c = mdec::plan(p.Hs, p.Hk, p.Ho, p.Hv, p.DP, p.DVP);
  if (c.kt == 0 || p.splits > 64 || p.rows != p.B * p.q_len) return -2;
  const int rc = c.kt == 32 ? launch_mixed_decode_kt<32>(p, c, stream) : launch_mixed_decode_kt<16>(p, c, stream);
  if (rc != 0 || p.splits == 1) return rc;
  return launch_pdl(mixed_merge_kernel, dim3(p.Ho, p.rows), dim3(kMergeWarps * 32), kMergeWarps * p.DVP * sizeof(float), stream,
                    1, p) == cudaSuccess ? 0 : -22;
}

}  // namespace b200
