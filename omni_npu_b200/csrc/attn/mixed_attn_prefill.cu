// Prompt portions of the attention with mixed heads (mixed_attn.cuh), bf16.  A key's score in one head needs all
// heads' products of that (query, key) pair, so the work is cut twice:
//
//   mixed_scores_kernel   16 queries x a range of keys, all heads: Q K^T on mma.sync with the queries of a warp's heads in
//                         registers, capped and lowered into shared memory, then the mixture as fp32 outer products
//                         (8 output heads x 4 keys per thread); mixed scores to memory in fp32.  The distance bias of a
//                         tile has 15 + keys values per head: a table, made while the tile before is mixed
//   mixed_values_kernel   128 rows = tokens x heads of a value head: online softmax over the stored scores, sink, P V
//
// The scores of as many query tiles as fit into the given buffer are made per call.

#include <type_traits>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "attn_common.cuh"
#include "attn_params.cuh"
#include "mixed_attn.cuh"

namespace b200 {

namespace mpre {
constexpr int BQ = 16;                   // queries of a score tile
constexpr int RANGE = 256;               // keys of a score CTA

__device__ __forceinline__ uint32_t piece(int row, int chunk, int width) {
  return static_cast<uint32_t>(row * width * 2 + ((chunk ^ (row & 7)) << 4));
}

struct Layout {
  int dk, ho8, s_pitch, d_pitch, k_bytes, s_off, t_off, d_off, bytes;
};
// ring of `stages` key tiles | scores [Hs][16][s_pitch] | talk^T [Hs][ho8] | distance bias [2][Hs][d_pitch]
__host__ __device__ inline Layout layout(int Hs, int Hk, int Ho, int DP, int bk, int stages) {
  Layout l;
  l.dk = DP <= 64 ? 64 : DP <= 128 ? 128 : 256;            // 16 times the kernel's KS
  l.ho8 = (Ho + 7) / 8 * 8;
  l.s_pitch = bk + 8;
  l.k_bytes = Hk * bk * l.dk * 2;
  l.s_off = stages * l.k_bytes;
  l.t_off = l.s_off + Hs * BQ * l.s_pitch * 4;
  l.d_pitch = bk + BQ;
  l.d_off = l.t_off + Hs * l.ho8 * 4;
  l.bytes = l.d_off + 2 * Hs * l.d_pitch * 4;
  return l;
}

struct Plan {
  int bk, stages, warps, ks;
};
inline Plan plan(int Hs, int Hk, int Ho, int DP) {
  if (DP > 256) return {0, 0, 0, 0};
  const int warps = Hs <= 16 ? 8 : 16, ks = DP <= 64 ? 4 : DP <= 128 ? 8 : 16;
  const int order[5][3] = {{32, 2, 112}, {32, 2, 226}, {32, 1, 226}, {16, 2, 226}, {16, 1, 226}};
  for (const auto& o : order)
    if (layout(Hs, Hk, Ho, DP, o[0], o[1]).bytes <= o[2] * 1024) return {o[0], o[1], warps, ks};
  return {0, 0, 0, 0};
}
}  // namespace mpre

bool mixed_prefill_fits(int Hs, int Hk, int Ho, int Hv, int DP, int DVP) {
  return DVP <= 256 && mpre::plan(Hs, Hk, Ho, DP).bk > 0;
}

// ------------------------------------------------------------- scores
// KS: steps of 16 along the head size; HPW: heads per warp and pass (16 registers of query per head and 4 steps)
template <int WARPS, int KS, int HPW, int BK>
__global__ void __launch_bounds__(WARPS * 32, WARPS == 8 ? 2 : 1) mixed_scores_kernel(const MixedAttnParams p, const int stages) {
  using namespace mpre;
  constexpr int THREADS = WARPS * 32, DK = KS * 16;
  extern __shared__ __align__(128) uint8_t smem[];
  const Layout L = layout(p.Hs, p.Hk, p.Ho, p.DP, BK, stages);
  float* sS = reinterpret_cast<float*>(smem + L.s_off);
  float* sT = reinterpret_cast<float*>(smem + L.t_off);
  float* sD = reinterpret_cast<float*>(smem + L.d_off);
  const uint32_t ring = smem_u32(smem);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z;
  const long long q_begin = p.cu_q[b];
  const int q_len = static_cast<int>(p.cu_q[b + 1] - q_begin);
  const int tok0 = (p.tile0 + blockIdx.x) * BQ;
  if (tok0 >= q_len) return;
  const int ctx = p.seq_lens[b] - q_len;
  const int hi = ctx + min(q_len, tok0 + BQ);                      // keys that some row sees
  const int k_begin = blockIdx.y * RANGE, k_end = min(hi, k_begin + RANGE);
  if (k_begin >= k_end) return;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q);
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(p.k_cache);
  const int per = p.Hs / p.Hk;

  // `1 << ll` threads share a row, a thread has the same keys of every tile and walks over the heads
  const int chunks = p.DP >> 3;
  int ll = 0;
  while (ll < 5 && (1 << ll) < chunks) ++ll;
  const int slots = THREADS >> ll, kstep = min(slots, BK), slot = tid >> ll, li = tid & ((1 << ll) - 1);
  const int g0 = slots > BK ? slot / BK : 0, gstep = slots > BK ? slots / BK : 1;
  auto issue = [&](int i) {
    const int n0 = k_begin + i * BK;
    if (n0 < k_end) {
      const uint32_t dst = ring + (stages == 2 ? i & 1 : 0) * L.k_bytes;
      for (int j = slot & (kstep - 1); j < BK; j += kstep) {
        const int key = n0 + j;
        const bool ok = key < k_end;
        const __nv_bfloat16* row0 = ok ? kc + cache_row(p, bt, key, g0, p.Hk) * p.DP : kc;
        const long long step = ok ? static_cast<long long>(gstep) * p.block_size * p.DP : 0;
        const int sz = ok ? 16 : 0;
        for (int c = li; c < chunks; c += 1 << ll) {
          const __nv_bfloat16* src = ok ? row0 + c * 8 : row0;
          uint32_t to = dst + piece(g0 * BK + j, c, DK);
#pragma unroll 4
          for (int g = g0; g < p.Hk; g += gstep, src += step, to += gstep * BK * DK * 2)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(to), "l"(src), "r"(sz) : "memory");
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  if (stages == 2) issue(0);
  for (int i = tid; i < p.Hs * L.ho8; i += THREADS) {
    const int g = i / L.ho8, h = i - g * L.ho8;
    sT[i] = h < p.Ho ? p.talk[h * p.Hs + g] * kLog2e : 0.f;
  }
  // distance bias of tile i: entry x of a head is for distance base + x, base = first query - last key
  auto make_bias = [&](int i) {
    if (k_begin + i * BK >= k_end) return;
    const int base = ctx + tok0 - (k_begin + i * BK + BK - 1);
    float* dst = sD + (i & 1) * p.Hs * L.d_pitch;
    for (int e = tid; e < p.Hs * (BK + BQ); e += THREADS) {
      const int g = e / (BK + BQ), x = e - g * (BK + BQ);
      dst[e] = p.r1 ? distance_bias(__ldg(p.r1 + g) * kLn2, __ldg(p.r2 + g), fmaxf(static_cast<float>(base + x), 0.f)) : 0.f;
    }
  };
  make_bias(0);

  // query fragments of the heads of a pass, straight from memory
  uint32_t qf[HPW][KS][4];
  const bool pairs = (p.D & 1) == 0 && (p.q_stride & 1) == 0 && (reinterpret_cast<uintptr_t>(q) & 3) == 0;
  const int tok_a = min(tok0 + (lane >> 2), q_len - 1), tok_b = min(tok0 + (lane >> 2) + 8, q_len - 1);
  auto load_q = [&](int pass) {                            // (rows beyond the portion repeat its last one)
#pragma unroll
    for (int j = 0; j < HPW; ++j) {
      const int g = (pass * WARPS + warp) * HPW + j;
      if (g >= p.Hs) continue;
      const __nv_bfloat16* at = q + static_cast<long long>(g) * p.D + (lane & 3) * 2;
      const __nv_bfloat16* src[2] = {at + (q_begin + tok_a) * p.q_stride, at + (q_begin + tok_b) * p.q_stride};
#pragma unroll
      for (int ks = 0; ks < KS; ++ks)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int d = ks * 16 + (e >> 1) * 8;
          uint32_t v = 0u;
          if (d + (lane & 3) * 2 < p.D) {
            if (pairs) {
              v = *reinterpret_cast<const uint32_t*>(src[e & 1] + d);
            } else {
              v = __bfloat16_as_ushort(src[e & 1][d]);
              if (d + (lane & 3) * 2 + 1 < p.D) v |= static_cast<uint32_t>(__bfloat16_as_ushort(src[e & 1][d + 1])) << 16;
            }
          }
          qf[j][ks][e] = v;
        }
    }
  };
  const int passes = (p.Hs + WARPS * HPW - 1) / (WARPS * HPW);
  if (passes == 1) load_q(0);

  const ScoreConst c = score_const(p);
  const int tiles = (k_end - k_begin + BK - 1) / BK;
  const int ks_used = p.DP >> 4;
  uint32_t kx[4];                                          // swizzled chunk of a row, by step modulo 4
#pragma unroll
  for (int i = 0; i < 4; ++i) kx[i] = ((i * 2 + ((lane >> 3) & 1)) ^ (lane & 7)) << 4;
  for (int it = 0; it < tiles; ++it) {
    if (stages == 1) {
      if (it) __syncthreads();
      issue(it);
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (stages == 2) issue(it + 1);
    const uint32_t kt = ring + (stages == 2 ? it & 1 : 0) * L.k_bytes;
    const int n0 = k_begin + it * BK;

    for (int pass = 0; pass < passes; ++pass) {
      if (passes > 1) load_q(pass);
#pragma unroll
      for (int j = 0; j < HPW; ++j) {
        const int g = (pass * WARPS + warp) * HPW + j;
        if (g >= p.Hs) continue;
        const uint32_t k_at = kt + ((g / per) * BK + (lane & 7) + ((lane >> 4) << 3)) * DK * 2;
        float s[BK / 8][4];
#pragma unroll
        for (int n = 0; n < BK / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          if (ks < ks_used) {
#pragma unroll
            for (int n = 0; n < BK / 16; ++n) {
              uint32_t kf[4];
              ldmatrix_x4(kf, k_at + n * 16 * DK * 2 + (ks >> 2) * 128 + kx[ks & 3]);
              mma_bf16_16816(s[2 * n], qf[j][ks], kf[0], kf[1]);
              mma_bf16_16816(s[2 * n + 1], qf[j][ks], kf[2], kf[3]);
            }
          }
        }
        float* dst = sS + g * BQ * L.s_pitch + (lane >> 2) * L.s_pitch + (lane & 3) * 2;
        const float* bias = sD + ((it & 1) * p.Hs + g) * L.d_pitch + BK - 1 + (lane >> 2) - (lane & 3) * 2;
        auto put = [&](auto cap) {
#pragma unroll
          for (int n = 0; n < BK / 8; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r)
              *reinterpret_cast<float2*>(dst + r * 8 * L.s_pitch + n * 8) =
                  make_float2(capped_score<decltype(cap)::value>(c, s[n][2 * r]) - bias[r * 8 - n * 8],
                              capped_score<decltype(cap)::value>(c, s[n][2 * r + 1]) - bias[r * 8 - n * 8 - 1]);
        };
        if (c.cap > 0.f) put(std::true_type{});
        else put(std::false_type{});
      }
    }
    __syncthreads();
    make_bias(it + 1);

    // ---- mixture: an item = 8 output heads x 4 keys of a query
    constexpr int GROUPS = BQ * BK / 4;
    const int items = (L.ho8 >> 3) * GROUPS;
    for (int item = tid; item < items; item += THREADS) {
      const int hc = item / GROUPS * 8, grp = item % GROUPS;
      const int row = grp / (BK / 4), key = grp % (BK / 4) * 4;
      float o[8][4];
#pragma unroll
      for (int h = 0; h < 8; ++h)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[h][e] = 0.f;
      const float* src = sS + row * L.s_pitch + key;
      const float* t = sT + hc;
#pragma unroll 4
      for (int g = 0; g < p.Hs; ++g) {
        const float4 a = *reinterpret_cast<const float4*>(src + g * BQ * L.s_pitch);
        const float4 w0 = *reinterpret_cast<const float4*>(t + g * L.ho8), w1 = *reinterpret_cast<const float4*>(t + g * L.ho8 + 4);
        const float w[8] = {w0.x, w0.y, w0.z, w0.w, w1.x, w1.y, w1.z, w1.w};
#pragma unroll
        for (int h = 0; h < 8; ++h) {
          o[h][0] = fmaf(w[h], a.x, o[h][0]);
          o[h][1] = fmaf(w[h], a.y, o[h][1]);
          o[h][2] = fmaf(w[h], a.z, o[h][2]);
          o[h][3] = fmaf(w[h], a.w, o[h][3]);
        }
      }
      if (tok0 + row < q_len) {
        float* dst = p.scratch +
                     (((static_cast<long long>(b) * p.tiles + blockIdx.x) * BQ + row) * p.Ho + hc) * p.pitch + n0 + key;
#pragma unroll
        for (int h = 0; h < 8; ++h)
          if (hc + h < p.Ho)
            *reinterpret_cast<float4*>(dst + h * p.pitch) = make_float4(o[h][0], o[h][1], o[h][2], o[h][3]);
      }
    }
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
}

// ------------------------------------------------------------- softmax and values
namespace mval {
constexpr int BM = 128, BN = 64, THREADS = 256;
constexpr int S_PITCH = BN + 8;          // floats
constexpr int S_BYTES = BM * S_PITCH * 4;
}

// DV: upper bound of the padded value size
template <int DV>
__global__ void __launch_bounds__(mval::THREADS, DV > 128 ? 1 : 2) mixed_values_kernel(const MixedAttnParams p,
                                                                                       const int heads_per_tile) {
  using namespace mval;
  extern __shared__ __align__(128) uint8_t smem[];
  constexpr int V_BYTES = BN * DV * 2;
  const uint32_t v0 = smem_u32(smem), s0 = v0 + 2 * V_BYTES;
  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int per = p.Ho / p.Hv;
  const int hchunks = (per + heads_per_tile - 1) / heads_per_tile;
  const int vh = blockIdx.y / hchunks, head0 = (blockIdx.y % hchunks) * heads_per_tile;
  const int hc = min(heads_per_tile, per - head0);
  const int tt = BM / hc;
  const long long q_begin = p.cu_q[b];
  const int q_len = static_cast<int>(p.cu_q[b + 1] - q_begin);
  const int first = p.tile0 * mpre::BQ;
  const int last = min(q_len, first + p.tiles * mpre::BQ);
  const int m0 = first + (gridDim.x - 1 - blockIdx.x) * tt;        // (the tiles with most keys first)
  if (m0 >= last) return;
  const int tok_end = min(last, m0 + tt);
  const int ctx = p.seq_lens[b] - q_len, hi = ctx + tok_end;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(p.v_cache);
  const int tiles = (hi + BN - 1) / BN;

  const int rows_live = (tok_end - m0) * hc;                       // rows: (token, head of the group)
  const float* sbase = p.scratch + ((static_cast<long long>(b) * p.tiles * mpre::BQ + (m0 - first)) * p.Ho +
                                    vh * per + head0) * p.pitch;
  auto srow = [&](int r) {
    const int tok = r / hc;
    return sbase + (static_cast<long long>(tok) * p.Ho + (r - tok * hc)) * p.pitch;
  };
  auto issue = [&](int it) {
    if (it < tiles) {
      // four threads per key row, 16-byte pieces dealt out in turn
      const int r = tid >> 2, key = it * BN + r;
      const bool ok = key < hi;
      const __nv_bfloat16* src = ok ? vc + cache_row(p, bt, key, vh, p.Hv) * p.DVP : vc;
      const int sz = ok ? 16 : 0;
      const uint32_t dst = v0 + (it & 1) * V_BYTES;
      for (int c = tid & 3; c < (p.DVP >> 3); c += 4)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + tile_offset<DV>(r, c)),
                     "l"(ok ? src + c * 8 : src), "r"(sz) : "memory");
      // 16 threads per row of scores (all within the row's pitch; what lies beyond a row's position is masked)
      const uint32_t sdst = s0 + (it & 1) * S_BYTES + (tid & 15) * 16;
#pragma unroll
      for (int i = 0; i < BM / 16; ++i) {
        const int rr = (tid >> 4) + i * 16;
        if (rows_live > rr)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(sdst + rr * S_PITCH * 4),
                       "l"(srow(rr) + it * BN + (tid & 15) * 4) : "memory");
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0);

  float o_acc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o_acc[i][j] = 0.f;
  float row_max[2], row_sum[2];
  int pos[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int row = warp * 16 + (lane >> 2) + r * 8;
    const int tok = m0 + row / hc, h = vh * per + head0 + row % hc;
    const bool ok = row < tt * hc && tok < tok_end;
    pos[r] = ok ? ctx + tok : -1;
    // the sink is a key seen from the start: maximum = its score, sum = 1 (summed over the quad at the end)
    row_max[r] = ok && p.sink ? p.sink[h] * kLog2e : -INFINITY;
    row_sum[r] = ok && p.sink && (lane & 3) == 0 ? 1.f : 0.f;
  }
  const int w_hi = min(ctx + tok_end - 1, ctx + m0 + (warp * 16 + 15) / hc);       // last position of this warp's rows

  for (int it = 0; it < tiles; ++it) {
    issue(it + 1);
    const int n0 = it * BN;
    const bool seen = n0 <= w_hi;
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    if (seen) {
      float s[BN / 8][4];
      const float* st = reinterpret_cast<const float*>(smem + 2 * V_BYTES + (it & 1) * S_BYTES) +
                        (warp * 16 + (lane >> 2)) * S_PITCH + (lane & 3) * 2;
      const bool interior = n0 + BN - 1 <= ctx + m0 && (warp * 16 + 15) < rows_live;
#pragma unroll
      for (int i = 0; i < BN / 8; ++i)
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const float2 x = *reinterpret_cast<const float2*>(st + r * 8 * S_PITCH + i * 8);
          const int key = n0 + i * 8 + (lane & 3) * 2;
          s[i][2 * r] = interior || key <= pos[r] ? x.x : -INFINITY;
          s[i][2 * r + 1] = interior || key + 1 <= pos[r] ? x.y : -INFINITY;
        }
      const uint32_t vt = v0 + (it & 1) * V_BYTES;
      float corr[2], m_use[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        float m = -INFINITY;
#pragma unroll
        for (int i = 0; i < BN / 8; ++i) m = fmaxf(m, fmaxf(s[i][2 * r], s[i][2 * r + 1]));
        const float nm = fmaxf(row_max[r], quad_max(m));
        corr[r] = nm == -INFINITY ? 1.f : exp2f(row_max[r] - nm);
        m_use[r] = nm == -INFINITY ? 0.f : nm;
        row_max[r] = nm;
        row_sum[r] *= corr[r];
      }
#pragma unroll
      for (int i = 0; i < BN / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          s[i][j] = exp2f(s[i][j] - m_use[j >> 1]);
          row_sum[j >> 1] += s[i][j];
        }
      if (corr[0] != 1.f || corr[1] != 1.f) {
#pragma unroll
        for (int i = 0; i < DV / 8; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) o_acc[i][j] *= corr[j >> 1];
      }
#pragma unroll
      for (int ks = 0; ks < BN / 16; ++ks) {
        uint32_t pa[4];
        pa[0] = pack_bf16x2(s[2 * ks][0], s[2 * ks][1]);
        pa[1] = pack_bf16x2(s[2 * ks][2], s[2 * ks][3]);
        pa[2] = pack_bf16x2(s[2 * ks + 1][0], s[2 * ks + 1][1]);
        pa[3] = pack_bf16x2(s[2 * ks + 1][2], s[2 * ks + 1][3]);
#pragma unroll
        for (int dt = 0; dt < DV / 16; ++dt) {
          if (dt * 16 < p.DVP) {
            uint32_t vf[4];
            ldmatrix_x4_trans(vf, vt + tile_offset<DV>(ks * 16 + (lane & 15), dt * 2 + (lane >> 4)));
            mma_bf16_16816(o_acc[2 * dt], pa, vf[0], vf[1]);
            mma_bf16_16816(o_acc[2 * dt + 1], pa, vf[2], vf[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");

#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const float l = quad_sum(row_sum[r]);
    if (pos[r] < 0) continue;
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const int row = warp * 16 + (lane >> 2) + r * 8;
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + (q_begin + m0 + row / hc) * p.out_stride +
                         static_cast<long long>(vh * per + head0 + row % hc) * p.DV;
    const bool pairs = (reinterpret_cast<uintptr_t>(dst) & 3) == 0;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      const int d = i * 8 + (lane & 3) * 2;
      if (d >= p.DV) continue;
      const float o0 = o_acc[i][2 * r] * inv, o1 = o_acc[i][2 * r + 1] * inv;
      if (pairs && d + 1 < p.DV) {
        *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16x2(o0, o1);
      } else {
        dst[d] = __float2bfloat16(o0);
        if (d + 1 < p.DV) dst[d + 1] = __float2bfloat16(o1);
      }
    }
  }
}

template <int WARPS, int KS, int HPW, int BK>
static int launch_scores(const MixedAttnParams& p, int stages, cudaStream_t stream) {
  auto kern = mixed_scores_kernel<WARPS, KS, HPW, BK>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -20;
    once.mark(dev);
  }
  const int bytes = mpre::layout(p.Hs, p.Hk, p.Ho, p.DP, BK, stages).bytes;
  const dim3 grid(p.tiles, (p.max_keys + mpre::RANGE - 1) / mpre::RANGE, p.B);
  return launch_pdl(kern, grid, dim3(WARPS * 32), bytes, stream, 1, p, stages) == cudaSuccess ? 0 : -21;
}

template <int WARPS, int BK>
static int launch_scores_ks(const MixedAttnParams& p, const mpre::Plan& c, cudaStream_t stream) {
  if (c.ks == 4) return launch_scores<WARPS, 4, 4, BK>(p, c.stages, stream);
  if (c.ks == 8) return launch_scores<WARPS, 8, 2, BK>(p, c.stages, stream);
  return launch_scores<WARPS, 16, 1, BK>(p, c.stages, stream);
}

template <int DV>
static int launch_values(const MixedAttnParams& p, cudaStream_t stream) {
  auto kern = mixed_values_kernel<DV>;
  static DeviceOnce once;
  int dev = 0;
  constexpr int SMEM = 2 * mval::BN * DV * 2 + 2 * mval::S_BYTES;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM) != cudaSuccess) return -20;
    once.mark(dev);
  }
  const int per = p.Ho / p.Hv, heads = per < mval::BM ? per : mval::BM;
  const int hchunks = (per + heads - 1) / heads, tt = mval::BM / heads;
  const int toks = p.tiles * mpre::BQ;
  const dim3 grid((toks + tt - 1) / tt, p.Hv * hchunks, p.B);
  return launch_pdl(kern, grid, dim3(mval::THREADS), SMEM, stream, 1, p, heads) == cudaSuccess ? 0 : -21;
}

int mixed_prefill(const MixedAttnParams& p, cudaStream_t stream) {
  const mpre::Plan c = mpre::plan(p.Hs, p.Hk, p.Ho, p.DP);
  if (c.bk == 0 || p.DVP > 256) return -2;
  int rc;
  if (c.bk == 32) rc = c.warps == 8 ? launch_scores_ks<8, 32>(p, c, stream) : launch_scores_ks<16, 32>(p, c, stream);
  else rc = c.warps == 8 ? launch_scores_ks<8, 16>(p, c, stream) : launch_scores_ks<16, 16>(p, c, stream);
  if (rc) return rc;
  if (p.DVP <= 64) return launch_values<64>(p, stream);
  if (p.DVP <= 128) return launch_values<128>(p, stream);
  return launch_values<256>(p, stream);
}

}  // namespace b200
