// Prompt portions of the attention with mixed heads (mixed_attn.cuh), bf16.  A key's score in one head needs all
// heads' products of that (query, key) pair, so the work is cut twice:
//
//   mixed_scores_kernel   16 queries x a range of keys, all heads: Q K^T on mma.sync with the queries of a warp's heads in
//                         registers; capped and lowered, a score goes to shared memory as a sum of three bf16 numbers
//                         (24 bits: all of an fp32 significand), so that the mixture is mma.sync products with fp32
//                         sums as well; mixed scores to memory in fp32.  The distance bias of a tile has 15 + keys
//                         values per head: a table, made while the tile before is mixed
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
constexpr int PLANES = 3;                // bf16 numbers that make up a score

__device__ __forceinline__ uint32_t piece(int row, int chunk, int width) {
  return static_cast<uint32_t>(row * width * 2 + ((chunk ^ (row & 7)) << 4));
}

struct Layout {
  int hs16, ho16, row, head, plane;      // bytes of a query's keys, of a head, of a plane of scores
  int t_row, t_plane;                    // bytes of a row and of a plane of the mixture
  int d_pitch, s_off, t_off, d_off, bytes;
  int per_k;                             // score heads of a key head
  long long row_step;                    // floats between the rows of scores that a warp writes one after another
};
// key tile [Hk][bk][dk] | scores, planes of [hs16][16][bk] | mixture, planes of [ho16][hs16] | distance bias [2][Hs][d_pitch]
inline Layout layout(int Hs, int Hk, int Ho, int DP, int bk, int terms) {
  Layout l{};
  const int dk = DP <= 64 ? 64 : DP <= 128 ? 128 : 256;
  l.hs16 = (Hs + 15) / 16 * 16;
  l.ho16 = (Ho + 15) / 16 * 16;
  l.row = bk * 2 + 16;                   // (the padding keeps fragment reads and writes off each other's banks)
  l.head = BQ * l.row + 16;
  l.plane = l.hs16 * l.head;
  l.t_row = l.hs16 * 2 + 16;
  l.t_plane = l.ho16 * l.t_row;
  l.d_pitch = bk + BQ;
  l.s_off = Hk * bk * dk * 2;
  l.t_off = l.s_off + PLANES * l.plane;
  l.d_off = l.t_off + terms * l.t_plane;
  l.bytes = l.d_off + 2 * Hs * l.d_pitch * 4;
  return l;
}

struct Plan {
  int bk, warps, ks;
};
inline Plan plan(int Hs, int Hk, int Ho, int DP, int terms) {
  if (DP > 256) return {0, 0, 0};
  const int warps = Hs <= 16 ? 8 : 16, ks = DP <= 64 ? 4 : DP <= 128 ? 8 : 16;
  const int order[4][2] = {{32, 112}, {16, 112}, {32, 226}, {16, 226}};
  for (const auto& o : order)
    if ((warps == 8 || o[1] > 112) && layout(Hs, Hk, Ho, DP, o[0], terms).bytes <= o[1] * 1024) return {o[0], warps, ks};
  return {0, 0, 0};
}

// Query tiles of the sequences before b.
__device__ __forceinline__ int tiles_before(const int* cu_q, int b, int lane) {
  int n = 0;
  for (int i = lane; i < b; i += 32) n += (cu_q[i + 1] - cu_q[i] + BQ - 1) / BQ;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) n += __shfl_xor_sync(0xffffffffu, n, o);
  return n;
}
// The sequence that query tile `tile` belongs to (-1: none), and the tile's number in it.
__device__ __forceinline__ int tile_owner(const int* cu_q, int B, int tile, int lane, int* local) {
  for (int base = 0; base < B; base += 32) {
    const int i = base + lane;
    const int mine = i < B ? (cu_q[i + 1] - cu_q[i] + BQ - 1) / BQ : 0;
    int upto = mine;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int v = __shfl_up_sync(0xffffffffu, upto, o);
      if (lane >= o) upto += v;
    }
    const unsigned past = __ballot_sync(0xffffffffu, upto > tile);
    if (past) {
      const int l = __ffs(past) - 1;
      *local = tile - __shfl_sync(0xffffffffu, upto - mine, l);
      return base + l;
    }
    tile -= __shfl_sync(0xffffffffu, upto, 31);
  }
  return -1;
}

// x0, x1 as sums of three bf16 numbers each
__device__ __forceinline__ void split3(float x0, float x1, uint32_t (&w)[PLANES]) {
#pragma unroll
  for (int i = 0; i < PLANES; ++i) {
    w[i] = pack_bf16x2(x0, x1);
    x0 -= __uint_as_float(w[i] << 16);
    x1 -= __uint_as_float(w[i] & 0xffff0000u);
  }
}
}  // namespace mpre

bool mixed_prefill_fits(int Hs, int Hk, int Ho, int Hv, int DP, int DVP) {
  return DVP <= 256 && mpre::plan(Hs, Hk, Ho, DP, mpre::PLANES).bk > 0;
}

// ------------------------------------------------------------- scores
// KS: steps of 16 along the head size; HPW: heads per warp and pass (16 registers of query per head and 4 steps)
template <int WARPS, int KS, int HPW, int BK>
__global__ void __launch_bounds__(WARPS * 32, WARPS == 8 ? 2 : 1)
mixed_scores_kernel(const MixedAttnParams p, const mpre::Layout L) {
  using namespace mpre;
  constexpr int THREADS = WARPS * 32, DK = KS * 16;
  extern __shared__ __align__(128) uint8_t smem[];
  float* sD = reinterpret_cast<float*>(smem + L.d_off);
  const uint32_t kt = smem_u32(smem), st = kt + L.s_off, tt = kt + L.t_off;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;

  pdl_trigger();
  pdl_wait();
  const int tile = gridDim.x - 1 - blockIdx.x;             // (the tiles with most keys first)
  int local = 0;
  const int b = tile_owner(p.cu_q, p.B, p.tile0 + tile, lane, &local);
  if (b < 0) return;
  const long long q_begin = p.cu_q[b];
  const int q_len = static_cast<int>(p.cu_q[b + 1] - q_begin);
  const int tok0 = local * BQ;
  const int ctx = p.seq_lens[b] - q_len;
  const int hi = ctx + min(q_len, tok0 + BQ);                      // keys that some row sees
  const int k_begin = blockIdx.y * p.range, k_end = min(hi, k_begin + p.range);
  if (k_begin >= k_end) return;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q);
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(p.k_cache);

  // DK / 8 threads share a row (32 at most), a thread has the same keys of every tile and walks over the heads
  constexpr int RT = DK / 8, SLOTS = THREADS / RT, KSTEP = SLOTS < BK ? SLOTS : BK, GSTEP = SLOTS > BK ? SLOTS / BK : 1;
  const int li = tid % RT, key0 = tid / RT % KSTEP, g0 = GSTEP > 1 ? tid / RT / KSTEP : 0;
  const bool li_used = li * 8 < p.DP;
  const uint32_t k_dst = kt + piece(g0 * BK + key0, li, DK);       // (KSTEP is a multiple of 8)
  const long long g_step = static_cast<long long>(GSTEP) * p.block_size * p.DP;
  auto issue = [&](int i) {
    const int n0 = k_begin + i * BK;
    if (n0 < k_end && li_used) {
#pragma unroll
      for (int j = 0; j < BK / KSTEP; ++j) {
        const int key = n0 + key0 + j * KSTEP;
        uint32_t to = k_dst + j * KSTEP * DK * 2;
        if (key < k_end) {
          const __nv_bfloat16* src = kc + cache_row(p, bt, key, g0, p.Hk) * p.DP + li * 8;
          for (int g = g0; g < p.Hk; g += GSTEP, src += g_step, to += GSTEP * BK * DK * 2)
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to), "l"(src) : "memory");
        } else {
          for (int g = g0; g < p.Hk; g += GSTEP, to += GSTEP * BK * DK * 2)
            asm volatile("st.shared.v4.u32 [%0], {%1, %1, %1, %1};" ::"r"(to), "r"(0) : "memory");
        }
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  issue(0);
  // the mixture (one plane when bf16 holds it exactly), zero beyond the heads; score rows beyond the heads
  for (int i = tid; i < L.ho16 * (L.hs16 >> 1); i += THREADS) {
    const int h = i / (L.hs16 >> 1), g = (i - h * (L.hs16 >> 1)) * 2;
    uint32_t w[PLANES];
    split3(h < p.Ho && g < p.Hs ? p.talk[h * p.Hs + g] : 0.f, h < p.Ho && g + 1 < p.Hs ? p.talk[h * p.Hs + g + 1] : 0.f, w);
#pragma unroll
    for (int t = 0; t < PLANES; ++t)
      if (t < p.talk_terms) *reinterpret_cast<uint32_t*>(smem + L.t_off + t * L.t_plane + h * L.t_row + g * 2) = w[t];
  }
  for (int t = 0; t < PLANES; ++t)
    for (int i = p.Hs * L.head + tid * 4; i < L.plane; i += THREADS * 4)
      *reinterpret_cast<uint32_t*>(smem + L.s_off + t * L.plane + i) = 0u;
  ScoreConst c = score_const(p);                           // scores in units of log2 e
  if (c.cap > 0.f) c.cap *= kLog2e;
  else c.in *= kLog2e;
  // what the score of tile i starts from, cap - distance bias: entry x of a head is for distance base + x, base =
  // first query - last key
  auto make_bias = [&](int i) {
    if (k_begin + i * BK >= k_end) return;
    const int base = ctx + tok0 - (k_begin + i * BK + BK - 1);
    constexpr int W = BK + BQ, GROUP = THREADS / 16;               // 16 threads per head, W / 16 entries each
    const int x0 = tid & 15;
    for (int g = tid >> 4; g < p.Hs; g += GROUP) {
      const float r1 = p.r1 ? __ldg(p.r1 + g) : 0.f, r2 = p.r1 ? __ldg(p.r2 + g) : 0.f;
      float* dst = sD + ((i & 1) * p.Hs + g) * W + x0;
#pragma unroll
      for (int x = 0; x < W; x += 16)
        dst[x] = c.cap - distance_bias(r1, r2, fmaxf(static_cast<float>(base + x0 + x), 0.f));
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

  uint32_t k_head[HPW];                                    // the key head of this warp's heads (of the first pass)
#pragma unroll
  for (int j = 0; j < HPW; ++j) k_head[j] = (warp * HPW + j) / L.per_k * BK * DK * 2;
  const uint32_t k_lane = kt + ((lane & 7) + ((lane >> 4) << 3)) * DK * 2;
  // the first row of scores that this warp writes, and where its fragments lie
  constexpr int HALVES = BK / 16, ROWS_STEP = WARPS / HALVES;
  const int row0 = warp / HALVES, k16 = warp % HALVES;
  const uint32_t s_lane = st + ((lane & 7) + ((lane >> 3) & 1) * 8) * L.head + row0 * (BK * 2 + 16) + k16 * 32 + (lane >> 4) * 16;
  const uint32_t t_lane = tt + (lane & 15) * L.t_row + (lane >> 4) * 16;
  float* out_tile = p.scratch + ((static_cast<long long>(tile) * BQ + row0) * p.Ho + (lane >> 2)) * p.pitch +
                    k_begin + k16 * 16 + (lane & 3) * 2;
  const int tiles = (k_end - k_begin + BK - 1) / BK;
  const int ks_used = p.DP >> 4;
  uint32_t kx[4];                                          // swizzled chunk of a row, by step modulo 4
#pragma unroll
  for (int i = 0; i < 4; ++i) kx[i] = ((i * 2 + ((lane >> 3) & 1)) ^ (lane & 7)) << 4;
  for (int it = 0; it < tiles; ++it) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();                                       // keys and bias are there; the scores before are used up
    const int n0 = k_begin + it * BK;

    for (int pass = 0; pass < passes; ++pass) {
      if (passes > 1) load_q(pass);
#pragma unroll
      for (int j = 0; j < HPW; ++j) {
        const int g = (pass * WARPS + warp) * HPW + j;
        if (g >= p.Hs) continue;
        const uint32_t k_at = k_lane + (pass == 0 ? k_head[j] : g / L.per_k * BK * DK * 2);
        float s[BK / 8][4];
#pragma unroll
        for (int n = 0; n < BK / 8; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
        const uint32_t k_of[4] = {k_at + kx[0], k_at + kx[1], k_at + kx[2], k_at + kx[3]};
        static_for<KS>([&](auto step) {
          constexpr int ks = decltype(step)::value;
          if (ks < ks_used) {
            static_for<BK / 16>([&](auto part) {
              constexpr int n = decltype(part)::value;
              uint32_t kf[4];
              ldmatrix_x4_at<n * 16 * DK * 2 + (ks >> 2) * 128>(kf, k_of[ks & 3]);
              mma_bf16_16816(s[2 * n], qf[j][ks], kf[0], kf[1]);
              mma_bf16_16816(s[2 * n + 1], qf[j][ks], kf[2], kf[3]);
            });
          }
        });
        uint8_t* dst = smem + L.s_off + g * L.head + (lane >> 2) * (BK * 2 + 16) + (lane & 3) * 4;
        const float* bias = sD + ((it & 1) * p.Hs + g) * (BK + BQ) + BK - 1 + (lane >> 2) - (lane & 3) * 2;
        auto put = [&](auto cap) {
#pragma unroll
          for (int n = 0; n < BK / 8; ++n)
#pragma unroll
            for (int r = 0; r < 2; ++r) {
              uint32_t w[PLANES];
              split3(biased_score<decltype(cap)::value>(c, s[n][2 * r], bias[r * 8 - n * 8]),
                     biased_score<decltype(cap)::value>(c, s[n][2 * r + 1], bias[r * 8 - n * 8 - 1]), w);
#pragma unroll
              for (int t = 0; t < PLANES; ++t)
                *reinterpret_cast<uint32_t*>(dst + t * L.plane + r * 8 * (BK * 2 + 16) + n * 16) = w[t];
            }
        };
        if (c.cap > 0.f) put(std::true_type{});
        else put(std::false_type{});
      }
    }
    __syncthreads();                                       // scores are there; the keys are used up
    issue(it + 1);
    make_bias(it + 1);

    // ---- mixture: 16 output heads x 16 keys of one or two queries per step
    constexpr int UNITS = BQ / ROWS_STEP >= 2 ? 2 : 1;
    float* out = out_tile;
    uint32_t s_at = s_lane;
#pragma unroll 1
    for (int row = row0; row < BQ; row += UNITS * ROWS_STEP, out += UNITS * L.row_step, s_at += UNITS * ROWS_STEP * (BK * 2 + 16)) {
      if (tok0 + row >= q_len) break;
      const bool second = tok0 + row + ROWS_STEP < q_len;
      uint32_t t_ob = t_lane;
      float* o_ob = out;
#pragma unroll 1
      for (int left = p.Ho - (lane >> 2), ob = 0; ob < L.ho16; ob += 16, left -= 16) {
        float o[UNITS][2][4];
#pragma unroll
        for (int u = 0; u < UNITS; ++u)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[u][0][e] = o[u][1][e] = 0.f;
        uint32_t s_kb = s_at, t_kb = t_ob;
#pragma unroll 1
        for (int kb = 0; kb < L.hs16; kb += 16, s_kb += 16 * L.head, t_kb += 32) {
          uint32_t sf[PLANES][UNITS][4], tf[4];
          ldmatrix_x4(tf, t_kb);
#pragma unroll
          for (int t = PLANES - 1; t >= 0; --t)
#pragma unroll
            for (int u = 0; u < UNITS; ++u) ldmatrix_x4_trans(sf[t][u], s_kb + t * L.plane + u * ROWS_STEP * (BK * 2 + 16));
          const auto add = [&](int t) {
#pragma unroll
            for (int u = 0; u < UNITS; ++u) {
              mma_bf16_16816(o[u][0], tf, sf[t][u][0], sf[t][u][1]);
              mma_bf16_16816(o[u][1], tf, sf[t][u][2], sf[t][u][3]);
            }
          };
#pragma unroll
          for (int t = PLANES - 1; t >= 0; --t) add(t);
          if (p.talk_terms > 1) {                          // (products below 2^-24 are left out)
            ldmatrix_x4(tf, t_kb + L.t_plane);
            add(1);
            add(0);
            ldmatrix_x4(tf, t_kb + 2 * L.t_plane);
            add(0);
          }
        }
        float* o_low = o_ob + 8 * p.pitch;
#pragma unroll
        for (int u = 0; u < UNITS; ++u) {
          if (u == 1 && !second) continue;
          if (left > 0) {
            *reinterpret_cast<float2*>(o_ob + u * L.row_step) = make_float2(o[u][0][0], o[u][0][1]);
            *reinterpret_cast<float2*>(o_ob + u * L.row_step + 8) = make_float2(o[u][1][0], o[u][1][1]);
          }
          if (left > 8) {
            *reinterpret_cast<float2*>(o_low + u * L.row_step) = make_float2(o[u][0][2], o[u][0][3]);
            *reinterpret_cast<float2*>(o_low + u * L.row_step + 8) = make_float2(o[u][1][2], o[u][1][3]);
          }
        }
        o_ob += 16 * p.pitch;
        t_ob += 16 * L.t_row;
      }
    }
    out_tile += BK;
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
__global__ void __launch_bounds__(mval::THREADS, DV > 128 ? 1 : 2)
mixed_values_kernel(const MixedAttnParams p, const int heads_per_tile) {
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
  // this sequence's share of the call's query tiles
  const int before = mpre::tiles_before(p.cu_q, b, lane);
  const int first = max(0, p.tile0 - before) * mpre::BQ;
  const int last = min(q_len, (p.tile0 + p.tiles - before) * mpre::BQ);
  const int m0 = first + (gridDim.x - 1 - blockIdx.x) * tt;        // (the tiles with most keys first)
  if (m0 >= last) return;
  const int tok_end = min(last, m0 + tt);
  const int ctx = p.seq_lens[b] - q_len, hi = ctx + tok_end;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(p.v_cache);
  const int tiles = (hi + BN - 1) / BN;

  const int rows_live = (tok_end - m0) * hc;                       // rows: (token, head of the group)
  const float* sbase = p.scratch + ((static_cast<long long>(before - p.tile0) * mpre::BQ + m0) * p.Ho + vh * per + head0) * p.pitch + (tid & 15) * 4;
  __shared__ int srow[BM];                                         // where the tile's rows of scores lie, -1: nowhere
  if (tid < BM) srow[tid] = tid < rows_live ? tid / hc * p.Ho + tid % hc : -1;
  __syncthreads();
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
        const int at = srow[(tid >> 4) + i * 16];
        if (at >= 0)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(sdst + ((tid >> 4) + i * 16) * S_PITCH * 4),
                       "l"(sbase + at * p.pitch + it * BN) : "memory");
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
  uint32_t vx[4];                                                  // swizzled chunk of a value row, by step modulo 4
#pragma unroll
  for (int i = 0; i < 4; ++i) vx[i] = (lane & 15) * DV * 2 + (((i * 2 + (lane >> 4)) ^ (lane & 7)) << 4);
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
          s[i][2 * r] = x.x;
          s[i][2 * r + 1] = x.y;
        }
      if (!interior) {
#pragma unroll
        for (int i = 0; i < BN / 8; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (n0 + i * 8 + (lane & 3) * 2 + (j & 1) > pos[j >> 1]) s[i][j] = -INFINITY;
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
      const uint32_t v_of[4] = {vt + vx[0], vt + vx[1], vt + vx[2], vt + vx[3]};
      static_for<BN / 16>([&](auto step) {
        constexpr int ks = decltype(step)::value;
        uint32_t pa[4];
        pa[0] = pack_bf16x2(s[2 * ks][0], s[2 * ks][1]);
        pa[1] = pack_bf16x2(s[2 * ks][2], s[2 * ks][3]);
        pa[2] = pack_bf16x2(s[2 * ks + 1][0], s[2 * ks + 1][1]);
        pa[3] = pack_bf16x2(s[2 * ks + 1][2], s[2 * ks + 1][3]);
        static_for<DV / 16>([&](auto part) {
          constexpr int dt = decltype(part)::value;
          if (dt * 16 < p.DVP) {
            uint32_t vf[4];
            ldmatrix_x4_trans_at<ks * 16 * DV * 2 + (dt >> 2) * 128>(vf, v_of[dt & 3]);
            mma_bf16_16816(o_acc[2 * dt], pa, vf[0], vf[1]);
            mma_bf16_16816(o_acc[2 * dt + 1], pa, vf[2], vf[3]);
          }
        });
      });
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
static int launch_scores(const MixedAttnParams& p, cudaStream_t stream) {
  auto kern = mixed_scores_kernel<WARPS, KS, HPW, BK>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024) != cudaSuccess) return -20;
    once.mark(dev);
  }
  mpre::Layout l = mpre::layout(p.Hs, p.Hk, p.Ho, p.DP, BK, p.talk_terms);
  l.per_k = p.Hs / p.Hk;
  l.row_step = WARPS / (BK / 16) * p.Ho * p.pitch;
  const dim3 grid(p.tiles, (p.max_keys + p.range - 1) / p.range);
  return launch_pdl(kern, grid, dim3(WARPS * 32), l.bytes, stream, 1, p, l) == cudaSuccess ? 0 : -21;
}

template <int WARPS, int BK>
static int launch_scores_ks(const MixedAttnParams& p, const mpre::Plan& c, cudaStream_t stream) {
  if (c.ks == 4) return launch_scores<WARPS, 4, 4, BK>(p, stream);
  if (c.ks == 8) return launch_scores<WARPS, 8, 2, BK>(p, stream);
  return launch_scores<WARPS, 16, 1, BK>(p, stream);
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
  const int own = (p.max_q_len + mpre::BQ - 1) / mpre::BQ, toks = (p.tiles < own ? p.tiles : own) * mpre::BQ;
  const dim3 grid((toks + tt - 1) / tt, p.Hv * hchunks, p.B);
  return launch_pdl(kern, grid, dim3(mval::THREADS), SMEM, stream, 1, p, heads) == cudaSuccess ? 0 : -21;
}

int mixed_prefill(const MixedAttnParams& in, cudaStream_t stream) {
  MixedAttnParams p = in;
  const mpre::Plan c = mpre::plan(p.Hs, p.Hk, p.Ho, p.DP, p.talk_terms);
  if (c.bk == 0 || p.DVP > 256 || (p.talk_terms != 1 && p.talk_terms != mpre::PLANES)) return -2;
  // keys of a score CTA: longer ranges where there are CTAs enough
  p.range = 128;
  while (p.range < 1024 && static_cast<long long>(p.tiles) * ((p.max_keys + 2 * p.range - 1) / (2 * p.range)) >= 888)
    p.range *= 2;
  int rc;
  if (c.bk == 32) rc = c.warps == 8 ? launch_scores_ks<8, 32>(p, c, stream) : launch_scores_ks<16, 32>(p, c, stream);
  else rc = c.warps == 8 ? launch_scores_ks<8, 16>(p, c, stream) : launch_scores_ks<16, 16>(p, c, stream);
  if (rc) return rc;
  if (p.DVP <= 64) return launch_values<64>(p, stream);
  if (p.DVP <= 128) return launch_values<128>(p, stream);
  return launch_values<256>(p, stream);
}

}  // namespace b200
