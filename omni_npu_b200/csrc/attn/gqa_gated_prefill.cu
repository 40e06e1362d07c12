// Prompt portions of the gated, windowed attention (gqa_gated.cuh), bf16, any head sizes up to 256, keys in
// cache blocks or contiguous.
//
// One CTA = 128 rows of one (sequence, key/value head): a row is one (token, head of the group), so a
// tile covers 128 / group tokens and its keys serve all heads of the group; with a window that is short
// against 128 tokens, far fewer keys are read and masked than with 128 tokens of a single head.  Eight
// warps x 16 rows; 64-key tiles of K and V are double-buffered with cp.async; S = Q K^T and O += P V on
// mma.sync with fp32 accumulators and an online softmax.  (Head size 128 takes the tcgen05 kernel of
// gqa_prefill_tcgen05.cu instead.)

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "attn_common.cuh"
#include "gqa_gated.cuh"

namespace b200 {

namespace gpre {
constexpr int BM = 128, BN = 64, THREADS = 256;
// DK, DV: upper bounds of the padded head sizes
template <int DK, int DV>
struct Cfg {
  static constexpr int Q_BYTES = BM * DK * 2;
  static constexpr int K_BYTES = BN * DK * 2;
  static constexpr int V_BYTES = BN * DV * 2;
  static constexpr int SMEM = Q_BYTES + 2 * K_BYTES + 2 * V_BYTES;
};
}  // namespace gpre

template <int DM>
__device__ __forceinline__ void load_gated_tile(uint32_t dst, const __nv_bfloat16* cache, const int* bt, int n0,
                                                int hi, int kvh, int Hk, int block_size, int width, int contiguous,
                                                int tid) {
  // four threads per key row, 16-byte chunks dealt out in turn
  const int row = tid >> 2;
  const int key = n0 + row;
  const bool ok = key < hi;
  const __nv_bfloat16* src = cache;
  if (ok && contiguous)
    src = cache + (static_cast<long long>(bt[0] + key) * Hk + kvh) * width;
  else if (ok)
    src = cache + ((static_cast<long long>(bt[key / block_size]) * Hk + kvh) * block_size + key % block_size) * width;
  const int sz = ok ? 16 : 0;
  for (int c = tid & 3; c < (width >> 3); c += 4)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst + tile_offset<DM>(row, c)),
                 "l"(src + c * 8), "r"(sz) : "memory");
}

// EXACT: the padded head sizes are DK and DV, and the query fragments stay in registers
template <int DK, int DV, bool EXACT>
__global__ void __launch_bounds__(gpre::THREADS, DK > 128 ? 1 : 2)
gqa_gated_prefill_kernel(const GatedAttnParams p, const int heads_per_tile) {
  using namespace gpre;
  using C = Cfg<DK, DV>;
  const int DP = EXACT ? DK : p.DP, DVP = EXACT ? DV : p.DVP;
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t* sQ = smem;
  const uint32_t kv0 = smem_u32(smem + C::Q_BYTES), v0 = kv0 + 2 * C::K_BYTES;

  pdl_trigger();
  pdl_wait();
  const int b = blockIdx.z;
  const int per = p.Hq / p.Hk;
  const int hchunks = (per + heads_per_tile - 1) / heads_per_tile;
  const int kvh = blockIdx.y / hchunks;
  const int head0 = (blockIdx.y % hchunks) * heads_per_tile;       // first head of the group in this tile
  const int hc = min(heads_per_tile, per - head0);
  const int tt = BM / hc;                                          // tokens per tile
  const long long q_begin = p.cu_q[b];
  const int q_len = static_cast<int>(p.cu_q[b + 1] - q_begin);
  // (the grid is laid out for heads_per_tile heads; a last, smaller chunk packs more tokens per tile)
  const int m0 = (gridDim.x - 1 - blockIdx.x) * tt;                // (the tiles with most keys first)
  if (m0 >= q_len) return;
  const int kv_len = p.seq_lens[b];
  const int ctx = kv_len - q_len;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q);
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(p.k_cache);
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(p.v_cache);

  const int tok_end = min(q_len, m0 + tt);
  const int hi = min(kv_len, ctx + tok_end);
  const int lo = p.window > 0 ? max(0, ctx + m0 - p.window + 1) / BN * BN : 0;
  const int tiles = (hi - lo + BN - 1) / BN;

  load_gated_tile<DK>(kv0, kc, bt, lo, hi, kvh, p.Hk, p.block_size, DP, p.contiguous, tid);
  load_gated_tile<DV>(v0, vc, bt, lo, hi, kvh, p.Hk, p.block_size, DVP, p.contiguous, tid);
  asm volatile("cp.async.commit_group;" ::: "memory");

  // ---- query rows -> shared: two threads per row
  {
    const int r = tid >> 1;
    const int tok = m0 + r / hc;
    const bool ok = r < tt * hc && tok < q_len;
    const __nv_bfloat16* src = q + (ok ? (q_begin + tok) * p.q_stride +
                                             static_cast<long long>(kvh * per + head0 + r % hc) * p.D : 0);
    const bool vec = (p.D & 7) == 0 && ((p.q_stride & 7) == 0) && ((reinterpret_cast<uintptr_t>(q) & 15) == 0);
    for (int c = tid & 1; c < (DP >> 3); c += 2) {
      uint4 u = make_uint4(0u, 0u, 0u, 0u);
      if (ok && vec) {
        if (c * 8 < p.D) u = *reinterpret_cast<const uint4*>(src + c * 8);
      } else if (ok) {
        __nv_bfloat16 h[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) h[j] = c * 8 + j < p.D ? src[c * 8 + j] : __float2bfloat16(0.f);
        uint32_t* w = reinterpret_cast<uint32_t*>(&u);
#pragma unroll
        for (int j = 0; j < 4; ++j)
          w[j] = static_cast<uint32_t>(__bfloat16_as_ushort(h[2 * j])) |
                 (static_cast<uint32_t>(__bfloat16_as_ushort(h[2 * j + 1])) << 16);
      }
      *reinterpret_cast<uint4*>(sQ + tile_offset<DK>(r, c)) = u;
    }
  }

  float o_acc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o_acc[i][j] = 0.f;
  uint32_t q_frag[EXACT ? DK / 16 : 1][4];
  // the sink is a key seen from the start: maximum = its score, sum = 1
  float row_max[2], row_sum[2];
  int pos[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    row_max[r] = p.has_sink ? p.sink_log2 : -INFINITY;
    row_sum[r] = p.has_sink && (lane & 3) == 0 ? 1.f : 0.f;        // summed over the quad at the end
    const int row = warp * 16 + (lane >> 2) + r * 8;
    pos[r] = row < tt * hc && m0 + row / hc < q_len ? ctx + m0 + row / hc : -1;
  }
  const int w_lo = ctx + m0 + warp * 16 / hc;                      // positions of this warp's rows
  const int w_hi = min(ctx + tok_end - 1, ctx + m0 + (warp * 16 + 15) / hc);

  for (int it = 0; it < tiles; ++it) {
    const int st = it & 1;
    if (it + 1 < tiles) {
      const int nn = lo + (it + 1) * BN;
      load_gated_tile<DK>(kv0 + (st ^ 1) * C::K_BYTES, kc, bt, nn, hi, kvh, p.Hk, p.block_size, DP, p.contiguous, tid);
      load_gated_tile<DV>(v0 + (st ^ 1) * C::V_BYTES, vc, bt, nn, hi, kvh, p.Hk, p.block_size, DVP, p.contiguous, tid);
      asm volatile("cp.async.commit_group;" ::: "memory");
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    if constexpr (EXACT) {
      if (it == 0) {
#pragma unroll
        for (int ks = 0; ks < DK / 16; ++ks)
          ldmatrix_x4(q_frag[ks], smem_u32(sQ) + tile_offset<DK>(warp * 16 + (lane & 15), ks * 2 + (lane >> 4)));
      }
    }
    const int n0 = lo + it * BN;
    // a warp none of whose rows sees a key of this tile has nothing to add
    const bool seen = n0 <= w_hi && (p.window <= 0 || n0 + BN - 1 > w_lo - p.window);
    if (seen) {
      const uint32_t kt = kv0 + st * C::K_BYTES, vt = v0 + st * C::V_BYTES;
      float s[BN / 8][4];
#pragma unroll
      for (int i = 0; i < BN / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DK / 16; ++ks) {
        if (EXACT || ks * 16 < DP) {
          uint32_t qf[4];
          if constexpr (EXACT) {
#pragma unroll
            for (int j = 0; j < 4; ++j) qf[j] = q_frag[ks][j];
          } else {
            ldmatrix_x4(qf, smem_u32(sQ) + tile_offset<DK>(warp * 16 + (lane & 15), ks * 2 + (lane >> 4)));
          }
#pragma unroll
          for (int nt = 0; nt < BN / 16; ++nt) {
            uint32_t kf[4];
            ldmatrix_x4(kf, kt + tile_offset<DK>(nt * 16 + (lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
            mma_bf16_16816(s[2 * nt], qf, kf[0], kf[1]);
            mma_bf16_16816(s[2 * nt + 1], qf, kf[2], kf[3]);
          }
        }
      }
      const bool interior = n0 + BN <= hi && n0 + BN - 1 <= w_lo && (p.window <= 0 || n0 > w_hi - p.window);
      float tmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int i = 0; i < BN / 8; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float v = s[i][j] * p.scale_log2;
          if (!interior) {
            const int key = n0 + i * 8 + (lane & 3) * 2 + (j & 1);
            const int ps = pos[j >> 1];
            if (!(key < hi && key <= ps && (p.window <= 0 || key > ps - p.window))) v = -INFINITY;
          }
          s[i][j] = v;
          tmax[j >> 1] = fmaxf(tmax[j >> 1], v);
        }
      float corr[2], m_use[2];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const float nm = fmaxf(row_max[r], quad_max(tmax[r]));
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
          if (EXACT || dt * 16 < DVP) {
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

  // ---- normalise, gate, store
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const float l = quad_sum(row_sum[r]);
    if (pos[r] < 0) continue;
    const float inv = l > 0.f ? 1.f / l : 0.f;
    const int row = warp * 16 + (lane >> 2) + r * 8;
    const long long tok = q_begin + m0 + row / hc;
    const long long col0 = static_cast<long long>(kvh * per + head0 + row % hc) * p.DV;
    const __nv_bfloat16* g = p.gate ? static_cast<const __nv_bfloat16*>(p.gate) + tok * p.g_stride + col0 : nullptr;
    __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + tok * p.out_stride + col0;
    const bool pairs = (reinterpret_cast<uintptr_t>(dst) & 3) == 0 && (reinterpret_cast<uintptr_t>(g) & 3) == 0;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      const int d = i * 8 + (lane & 3) * 2;
      if (d >= p.DV) continue;
      float o0 = o_acc[i][2 * r] * inv, o1 = o_acc[i][2 * r + 1] * inv;
      if (pairs && d + 1 < p.DV) {
        if (g) {
          const __nv_bfloat162 gv = *reinterpret_cast<const __nv_bfloat162*>(g + d);
          o0 *= gate_sigmoid(__low2float(gv));
          o1 *= gate_sigmoid(__high2float(gv));
        }
        *reinterpret_cast<uint32_t*>(dst + d) = pack_bf16x2(o0, o1);
      } else {
        dst[d] = __float2bfloat16(g ? o0 * gate_sigmoid(__bfloat162float(g[d])) : o0);
        if (d + 1 < p.DV) dst[d + 1] = __float2bfloat16(g ? o1 * gate_sigmoid(__bfloat162float(g[d + 1])) : o1);
      }
    }
  }
}

template <int DK, int DV, bool EXACT = false>
static int launch_gated_prefill(const GatedAttnParams& p, int max_q_len, cudaStream_t stream) {
  auto kern = gqa_gated_prefill_kernel<DK, DV, EXACT>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, gpre::Cfg<DK, DV>::SMEM) != cudaSuccess)
      return -20;
    once.mark(dev);
  }
  const int per = p.Hq / p.Hk;
  const int heads = per < gpre::BM ? per : gpre::BM;
  const int hchunks = (per + heads - 1) / heads;
  const int tt = gpre::BM / heads;
  const dim3 grid((max_q_len + tt - 1) / tt, p.Hk * hchunks, p.B);
  return launch_pdl(kern, grid, dim3(gpre::THREADS), gpre::Cfg<DK, DV>::SMEM, stream, 1, p, heads) == cudaSuccess ? 0
                                                                                                               : -21;
}

int gated_prefill(const GatedAttnParams& p, int max_q_len, cudaStream_t stream) {
  const int m = p.DP > p.DVP ? p.DP : p.DVP;
  if (m <= 64) return launch_gated_prefill<64, 64>(p, max_q_len, stream);
  if (m <= 128) return launch_gated_prefill<128, 128>(p, max_q_len, stream);
  if (p.DP == 192 && p.DVP == 128) return launch_gated_prefill<192, 128, true>(p, max_q_len, stream);
  if (p.DP <= 192 && p.DVP <= 128) return launch_gated_prefill<192, 128>(p, max_q_len, stream);
  if (m <= 256) return launch_gated_prefill<256, 256>(p, max_q_len, stream);
  return -2;
}

}  // namespace b200
