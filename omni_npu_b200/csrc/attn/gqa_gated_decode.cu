// Decode step of the gated, windowed attention (gqa_gated.cuh), bf16.
//
// One cluster = up to 16 query rows of one (sequence, key/value head): the heads of the group times the
// step's tokens.  Its `splits` CTAs share the visible keys.  Inside a CTA four warps take 16-key tiles
// in turn; each warp has its own ring of shared-memory stages fed by cp.async, so no barrier stands
// between its loads and its products.  S = Q K^T and O = P V run on mma.sync (16 rows are far from a
// tcgen05 tile and the step is bound by the cache stream).  The warps' partial results meet in shared
// memory, the CTAs' through distributed shared memory; the rows are then normalised (sink included),
// gated and stored.

#include <cooperative_groups.h>

#include "../common/device_once.h"
#include "../common/pdl.cuh"
#include "attn_common.cuh"
#include "gqa_gated.cuh"

namespace cg = cooperative_groups;

namespace b200 {

namespace gdec {
constexpr int WARPS = 4, THREADS = WARPS * 32, KEYS = 16, ROWS = 16;

// DM: upper bound of the padded head sizes (64, 128 or 256)
template <int DM>
struct Cfg {
  static constexpr int STAGES = 3;                              // (DM 128: two CTAs per SM)
  static constexpr int TILE = KEYS * DM * 2;                    // one K or V tile of a warp
  static constexpr int RING = WARPS * STAGES * 2 * TILE;
  static constexpr int Q_BYTES = ROWS * DM * 2;
  static constexpr int PART = ROWS * DM * 4;                    // fp32 partial output of a warp
  static constexpr int STAT = WARPS * ROWS * 2 * 4;             // their maxima and sums
  static constexpr int SMEM = Q_BYTES + RING + STAT + ROWS * 2 * 4;
  static_assert(WARPS * PART <= RING, "the partial outputs reuse the ring");
};
}  // namespace gdec

template <int DM>
__global__ void __launch_bounds__(gdec::THREADS) gqa_gated_decode_kernel(const GatedAttnParams p) {
  using namespace gdec;
  using C = Cfg<DM>;
  extern __shared__ __align__(128) uint8_t smem[];
  uint8_t* sQ = smem;
  uint8_t* ring = smem + C::Q_BYTES;
  float* part = reinterpret_cast<float*>(ring);                         // [WARPS][ROWS][DM]
  float* stat = reinterpret_cast<float*>(ring + C::RING);               // [WARPS][ROWS][2]
  float* cta_stat = stat + WARPS * ROWS * 2;                            // [ROWS][2]

  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int split = blockIdx.x % p.splits;
  const int b = blockIdx.x / p.splits;
  const int per = p.Hq / p.Hk;
  const int rows_all = p.q_len * per;
  const int chunks = (rows_all + ROWS - 1) / ROWS;
  const int kvh = blockIdx.y / chunks;
  const int r0 = (blockIdx.y % chunks) * ROWS;

  pdl_trigger();
  pdl_wait();

  const int kv_len = p.seq_lens[b];
  const int ctx = kv_len - p.q_len;
  const long long q_begin = static_cast<long long>(b) * p.q_len;
  const int* bt = p.block_tables + static_cast<long long>(b) * p.max_blocks;
  const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.q);
  const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(p.k_cache);
  const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(p.v_cache);

  // keys that some row of this tile sees, in 16-key tiles; this CTA's share of them
  const int tok_lo = r0 / per, tok_hi = min(rows_all, r0 + ROWS) - 1;
  const int hi = min(kv_len, ctx + tok_hi / per + 1);
  const int lo = p.window > 0 ? max(0, ctx + tok_lo - p.window + 1) : 0;
  const int t_lo = lo / KEYS, t_hi = (max(hi, lo) + KEYS - 1) / KEYS;
  const int share = (t_hi - t_lo + p.splits - 1) / p.splits;
  const int t_begin = min(t_hi, t_lo + split * share), t_end = min(t_hi, t_begin + share);
  const int mine = t_end - t_begin > warp ? (t_end - t_begin - warp + WARPS - 1) / WARPS : 0;

  const int kchunks = p.DP >> 3, vchunks = p.DVP >> 3;
  const int key_row = lane >> 1;
  // the cache block of this lane's key is looked up one tile ahead of its copies
  auto block_of = [&](int i) {
    const int key = (t_begin + warp + i * WARPS) * KEYS + key_row;
    return i < mine && key < hi ? bt[p.bs_shift >= 0 ? key >> p.bs_shift : key / p.block_size] : 0;
  };
  int blk = block_of(0);
  auto issue = [&](int i) {
    if (i < mine) {
      const int key = (t_begin + warp + i * WARPS) * KEYS + key_row;
      const bool ok = key < hi;
      const __nv_bfloat16* ks = kc;
      const __nv_bfloat16* vs = vc;
      if (ok) {
        const int off = p.bs_shift >= 0 ? key & (p.block_size - 1) : key % p.block_size;
        const long long row = (static_cast<long long>(blk) * p.Hk + kvh) * p.block_size + off;
        ks = kc + row * p.DP;
        vs = vc + row * p.DVP;
      }
      blk = block_of(i + 1);
      const int sz = ok ? 16 : 0;
      const uint32_t kt = smem_u32(ring + (warp * C::STAGES + i % C::STAGES) * 2 * C::TILE);
      const uint32_t vt = kt + C::TILE;
#pragma unroll
      for (int c = lane & 1, u = 0; u < DM / 16; ++u, c += 2)
        if (c < kchunks)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(kt + tile_offset<DM>(key_row, c)),
                       "l"(ks + c * 8), "r"(sz) : "memory");
#pragma unroll
      for (int c = lane & 1, u = 0; u < DM / 16; ++u, c += 2)
        if (c < vchunks)
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(vt + tile_offset<DM>(key_row, c)),
                       "l"(vs + c * 8), "r"(sz) : "memory");
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < C::STAGES - 1; ++i) issue(i);

  // query rows -> shared (zero beyond the head size and the last row)
  const bool vec_q = (p.D & 7) == 0 && (p.q_stride & 7) == 0 && (reinterpret_cast<uintptr_t>(q) & 15) == 0;
  if (vec_q) {
    // eight threads per row
    const int r = tid >> 3, R = r0 + r;
    const __nv_bfloat16* src =
        q + (R < rows_all ? (q_begin + R / per) * p.q_stride + static_cast<long long>(kvh * per + R % per) * p.D : 0);
    for (int c = tid & 7; c < kchunks; c += 8)
      *reinterpret_cast<uint4*>(sQ + tile_offset<DM>(r, c)) =
          R < rows_all && c * 8 < p.D ? *reinterpret_cast<const uint4*>(src + c * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
  for (int idx = tid; !vec_q && idx < ROWS * p.DP; idx += THREADS) {
    const int r = idx / p.DP, d = idx % p.DP;
    const int R = r0 + r;
    __nv_bfloat16 v = __float2bfloat16(0.f);
    if (R < rows_all && d < p.D)
      v = q[(q_begin + R / per) * p.q_stride + static_cast<long long>(kvh * per + R % per) * p.D + d];
    *reinterpret_cast<__nv_bfloat16*>(sQ + tile_offset<DM>(r, d >> 3) + (d & 7) * 2) = v;
  }
  __syncthreads();
  uint32_t q_frag[DM / 16][4];
#pragma unroll
  for (int ks = 0; ks < DM / 16; ++ks)
    if (ks * 16 < p.DP) ldmatrix_x4(q_frag[ks], smem_u32(sQ) + tile_offset<DM>(lane & 15, ks * 2 + (lane >> 4)));

  float o_acc[DM / 8][4];
#pragma unroll
  for (int i = 0; i < DM / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) o_acc[i][j] = 0.f;
  float row_max[2] = {-INFINITY, -INFINITY}, row_sum[2] = {0.f, 0.f};
  int pos[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int R = r0 + (lane >> 2) + r * 8;
    pos[r] = R < rows_all ? ctx + R / per : -1;            // -1: sees nothing
  }

  for (int i = 0; i < mine; ++i) {
    issue(i + C::STAGES - 1);
    asm volatile("cp.async.wait_group %0;" ::"n"(C::STAGES - 1) : "memory");
    __syncwarp();
    const int n0 = (t_begin + warp + i * WARPS) * KEYS;
    const uint32_t kt = smem_u32(ring + (warp * C::STAGES + i % C::STAGES) * 2 * C::TILE);
    const uint32_t vt = kt + C::TILE;
    float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int ks = 0; ks < DM / 16; ++ks) {
      if (ks * 16 < p.DP) {
        uint32_t kf[4];
        ldmatrix_x4(kf, kt + tile_offset<DM>((lane & 7) + ((lane >> 4) << 3), ks * 2 + ((lane >> 3) & 1)));
        mma_bf16_16816(s[0], q_frag[ks], kf[0], kf[1]);
        mma_bf16_16816(s[1], q_frag[ks], kf[2], kf[3]);
      }
    }
    float tmax[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int key = n0 + nt * 8 + (lane & 3) * 2 + (j & 1);
        const int ps = pos[j >> 1];
        const bool ok = key < kv_len && key <= ps && (p.window <= 0 || key > ps - p.window);
        s[nt][j] = ok ? s[nt][j] * p.scale_log2 : -INFINITY;
        tmax[j >> 1] = fmaxf(tmax[j >> 1], s[nt][j]);
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
    for (int nt = 0; nt < 2; ++nt)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        s[nt][j] = exp2f(s[nt][j] - m_use[j >> 1]);
        row_sum[j >> 1] += s[nt][j];
      }
    uint32_t pa[4];
    pa[0] = pack_bf16x2(s[0][0], s[0][1]);
    pa[1] = pack_bf16x2(s[0][2], s[0][3]);
    pa[2] = pack_bf16x2(s[1][0], s[1][1]);
    pa[3] = pack_bf16x2(s[1][2], s[1][3]);
#pragma unroll
    for (int dt = 0; dt < DM / 16; ++dt) {
      if (dt * 16 < p.DVP) {
#pragma unroll
        for (int h = 0; h < 2; ++h)
#pragma unroll
          for (int j = 0; j < 4; ++j) o_acc[2 * dt + h][j] *= corr[j >> 1];
        uint32_t vf[4];
        ldmatrix_x4_trans(vf, vt + tile_offset<DM>(lane & 15, dt * 2 + (lane >> 4)));
        mma_bf16_16816(o_acc[2 * dt], pa, vf[0], vf[1]);
        mma_bf16_16816(o_acc[2 * dt + 1], pa, vf[2], vf[3]);
      }
    }
    __syncwarp();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();                                         // every warp is done with its ring

  // ---- the warps' partial results -> shared
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const float l = quad_sum(row_sum[r]);
    const int row = (lane >> 2) + r * 8;
    if ((lane & 3) == 0) {
      stat[(warp * ROWS + row) * 2] = row_max[r];
      stat[(warp * ROWS + row) * 2 + 1] = l;
    }
#pragma unroll
    for (int i = 0; i < DM / 8; ++i)
      if (i * 8 < p.DVP)
        *reinterpret_cast<float2*>(part + (warp * ROWS + row) * DM + i * 8 + (lane & 3) * 2) =
            make_float2(o_acc[i][2 * r], o_acc[i][2 * r + 1]);
  }
  __syncthreads();
  // ---- joined in the first warp's area, scaled to the CTA's maximum: eight threads per row
  {
    const int row = tid >> 3;
    float m = -INFINITY, f[WARPS], l = 0.f;
#pragma unroll
    for (int w = 0; w < WARPS; ++w) m = fmaxf(m, stat[(w * ROWS + row) * 2]);
#pragma unroll
    for (int w = 0; w < WARPS; ++w) {
      const float mw = stat[(w * ROWS + row) * 2];
      f[w] = mw == -INFINITY ? 0.f : exp2f(mw - m);
      l += f[w] * stat[(w * ROWS + row) * 2 + 1];
    }
    if (r0 + row < rows_all) {
      for (int d = (tid & 7) * 2; d < p.DVP; d += 16) {
        float2 o = make_float2(0.f, 0.f);
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
          const float2 x = *reinterpret_cast<const float2*>(part + (w * ROWS + row) * DM + d);
          o.x += f[w] * x.x;
          o.y += f[w] * x.y;
        }
        *reinterpret_cast<float2*>(part + row * DM + d) = o;
      }
    }
    if ((tid & 7) == 0) {
      cta_stat[row * 2] = m;
      cta_stat[row * 2 + 1] = l;
    }
  }
  cg::cluster_group cluster = cg::this_cluster();
  if (p.splits > 1) cluster.sync();
  else __syncthreads();

  // ---- rows are dealt out over the CTAs of the cluster, eight threads per row and `splits` rows apart
  {
    const int row = tid >> 3, R = r0 + row;
    if (R < rows_all && row % p.splits == split) {
      float m = p.has_sink ? p.sink_log2 : -INFINITY;
      float mc[8];
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        mc[c] = -INFINITY;
        if (c < p.splits) mc[c] = (p.splits > 1 ? cluster.map_shared_rank(cta_stat, c) : cta_stat)[row * 2];
        m = fmaxf(m, mc[c]);
      }
      float l = p.has_sink ? exp2f(p.sink_log2 - m) : 0.f;
#pragma unroll
      for (int c = 0; c < 8; ++c) {
        if (mc[c] == -INFINITY) {
          mc[c] = 0.f;
          continue;
        }
        mc[c] = exp2f(mc[c] - m);
        l += mc[c] * (p.splits > 1 ? cluster.map_shared_rank(cta_stat, c) : cta_stat)[row * 2 + 1];
      }
      const float inv = l > 0.f ? 1.f / l : 0.f;
      const long long tok = q_begin + R / per;
      const long long col = static_cast<long long>(kvh * per + R % per) * p.DV;
      const __nv_bfloat16* gate = p.gate ? static_cast<const __nv_bfloat16*>(p.gate) + tok * p.g_stride + col : nullptr;
      __nv_bfloat16* dst = static_cast<__nv_bfloat16*>(p.out) + tok * p.out_stride + col;
      for (int d = tid & 7; d < p.DV; d += 8) {
        float o = 0.f;
#pragma unroll
        for (int c = 0; c < 8; ++c)
          if (c < p.splits && mc[c] != 0.f)
            o += mc[c] * (p.splits > 1 ? cluster.map_shared_rank(part, c) : part)[row * DM + d];
        o *= inv;
        if (gate) o *= gate_sigmoid(__bfloat162float(gate[d]));
        dst[d] = __float2bfloat16(o);
      }
    }
  }
  if (p.splits > 1) cluster.sync();                        // no CTA leaves while its memory is being read
}

template <int DM>
static int launch_gated_decode(const GatedAttnParams& p, cudaStream_t stream) {
  auto kern = gqa_gated_decode_kernel<DM>;
  static DeviceOnce once;
  int dev = 0;
  if (once.needed(&dev)) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, gdec::Cfg<DM>::SMEM) != cudaSuccess)
      return -20;
    once.mark(dev);
  }
  const int chunks = (p.q_len * (p.Hq / p.Hk) + gdec::ROWS - 1) / gdec::ROWS;
  return launch_pdl(kern, dim3(p.B * p.splits, p.Hk * chunks), dim3(gdec::THREADS), gdec::Cfg<DM>::SMEM, stream,
                    p.splits, p) == cudaSuccess ? 0 : -21;
}

// Head sizes up to 256 (padded); splits 1, 2, 4 or 8.
int gated_decode(const GatedAttnParams& p, cudaStream_t stream) {
  if (p.splits != 1 && p.splits != 2 && p.splits != 4 && p.splits != 8) return -1;
  const int m = p.DP > p.DVP ? p.DP : p.DVP;
  if (m <= 64) return launch_gated_decode<64>(p, stream);
  if (m <= 128) return launch_gated_decode<128>(p, stream);
  if (m <= 256) return launch_gated_decode<256>(p, stream);
  return -2;
}

}  // namespace b200
