// Mixture of experts: routing, rows in expert order, and one product per expert (see kernels.h for the routing rule).
//
// nfk_moe_route     one warp per token: scores, group limit, top experts and their weights; a counter per expert
//                   gives every chosen (token, expert) its rank.
// nfk_moe_permute   the tokens' rows in expert order (no gaps: a tensor-core tile may start at any row).
// nfk_moe_gemm      bf16: tcgen05 products over the experts' row ranges, operands by TMA, accumulators in TMEM,
//                   persistent over (expert, row tile, column tile). The tile list follows from the counters, which
//                   every CTA reads when it starts, so the host never learns the counts. fp32: FMA tiles.
//
// The weighted sum over a token's experts is part of the residual step (nfk_residual_norm).
#include "elem_io.cuh"
#include "gated_act.cuh"

namespace nf {
namespace {

constexpr int kMaxExperts = 1024;

// ---- routing ------------------------------------------------------------------------------------------------
constexpr int kRouteWarps = 4;

// Largest of one value per lane-owned candidate; ties go to the lower index. Every lane gets both.
__device__ __forceinline__ void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, o);
    const int oi = __shfl_xor_sync(0xffffffffu, i, o);
    if (ov > v || (ov == v && oi < i)) {
      v = ov;
      i = oi;
    }
  }
}

__global__ void __launch_bounds__(kRouteWarps * 32)
moe_route_kernel(nfk_moe_route_params p) {
  extern __shared__ float rsm[];                       // per warp: scores | choice scores | group scores
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int E = p.experts + p.identity, per = E / p.groups;
  float* s_s = rsm + warp * (2 * E + p.groups);
  float* c_s = s_s + E;
  float* g_s = c_s + E;
  const bool softmax = p.score == NFK_SCORE_SOFTMAX, whole = p.score == NFK_SCORE_SOFTMAX_ALL;
  for (int t = blockIdx.x * kRouteWarps + warp; t < p.T; t += gridDim.x * kRouteWarps) {
    const float* z = p.logits + t * p.ld;
    float z_max = -INFINITY, inv = 0.f;
    if (whole) {
      for (int e = lane; e < E; e += 32) z_max = fmaxf(z_max, z[e]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) z_max = fmaxf(z_max, __shfl_xor_sync(0xffffffffu, z_max, o));
      float all = 0.f;
      for (int e = lane; e < E; e += 32) all += expf(z[e] - z_max);
      inv = 1.f / warp_sum(all);
    }
    for (int e = lane; e < E; e += 32) {
      const float corr = p.correction != nullptr ? p.correction[e] : 0.f;
      const float s = softmax ? z[e] + corr : whole ? expf(z[e] - z_max) * inv : 1.f / (1.f + expf(-z[e]));
      s_s[e] = s;
      c_s[e] = softmax ? s : s + corr;
    }
    if (lane == 0 && p.gate_col >= 0) p.gate[t] = 1.f / (1.f + expf(-z[p.gate_col]));
    __syncwarp();
    if (p.groups > 1) {
      for (int g = lane; g < p.groups; g += 32) {
        float a = -INFINITY, b = -INFINITY;            // two largest
        for (int e = g * per; e < (g + 1) * per; ++e) {
          const float c = c_s[e];
          if (c > a) {
            b = a;
            a = c;
          } else if (c > b) {
            b = c;
          }
        }
        g_s[g] = per > 1 && p.group_max == 0 ? a + b : a;
      }
      __syncwarp();
      // a group stays if fewer than `keep` groups come before it
      for (int g = lane; g < p.groups; g += 32) {
        const float v = g_s[g];
        int before = 0;
        for (int o = 0; o < p.groups; ++o) before += (g_s[o] > v || (g_s[o] == v && o < g)) ? 1 : 0;
        if (before >= p.keep)
          for (int e = g * per; e < (g + 1) * per; ++e) c_s[e] = -INFINITY;
      }
      __syncwarp();
    }
    float sum = 0.f;
    int mine = -1;                                     // lane k keeps the k-th chosen expert
    for (int k = 0; k < p.top; ++k) {
      float v = -INFINITY;
      int i = E;
      for (int e = lane; e < E; e += 32)
        if (c_s[e] > v) {
          v = c_s[e];
          i = e;
        }
      warp_argmax(v, i);
      if (i >= E) i = 0;                               // fewer candidates than `top`: rejected by the launcher
      sum += s_s[i];
      if (lane == k) mine = i;
      __syncwarp();
      if (lane == 0) c_s[i] = -INFINITY;
      __syncwarp();
    }
    float share = mine >= 0 ? s_s[mine] : 0.f;
    if (softmax) {
      const float top = __shfl_sync(0xffffffffu, share, 0);        // the first one chosen has the largest logit
      share = mine >= 0 ? expf(share - top) : 0.f;
      share /= warp_sum(share);
    } else if (!whole) {
      share /= sum + 1e-20f;
    }
    if (lane < p.top) {
      const long long o = static_cast<long long>(t) * p.top + lane;
      p.expert[o] = mine;
      p.weight[o] = share * p.scale;
      p.rank[o] = mine < p.experts ? atomicAdd(p.counts + mine, 1) : 0;
    }
    if (p.identity > 0) {
      const float kept = warp_sum(lane < p.top && mine >= p.experts ? share * p.scale : 0.f);
      if (lane == 0) p.gate[t] = kept;
    }
    __syncwarp();
  }
}

// Exclusive prefix sums over the experts, by one warp: off[e] rows before expert e, and with tile sizes tiles[e] work
// tiles before it. Both have one more entry, the total.
__device__ __forceinline__ void expert_offsets(const int* counts, int experts, int* off, int* tiles, int tile_rows, int n_blocks) {
  const int lane = threadIdx.x & 31;
  int r0 = 0, t0 = 0;
  for (int e0 = 0; e0 < experts; e0 += 32) {
    const int c = e0 + lane < experts ? counts[e0 + lane] : 0;
    int r = c, t = (c + tile_rows - 1) / tile_rows * n_blocks;
    const int t_own = t;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int ur = __shfl_up_sync(0xffffffffu, r, o), ut = __shfl_up_sync(0xffffffffu, t, o);
      if (lane >= o) {
        r += ur;
        t += ut;
      }
    }
    if (e0 + lane < experts) {
      off[e0 + lane] = r0 + r - c;
      if (tiles != nullptr) tiles[e0 + lane] = t0 + t - t_own;
    }
    r0 += __shfl_sync(0xffffffffu, r, 31);
    t0 += __shfl_sync(0xffffffffu, t, 31);
  }
  if (lane == 0) {
    off[experts] = r0;
    if (tiles != nullptr) tiles[experts] = t0;
  }
}

// ---- rows in expert order -------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
moe_permute_kernel(nfk_moe_permute_params p, int row_chunks) {
  __shared__ int off[kMaxExperts + 1];
  if (threadIdx.x < 32) expert_offsets(p.counts, p.experts, off, nullptr, 1, 1);
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const long long ld_h = p.ld_h * (p.dtype == NFK_F32 ? 4 : 2) / 16, ld_o = p.ld_out * (p.dtype == NFK_F32 ? 4 : 2) / 16;
  for (int t = blockIdx.x * 8 + warp; t < p.T; t += gridDim.x * 8) {
    int slot = 0;
    if (lane < p.top) {
      const long long o = static_cast<long long>(t) * p.top + lane;
      const int e = p.expert[o];
      slot = e < p.experts ? off[e] + p.rank[o] : -1;
      p.slot[o] = slot;
    }
    const uint4* src = reinterpret_cast<const uint4*>(p.h) + t * ld_h;
    uint4* out = reinterpret_cast<uint4*>(p.out);
    for (int c0 = 0; c0 < row_chunks; c0 += 128) {
      const int c = c0 + lane;
      uint4 v[4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (c + j * 32 < row_chunks) v[j] = src[c + j * 32];
      for (int k = 0; k < p.top; ++k) {
        const long long s = __shfl_sync(0xffffffffu, slot, k);
        if (s < 0) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if (c + j * 32 < row_chunks) out[s * ld_o + c + j * 32] = v[j];
      }
    }
  }
}

// ---- one product per expert, tcgen05 ----------------------------------------------------------------------------
constexpr int BM = 128, BK = 64, kStages = 4, kThreads = 192;
constexpr int kATile = BM * BK * 2, kBTile = 256 * BK * 2, kStage = kATile + kBTile;
constexpr int kTables = 2 * (kMaxExperts + 1) * 4 + 8;
constexpr int kGemmSmem = 1024 + 1024 + (kTables + 1023) / 1024 * 1024 + kStages * kStage;

// Position in the tile list: tiles of one expert follow one another, its row tiles fastest (they share the
// weights' tile in L2).
struct TileWalk {
  int tile, e;
};
struct Tile {
  int expert, row0, row_end, n_blk;
};
__device__ __forceinline__ bool next_tile(TileWalk& w, const int* off, const int* tiles, int experts, int step, Tile& t) {
  if (w.tile >= tiles[experts]) return false;
  while (tiles[w.e + 1] <= w.tile) ++w.e;
  const int local = w.tile - tiles[w.e];
  const int m_tiles = (off[w.e + 1] - off[w.e] + BM - 1) / BM;
  t.expert = w.e;
  t.n_blk = local / m_tiles;
  t.row0 = off[w.e] + (local - t.n_blk * m_tiles) * BM;
  t.row_end = off[w.e + 1];
  w.tile += step;
  return true;
}

template <bool GATED>
__global__ void __launch_bounds__(kThreads, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tmA, const __grid_constant__ CUtensorMap tmA32,
                const __grid_constant__ CUtensorMap tmB0, const __grid_constant__ CUtensorMap tmB1, nfk_moe_gemm_params p,
                int bn) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem_al = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem_al);
  uint64_t* empty_bar = full_bar + kStages;
  uint64_t* tmem_full = empty_bar + kStages;
  uint64_t* tmem_empty = tmem_full + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tmem_empty + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* off = reinterpret_cast<int*>(smem_al + 1024);
  int* tiles = off + kMaxExperts + 1;
  uint8_t* ring = smem_al + 1024 + (kTables + 1023) / 1024 * 1024;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int out_bn = GATED ? bn / 2 : bn;
  const int n_blocks = (p.N + out_bn - 1) / out_bn, num_kb = (p.K + BK - 1) / BK;
  const int b_bytes = bn * BK * 2;

  if (threadIdx.x == 0) {
    for (int s = 0; s < kStages; ++s) {
      mbar_init(&full_bar[s], 1);
      mbar_init(&empty_bar[s], 1);
    }
    for (int a = 0; a < 2; ++a) {
      mbar_init(&tmem_full[a], 1);
      mbar_init(&tmem_empty[a], 4);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmA);
    tma_prefetch_desc(&tmA32);
    tma_prefetch_desc(&tmB0);
    if (GATED) tma_prefetch_desc(&tmB1);
  }
  if (warp == 2) expert_offsets(p.counts, p.experts, off, tiles, BM, n_blocks);
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  TileWalk walk{static_cast<int>(blockIdx.x), 0};
  Tile tl;
  const int step = gridDim.x;
  // counters that do not fit the buffers would send rows past their end
  const bool sane = off[p.experts] <= p.rows;
  if (!sane && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);

  if (!sane) {
  } else if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      uint32_t it = 0;
      bool ok = true;
      while (ok && next_tile(walk, off, tiles, p.experts, step, tl)) {
        // rows past the expert's last one are left as they are in shared memory: they only make rows of the product
        // that are not stored
        const int rows = min(BM, tl.row_end - tl.row0), boxes = (rows + 31) / 32;
        const int brow = tl.expert * p.N + tl.n_blk * out_bn;
        const uint32_t bytes = (boxes == 4 ? kATile : boxes * (32 * BK * 2)) + b_bytes;
        for (int kb = 0; kb < num_kb; ++kb, ++it) {
          const int s = it % kStages;
          if (!wait_or_abort(&empty_bar[s], ((it / kStages) & 1) ^ 1, abort_flag)) {
            report_status(p.status, NF_ST_TIMEOUT_SMEM_EMPTY);
            *abort_flag = 1;
            ok = false;
            break;
          }
          uint8_t* sa = ring + s * kStage;
          uint8_t* sb = sa + kATile;
          mbar_expect_tx(&full_bar[s], bytes);
          tma_load_2d(sb, &tmB0, &full_bar[s], kb * BK, brow);
          if (GATED) tma_load_2d(sb + b_bytes / 2, &tmB1, &full_bar[s], kb * BK, brow);
          if (boxes == 4) {
            tma_load_2d(sa, &tmA, &full_bar[s], kb * BK, tl.row0);
          } else {
            for (int b = 0; b < boxes; ++b) tma_load_2d(sa + b * (32 * BK * 2), &tmA32, &full_bar[s], kb * BK, tl.row0 + b * 32);
          }
        }
      }
      if (!ok) {
        // give loads already in flight a bounded chance to land before the CTA exits
        const uint32_t back = it < kStages ? it : kStages;
        for (uint32_t j = it - back; j < it; ++j) (void)mbar_wait(&full_bar[j % kStages], (j / kStages) & 1);
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      const uint32_t idesc = umma_idesc_bf16(BM, bn);
      uint32_t it = 0, n_tile = 0;
      bool ok = true;
      while (ok && next_tile(walk, off, tiles, p.experts, step, tl)) {
        const uint32_t acc = n_tile & 1;
        if (!wait_or_abort(&tmem_empty[acc], ((n_tile >> 1) & 1) ^ 1, abort_flag)) {
          report_status(p.status, NF_ST_TIMEOUT_TMEM_EMPTY);
          *abort_flag = 1;
          break;
        }
        tc_fence_after();
        for (int kb = 0; kb < num_kb; ++kb, ++it) {
          const int s = it % kStages;
          if (!wait_or_abort(&full_bar[s], (it / kStages) & 1, abort_flag)) {
            report_status(p.status, NF_ST_TIMEOUT_SMEM_FULL);
            *abort_flag = 1;
            ok = false;
            break;
          }
          tc_fence_after();
          const uint32_t a = smem_u32(ring + s * kStage), b = a + kATile;
#pragma unroll
          for (int k = 0; k < BK / 16; ++k)
            umma_bf16_ss(tmem + acc * 256, umma_desc_k_sw128(a + k * 32), umma_desc_k_sw128(b + k * 32), idesc,
                         (kb | k) ? 1u : 0u);
          umma_commit(&empty_bar[s]);
        }
        if (ok) umma_commit(&tmem_full[acc]);
        ++n_tile;
      }
    }
  } else {
    // ---------------- epilogue ----------------
    const int q = warp & 3;
    const GatedAct act{p.act, p.act_limit, p.act_alpha, p.act_shift};
    __nv_bfloat16* D = reinterpret_cast<__nv_bfloat16*>(p.D);
    uint32_t n_tile = 0;
    while (next_tile(walk, off, tiles, p.experts, step, tl)) {
      const uint32_t acc = n_tile & 1;
      if (!wait_or_abort(&tmem_full[acc], (n_tile >> 1) & 1, abort_flag)) {
        if (lane == 0) report_status(p.status, NF_ST_TIMEOUT_TMEM_FULL);
        *abort_flag = 1;
        break;
      }
      ++n_tile;
      __syncwarp();
      tc_fence_after();
      const uint32_t t_lane = tmem + (static_cast<uint32_t>(q * 32) << 16) + acc * 256;
      const int row = tl.row0 + q * 32 + lane;
      const bool row_ok = row < tl.row_end;
      __nv_bfloat16* dst = D + static_cast<long long>(row) * p.ldd;
      if (tl.row0 + q * 32 < tl.row_end) {
#pragma unroll 1
        for (int c = 0; c * 16 < out_bn; c += 2) {
          const bool half = c * 16 + 16 == out_bn;       // width = 32 k + 16
          uint32_t r[32], u[32];
          float v[32];
          if (half) tmem_ld_32x32b_x16(t_lane + c * 16, r);
          else tmem_ld_32x32b_x32(t_lane + c * 16, r);
          if (GATED) {
            if (half) tmem_ld_32x32b_x16(t_lane + bn / 2 + c * 16, u);
            else tmem_ld_32x32b_x32(t_lane + bn / 2 + c * 16, u);
          }
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j)
            v[j] = GATED ? gated_act(__uint_as_float(r[j]), __uint_as_float(u[j]), act) : __uint_as_float(r[j]);
          if (!GATED && p.lin_act != NFK_LIN_NONE) {
#pragma unroll
            for (int j = 0; j < 32; ++j) v[j] = lin_act_of(v[j], p.lin_act);
          }
          if (row_ok) {
#pragma unroll
            for (int g = 0; g < 4; ++g) {
              const int cl = c * 16 + g * 8, col = tl.n_blk * out_bn + cl;
              if (cl < out_bn && col < p.N)
                *reinterpret_cast<uint4*>(dst + col) =
                    make_uint4(pack_bf16x2(v[g * 8], v[g * 8 + 1]), pack_bf16x2(v[g * 8 + 2], v[g * 8 + 3]),
                               pack_bf16x2(v[g * 8 + 4], v[g * 8 + 5]), pack_bf16x2(v[g * 8 + 6], v[g * 8 + 7]));
            }
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tmem_empty[acc]);
    }
  }
  tc_fence_before();
  __syncwarp();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 512);
  }
}

// ---- one product per expert, fp32 -----------------------------------------------------------------------------------
constexpr int kFt = 64, kFk = 16, kFthr = 256;

template <bool GATED>
__global__ void __launch_bounds__(kFthr)
moe_gemm_f32_kernel(nfk_moe_gemm_params p) {
  __shared__ int off[kMaxExperts + 1], tiles[kMaxExperts + 1];
  __shared__ float sa[kFk][kFt + 4], sb[kFk][kFt + 4], sc[GATED ? kFk : 1][kFt + 4];
  if (threadIdx.x < 32) expert_offsets(p.counts, p.experts, off, tiles, kFt, 1);
  __syncthreads();
  const int tile = blockIdx.y;
  if (tile >= tiles[p.experts]) return;
  if (off[p.experts] > p.rows) {
    if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    return;
  }
  int e = 0;
  while (tiles[e + 1] <= tile) ++e;
  const int row0 = off[e] + (tile - tiles[e]) * kFt, row_end = off[e + 1];
  const int col0 = blockIdx.x * kFt;
  const float* A = reinterpret_cast<const float*>(p.A);
  const float* B = reinterpret_cast<const float*>(p.B) + static_cast<long long>(e) * p.N * p.ldb;
  const float* B2 = GATED ? reinterpret_cast<const float*>(p.B2) + static_cast<long long>(e) * p.N * p.ldb : nullptr;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {}, up[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kFk) {
    for (int i = threadIdx.x; i < kFt * kFk; i += kFthr) {
      const int r = i / kFk, k = i % kFk;
      const bool kin = k0 + k < p.K;
      sa[k][r] = (kin && row0 + r < row_end) ? A[static_cast<long long>(row0 + r) * p.lda + k0 + k] : 0.f;
      const bool in = kin && col0 + r < p.N;
      const long long bo = static_cast<long long>(col0 + r) * p.ldb + k0 + k;
      sb[k][r] = in ? B[bo] : 0.f;
      if (GATED) sc[k][r] = in ? B2[bo] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kFk; ++k) {
      float a[4], b[4], c[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sa[k][ty * 4 + i];
        b[i] = sb[k][tx * 4 + i];
        if (GATED) c[i] = sc[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
          if (GATED) up[i][j] = fmaf(a[i], c[j], up[i][j]);
        }
    }
    __syncthreads();
  }
  const GatedAct act{p.act, p.act_limit, p.act_alpha, p.act_shift};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = row0 + ty * 4 + i;
    if (row >= row_end) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = col0 + tx * 4 + j;
      if (col < p.N)
        reinterpret_cast<float*>(p.D)[static_cast<long long>(row) * p.ldd + col] =
            GATED ? gated_act_of<true>(acc[i][j], up[i][j], act) : lin_act_of(acc[i][j], p.lin_act);
    }
  }
}

template <bool GATED>
int launch_moe_gemm(const nfk_moe_gemm_params& p, cudaStream_t stream) {
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    if (cudaFuncSetAttribute(moe_gemm_kernel<GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, kGemmSmem) != cudaSuccess)
      return NF_ERR_CUDA;
    attr = true;
  }
  const int want = (p.N + 31) / 32 * 32 * (GATED ? 2 : 1);
  const int bn = want < 256 ? want : 256;
  CUtensorMap tmA, tmA32, tmB0, tmB1;
  int rc = make_tmap_bf16_2d(&tmA, p.A, p.rows, p.K, p.lda, BM, BK);
  if (rc == NF_OK) rc = make_tmap_bf16_2d(&tmA32, p.A, p.rows, p.K, p.lda, 32, BK);
  if (rc == NF_OK) rc = make_tmap_bf16_2d(&tmB0, p.B, static_cast<uint64_t>(p.experts) * p.N, p.K, p.ldb, GATED ? bn / 2 : bn, BK);
  if (rc == NF_OK && GATED) rc = make_tmap_bf16_2d(&tmB1, p.B2, static_cast<uint64_t>(p.experts) * p.N, p.K, p.ldb, bn / 2, BK);
  if (rc != NF_OK) return rc;
  if (!GATED) tmB1 = tmB0;
  const int out_bn = GATED ? bn / 2 : bn;
  // no more CTAs than there can be tiles
  const long long most = (static_cast<long long>(p.rows / BM) + (p.rows < p.experts ? p.rows : p.experts)) * ((p.N + out_bn - 1) / out_bn);
  long long ctas = p.num_ctas > 0 ? p.num_ctas : device_sm_count();
  if (ctas > most) ctas = most;
  if (ctas < 1) ctas = 1;
  moe_gemm_kernel<GATED><<<static_cast<int>(ctas), kThreads, kGemmSmem, stream>>>(tmA, tmA32, tmB0, tmB1, p, bn);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_moe_route(const nfk_moe_route_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == 0) return NF_OK;
  if (!p->logits || !p->expert || !p->weight || !p->rank || !p->counts || p->T < 0 || p->experts <= 0 ||
      p->identity < 0 || p->experts + p->identity > kMaxExperts || p->groups <= 0 || (p->experts + p->identity) % p->groups != 0 ||
      p->keep <= 0 || p->keep > p->groups || p->top <= 0 || p->top > 32 ||
      p->top > p->keep * ((p->experts + p->identity) / p->groups) || ((p->gate_col >= 0 || p->identity > 0) && !p->gate) ||
      (p->gate_col >= 0 && p->identity > 0) || p->score < NFK_SCORE_SIGMOID || p->score > NFK_SCORE_SOFTMAX_ALL)
    return NF_ERR_BAD_ARG;
  const size_t sm = static_cast<size_t>(kRouteWarps) * (2 * (p->experts + p->identity) + p->groups) * 4;
  if (sm > 48 * 1024) return NF_ERR_UNSUPPORTED;
  int grid = (p->T + kRouteWarps - 1) / kRouteWarps;
  if (grid > 16 * device_sm_count()) grid = 16 * device_sm_count();
  moe_route_kernel<<<grid, kRouteWarps * 32, sm, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_moe_permute(const nfk_moe_permute_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == 0) return NF_OK;
  if (!p->h || !p->out || !p->expert || !p->rank || !p->counts || !p->slot || p->T < 0 || p->top <= 0 || p->top > 32 ||
      p->experts <= 0 || p->experts > kMaxExperts || p->cols <= 0 || p->cols % 8 != 0 || p->ld_h % 8 != 0 ||
      p->ld_out % 8 != 0 || ((reinterpret_cast<uintptr_t>(p->h) | reinterpret_cast<uintptr_t>(p->out)) & 15) != 0)
    return NF_ERR_BAD_ARG;
  int grid = (p->T + 7) / 8;
  if (grid > 8 * device_sm_count()) grid = 8 * device_sm_count();
  moe_permute_kernel<<<grid, 256, 0, stream>>>(*p, p->cols * (p->dtype == NFK_F32 ? 4 : 2) / 16);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_moe_gemm(const nfk_moe_gemm_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->rows == 0) return NF_OK;
  if (!p->A || !p->B || !p->D || !p->counts || p->rows < 0 || p->experts <= 0 || p->experts > kMaxExperts || p->N <= 0 ||
      p->K <= 0 || p->N % 8 != 0 || p->K % 8 != 0 || p->lda % 8 != 0 || p->ldb % 8 != 0 || p->ldd % 8 != 0 ||
      p->act < NFK_ACT_SILU || p->act > NFK_ACT_CAPPED || p->lin_act < NFK_LIN_NONE || p->lin_act > NFK_LIN_RELU2 || (reinterpret_cast<uintptr_t>(p->D) & 15) != 0)
    return NF_ERR_BAD_ARG;
  if (p->dtype == NFK_F32) {
    const long long m_tiles = p->rows / kFt + (p->rows < p->experts ? p->rows : p->experts);
    if (m_tiles > 65535) return NF_ERR_BAD_ARG;
    const dim3 grid((p->N + kFt - 1) / kFt, static_cast<unsigned>(m_tiles));
    if (p->B2 != nullptr) moe_gemm_f32_kernel<true><<<grid, kFthr, 0, stream>>>(*p);
    else moe_gemm_f32_kernel<false><<<grid, kFthr, 0, stream>>>(*p);
    return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
  }
  return p->B2 != nullptr ? launch_moe_gemm<true>(*p, stream) : launch_moe_gemm<false>(*p, stream);
}
