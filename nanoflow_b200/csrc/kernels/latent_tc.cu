// Latent attention of single tokens on the 5th-generation tensor cores, in transposed form: a token's heads are
// the columns of the products instead of the rows, so up to 32 heads do not leave most of a 128-row tile empty.
//
//   S^T [keys x heads]    = C [keys x ld] Q^T              keys are the rows (K-major operand, as TMA leaves it)
//   O^T [ld x heads]     += C^T [ld x keys] P^T            latent columns are the rows (the same tile, MN-major)
//
// A CTA takes one token, 32 of its heads and a range of keys, in tiles of 64 keys (whole pages, by TMA). P^T has 64
// columns: the high bf16 parts of the 32 heads' probabilities and their low parts, which go to columns of their own
// and are added at the end, so the second product keeps about 16 bits without a second pass over the tile.
// Rows 64-127 of the score product read whatever follows the tile; nobody looks at them.
//
// Roles (12 warps): 0, 1 and 4, 5 softmax of 16 heads each, one thread per key (TMEM lanes 0-63; maxima over keys by
// shuffles, the reference maximum of a head moves only when it is outgrown by 2^8); 2 MMA issue and TMEM; 3 TMA;
// 8-11 rescale O^T when a reference maximum moved, and write the output. Every wait is bounded; one that runs out
// sets the status word and an abort flag, after which all roles run through without waiting.
#include "latent_tc.h"
#include "attn_mma.cuh"

namespace nf {
namespace {

constexpr int kTile = 64, kThr = 384, kHeads = 32;
constexpr float kGap = 8.f;

template <int D>
struct TcCfg {
  // a key tile holds pages as the pool stores them: [8-key group][64-column block][8 keys][128 bytes]
  static constexpr int BLK = 1024, GRP = D / 64 * BLK;
  static constexpr int TILE = kTile / 8 * GRP;
  static constexpr int STAGES = D <= 256 ? 4 : (D == 384 ? 3 : 2);
  static constexpr int QBLK = kHeads * 128;
  static constexpr int Q_OFF = STAGES * TILE;
  static constexpr int P_OFF = Q_OFF + D / 64 * QBLK;     // two buffers [64 keys][64]
  static constexpr int F_OFF = P_OFF + 2 * kTile * 128;
  // fp32: maxima [2 groups][2 warps][16], alpha [2 parities][32], l [2 groups][2 warps][16], inverse [32], m [32]
  static constexpr int BAR_OFF = F_OFF + (64 + 64 + 64 + 64) * 4;
  // rows 64-127 of the last stage's score product read one tile further: that has to be shared memory, too
  static constexpr int END = BAR_OFF + 256 > (STAGES + 1) * TILE ? BAR_OFF + 256 : (STAGES + 1) * TILE;
  static constexpr int SMEM = END + 1024;
  static constexpr int O_COL = 64;                        // TMEM: S^T of even / odd tiles, then O^T blocks of 64
  static constexpr int NCB = D / 128;
  static constexpr int TMEM_COLS = O_COL + NCB * 64 <= 128 ? 128 : (O_COL + NCB * 64 <= 256 ? 256 : 512);
};

enum TBar : int { FULL0 = 0, EMPTY0 = 4, S_FULL0 = 8, P_FULL0 = 10, CORR0 = 12, PV0 = 14, NUM_TBARS = 16 };

// K-major operand in the 128-byte swizzle, `sbo` bytes between groups of eight rows.
__device__ __forceinline__ uint64_t desc_k(uint32_t addr, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>(1) << 16;
  d |= static_cast<uint64_t>((sbo >> 4) & 0x3FFF) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
// MN-major operand: `lbo` bytes between blocks of 64 along M / N, `sbo` between groups of eight k indices.
__device__ __forceinline__ uint64_t desc_mn(uint32_t addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>((lbo >> 4) & 0x3FFF) << 16;
  d |= static_cast<uint64_t>((sbo >> 4) & 0x3FFF) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
__device__ __forceinline__ void pair_sync(int g) { asm volatile("bar.sync %0, 64;" ::"r"(g + 1) : "memory"); }

// v[0..15] of 32 lanes -> lane i holds the reduction (over all lanes) of v[i >> 1].
template <class Op>
__device__ __forceinline__ float reduce16(const float (&v)[16], Op op) {
  const int lane = threadIdx.x & 31;
  float a[8], b[4], c[2];
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const bool up = lane & 16;
    const float keep = up ? v[8 + i] : v[i], send = up ? v[i] : v[8 + i];
    a[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 16));
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const bool up = lane & 8;
    const float keep = up ? a[4 + i] : a[i], send = up ? a[i] : a[4 + i];
    b[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 8));
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const bool up = lane & 4;
    const float keep = up ? b[2 + i] : b[i], send = up ? b[i] : b[2 + i];
    c[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, 4));
  }
  const bool up = lane & 2;
  const float keep = up ? c[1] : c[0], send = up ? c[0] : c[1];
  const float d = op(keep, __shfl_xor_sync(0xffffffffu, send, 2));
  return op(d, __shfl_xor_sync(0xffffffffu, d, 1));
}

template <int D>
__global__ void __launch_bounds__(kThr, 1)
latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tmC, nfk_latent_attn_params p) {
  using C = TcCfg<D>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t sb = smem_u32(smem);
  float* max_s = reinterpret_cast<float*>(smem + C::F_OFF);   // [group][warp][16]
  float* alpha_s = max_s + 64;                                // [parity][32]
  float* l_s = alpha_s + 64;                                  // [group][warp][16]
  float* inv_s = l_s + 64;                                    // [32] 1 / l (or l, with splits)
  float* m_s = inv_s + 32;                                    // [32]
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + C::BAR_OFF);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + NUM_TBARS);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  volatile int* rescale_s = reinterpret_cast<volatile int*>(tmem_slot + 2);   // [parity][group]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hgroups = (p.heads + kHeads - 1) / kHeads;
  const int head0 = (blockIdx.x % hgroups) * kHeads;
  const int split = (blockIdx.x / hgroups) % p.splits;
  const int ti = blockIdx.x / (hgroups * p.splits);
  const int tok = p.tokens[ti];
  const int pos = p.positions[tok], req = p.token_req[tok];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int key0 = lo / kPage * kPage;                         // tiles start on a page
  const int n_all = (pos - key0) / kTile + 1;
  const int per = (n_all + p.splits - 1) / p.splits;
  const int t_begin = min(n_all, split * per), n_tiles = min(n_all, t_begin + per) - t_begin;

  if (threadIdx.x == 0) {
    for (int b = 0; b < NUM_TBARS; ++b) mbar_init(&bars[b], (b >= P_FULL0 && b < PV0) ? 4 : 1);
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmC);
  }
  // queries: [D / 64][32 heads][64 columns], 128-byte swizzle; heads past the last one are zero
  for (int i = threadIdx.x; i < kHeads * (D / 8); i += kThr) {
    const int r = i / (D / 8), ch = i % (D / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (head0 + r < p.heads)
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(tok) * p.ld_q +
                                          static_cast<long long>(head0 + r) * D + ch * 8);
    *reinterpret_cast<uint4*>(smem + C::Q_OFF + (ch >> 3) * C::QBLK + r * 128 + (((ch ^ r) & 7) << 4)) = v;
  }
  fence_proxy_async_smem();
  if (warp == 2) {
    tmem_alloc(tmem_slot, C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  auto wait = [&](int b, int parity, unsigned int code) -> bool {
    if (*abort_flag) return false;
    if (mbar_wait(&bars[b], parity)) return true;
    report_status(p.status, code);
    *abort_flag = 1;
    return false;
  };

  if (warp == 3) {
    // ------------------------------------------------------------------ copies: lanes 0-3 one page each
    const int pg0 = p.kv_indptr[req], np = p.kv_indptr[req + 1] - pg0;
    const int first = p.kv_first != nullptr ? p.kv_first[req] : 0;
    auto page_at = [&](int t) {
      const int slot = min((key0 + (t_begin + t) * kTile) / kPage + lane, pos / kPage) - first;   // past the end: the last page
      return (lane < 4 && slot >= 0 && slot < np) ? p.kv_indices[pg0 + slot] : -1;
    };
    int next = n_tiles > 0 ? page_at(0) : 0, issued = 0;
    for (int t = 0; t < n_tiles; ++t) {
      int page = next;
      if (t + 1 < n_tiles) next = page_at(t + 1);
      const int s = t % C::STAGES;
      int ok = 1;
      if (lane == 0) {
        ok = wait(EMPTY0 + s, ((t / C::STAGES) & 1) ^ 1, NF_ST_TIMEOUT_SMEM_EMPTY);
        if (ok) mbar_expect_tx(&bars[FULL0 + s], C::TILE);
      }
      if (__shfl_sync(0xffffffffu, ok, 0) == 0) break;
      if (lane < 4) {
        if (page < 0 || page >= p.num_pages) {
          report_status(p.status, NF_ST_BAD_INDEX);
          page = 0;
        }
        tma_load_2d(smem + s * C::TILE + lane * (kPage * D * 2), &tmC, &bars[FULL0 + s], 0, page * (kPage * D / 64));
      }
      ++issued;
    }
    // copies still in flight must have landed before the CTA gives its shared memory back
    if (lane == 0)
      for (int t = max(0, issued - C::STAGES); t < issued; ++t) (void)mbar_wait(&bars[FULL0 + t % C::STAGES], (t / C::STAGES) & 1);
  } else if (warp == 2) {
    // ------------------------------------------------------------------ MMA issue
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(128, kHeads);
      const uint32_t idesc_o = umma_idesc_bf16(128, 2 * kHeads) | (1u << 15) | (1u << 16);   // both operands MN-major
      auto issue_s = [&](int t) -> bool {
        const int s = t % C::STAGES;
        if (!wait(FULL0 + s, (t / C::STAGES) & 1, NF_ST_TIMEOUT_SMEM_FULL)) return false;
        tc_fence_after();
        const uint32_t kb = sb + s * C::TILE;
#pragma unroll 8
        for (int k = 0; k < D / 16; ++k)
          umma_bf16_ss(tmem + (t & 1) * kHeads, desc_k(kb + (k >> 2) * C::BLK + (k & 3) * 32, C::GRP),
                       umma_desc_k_sw128(sb + C::Q_OFF + (k >> 2) * C::QBLK + (k & 3) * 32), idesc_s, k ? 1u : 0u);
        umma_commit(&bars[S_FULL0 + (t & 1)]);
        return true;
      };
      bool ok = n_tiles > 0 && issue_s(0);
      for (int t = 0; t < n_tiles && ok; ++t) {
        if (t + 1 < n_tiles && !issue_s(t + 1)) break;
        const int par = t & 1, ph = (t >> 1) & 1, s = t % C::STAGES;
        ok = wait(P_FULL0 + par, ph, NF_ST_TIMEOUT_SMEM_FULL) && wait(CORR0 + par, ph, NF_ST_TIMEOUT_TMEM_EMPTY);
        if (!ok) break;
        tc_fence_after();
        const uint32_t kb = sb + s * C::TILE, pb = sb + C::P_OFF + par * (kTile * 128);
#pragma unroll
        for (int cb = 0; cb < C::NCB; ++cb)
#pragma unroll
          for (int k = 0; k < kTile / 16; ++k)
            umma_bf16_ss(tmem + C::O_COL + cb * (2 * kHeads), desc_mn(kb + 2 * cb * C::BLK + k * 2 * C::GRP, C::BLK, C::GRP),
                         desc_mn(pb + k * 2048, 8192, 1024), idesc_o, (t | k) ? 1u : 0u);
        umma_commit(&bars[EMPTY0 + s]);
        umma_commit(&bars[PV0 + par]);
      }
    }
  } else if (warp < 6) {
    // ------------------------------------------------------------------ softmax: key = lane of a warp pair, 16 heads
    const int g = warp >> 2, w = warp & 3;                  // w: 0 or 1, keys 32 w ...
    const int hb = g * 16;
    const float scale = p.scale * kLog2e;
    float m[16], l[16];
#pragma unroll
    for (int h = 0; h < 16; ++h) {
      const int head = head0 + hb + h;
      const bool sink = p.sinks != nullptr && split == 0 && head < p.heads;
      m[h] = sink ? p.sinks[head] * kLog2e : -INFINITY;
      l[h] = (sink && w == 0 && lane == 0) ? 1.f : 0.f;
    }
    for (int t = 0; t < n_tiles; ++t) {
      const int par = t & 1;
      (void)wait(S_FULL0 + par, (t >> 1) & 1, NF_ST_TIMEOUT_TMEM_FULL);
      __syncwarp();
      tc_fence_after();
      uint32_t r[32];
      tmem_ld_32x32b_x16(tmem + (static_cast<uint32_t>(w * 32) << 16) + par * kHeads + hb, r);
      tmem_ld_wait();
      const int key = key0 + (t_begin + t) * kTile + w * 32 + lane;
      const bool seen = key >= lo && key <= pos;
      float x[16];
#pragma unroll
      for (int h = 0; h < 16; ++h) x[h] = seen ? __uint_as_float(r[h]) * scale : -INFINITY;
      const float mx = reduce16(x, [](float a, float b) { return fmaxf(a, b); });
      float* mine = max_s + (g * 2 + w) * 16;
      if ((lane & 1) == 0) mine[lane >> 1] = mx;
      pair_sync(g);
      const float* m0 = max_s + g * 32;
      bool any = false;
      float al[16];
#pragma unroll
      for (int h = 0; h < 16; ++h) {
        const float top = fmaxf(m0[h], m0[16 + h]);
        const bool grow = top > m[h] + kGap || m[h] == -INFINITY;
        al[h] = grow ? fast_exp2(m[h] - top) : 1.f;          // the first maximum: exp2(-inf) = 0
        any |= grow;
        if (grow) {
          m[h] = top;
          l[h] *= al[h];
        }
      }
      if (w == 0 && lane == 0) rescale_s[par * 2 + g] = (any && t > 0) ? 1 : 0;
      if (w == 0 && any) {
#pragma unroll
        for (int h = 0; h < 16; ++h)
          if (lane == h) alpha_s[par * kHeads + hb + h] = al[h];
      } else if (w == 0 && lane < 16) {
        alpha_s[par * kHeads + hb + lane] = 1.f;
      }
      uint32_t hi[8], lw[8];
#pragma unroll
      for (int h = 0; h < 16; h += 2) {
        const float e0 = fast_exp2(x[h] - m[h]), e1 = fast_exp2(x[h + 1] - m[h + 1]);
        l[h] += e0;
        l[h + 1] += e1;
        hi[h >> 1] = pack_bf16x2(e0, e1);
        const float2 f = unpack_bf16x2(hi[h >> 1]);
        lw[h >> 1] = pack_bf16x2(e0 - f.x, e1 - f.y);
      }
      // this key's row of P^T: high parts of all heads in columns 0-31, low parts in 32-63
      const int row = w * 32 + lane;
      uint8_t* prow = smem + C::P_OFF + par * (kTile * 128) + row * 128;
#pragma unroll
      for (int q = 0; q < 2; ++q) {
        *reinterpret_cast<uint4*>(prow + (((g * 2 + q) ^ (row & 7)) << 4)) = make_uint4(hi[4 * q], hi[4 * q + 1], hi[4 * q + 2], hi[4 * q + 3]);
        *reinterpret_cast<uint4*>(prow + (((4 + g * 2 + q) ^ (row & 7)) << 4)) = make_uint4(lw[4 * q], lw[4 * q + 1], lw[4 * q + 2], lw[4 * q + 3]);
      }
      fence_proxy_async_smem();
      tc_fence_before();
      pair_sync(g);               // the pair's maxima have been read, its rows are written
      if (lane == 0) mbar_arrive(&bars[P_FULL0 + par]);
    }
    const float ls = reduce16(l, [](float a, float b) { return a + b; });
    if ((lane & 1) == 0) l_s[(g * 2 + w) * 16 + (lane >> 1)] = ls;
    pair_sync(g);
    if (w == 0) {
#pragma unroll
      for (int h = 0; h < 16; ++h)
        if (lane == h) {
          const float sum = l_s[g * 32 + h] + l_s[g * 32 + 16 + h];
          inv_s[hb + h] = p.splits == 1 ? (sum > 0.f ? 1.f / sum : 0.f) : sum;
          m_s[hb + h] = m[h];
        }
    }
  }
  if (warp >= 8) {
    // ------------------------------------------------------------------ O^T: rescaling, one latent column per thread
    const int qd = warp & 3;
    const uint32_t t_lane = tmem + (static_cast<uint32_t>(qd * 32) << 16) + C::O_COL;
    for (int t = 0; t < n_tiles; ++t) {
      const int par = t & 1;
      (void)wait(P_FULL0 + par, (t >> 1) & 1, NF_ST_TIMEOUT_TMEM_FULL);
      __syncwarp();
      if ((rescale_s[par * 2] | rescale_s[par * 2 + 1]) != 0) {
        (void)wait(PV0 + ((t - 1) & 1), ((t - 1) >> 1) & 1, NF_ST_TIMEOUT_TMEM_FULL);
        __syncwarp();
        tc_fence_after();
#pragma unroll 1
        for (int c = 0; c < 2 * C::NCB; ++c) {
          uint32_t ov[32];
          tmem_ld_32x32b_x32(t_lane + c * 32, ov);
          tmem_ld_wait();
#pragma unroll
          for (int h = 0; h < 32; ++h) ov[h] = __float_as_uint(__uint_as_float(ov[h]) * alpha_s[par * kHeads + h]);
          tmem_st_32x32b_x32(t_lane + c * 32, ov);
        }
        tmem_st_wait();
        tc_fence_before();
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars[CORR0 + par]);
    }
    if (n_tiles > 0) (void)wait(PV0 + ((n_tiles - 1) & 1), ((n_tiles - 1) >> 1) & 1, NF_ST_TIMEOUT_TMEM_FULL);
    __syncwarp();
    tc_fence_after();
  }
  __syncwarp();
  __syncthreads();                 // the sums and maxima are in shared memory
  if (warp >= 8) {
    const int qd = warp & 3;
    const uint32_t t_lane = tmem + (static_cast<uint32_t>(qd * 32) << 16) + C::O_COL;
    float* ws = p.splits == 1 ? nullptr
                              : p.workspace + ((static_cast<long long>(ti) * p.splits + split) * p.heads + head0) * (D + 2);
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(tok) * p.ld_out +
                         static_cast<long long>(head0) * D;
    if (n_tiles > 0 || p.splits > 1) {
#pragma unroll 1
      for (int cb = 0; cb < C::NCB; ++cb) {
        uint32_t a[32], b[32];
        tmem_ld_32x32b_x32(t_lane + cb * 64, a);
        tmem_ld_32x32b_x32(t_lane + cb * 64 + 32, b);
        tmem_ld_wait();
        const int col = cb * 128 + qd * 32 + lane;
#pragma unroll
        for (int h = 0; h < 32; ++h) {
          if (head0 + h >= p.heads) break;
          const float v = n_tiles > 0 ? __uint_as_float(a[h]) + __uint_as_float(b[h]) : 0.f;
          if (ws == nullptr) dst[static_cast<long long>(h) * D + col] = __float2bfloat16(v * inv_s[h]);
          else ws[static_cast<long long>(h) * (D + 2) + col] = v;
        }
      }
    }
    if (ws != nullptr && qd == 0 && head0 + lane < p.heads) {
      ws[static_cast<long long>(lane) * (D + 2) + D] = m_s[lane];
      ws[static_cast<long long>(lane) * (D + 2) + D + 1] = inv_s[lane];
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 2) {
    tc_fence_after();
    tmem_dealloc(tmem, C::TMEM_COLS);
  }
}

template <int D>
int launch(const nfk_latent_attn_params& p, cudaStream_t stream) {
  using C = TcCfg<D>;
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    if (cudaFuncSetAttribute(latent_attn_tc_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::SMEM) != cudaSuccess)
      return NF_ERR_CUDA;
    attr = true;
  }
  CUtensorMap tm;
  const int rc = make_tmap_bf16_2d(&tm, p.pool, static_cast<uint64_t>(p.num_pages) * kPage * (D / 64), 64, 64, kPage * (D / 64), 64);
  if (rc != NF_OK) return rc;
  const long long grid = static_cast<long long>(p.n_tokens) * p.splits * ((p.heads + kHeads - 1) / kHeads);
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  latent_attn_tc_kernel<D><<<static_cast<int>(grid), kThr, C::SMEM, stream>>>(tm, p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace

bool latent_tc_built(long long ld) { return ld == 128 || ld == 256 || ld == 384 || ld == 512; }

int latent_tc_launch(const nfk_latent_attn_params& p, cudaStream_t stream) {
  switch (p.ld) {
    case 128: return launch<128>(p, stream);
    case 256: return launch<256>(p, stream);
    case 384: return launch<384>(p, stream);
    case 512: return launch<512>(p, stream);
    default: return NF_ERR_UNSUPPORTED;
  }
}

}  // namespace nf
