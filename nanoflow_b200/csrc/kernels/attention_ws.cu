// Chunked-prefill attention on the 5th-generation tensor cores (head_dim 128), warp-specialised.
//
// A work item is (request, first token, token count <= 128/group) x kv head, as in nfk_attn_prefill: the
// item's query rows r = token * group + head fill one 128-row MMA tile, and the item walks its keys in
// tiles of 64 tokens. Three roles share a 192-thread CTA and meet only through mbarriers:
//
//   warp 4, one thread   loads: TMA copies (no multicast) of the Q rows and of whole K / V pages from the
//                        paged pool into 128B-swizzled shared memory, two K and two V tiles in flight;
//                        the page ids of the next tile are fetched while the current one is issued
//   warp 5, one thread   tcgen05.mma: S(t+1) = Q K(t+1)^T is issued before P(t) is waited for, into the
//                        other of two S accumulators in TMEM, so the tensor cores work on the next tile's
//                        scores while the softmax warps are still busy with this tile; then
//                        O += P(t) V(t) with P read from TMEM (A operand in tensor memory) and V read
//                        token-major from shared memory (MN-major B operand: no transpose pass)
//   warps 0-3            softmax: one thread per query row reads its 64 scores from TMEM, keeps the
//                        running maximum and sum, and writes P (bf16, two per column) back over the first 32
//                        columns of the S accumulator it came from: P never passes through shared memory
//
// S(t+2) goes into the accumulator that held S(t) / P(t), so the MMA thread issues it only once
// O += P(t) V(t) has completed (products into different accumulators are not ordered against each other's
// operand reads); S(t+2) is needed a whole softmax pass later, so that wait is off the critical path.
//
// O stays in TMEM for the whole item: P is taken relative to a reference maximum that only moves (and O
// is rescaled in TMEM) when a row's maximum outgrows it by more than 2^8. Two CTAs fit an SM (97 KB of
// shared memory, 256 TMEM columns each). Every wait is bounded; a wait that runs out sets the status
// word and all roles leave through the common exit, which frees TMEM.
//
// EXT adds what other attention designs need, in an instantiation of its own: a sliding window (tiles before
// the first row's window are never loaded), a sink in the softmax denominator, K / V as columns of plain
// rows instead of pool pages (keys expanded from a latent cache), and probabilities that enter the second
// product as a bf16 pair: the high parts over the first half of the S accumulator, the low parts over the
// second half; also chunks (a position sees its own chunk only), and page lists that start inside the sequence.
// CAP adds capped scores (cap tanh(score / cap)), DIST scores that lose a ln(1 + b distance) with two numbers per head;
// with any of these, head_dim 64 is built as well.
//
// Takes the place of the reference's FlashInfer BatchPrefillWithPagedKVCacheKernel
// (gemv/include/attention/prefill.cuh:1066-1374, mma.sync m16n16k16 + ldmatrix on sm_80).
#include "common.cuh"
#include "kernels.h"
#include "softcap.cuh"

namespace nf {
namespace {

constexpr int kPage = 16;
constexpr int kTile = 64;             // kv tokens per tile
constexpr int kThreads = 192;         // warps 0-3 softmax (TMEM lane quarter = warp index), 4 loads, 5 MMA
constexpr float kLog2e = 1.4426950408889634f;
constexpr float kRescaleGap = 8.0f;   // log2 of how far a row maximum may outgrow its reference

// Shared-memory map (bytes from the 1024-aligned base); every operand region is 1024-aligned. Operands are cut into
// blocks of 64 columns ("halves" at head_dim 128).
constexpr int kHalfBytes = 8192;               // [64 tok][64 hd]
template <int HD>
struct WsCfg {
  static constexpr int NH = HD / 64;
  static constexpr int Q_OFF = 0;                       // NH x [128 rows][64 hd]
  static constexpr int K_OFF = NH * 16384;              // 2 stages x NH x [64 tok][64 hd]
  static constexpr int kStageBytes = NH * kHalfBytes;   // one K (or V) tile
  static constexpr int V_OFF = K_OFF + 2 * kStageBytes; // 2 stages x NH x [64 tok][64 hd]
  static constexpr int BAR_OFF = V_OFF + 2 * kStageBytes;
  static constexpr int kSmemBytes = BAR_OFF + 256;
};

enum Bar : int {
  Q_FULL = 0, Q_EMPTY, K_FULL0, K_FULL1, K_EMPTY0, K_EMPTY1, V_FULL0, V_FULL1, V_EMPTY0, V_EMPTY1,
  S_FULL0, S_FULL1, P_FULL0, P_FULL1, PV_DONE0, PV_DONE1, O_FREE, NUM_BARS
};

__device__ __forceinline__ float fast_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void st_shared_v4(uint32_t addr, uint32_t a, uint32_t b, uint32_t c, uint32_t d) {
  asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(a), "r"(b), "r"(c), "r"(d) : "memory");
}
// Shared-memory descriptor of an MN-major operand in the 128-byte swizzle: 64 elements along M/N are
// contiguous (one 128-byte row per k index), `lbo` bytes lead to the next 64 elements along M/N, `sbo`
// bytes to the next group of eight k indices.
__device__ __forceinline__ uint64_t umma_desc_mn_sw128(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  uint64_t d = 0;
  d |= static_cast<uint64_t>((smem_addr & 0x3FFFF) >> 4);
  d |= static_cast<uint64_t>((lbo >> 4) & 0x3FFF) << 16;
  d |= static_cast<uint64_t>((sbo >> 4) & 0x3FFF) << 32;
  d |= static_cast<uint64_t>(1) << 46;
  d |= static_cast<uint64_t>(2) << 61;
  return d;
}
constexpr uint32_t kIdescBMnMajor = 1u << 16;

struct Item {
  int req, tok0, ntok, kvh, pg0, np, kv_len, q_end, n_tiles;
  int t_first;      // first key tile (EXT: the one the first row's window or chunk starts in)
  int pg_first;     // page slot of the sequence that the page list starts with
  bool valid;
};
template <bool EXT>
__device__ __forceinline__ Item read_item(const nfk_attn_params& p, long long w) {
  Item it;
  const int item = static_cast<int>(w / p.kv_heads);
  it.kvh = static_cast<int>(w % p.kv_heads);
  it.req = p.items[item * 3 + 0];
  it.tok0 = p.items[item * 3 + 1];
  it.ntok = p.items[item * 3 + 2];
  it.pg0 = p.kv_indptr[it.req];
  it.np = p.kv_indptr[it.req + 1] - it.pg0;
  it.pg_first = EXT && p.kv_first != nullptr ? p.kv_first[it.req] : 0;
  it.kv_len = (it.pg_first + it.np - 1) * kPage + p.kv_last_page_len[it.req];
  it.q_end = p.qo_indptr[it.req + 1];
  // absolute position of global token t of this request: kv_len - (q_end - t)
  const int kv_hi = it.kv_len - (it.q_end - (it.tok0 + it.ntok - 1)) + 1;   // keys visible to the last row
  it.valid = it.ntok > 0 && it.np > 0 && kv_hi > 0;
  it.n_tiles = it.valid ? (kv_hi + kTile - 1) / kTile : 0;
  it.t_first = 0;
  if (EXT && p.window > 0 && it.valid) {
    const int lo = it.kv_len - (it.q_end - it.tok0) - p.window + 1;     // first key of the first row
    if (lo > 0) it.t_first = lo / kTile;
    it.n_tiles -= it.t_first;
  } else if (EXT && p.chunk > 0 && it.valid) {
    it.t_first = (it.kv_len - (it.q_end - it.tok0)) / p.chunk * p.chunk / kTile;
    it.n_tiles -= it.t_first;
  }
  return it;
}

// The CTA's work in round k, -1 if there is none. Later items of a request see more keys (and callers may order all items by
// that), so the last ones go first, and every other round deals them out in reverse: each CTA's share is of nearly the same
// length.
__device__ __forceinline__ long long work_index(int k, long long total) {
  const long long g = gridDim.x, i = k * g + ((k & 1) != 0 ? g - 1 - blockIdx.x : blockIdx.x);
  return i < total ? total - 1 - i : -1;
}

template <int HD, bool EXT, bool CAP, bool DIST>
__global__ void __launch_bounds__(kThreads, 2)
attn_prefill_ws_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmKV,
                       nfk_attn_params p) {
  using C = WsCfg<HD>;
  constexpr int NH = C::NH, Q_OFF = C::Q_OFF, K_OFF = C::K_OFF, V_OFF = C::V_OFF, BAR_OFF = C::BAR_OFF;
  constexpr int kStageBytes = C::kStageBytes;
  extern __shared__ __align__(1024) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + BAR_OFF);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + NUM_BARS);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if ((sb & 1023u) != 0u) {
    // the operand layouts assume a 1024-aligned base; report instead of computing garbage
    if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    return;
  }

  if (threadIdx.x == 0) {
    for (int b = 0; b < NUM_BARS; ++b) {
      const bool warps4 = b == P_FULL0 || b == P_FULL1 || b == O_FREE;
      mbar_init(&bars[b], warps4 ? 4 : 1);
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmKV);
  }
  // Q rows past an item's last token are never loaded; start them (and everything else) from zero so
  // that what the tensor cores read there is always finite
  for (int i = threadIdx.x; i < BAR_OFF / 16; i += kThreads) st_shared_v4(sb + i * 16, 0u, 0u, 0u, 0u);
  fence_proxy_async_smem();
  if (warp == 5) {
    tmem_alloc(tmem_slot, 256);   // S0: columns [0,64), S1: [64,128), O: [128,256)
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  const int group = p.q_heads / p.kv_heads;
  const long long total = static_cast<long long>(p.num_items) * p.kv_heads;
  const int rounds = static_cast<int>((total + gridDim.x - 1) / gridDim.x);
  auto fail = [&](unsigned int code) {
    report_status(p.status, code);
    *abort_flag = 1;
  };

  if (warp == 4) {
    // ------------------------------------------------------------------ loads
    if (lane == 0) {
      uint32_t g = 0, n_item = 0;          // tiles / items issued so far by this CTA
      uint32_t issued[NUM_BARS];           // per "full" barrier: loads issued on it
      for (int b = 0; b < NUM_BARS; ++b) issued[b] = 0;
      bool ok = true;
      for (int k = 0; k < rounds && ok; ++k) {
        const long long w = work_index(k, total);
        if (w < 0) continue;
        const Item it = read_item<EXT>(p, w);
        if (!it.valid) continue;
        if (!mbar_wait(&bars[Q_EMPTY], (n_item & 1) ^ 1) || *abort_flag) { fail(NF_ST_TIMEOUT_SMEM_EMPTY); break; }
        if (EXT && p.q_rows > 0) {
          // one head per query row tile: 128 rows in two boxes; rows past the item's tokens are other tokens' (or
          // zero past the buffer) and are never stored
          mbar_expect_tx(&bars[Q_FULL], 128u * HD * 2);
#pragma unroll
          for (int h = 0; h < NH; ++h)
            tma_load_2d(smem + Q_OFF + h * 16384, &tmQ, &bars[Q_FULL], it.kvh * HD + h * 64, it.tok0);
        } else {
        mbar_expect_tx(&bars[Q_FULL], static_cast<uint32_t>(it.ntok * group) * HD * 2);
        for (int tl = 0; tl < it.ntok; ++tl) {
          // row of the [T * heads per row][HD] view
          const int grow = (it.tok0 + tl) * (EXT && p.ld_q > 0 ? p.ld_q / HD : p.q_heads) + it.kvh * group;
#pragma unroll
          for (int h = 0; h < NH; ++h)
            tma_load_2d(smem + Q_OFF + h * 16384 + tl * group * 128, &tmQ, &bars[Q_FULL], h * 64, grow);
        }
        }
        ++issued[Q_FULL];
        ++n_item;
        int pages[4];
        auto fetch_pages = [&](int t) {
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            int pslot = (it.t_first + t) * (kTile / kPage) + j - it.pg_first;
            // past the sequence, or given back since nobody sees it: a valid page, masked by position
            if (pslot < 0 || pslot >= it.np) pslot = 0;
            int page = p.kv_indices[it.pg0 + pslot];
            if (page < 0 || page >= p.num_pages) {
              report_status(p.status, NF_ST_BAD_INDEX);
              page = 0;
            }
            pages[j] = page;
          }
        };
        fetch_pages(0);
        for (int t = 0; t < it.n_tiles; ++t, ++g) {
          const int s = g & 1;
          const uint32_t ph = ((g >> 1) & 1) ^ 1;
          int cur[4] = {pages[0], pages[1], pages[2], pages[3]};
          if (t + 1 < it.n_tiles) fetch_pages(t + 1);     // in flight while this tile's copies are issued
          if (!mbar_wait(&bars[K_EMPTY0 + s], ph) || *abort_flag) { fail(NF_ST_TIMEOUT_SMEM_EMPTY); ok = false; break; }
          mbar_expect_tx(&bars[K_FULL0 + s], kStageBytes);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            // row of the [pages*2*kv_heads*16][128] view, or row and column of the plain [rows][kv_ld] one
            const bool plain = EXT && p.kv_ld > 0;
            const int row0 = plain ? cur[j] * kPage : ((cur[j] * 2) * p.kv_heads + it.kvh) * kPage;
            const int col0 = plain ? p.k_col + it.kvh * HD : 0;
            uint8_t* dst = smem + K_OFF + s * kStageBytes + j * 2048;
#pragma unroll
            for (int h = 0; h < NH; ++h) tma_load_2d(dst + h * kHalfBytes, &tmKV, &bars[K_FULL0 + s], col0 + h * 64, row0);
          }
          ++issued[K_FULL0 + s];
          if (!mbar_wait(&bars[V_EMPTY0 + s], ph) || *abort_flag) { fail(NF_ST_TIMEOUT_SMEM_EMPTY); ok = false; break; }
          mbar_expect_tx(&bars[V_FULL0 + s], kStageBytes);
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const bool plain = EXT && p.kv_ld > 0;
            const int row0 = plain ? cur[j] * kPage : ((cur[j] * 2 + 1) * p.kv_heads + it.kvh) * kPage;
            const int col0 = plain ? p.v_col + it.kvh * HD : 0;
            uint8_t* dst = smem + V_OFF + s * kStageBytes + j * 2048;
#pragma unroll
            for (int h = 0; h < NH; ++h) tma_load_2d(dst + h * kHalfBytes, &tmKV, &bars[V_FULL0 + s], col0 + h * 64, row0);
          }
          ++issued[V_FULL0 + s];
        }
      }
      // copies still in flight must have landed before the CTA gives its shared memory back
      const int fulls[5] = {Q_FULL, K_FULL0, K_FULL1, V_FULL0, V_FULL1};
      for (int i = 0; i < 5; ++i) {
        const int b = fulls[i];
        if (issued[b] > 0) (void)mbar_wait(&bars[b], (issued[b] - 1) & 1);
      }
    }
  } else if (warp == 5) {
    // ------------------------------------------------------------------ MMA issue
    if (lane == 0) {
      const uint32_t idesc_s = umma_idesc_bf16(128, kTile);
      const uint32_t idesc_o = umma_idesc_bf16(128, HD) | kIdescBMnMajor;
      uint32_t g = 0, n_item = 0;
      // `pv_issued`: PV products issued so far by this CTA. The S accumulator that S(gt) goes into held P(gt-2),
      // the A operand of PV(gt-2); products with different accumulators are not ordered against each other's
      // operand reads, so the latest PV issued (gt-2 inside an item, gt-1 at its start) must have completed.
      auto issue_s = [&](uint32_t gt, uint32_t pv_issued) -> bool {
        const int s = gt & 1;
        const uint32_t ph = (gt >> 1) & 1;
        if (pv_issued > 0 && !mbar_wait(&bars[PV_DONE0 + ((pv_issued - 1) & 1)], ((pv_issued - 1) >> 1) & 1)) return false;
        if (!mbar_wait(&bars[K_FULL0 + s], ph)) return false;
        tc_fence_after();
        const uint32_t kb = sb + K_OFF + s * kStageBytes;
#pragma unroll
        for (int h = 0; h < NH; ++h)
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ss(tmem + s * kTile, umma_desc_k_sw128(sb + Q_OFF + h * 16384 + k * 32),
                         umma_desc_k_sw128(kb + h * kHalfBytes + k * 32), idesc_s, (h | k) ? 1u : 0u);
        umma_commit(&bars[K_EMPTY0 + s]);
        umma_commit(&bars[S_FULL0 + s]);
        return true;
      };
      bool ok = true;
      for (int k = 0; k < rounds && ok; ++k) {
        const long long w = work_index(k, total);
        if (w < 0) continue;
        const Item it = read_item<EXT>(p, w);
        if (!it.valid) continue;
        if (!mbar_wait(&bars[Q_FULL], n_item & 1) || *abort_flag) { fail(NF_ST_TIMEOUT_SMEM_FULL); break; }
        if (!issue_s(g, g)) { fail(NF_ST_TIMEOUT_SMEM_FULL); break; }
        for (int t = 0; t < it.n_tiles; ++t) {
          const uint32_t gt = g + t;
          if (t + 1 < it.n_tiles) {
            if (!issue_s(gt + 1, gt)) { fail(NF_ST_TIMEOUT_SMEM_FULL); ok = false; break; }
          } else {
            umma_commit(&bars[Q_EMPTY]);     // the last S product of the item has been issued
          }
          // the previous item's O must have been read out before this item's first PV overwrites it
          if (t == 0 && !mbar_wait(&bars[O_FREE], (n_item & 1) ^ 1)) { fail(NF_ST_TIMEOUT_TMEM_EMPTY); ok = false; break; }
          const int s = gt & 1;
          if (!mbar_wait(&bars[P_FULL0 + s], (gt >> 1) & 1) || !mbar_wait(&bars[V_FULL0 + s], (gt >> 1) & 1) || *abort_flag) {
            fail(NF_ST_TIMEOUT_SMEM_FULL);
            ok = false;
            break;
          }
          tc_fence_after();
          const uint32_t vb = sb + V_OFF + s * kStageBytes;
#pragma unroll
          for (int k = 0; k < 4; ++k)
            umma_bf16_ts(tmem + 2 * kTile, tmem + s * kTile + k * 8,      // P(t): 16 tokens = 8 columns per step
                         umma_desc_mn_sw128(vb + k * 2048, kHalfBytes, 1024), idesc_o, (t | k) ? 1u : 0u);
          if (EXT) {
#pragma unroll
            for (int k = 0; k < 4; ++k)                                   // the low parts of P(t)
              umma_bf16_ts(tmem + 2 * kTile, tmem + s * kTile + 32 + k * 8,
                           umma_desc_mn_sw128(vb + k * 2048, kHalfBytes, 1024), idesc_o, 1u);
          }
          umma_commit(&bars[V_EMPTY0 + s]);
          umma_commit(&bars[PV_DONE0 + s]);
        }
        g += it.n_tiles;
        ++n_item;
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax (one thread per query row)
    const int row = warp * 32 + lane;                  // query row = TMEM lane
    const uint32_t t_lane = tmem + (static_cast<uint32_t>(warp * 32) << 16);
    __nv_bfloat16* outp = reinterpret_cast<__nv_bfloat16*>(p.out);
    // CAP: capped scores carry the scale themselves
    const float scale = CAP || DIST ? 1.f : p.sm_scale * kLog2e;
    const float cap_in = CAP ? p.sm_scale / p.softcap : 0.f, cap_out = CAP ? p.softcap * kLog2e : 0.f;
    uint32_t g = 0, n_item = 0;
    bool ok = true;
    for (int k = 0; k < rounds && ok; ++k) {
        const long long w = work_index(k, total);
        if (w < 0) continue;
      const Item it = read_item<EXT>(p, w);
      if (!it.valid) continue;
      const int tl = row / group, hh = row % group;
      const bool row_valid = tl < it.ntok;
      const int pos = row_valid ? it.kv_len - (it.q_end - (it.tok0 + tl)) : -1;
      const int chunk_lo = EXT && p.chunk > 0 && row_valid ? pos / p.chunk * p.chunk : 0;
      float2 far = make_float2(0.f, 0.f);
      if (DIST && row_valid) far = reinterpret_cast<const float2*>(p.dist)[it.kvh * group + hh];
      float m_ref = -INFINITY, l = 0.f;
      for (int t = 0; t < it.n_tiles; ++t) {
        const uint32_t gt = g + t;
        const int s = gt & 1;
        const int cbase = (it.t_first + t) * kTile;
        float loss[DIST ? 64 : 1];                             // does not depend on the scores: while they are formed
        if (DIST) {
          const float d0 = static_cast<float>(pos - cbase);
#pragma unroll
          for (int j = 0; j < 64; ++j) loss[DIST ? j : 0] = distance_loss(far, d0 - j);     // (keys behind the row are masked below)
        }
        if (!mbar_wait(&bars[S_FULL0 + s], (gt >> 1) & 1) || *abort_flag) { fail(NF_ST_TIMEOUT_TMEM_FULL); ok = false; break; }
        tc_fence_after();
        uint32_t r0[32], r1[32];
        tmem_ld_32x32b_x32(t_lane + s * kTile, r0);
        tmem_ld_32x32b_x32(t_lane + s * kTile + 32, r1);
        tmem_ld_wait();
        if (CAP) {
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            r0[j] = __float_as_uint(cap_out * tanh_by_exp(__uint_as_float(r0[j]) * cap_in));
            r1[j] = __float_as_uint(cap_out * tanh_by_exp(__uint_as_float(r1[j]) * cap_in));
          }
        }
        if (DIST) {
          const float in = p.sm_scale * kLog2e;
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            r0[j] = __float_as_uint(fmaf(__uint_as_float(r0[j]), in, -loss[DIST ? j : 0]));
            r1[j] = __float_as_uint(fmaf(__uint_as_float(r1[j]), in, -loss[DIST ? 32 + j : 0]));
          }
        }
        if (cbase + kTile - 1 > pos) {                        // only tiles on the diagonal need the mask
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            if (cbase + j > pos) r0[j] = 0xff800000u;         // -inf
            if (cbase + 32 + j > pos) r1[j] = 0xff800000u;
          }
        }
        if (EXT && p.window > 0 && cbase <= pos - p.window) {   // tiles on the window's lower edge
          const int lo = pos - p.window + 1;
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            if (cbase + j < lo) r0[j] = 0xff800000u;
            if (cbase + 32 + j < lo) r1[j] = 0xff800000u;
          }
        }
        if (EXT && cbase < chunk_lo) {                          // tiles that start before the row's chunk
#pragma unroll
          for (int j = 0; j < 32; ++j) {
            if (cbase + j < chunk_lo) r0[j] = 0xff800000u;
            if (cbase + 32 + j < chunk_lo) r1[j] = 0xff800000u;
          }
        }
        float mxp = -INFINITY;
#pragma unroll
        for (int j = 0; j < 32; ++j) mxp = fmaxf(mxp, fmaxf(__uint_as_float(r0[j]), __uint_as_float(r1[j])));
        const float mx = mxp * scale;
        const bool grow = mx > m_ref + kRescaleGap || (m_ref == -INFINITY && mx > -INFINITY);
        if (t == 0) {
          m_ref = mx;
        } else if (__any_sync(0xffffffffu, grow)) {
          // bring O (in TMEM) and the row sum to the new reference maximum; warp-wide because the TMEM
          // accesses are, rows that did not grow scale by one. O may only be touched between two PV
          // products: PV(t-1) is the last one issued (PV(t) needs this tile's P), so once it is done O is still
          if (!mbar_wait(&bars[PV_DONE0 + ((gt - 1) & 1)], ((gt - 1) >> 1) & 1) || *abort_flag) {
            fail(NF_ST_TIMEOUT_TMEM_FULL);
            ok = false;
            break;
          }
          tc_fence_after();
          const float alpha = grow ? (m_ref == -INFINITY ? 0.f : fast_exp2(m_ref - mx)) : 1.f;
#pragma unroll 1
          for (int c = 0; c < HD / 32; ++c) {
            uint32_t ov[32];
            tmem_ld_32x32b_x32(t_lane + 2 * kTile + c * 32, ov);
            tmem_ld_wait();
#pragma unroll
            for (int j = 0; j < 32; ++j) ov[j] = __float_as_uint(__uint_as_float(ov[j]) * alpha);
            tmem_st_32x32b_x32(t_lane + 2 * kTile + c * 32, ov);
          }
          tmem_st_wait();
          l *= alpha;
          if (grow) m_ref = mx;
        }
        const float ms = m_ref == -INFINITY ? 0.f : m_ref;
        float rs = 0.f;
        uint32_t pk[32];                                      // column j: tokens 2j, 2j + 1 of the tile
        uint32_t pl[EXT ? 32 : 1];                            // low parts
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const float x0 = fast_exp2(fmaf(__uint_as_float(r0[2 * j]), scale, -ms));
          const float x1 = fast_exp2(fmaf(__uint_as_float(r0[2 * j + 1]), scale, -ms));
          const float y0 = fast_exp2(fmaf(__uint_as_float(r1[2 * j]), scale, -ms));
          const float y1 = fast_exp2(fmaf(__uint_as_float(r1[2 * j + 1]), scale, -ms));
          rs += (x0 + x1) + (y0 + y1);
          pk[j] = pack_bf16x2(x0, x1);
          pk[16 + j] = pack_bf16x2(y0, y1);
          if (EXT) {
            const float2 xh = unpack_bf16x2(pk[j]), yh = unpack_bf16x2(pk[16 + j]);
            pl[EXT ? j : 0] = pack_bf16x2(x0 - xh.x, x1 - xh.y);
            pl[EXT ? 16 + j : 0] = pack_bf16x2(y0 - yh.x, y1 - yh.y);
          }
        }
        l += rs;
        // P(t) goes over the first half of the S accumulator it was computed from (all 64 scores are in
        // registers); the other accumulator holds P(t-1) / S(t+1), so nothing has to be waited for
        tmem_st_32x32b_x32(t_lane + s * kTile, pk);
        if constexpr (EXT) tmem_st_32x32b_x32(t_lane + s * kTile + 32, pl);
        tmem_st_wait();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bars[P_FULL0 + s]);
      }
      if (!ok) break;
      g += it.n_tiles;
      // ---- the item's last PV product, then O / l to global memory ----
      // (one barrier per S accumulator: the softmax warps do not wait for every product, and up to two can be
      // outstanding here, which a single barrier's phase bit could not tell apart)
      if (!mbar_wait(&bars[PV_DONE0 + ((g - 1) & 1)], ((g - 1) >> 1) & 1) || *abort_flag) { fail(NF_ST_TIMEOUT_TMEM_FULL); break; }
      tc_fence_after();
      // a far larger sink makes the sum infinite and the row zero, as it should be
      if (EXT && p.sinks != nullptr && row_valid) l += fast_exp2(p.sinks[it.kvh * group + hh] * kLog2e - m_ref);
      const float inv = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* dst = outp + (static_cast<long long>(it.tok0 + tl) * p.q_heads + it.kvh * group + hh) * HD;
#pragma unroll 1
      for (int c = 0; c < HD / 32; ++c) {
        uint32_t r[32];
        tmem_ld_32x32b_x32(t_lane + 2 * kTile + c * 32, r);
        tmem_ld_wait();
        if (row_valid) {
#pragma unroll
          for (int g8 = 0; g8 < 4; ++g8) {
            uint4 v;
            v.x = pack_bf16x2(__uint_as_float(r[g8 * 8 + 0]) * inv, __uint_as_float(r[g8 * 8 + 1]) * inv);
            v.y = pack_bf16x2(__uint_as_float(r[g8 * 8 + 2]) * inv, __uint_as_float(r[g8 * 8 + 3]) * inv);
            v.z = pack_bf16x2(__uint_as_float(r[g8 * 8 + 4]) * inv, __uint_as_float(r[g8 * 8 + 5]) * inv);
            v.w = pack_bf16x2(__uint_as_float(r[g8 * 8 + 6]) * inv, __uint_as_float(r[g8 * 8 + 7]) * inv);
            *reinterpret_cast<uint4*>(dst + c * 32 + g8 * 8) = v;
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars[O_FREE]);
      ++n_item;
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 5) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

template <int HD, bool EXT, bool CAP, bool DIST = false>
int launch_ws(const nfk_attn_params& p, const CUtensorMap& tmQ, const CUtensorMap& tmKV, cudaStream_t stream) {
  constexpr int bytes = WsCfg<HD>::kSmemBytes;
  static bool attr_dev[kMaxDevices] = {false};   // the attribute is per device
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    if (cudaFuncSetAttribute(attn_prefill_ws_kernel<HD, EXT, CAP, DIST>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) !=
        cudaSuccess)
      return NF_ERR_CUDA;
    attr = true;
  }
  const long long total = static_cast<long long>(p.num_items) * p.kv_heads;
  long long ctas = p.num_ctas > 0 ? p.num_ctas : 2LL * device_sm_count();   // two resident CTAs per SM
  if (ctas > total) ctas = total;
  attn_prefill_ws_kernel<HD, EXT, CAP, DIST><<<static_cast<int>(ctas), kThreads, bytes, stream>>>(tmQ, tmKV, p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_attn_prefill_ws(const nfk_attn_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (!p->q || !p->out || !p->kv_pool || !p->qo_indptr || !p->kv_indptr || !p->kv_indices || !p->kv_last_page_len)
    return NF_ERR_BAD_ARG;
  if (p->kv_heads <= 0 || p->q_heads % p->kv_heads != 0 || p->num_pages <= 0) return NF_ERR_BAD_ARG;
  const int group = p->q_heads / p->kv_heads;
  // `precise` and the extensions run in the EXT instantiations, capped scores and head_dim 64 in one of their own
  const bool cap = p->softcap > 0.f, dist = p->dist != nullptr;
  const bool ext = p->window > 0 || p->sinks != nullptr || p->kv_ld > 0 || p->q_rows > 0 || cap || p->precise != 0;
  if (p->page_size != kPage || p->softcap < 0.f || (cap && dist)) return NF_ERR_UNSUPPORTED;
  if (p->chunk < 0 || (p->chunk > 0 && p->window > 0)) return NF_ERR_BAD_ARG;
  if ((dist || p->chunk > 0 || p->kv_first != nullptr) && p->precise == 0) return NF_ERR_UNSUPPORTED;
  if (p->head_dim != 128 && !(p->head_dim == 64 && ext)) return NF_ERR_UNSUPPORTED;
  if (ext ? group > 128 : (group > 16 || (16 % group) != 0)) return NF_ERR_UNSUPPORTED;
  const uint64_t HD = static_cast<uint64_t>(p->head_dim);
  if (p->num_items == 0) return NF_OK;
  if (p->num_items < 0 || p->items == nullptr) return NF_ERR_BAD_ARG;
  // Q as [tokens * q_heads][128] (the token count is not known here: any row the items name is inside
  // the caller's buffer, the map's row bound only has to be large enough); the pool as
  // [pages * 2 * kv_heads * 16][128]. Boxes: the `group` rows of one token, one page of one head; 64 columns.
  // With q_rows the queries are [q_rows][q_heads * 128] and a box is 128 tokens of one head; with kv_ld the
  // keys and values are columns of [num_pages * 16][kv_ld] rows.
  if (p->window < 0 || (p->q_rows > 0 && group != 1)) return NF_ERR_BAD_ARG;
  if (p->q_rows == 0 && p->ld_q != 0 && (p->precise == 0 || p->ld_q % p->head_dim != 0 || p->ld_q < p->q_heads * p->head_dim))
    return NF_ERR_BAD_ARG;
  if (p->kv_ld > 0 && (p->kv_ld % 8 != 0 || p->k_col < 0 || p->v_col < 0 || p->k_col % 8 != 0 || p->v_col % 8 != 0))
    return NF_ERR_BAD_ARG;
  CUtensorMap tmQ, tmKV;
  int rc = p->q_rows > 0 ? make_tmap_bf16_2d(&tmQ, p->q, p->q_rows, static_cast<uint64_t>(p->q_heads) * HD,
                                             p->ld_q > 0 ? p->ld_q : static_cast<uint64_t>(p->q_heads) * HD, 128, 64)
                         : make_tmap_bf16_2d(&tmQ, p->q, 1ull << 26, HD, HD, static_cast<uint32_t>(group), 64);
  if (rc != NF_OK) return rc;
  rc = p->kv_ld > 0 ? make_tmap_bf16_2d(&tmKV, p->kv_pool, static_cast<uint64_t>(p->num_pages) * kPage, p->kv_ld, p->kv_ld, kPage, 64)
                    : make_tmap_bf16_2d(&tmKV, p->kv_pool, static_cast<uint64_t>(p->num_pages) * 2 * p->kv_heads * kPage, HD, HD, kPage, 64);
  if (rc != NF_OK) return rc;
  if (dist) return p->head_dim == 64 ? launch_ws<64, true, false, true>(*p, tmQ, tmKV, stream) : launch_ws<128, true, false, true>(*p, tmQ, tmKV, stream);
  if (p->head_dim == 64) return cap ? launch_ws<64, true, true>(*p, tmQ, tmKV, stream) : launch_ws<64, true, false>(*p, tmQ, tmKV, stream);
  if (cap) return launch_ws<128, true, true>(*p, tmQ, tmKV, stream);
  return ext ? launch_ws<128, true, false>(*p, tmQ, tmKV, stream) : launch_ws<128, false, false>(*p, tmQ, tmKV, stream);
}
