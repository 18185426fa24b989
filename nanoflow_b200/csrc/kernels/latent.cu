// Latent attention: the cache holds one low-rank row per token, shared by all heads (see kernels.h for the
// pool layout).
//
// nfk_latent_append   RMS norm of a token's latent row, written to its page slot
// nfk_latent_gather   pages back to plain rows (for the expansion to keys and values)
// nfk_latent_attn     attention of listed tokens in latent space (queries already multiplied by their heads'
//                     key matrices, so the cached row is key and value at once), sliding window, sink.
//                     Used for decoding, for prompt tokens whose keys are not expanded, and in 32-bit.
//
// Two kernels for the attention. The tensor-core one (bf16): a CTA takes one token, 16 or 32 of its heads (the
// rows of its MMA tiles) and a range of keys; every latent row is fetched once for all those heads, in whole
// pages by TMA. Two groups of eight warps work on 16 heads each (or on alternate key tiles of the same heads),
// so that one group's softmax runs under the other's products. Per tile of 64 keys a group first splits the
// scores by (column quarter, half of the keys), with the warp's part of the queries in registers, then the
// softmax by row, then the output by column. Probabilities enter the second product as a bf16 pair (high and
// low part), which keeps them to about 16 bits. The simple one (bf16 or fp32, any size): one CTA per token and head.
#include "attn_mma.cuh"
#include "elem_io.cuh"

namespace nf {
namespace {

// ---- append ---------------------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(128)
latent_append_kernel(nfk_latent_append_params p) {
  const int lane = threadIdx.x & 31;
  // columns moved four at a time: all whole groups of four when every row starts on such a group
  const bool vec = p.ld_src % 4 == 0 && p.ld % 4 == 0 && (reinterpret_cast<uintptr_t>(p.src) & 15) == 0 &&
                   (reinterpret_cast<uintptr_t>(p.w) & 15) == 0 && (reinterpret_cast<uintptr_t>(p.pool) & 15) == 0;
  const int n4 = vec ? p.rank / 4 * 4 : 0;
  const bool tiled = latent_tiled(p.dtype, p.ld, p.page_size);
  for (int t = blockIdx.x * 4 + (threadIdx.x >> 5); t < p.T; t += gridDim.x * 4) {
    const T* src = reinterpret_cast<const T*>(p.src) + static_cast<long long>(t) * p.ld_src;
    const int pos = p.positions[t];
    const int page = page_of(pos, p.token_req[t], p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages,
                             p.status);
    float ss = 0.f;
    for (int c = lane * 4; c < n4; c += 128) {
      const float4 v = load4(src + c);
      ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
    for (int c = n4 + lane; c < p.rank; c += 32) {
      const float v = to_f32(src[c]);
      ss += v * v;
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(p.rank) + p.eps);
    if (page < 0) continue;
    T* pool = reinterpret_cast<T*>(p.pool);
    auto at = [&](int c) { return pool + latent_offset(page, pos % p.page_size, c, p.page_size, p.ld, tiled); };
    for (int c = lane * 4; c < n4; c += 128) {
      const float4 v = load4(src + c), w = load4(p.w + c);
      store4(at(c), make_float4(v.x * inv * w.x, v.y * inv * w.y, v.z * inv * w.z, v.w * inv * w.w));
    }
    for (int c = n4 + lane; c < p.rank; c += 32) put(at(c), to_f32(src[c]) * inv * p.w[c]);
  }
}

// ---- gather -----------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256)
latent_gather_kernel(nfk_latent_gather_params p, int elem_bytes) {
  const int per16 = 16 / elem_bytes, chunks = static_cast<int>(p.ld) / per16;
  const bool tiled = latent_tiled(p.dtype, p.ld, p.page_size);
  for (int i = blockIdx.x; i < p.n_pages; i += gridDim.x) {
    const int page = p.page_ids[i];
    if (page < 0 || page >= p.num_pages) {
      if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
      continue;
    }
    for (int k = threadIdx.x; k < p.page_size * chunks; k += blockDim.x) {
      const int r = k / chunks, ch = k % chunks;
      const long long src = latent_offset(page, r, ch * per16, p.page_size, p.ld, tiled);
      const long long dst = (static_cast<long long>(i) * p.page_size + r) * p.ld + ch * per16;
      *reinterpret_cast<uint4*>(reinterpret_cast<char*>(p.out) + dst * elem_bytes) =
          *reinterpret_cast<const uint4*>(reinterpret_cast<const char*>(p.pool) + src * elem_bytes);
    }
  }
}

// ---- simple kernel ----------------------------------------------------------------------------------
constexpr int kSimpleThreads = 128, kSimpleTile = 64, kSimpleCols = 16;   // up to 128 * 16 latent columns

template <class T>
__global__ void __launch_bounds__(kSimpleThreads)
latent_attn_simple_kernel(nfk_latent_attn_params p) {
  extern __shared__ float q_s[];                      // [ld]
  __shared__ float s_s[kSimpleTile];
  __shared__ int row_s[kSimpleTile];                  // page * page_size + row, or -1
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int ld = static_cast<int>(p.ld);
  const T* pool = reinterpret_cast<const T*>(p.pool);
  const int head = blockIdx.x % p.heads;
  const int tok = p.tokens[blockIdx.x / p.heads];
  const int pos = p.positions[tok], req = p.token_req[tok];
  const T* q = reinterpret_cast<const T*>(p.q) + static_cast<long long>(tok) * p.ld_q + static_cast<long long>(head) * ld;
  for (int c = threadIdx.x; c < ld; c += kSimpleThreads) q_s[c] = to_f32(q[c]);
  float acc[kSimpleCols];
#pragma unroll
  for (int i = 0; i < kSimpleCols; ++i) acc[i] = 0.f;
  float m = p.sinks != nullptr ? p.sinks[head] : -INFINITY, l = p.sinks != nullptr ? 1.f : 0.f;
  const bool tiled = latent_tiled(p.dtype, p.ld, p.page_size);
  auto at = [&](int k, int c) { return pool + latent_offset(row_s[k] / p.page_size, row_s[k] % p.page_size, c, p.page_size, ld, tiled); };
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  for (int j0 = lo; j0 <= pos; j0 += kSimpleTile) {
    const int n = min(kSimpleTile, pos + 1 - j0);
    __syncthreads();
    if (threadIdx.x < n) {
      const int j = j0 + threadIdx.x;
      const int page = page_of(j, req, p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages, p.status);
      row_s[threadIdx.x] = page < 0 ? -1 : page * p.page_size + j % p.page_size;
    }
    __syncthreads();
    for (int k = warp; k < n; k += kSimpleThreads / 32) {
      float d = 0.f;
      if (row_s[k] >= 0) {
        for (int i = lane; i < ld; i += 32) d += q_s[i] * to_f32(*at(k, i));
      }
      d = warp_sum(d);
      if (lane == 0) s_s[k] = row_s[k] >= 0 ? d * p.scale : -INFINITY;
    }
    __syncthreads();
    float mx = m;
    for (int k = 0; k < n; ++k) mx = fmaxf(mx, s_s[k]);
    if (mx == -INFINITY) continue;
    const float alpha = expf(m - mx);
    m = mx;
    l *= alpha;
#pragma unroll
    for (int i = 0; i < kSimpleCols; ++i) acc[i] *= alpha;
    for (int k = 0; k < n; ++k) {
      if (row_s[k] < 0) continue;
      const float w = expf(s_s[k] - m);
      l += w;
#pragma unroll
      for (int i = 0; i < kSimpleCols; ++i) {
        const int col = threadIdx.x + i * kSimpleThreads;
        if (col < ld) acc[i] += w * to_f32(*at(k, col));
      }
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* out = reinterpret_cast<T*>(p.out) + static_cast<long long>(tok) * p.ld_out + static_cast<long long>(head) * ld;
#pragma unroll
  for (int i = 0; i < kSimpleCols; ++i) {
    const int col = threadIdx.x + i * kSimpleThreads;
    if (col < ld) put(out + col, acc[i] * inv);
  }
}

// ---- tensor-core kernel -------------------------------------------------------------------------------
constexpr int kLTile = 64;
constexpr int kLGroup = 256, kLThreads = 2 * kLGroup;   // two groups of eight warps

template <int DW, bool KSPLIT>
struct LCfg {
  static constexpr int D = DW * 64;                       // latent columns
  static constexpr int ROWS = KSPLIT ? 16 : 32;           // heads per CTA, 16 per group
  static constexpr int TILE_BYTES = kLTile * D * 2;       // 128-byte swizzle, see key_off
  static constexpr int S_LD = kLTile + 8;
  static constexpr int S_BYTES = 4 * 16 * S_LD * 4;       // per group: score parts of the four column quarters
  static constexpr int P_BYTES = 16 * kLTile * 2;         // per group: one part (high or low)
  static constexpr int O_LD = D + 4;
  static constexpr int GROUP_BYTES = S_BYTES + 2 * P_BYTES + 2 * 16 * 4;
  static constexpr int FIXED = 2 * GROUP_BYTES + 128;
  static constexpr int STAGES = 4 * TILE_BYTES + FIXED <= 200 * 1024 ? 4 : (3 * TILE_BYTES + FIXED <= 200 * 1024 ? 3 : 2);
  static constexpr int SMEM = FIXED + STAGES * TILE_BYTES + 1024;
  static_assert(16 * O_LD * 4 <= STAGES * TILE_BYTES, "the merge of the two groups reuses the key tiles");
};

// Byte offset of 16-byte chunk `ch` of row `row` in a tile of `row_bytes`-byte rows.
__device__ __forceinline__ uint32_t sw_off(int row, int ch, int row_bytes) {
  return static_cast<uint32_t>(row * row_bytes + ((ch ^ (row & 7)) << 4));
}
// ... in a key tile: pages as the pool stores them, [8-key group][64-column block][8 keys][128 bytes].
template <int DW>
__device__ __forceinline__ uint32_t key_off(int key, int ch) {
  return static_cast<uint32_t>((key >> 3) * (DW * 1024) + (ch >> 3) * 1024 + (key & 7) * 128 + (((ch ^ key) & 7) << 4));
}
// A fragment (16 rows x 16 k) of a row-major tile.
__device__ __forceinline__ void load_a(uint32_t (&a)[4], uint32_t base, int row0, int ks, int row_bytes) {
  const int lane = threadIdx.x & 31;
  ldsm_x4(base + sw_off(row0 + (lane & 15), 2 * ks + (lane >> 4), row_bytes), a[0], a[1], a[2], a[3]);
}
__device__ __forceinline__ void group_sync(int g) { asm volatile("bar.sync %0, 256;" ::"r"(g + 1) : "memory"); }
// Count of the warps that are done with a key tile; orders their reads before what the last one does next.
__device__ __forceinline__ int count_done(uint32_t addr) {
  int old;
  asm volatile("atom.acq_rel.cta.shared::cta.add.s32 %0, [%1], 1;" : "=r"(old) : "r"(addr) : "memory");
  return old + 1;
}

// KSPLIT false: the groups take different heads (rows 0-15 and 16-31) over the same key tiles; true (at most 16
// heads): they take alternate key tiles and are merged at the end. Either way they only share the tiles, so
// one group's softmax runs under the other's products. The warp that is last to finish with a tile starts
// the copy of the tile that takes its place.
template <int DW, bool KSPLIT>
__global__ void __launch_bounds__(kLThreads, 1)
latent_attn_mma_kernel(const __grid_constant__ CUtensorMap tmC, nfk_latent_attn_params p) {
  using Cfg = LCfg<DW, KSPLIT>;
  constexpr int D = Cfg::D, ROWS = Cfg::ROWS;
  constexpr int kDone = KSPLIT ? kLGroup / 32 : kLThreads / 32;    // warps that read a tile
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t sb = smem_u32(smem);
  const int warp = (threadIdx.x >> 5) & 7, lane = threadIdx.x & 31, grp = threadIdx.x / kLGroup;
  uint8_t* fixed = smem + Cfg::STAGES * Cfg::TILE_BYTES;
  float* s_s = reinterpret_cast<float*>(fixed + grp * Cfg::GROUP_BYTES);
  uint8_t* p_ptr = fixed + grp * Cfg::GROUP_BYTES + Cfg::S_BYTES;
  const uint32_t p_hi = smem_u32(p_ptr), p_lo = p_hi + Cfg::P_BYTES;
  float* alpha_s = reinterpret_cast<float*>(p_ptr + 2 * Cfg::P_BYTES);
  float* l_s = alpha_s + 16;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(fixed + 2 * Cfg::GROUP_BYTES);
  int* done_s = reinterpret_cast<int*>(full_bar + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(done_s + 4);
  const int hgroups = (p.heads + ROWS - 1) / ROWS;
  const int hg = blockIdx.x % hgroups;
  const int split = (blockIdx.x / hgroups) % p.splits;
  const int ti = blockIdx.x / (hgroups * p.splits);
  const int tok = p.tokens[ti];
  const int pos = p.positions[tok], req = p.token_req[tok];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int key0 = lo / kPage * kPage;                         // tiles start on a page
  const int n_all = (pos - key0) / kLTile + 1;
  const int per = (n_all + p.splits - 1) / p.splits;
  const int t_begin = min(n_all, split * per), n_tiles = min(n_all, t_begin + per) - t_begin;
  const int head0 = hg * ROWS + (KSPLIT ? 0 : grp * 16);       // first head of this group

  if (threadIdx.x == 0) {
    for (int s = 0; s < Cfg::STAGES; ++s) {
      mbar_init(&full_bar[s], 1);
      done_s[s] = 0;
    }
    *abort_flag = 0;
    mbar_fence_init();
    tma_prefetch_desc(&tmC);
  }
  __syncthreads();

  // ---- copies: whole pages, lanes 0-3 one page of the tile each ----
  const int pg0 = p.kv_indptr[req], np = p.kv_indptr[req + 1] - pg0;
  const int first = p.kv_first != nullptr ? p.kv_first[req] : 0;
  auto page_at = [&](int t) {
    // past the last key: the last page again, masked by position
    const int slot = min((key0 + (t_begin + t) * kLTile) / kPage + lane, pos / kPage) - first;
    return (slot >= 0 && slot < np) ? p.kv_indices[pg0 + slot] : -1;    // looked at when the copy starts, not before
  };
  auto copy_tile = [&](int t, int page) {       // one whole warp
    const int s = t % Cfg::STAGES;
    if (page < 0 || page >= p.num_pages) {
      report_status(p.status, NF_ST_BAD_INDEX);
      page = 0;
    }
    if (lane == 0) mbar_expect_tx(&full_bar[s], Cfg::TILE_BYTES);
    __syncwarp();
    if (lane < 4) {
      tma_load_2d(smem + s * Cfg::TILE_BYTES + lane * (kPage * D * 2), &tmC, &full_bar[s], 0, page * (kPage * DW));
    }
  };
  if (threadIdx.x < 32) {
    for (int t = 0; t < min(n_tiles, Cfg::STAGES); ++t) copy_tile(t, lane < 4 ? page_at(t) : 0);
  }

  // ---- scores by (column quarter, key half), softmax by row, output by column ----
  const int kq = warp >> 1, kh = warp & 1;
  uint32_t qa[DW][4];                                          // this quarter's columns of the group's rows
  {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(tok) * p.ld_q;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int head = head0 + half * 8 + (lane >> 2);
      const __nv_bfloat16* row = q + static_cast<long long>(head) * D + kq * (DW * 16) + (lane & 3) * 2;
#pragma unroll
      for (int ks = 0; ks < DW; ++ks) {
        qa[ks][half] = head < p.heads ? *reinterpret_cast<const uint32_t*>(row + ks * 16) : 0u;
        qa[ks][half + 2] = head < p.heads ? *reinterpret_cast<const uint32_t*>(row + ks * 16 + 8) : 0u;
      }
    }
  }
  float o[DW][4];
#pragma unroll
  for (int b = 0; b < DW; ++b) o[b][0] = o[b][1] = o[b][2] = o[b][3] = 0.f;
  const int row_r = warp * 2 + (lane >> 4);                    // softmax row of this half warp
  float m_r = -INFINITY, l_r = 0.f;
  {
    const int head = head0 + row_r;
    if (p.sinks != nullptr && head < p.heads && split == 0 && !(KSPLIT && grp == 1)) {
      m_r = p.sinks[head] * kLog2e;
      l_r = (lane & 15) == 0 ? 1.f : 0.f;
    }
  }
  const float scale = p.scale * kLog2e;
  const int mm = lane >> 3, rr = lane & 7;

  for (int t = KSPLIT ? grp : 0; t < n_tiles; t += KSPLIT ? 2 : 1) {
    const int s = t % Cfg::STAGES;
    const uint32_t st = sb + s * Cfg::TILE_BYTES;
    // page of the tile that will take this one's place, in case this warp is the one to copy it
    const int page = (lane < 4 && t + Cfg::STAGES < n_tiles) ? page_at(t + Cfg::STAGES) : 0;
    // a wait that runs out is reported; the warps go on in step, so that they meet at their barriers
    if (*abort_flag == 0 && !mbar_wait(&full_bar[s], (t / Cfg::STAGES) & 1)) {
      if (lane == 0) report_status(p.status, NF_ST_TIMEOUT_SMEM_FULL);
      *abort_flag = 1;
    }
    __syncwarp();
    // 1. scores of 32 keys over a quarter of the columns
    {
      float sc[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j) sc[j][0] = sc[j][1] = sc[j][2] = sc[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < DW; ++ks) {
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          uint32_t b0, b1, b2, b3;
          ldsm_x4(st + key_off<DW>(kh * 32 + g * 16 + (mm >> 1) * 8 + rr, (kq * DW + ks) * 2 + (mm & 1)), b0, b1, b2, b3);
          mma_bf16(sc[2 * g], qa[ks], b0, b1);
          mma_bf16(sc[2 * g + 1], qa[ks], b2, b3);
        }
      }
      float* dst = s_s + (kq * 16 + (lane >> 2)) * Cfg::S_LD + kh * 32 + (lane & 3) * 2;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        *reinterpret_cast<float2*>(dst + j * 8) = make_float2(sc[j][0], sc[j][1]);
        *reinterpret_cast<float2*>(dst + 8 * Cfg::S_LD + j * 8) = make_float2(sc[j][2], sc[j][3]);
      }
    }
    group_sync(grp);
    // 2. softmax of this warp's two rows: half a warp per row, four keys per lane
    {
      const int key = key0 + (t_begin + t) * kLTile + (lane & 15) * 4;
      const float* src = s_s + row_r * Cfg::S_LD + (lane & 15) * 4;
      float4 v = *reinterpret_cast<const float4*>(src);
#pragma unroll
      for (int k = 1; k < 4; ++k) {
        const float4 w = *reinterpret_cast<const float4*>(src + k * 16 * Cfg::S_LD);
        v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
      }
      v.x = (key >= lo && key <= pos) ? v.x * scale : -INFINITY;
      v.y = (key + 1 >= lo && key + 1 <= pos) ? v.y * scale : -INFINITY;
      v.z = (key + 2 >= lo && key + 2 <= pos) ? v.z * scale : -INFINITY;
      v.w = (key + 3 >= lo && key + 3 <= pos) ? v.w * scale : -INFINITY;
      float mx = fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w));
#pragma unroll
      for (int off = 8; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
      const float mn = fmaxf(m_r, mx);
      const float ms = mn == -INFINITY ? 0.f : mn;
      const float al = fast_exp2(m_r - ms);
      m_r = mn;
      const float e0 = fast_exp2(v.x - ms), e1 = fast_exp2(v.y - ms), e2 = fast_exp2(v.z - ms), e3 = fast_exp2(v.w - ms);
      l_r = l_r * al + ((e0 + e1) + (e2 + e3));      // this lane's keys; the row's lanes are added up at the end
      const uint32_t h0 = pack_bf16x2(e0, e1), h1 = pack_bf16x2(e2, e3);
      const float2 f0 = unpack_bf16x2(h0), f1 = unpack_bf16x2(h1);
      const uint32_t off = sw_off(row_r, (lane & 15) >> 1, kLTile * 2) + (lane & 1) * 8;
      *reinterpret_cast<uint2*>(p_ptr + off) = make_uint2(h0, h1);
      *reinterpret_cast<uint2*>(p_ptr + Cfg::P_BYTES + off) =
          make_uint2(pack_bf16x2(e0 - f0.x, e1 - f0.y), pack_bf16x2(e2 - f1.x, e3 - f1.y));
      if ((lane & 15) == 0) alpha_s[row_r] = al;
    }
    group_sync(grp);
    // 3. output: DW * 8 columns per warp
    {
      const float al0 = alpha_s[lane >> 2], al1 = alpha_s[8 + (lane >> 2)];
      if (__any_sync(0xffffffffu, al0 != 1.f || al1 != 1.f)) {
#pragma unroll
        for (int b = 0; b < DW; ++b) {
          o[b][0] *= al0; o[b][1] *= al0; o[b][2] *= al1; o[b][3] *= al1;
        }
      }
    }
#pragma unroll
    for (int ks = 0; ks < kLTile / 16; ++ks) {
      uint32_t ph[4], pl[4];
      load_a(ph, p_hi, 0, ks, kLTile * 2);
      load_a(pl, p_lo, 0, ks, kLTile * 2);
      const int key = ks * 16 + (mm & 1) * 8 + rr;
#pragma unroll
      for (int b = 0; b < DW; b += 2) {
        const int ch = min(warp * DW + b + (mm >> 1), D / 8 - 1);   // odd DW: the second half is not used
        uint32_t b0, b1, b2, b3;
        ldsm_x4_trans(st + key_off<DW>(key, ch), b0, b1, b2, b3);
        mma_bf16(o[b], ph, b0, b1);
        if (b + 1 < DW) mma_bf16(o[b + 1 < DW ? b + 1 : b], ph, b2, b3);
        mma_bf16(o[b], pl, b0, b1);
        if (b + 1 < DW) mma_bf16(o[b + 1 < DW ? b + 1 : b], pl, b2, b3);
      }
    }
    __syncwarp();
    int last = 0;
    if (lane == 0) {
      last = count_done(smem_u32(&done_s[s])) == kDone;
      if (last) done_s[s] = 0;
    }
    if (__shfl_sync(0xffffffffu, last, 0) != 0 && t + Cfg::STAGES < n_tiles) copy_tile(t + Cfg::STAGES, page);
  }
  if (*abort_flag != 0 && threadIdx.x == 0) {
    // a wait ran out: give copies still in flight a bounded chance to land before the CTA ends
    for (int t = max(0, n_tiles - Cfg::STAGES); t < n_tiles; ++t) (void)mbar_wait(&full_bar[t % Cfg::STAGES], (t / Cfg::STAGES) & 1);
  }
  // row sums and reference maxima to every warp of the group
#pragma unroll
  for (int off = 8; off > 0; off >>= 1) l_r += __shfl_xor_sync(0xffffffffu, l_r, off);
  group_sync(grp);            // the last tile's rescaling factors have been read
  if ((lane & 15) == 0) {
    l_s[row_r] = l_r;
    alpha_s[row_r] = m_r;
  }
  if (KSPLIT) {
    // merge: group 1 leaves its output over the key tiles, group 0 brings both to the larger maximum
    __syncthreads();
    float* mo = reinterpret_cast<float*>(smem);
    const float* other_m = reinterpret_cast<const float*>(fixed + Cfg::GROUP_BYTES + Cfg::S_BYTES + 2 * Cfg::P_BYTES);
    const int c0 = warp * DW * 8 + (lane & 3) * 2;
    if (grp == 1) {
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int b = 0; b < DW; ++b)
          *reinterpret_cast<float2*>(mo + (half * 8 + (lane >> 2)) * Cfg::O_LD + c0 + b * 8) = make_float2(o[b][2 * half], o[b][2 * half + 1]);
    }
    __syncthreads();
    if (grp == 1) return;
    float ms[2], f0[2], f1[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = half * 8 + (lane >> 2);
      const float m0 = alpha_s[row], m1 = other_m[row];
      ms[half] = fmaxf(m0, m1);
      const float msafe = ms[half] == -INFINITY ? 0.f : ms[half];
      f0[half] = fast_exp2(m0 - msafe);
      f1[half] = fast_exp2(m1 - msafe);
#pragma unroll
      for (int b = 0; b < DW; ++b) {
        const float2 v = *reinterpret_cast<const float2*>(mo + row * Cfg::O_LD + c0 + b * 8);
        o[b][2 * half] = o[b][2 * half] * f0[half] + v.x * f1[half];
        o[b][2 * half + 1] = o[b][2 * half + 1] * f0[half] + v.y * f1[half];
      }
    }
    float l[2];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = half * 8 + (lane >> 2);
      l[half] = l_s[row] * f0[half] + other_m[16 + row] * f1[half];
    }
    group_sync(0);            // everyone has read the maxima and sums
    if (warp == 0 && (lane & 3) == 0) {
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        l_s[half * 8 + (lane >> 2)] = l[half];
        alpha_s[half * 8 + (lane >> 2)] = ms[half];
      }
    }
  }
  group_sync(grp);
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int row = half * 8 + (lane >> 2), head = head0 + row;
    if (head >= p.heads) continue;
    const float l = l_s[row], inv = l > 0.f ? 1.f / l : 0.f;
    const int c0 = warp * DW * 8 + (lane & 3) * 2;
    if (p.splits == 1) {
      __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(tok) * p.ld_out +
                           static_cast<long long>(head) * D;
#pragma unroll
      for (int b = 0; b < DW; ++b)
        *reinterpret_cast<uint32_t*>(dst + c0 + b * 8) = pack_bf16x2(o[b][2 * half] * inv, o[b][2 * half + 1] * inv);
    } else {
      float* ws = p.workspace + ((static_cast<long long>(ti) * p.splits + split) * p.heads + head) * (D + 2);
#pragma unroll
      for (int b = 0; b < DW; ++b)
        *reinterpret_cast<float2*>(ws + c0 + b * 8) = make_float2(o[b][2 * half], o[b][2 * half + 1]);
      if (warp == 0 && (lane & 3) == 0) {
        ws[D] = alpha_s[row];
        ws[D + 1] = l;
      }
    }
  }
}

__global__ void __launch_bounds__(128)
latent_attn_merge_kernel(nfk_latent_attn_params p) {
  const int head = blockIdx.x % p.heads, ti = blockIdx.x / p.heads;
  const int D = static_cast<int>(p.ld);
  const float* ws = p.workspace + (static_cast<long long>(ti) * p.splits * p.heads + head) * (D + 2);
  const long long step = static_cast<long long>(p.heads) * (D + 2);
  float m = -INFINITY, l = 0.f;
  for (int s = 0; s < p.splits; ++s) m = fmaxf(m, ws[s * step + D]);
  const float ms = m == -INFINITY ? 0.f : m;
  for (int s = 0; s < p.splits; ++s) l += ws[s * step + D + 1] * fast_exp2(ws[s * step + D] - ms);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  const int tok = p.tokens[ti];
  __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(tok) * p.ld_out +
                       static_cast<long long>(head) * D;
  for (int c = threadIdx.x * 2; c < D; c += 256) {
    float x = 0.f, y = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float w = fast_exp2(ws[s * step + D] - ms);
      const float2 v = *reinterpret_cast<const float2*>(ws + s * step + c);
      x += v.x * w;
      y += v.y * w;
    }
    *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(x * inv, y * inv);
  }
}

template <int DW, bool KSPLIT>
int launch_latent(const nfk_latent_attn_params& p, cudaStream_t stream) {
  using Cfg = LCfg<DW, KSPLIT>;
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    if (cudaFuncSetAttribute(latent_attn_mma_kernel<DW, KSPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM) !=
        cudaSuccess)
      return NF_ERR_CUDA;
    attr = true;
  }
  CUtensorMap tm;
  const int rc = make_tmap_bf16_2d(&tm, p.pool, static_cast<uint64_t>(p.num_pages) * kPage * DW, 64, 64, kPage * DW, 64);
  if (rc != NF_OK) return rc;
  const int hgroups = (p.heads + Cfg::ROWS - 1) / Cfg::ROWS;
  const long long grid = static_cast<long long>(p.n_tokens) * p.splits * hgroups;
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  latent_attn_mma_kernel<DW, KSPLIT><<<static_cast<int>(grid), kLThreads, Cfg::SMEM, stream>>>(tm, p);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  if (p.splits > 1) {
    latent_attn_merge_kernel<<<p.n_tokens * p.heads, 128, 0, stream>>>(p);
    if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  }
  return NF_OK;
}
template <int DW>
int launch_latent_mt(const nfk_latent_attn_params& p, cudaStream_t stream) {
  return p.heads <= 16 ? launch_latent<DW, true>(p, stream) : launch_latent<DW, false>(p, stream);
}

bool mma_ok(const nfk_latent_attn_params& p) {
  const bool size = p.ld == 64 || p.ld == 128 || p.ld == 192 || p.ld == 256 || p.ld == 384 || p.ld == 512;
  return p.dtype == NFK_BF16 && size && p.page_size == kPage && p.ld_q % 8 == 0 && p.ld_out % 2 == 0 &&
         (reinterpret_cast<uintptr_t>(p.q) & 15) == 0 && (reinterpret_cast<uintptr_t>(p.pool) & 15) == 0;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_latent_append(const nfk_latent_append_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == 0) return NF_OK;
  if (!p->src || !p->w || !p->pool || !p->positions || !p->token_req || !p->kv_indptr || !p->kv_indices || p->T < 0 ||
      p->rank <= 0 || p->ld < p->rank || p->page_size <= 0 || p->num_pages <= 0)
    return NF_ERR_BAD_ARG;
  int grid = (p->T + 3) / 4;
  if (grid > 16 * device_sm_count()) grid = 16 * device_sm_count();
  if (p->dtype == NFK_F32) latent_append_kernel<float><<<grid, 128, 0, stream>>>(*p);
  else latent_append_kernel<__nv_bfloat16><<<grid, 128, 0, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_latent_gather(const nfk_latent_gather_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->n_pages == 0) return NF_OK;
  const int es = p->dtype == NFK_F32 ? 4 : 2;
  if (!p->pool || !p->out || !p->page_ids || p->n_pages < 0 || p->page_size <= 0 || p->num_pages <= 0 || p->ld <= 0 ||
      p->ld * es % 16 != 0 || (reinterpret_cast<uintptr_t>(p->pool) & 15) != 0 || (reinterpret_cast<uintptr_t>(p->out) & 15) != 0)
    return NF_ERR_BAD_ARG;
  int grid = 8 * device_sm_count();
  if (grid > p->n_pages) grid = p->n_pages;
  latent_gather_kernel<<<grid, 256, 0, stream>>>(*p, es);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_latent_attn(const nfk_latent_attn_params* pp, cudaStream_t stream) {
  using namespace nf;
  if (pp == nullptr) return NF_ERR_BAD_ARG;
  nfk_latent_attn_params p = *pp;
  if (p.n_tokens == 0) return NF_OK;
  if (!p.q || !p.pool || !p.out || !p.tokens || !p.positions || !p.token_req || !p.kv_indptr || !p.kv_indices ||
      p.n_tokens < 0 || p.heads <= 0 || p.ld <= 0 || p.ld > kSimpleThreads * kSimpleCols || p.page_size <= 0 ||
      p.num_pages <= 0 || p.window < 0)
    return NF_ERR_BAD_ARG;
  if (p.splits < 1) p.splits = 1;
  if (p.impl < 0 || p.impl > 2) return NF_ERR_BAD_ARG;
  if (p.impl == 2 && !mma_ok(p)) return NF_ERR_UNSUPPORTED;
  if (p.impl != 1 && mma_ok(p)) {
    if (p.splits > 1 && (p.workspace == nullptr || static_cast<long long>(p.n_tokens) * p.splits * p.heads * (p.ld + 2) >
                                                       p.workspace_floats))
      p.splits = 1;
    switch (p.ld / 64) {
      case 1: return launch_latent_mt<1>(p, stream);
      case 2: return launch_latent_mt<2>(p, stream);
      case 3: return launch_latent_mt<3>(p, stream);
      case 4: return launch_latent_mt<4>(p, stream);
      case 6: return launch_latent_mt<6>(p, stream);
      default: return launch_latent_mt<8>(p, stream);
    }
  }
  const long long grid = static_cast<long long>(p.n_tokens) * p.heads;
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  const size_t sm = static_cast<size_t>(p.ld) * 4;
  if (p.dtype == NFK_F32)
    latent_attn_simple_kernel<float><<<static_cast<int>(grid), kSimpleThreads, sm, stream>>>(p);
  else
    latent_attn_simple_kernel<__nv_bfloat16><<<static_cast<int>(grid), kSimpleThreads, sm, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}
