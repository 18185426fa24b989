// Latent attention: the cache holds one low-rank row per token, shared by all heads (see kernels.h for the
// pool layout).
//
// nfk_latent_append   RMS norm of a token's latent row, written to its page slot
// nfk_latent_attn     attention of listed tokens in latent space (queries already multiplied by their heads'
//                     key matrices, so the cached row is key and value at once), sliding window, sink.
//                     Used for decoding, for prompt tokens whose keys are not expanded, and in 32-bit.
//
// Two kernels for the attention. The tensor-core one (bf16): a CTA takes one token, 16 or 32 of its heads (the
// rows of its MMA tiles) and a range of keys; every latent row is fetched once for all those heads. Per tile
// of 64 keys the eight warps first split the scores by key, then the softmax by row, then the output by
// column; probabilities enter the second product as a bf16 pair (high and low part), which keeps them to about
// 16 bits. The simple one (bf16 or fp32, any size): one CTA per token and head.
#include "attn_mma.cuh"
#include "elem_io.cuh"

namespace nf {
namespace {

// ---- append ---------------------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(128)
latent_append_kernel(nfk_latent_append_params p) {
  const int lane = threadIdx.x & 31;
  for (int t = blockIdx.x * 4 + (threadIdx.x >> 5); t < p.T; t += gridDim.x * 4) {
    const T* src = reinterpret_cast<const T*>(p.src) + static_cast<long long>(t) * p.ld_src;
    float ss = 0.f;
    for (int c = lane; c < p.rank; c += 32) {
      const float v = to_f32(src[c]);
      ss += v * v;
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(p.rank) + p.eps);
    const int pos = p.positions[t];
    const int page = page_of(pos, p.token_req[t], p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages,
                             p.status);
    if (page < 0) continue;
    T* dst = reinterpret_cast<T*>(p.pool) + (static_cast<long long>(page) * p.page_size + pos % p.page_size) * p.ld;
    for (int c = lane; c < p.rank; c += 32) put(dst + c, to_f32(src[c]) * inv * p.w[c]);
  }
}

// ---- simple kernel ----------------------------------------------------------------------------------
constexpr int kSimpleThreads = 128, kSimpleTile = 64, kSimpleCols = 16;   // up to 128 * 16 latent columns

template <class T>
__global__ void __launch_bounds__(kSimpleThreads)
latent_attn_simple_kernel(nfk_latent_attn_params p) {
  extern __shared__ float q_s[];                      // [ld]
  __shared__ float s_s[kSimpleTile];
  __shared__ int row_s[kSimpleTile];
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
        const T* c = pool + static_cast<long long>(row_s[k]) * ld;
        for (int i = lane; i < ld; i += 32) d += q_s[i] * to_f32(c[i]);
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
      const T* c = pool + static_cast<long long>(row_s[k]) * ld;
#pragma unroll
      for (int i = 0; i < kSimpleCols; ++i) {
        const int col = threadIdx.x + i * kSimpleThreads;
        if (col < ld) acc[i] += w * to_f32(c[col]);
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
constexpr int kLThreads = 256, kLTile = 64;

template <int DW, int MT>
struct LCfg {
  static constexpr int D = DW * 64;                       // latent columns
  static constexpr int ROWS = MT * 16;
  static constexpr int TILE_BYTES = kLTile * D * 2;
  static constexpr int Q_BYTES = ROWS * D * 2;
  static constexpr int S_LD = kLTile + 4;
  static constexpr int S_BYTES = ROWS * S_LD * 4;
  static constexpr int P_BYTES = ROWS * kLTile * 2;       // one part (high or low)
  static constexpr int FIXED = Q_BYTES + S_BYTES + 2 * P_BYTES + 2 * ROWS * 4;
  static constexpr int STAGES = 3 * TILE_BYTES + FIXED <= 110 * 1024 ? 3 : 2;
  static constexpr int SMEM = FIXED + STAGES * TILE_BYTES;
};

// Byte offset of 16-byte chunk `ch` of row `row` in a tile of `row_bytes`-byte rows.
__device__ __forceinline__ uint32_t sw_off(int row, int ch, int row_bytes) {
  return static_cast<uint32_t>(row * row_bytes + ((ch ^ (row & 7)) << 4));
}
// A fragment (16 rows x 16 k) of a row-major tile.
__device__ __forceinline__ void load_a(uint32_t (&a)[4], uint32_t base, int row0, int ks, int row_bytes) {
  const int lane = threadIdx.x & 31;
  ldsm_x4(base + sw_off(row0 + (lane & 15), 2 * ks + (lane >> 4), row_bytes), a[0], a[1], a[2], a[3]);
}

template <int DW, int MT>
__global__ void __launch_bounds__(kLThreads, 1)
latent_attn_mma_kernel(nfk_latent_attn_params p) {
  using Cfg = LCfg<DW, MT>;
  constexpr int D = Cfg::D, ROWS = Cfg::ROWS;
  extern __shared__ __align__(128) uint8_t smem[];
  const uint32_t sb = smem_u32(smem);
  const uint32_t q_base = sb + Cfg::STAGES * Cfg::TILE_BYTES;
  float* s_s = reinterpret_cast<float*>(smem + Cfg::STAGES * Cfg::TILE_BYTES + Cfg::Q_BYTES);
  const uint32_t p_hi = q_base + Cfg::Q_BYTES + Cfg::S_BYTES, p_lo = p_hi + Cfg::P_BYTES;
  uint8_t* p_ptr = smem + Cfg::STAGES * Cfg::TILE_BYTES + Cfg::Q_BYTES + Cfg::S_BYTES;
  float* alpha_s = reinterpret_cast<float*>(p_ptr + 2 * Cfg::P_BYTES);
  float* l_s = alpha_s + ROWS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hgroups = (p.heads + ROWS - 1) / ROWS;
  const int hg = blockIdx.x % hgroups;
  const int split = (blockIdx.x / hgroups) % p.splits;
  const int ti = blockIdx.x / (hgroups * p.splits);
  const int tok = p.tokens[ti];
  const int pos = p.positions[tok], req = p.token_req[tok];
  const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(p.pool);
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int key0 = lo / kPage * kPage;                         // tiles start on a page
  const int n_all = (pos - key0) / kLTile + 1;
  const int per = (n_all + p.splits - 1) / p.splits;
  const int t_begin = split * per, t_end = min(n_all, t_begin + per);
  const int pg0 = p.kv_indptr[req], np = p.kv_indptr[req + 1] - pg0;
  const int first = p.kv_first != nullptr ? p.kv_first[req] : 0;

  // queries of this CTA's heads (rows past the last head are zero)
  for (int i = threadIdx.x; i < ROWS * (D / 8); i += kLThreads) {
    const int r = i / (D / 8), ch = i % (D / 8), head = hg * ROWS + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (head < p.heads)
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p.q) +
                                          static_cast<long long>(tok) * p.ld_q + static_cast<long long>(head) * D + ch * 8);
    *reinterpret_cast<uint4*>(smem + Cfg::STAGES * Cfg::TILE_BYTES + sw_off(r, ch, D * 2)) = v;
  }
  auto issue = [&](int t) {
    if (t < t_end) {
      const uint32_t st = sb + ((t - t_begin) % Cfg::STAGES) * Cfg::TILE_BYTES;
#pragma unroll
      for (int j = 0; j < kLTile * (D / 8) / kLThreads; ++j) {
        const int idx = threadIdx.x + kLThreads * j;
        const int row = idx / (D / 8), ch = idx % (D / 8);
        const int key = min(key0 + t * kLTile + row, pos);     // past the last key: any valid row, masked below
        int slot = key / kPage - first;
        if (slot < 0 || slot >= np) {
          report_status(p.status, NF_ST_BAD_INDEX);
          slot = 0;
        }
        int page = p.kv_indices[pg0 + slot];
        if (page < 0 || page >= p.num_pages) {
          report_status(p.status, NF_ST_BAD_INDEX);
          page = 0;
        }
        cp_async16(st + sw_off(row, ch, D * 2),
                   pool + (static_cast<long long>(page) * kPage + key % kPage) * D + ch * 8);
      }
    }
    cp_async_commit();
  };
#pragma unroll
  for (int s = 0; s < Cfg::STAGES - 1; ++s) issue(t_begin + s);

  float o[MT][DW][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int b = 0; b < DW; ++b) o[a][b][0] = o[a][b][1] = o[a][b][2] = o[a][b][3] = 0.f;
  // softmax rows of this warp: 2 * MT of them, state replicated in its lanes
  constexpr int RW = ROWS / 8;
  float m_r[RW], l_r[RW];
#pragma unroll
  for (int r = 0; r < RW; ++r) {
    const int head = hg * ROWS + warp * RW + r;
    const bool sink = p.sinks != nullptr && head < p.heads && split == 0;
    m_r[r] = sink ? p.sinks[head] * kLog2e : -INFINITY;
    l_r[r] = sink ? 1.f : 0.f;
  }
  const float scale = p.scale * kLog2e;

  for (int t = t_begin; t < t_end; ++t) {
    cp_async_wait<Cfg::STAGES - 2>();
    __syncthreads();           // tile t is in shared memory, every warp is done with tile t - 1
    issue(t + Cfg::STAGES - 1);
    const uint32_t st = sb + ((t - t_begin) % Cfg::STAGES) * Cfg::TILE_BYTES;
    // 1. scores: MT = 2: 16 keys x one row tile per warp; MT = 1: 8 keys per warp
    {
      const int mt = MT == 2 ? (warp & 1) : 0;
      const int k0 = MT == 2 ? (warp >> 1) * 16 : warp * 8;
      float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
      const int mm = lane >> 3, rr = lane & 7;
#pragma unroll 4
      for (int ks = 0; ks < D / 16; ks += 2) {
        uint32_t a0[4], a1[4], b0, b1, b2, b3;
        load_a(a0, q_base, mt * 16, ks, D * 2);
        load_a(a1, q_base, mt * 16, ks + 1, D * 2);
        if (MT == 2) {
          ldsm_x4(st + sw_off(k0 + (mm >> 1) * 8 + rr, 2 * ks + (mm & 1), D * 2), b0, b1, b2, b3);
          mma_bf16(s0, a0, b0, b1);
          mma_bf16(s1, a0, b2, b3);
          ldsm_x4(st + sw_off(k0 + (mm >> 1) * 8 + rr, 2 * ks + 2 + (mm & 1), D * 2), b0, b1, b2, b3);
          mma_bf16(s0, a1, b0, b1);
          mma_bf16(s1, a1, b2, b3);
        } else {
          ldsm_x4(st + sw_off(k0 + rr, 2 * ks + mm, D * 2), b0, b1, b2, b3);
          mma_bf16(s0, a0, b0, b1);
          mma_bf16(s0, a1, b2, b3);
        }
      }
      const int r0 = mt * 16 + (lane >> 2), c0 = k0 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(s_s + r0 * Cfg::S_LD + c0) = make_float2(s0[0], s0[1]);
      *reinterpret_cast<float2*>(s_s + (r0 + 8) * Cfg::S_LD + c0) = make_float2(s0[2], s0[3]);
      if (MT == 2) {
        *reinterpret_cast<float2*>(s_s + r0 * Cfg::S_LD + c0 + 8) = make_float2(s1[0], s1[1]);
        *reinterpret_cast<float2*>(s_s + (r0 + 8) * Cfg::S_LD + c0 + 8) = make_float2(s1[2], s1[3]);
      }
    }
    __syncthreads();
    // 2. softmax of this warp's rows, two keys per lane
    {
      const int key = key0 + t * kLTile + lane * 2;
      const bool in0 = key >= lo && key <= pos, in1 = key + 1 >= lo && key + 1 <= pos;
#pragma unroll
      for (int r = 0; r < RW; ++r) {
        const int row = warp * RW + r;
        const float2 s = *reinterpret_cast<const float2*>(s_s + row * Cfg::S_LD + lane * 2);
        const float x0 = in0 ? s.x * scale : -INFINITY, x1 = in1 ? s.y * scale : -INFINITY;
        float mx = fmaxf(x0, x1);
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, off));
        const float mn = fmaxf(m_r[r], mx);
        const float ms = mn == -INFINITY ? 0.f : mn;
        const float al = exp2f(m_r[r] - ms);
        m_r[r] = mn;
        const float e0 = exp2f(x0 - ms), e1 = exp2f(x1 - ms);
        l_r[r] = l_r[r] * al + warp_sum(e0 + e1);
        const uint32_t hi = pack_bf16x2(e0, e1);
        const float2 hf = unpack_bf16x2(hi);
        const uint32_t off = sw_off(row, lane >> 2, kLTile * 2) + (lane & 3) * 4;
        *reinterpret_cast<uint32_t*>(p_ptr + off) = hi;
        *reinterpret_cast<uint32_t*>(p_ptr + Cfg::P_BYTES + off) = pack_bf16x2(e0 - hf.x, e1 - hf.y);
        if (lane == 0) alpha_s[row] = al;
      }
    }
    __syncthreads();
    // 3. output: DW * 8 columns per warp
    {
      const int mm = lane >> 3, rr = lane & 7;
#pragma unroll
      for (int a = 0; a < MT; ++a) {
        const float al0 = alpha_s[a * 16 + (lane >> 2)], al1 = alpha_s[a * 16 + 8 + (lane >> 2)];
#pragma unroll
        for (int b = 0; b < DW; ++b) {
          o[a][b][0] *= al0; o[a][b][1] *= al0; o[a][b][2] *= al1; o[a][b][3] *= al1;
        }
      }
#pragma unroll
      for (int ks = 0; ks < kLTile / 16; ++ks) {
        uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
        for (int a = 0; a < MT; ++a) {
          load_a(ph[a], p_hi, a * 16, ks, kLTile * 2);
          load_a(pl[a], p_lo, a * 16, ks, kLTile * 2);
        }
        const int key = ks * 16 + (mm & 1) * 8 + rr;
#pragma unroll
        for (int b = 0; b < DW; b += 2) {
          const int ch = min(warp * DW + b + (mm >> 1), D / 8 - 1);   // odd DW: the second half is not used
          uint32_t b0, b1, b2, b3;
          ldsm_x4_trans(st + sw_off(key, ch, D * 2), b0, b1, b2, b3);
#pragma unroll
          for (int a = 0; a < MT; ++a) {
            mma_bf16(o[a][b], ph[a], b0, b1);
            mma_bf16(o[a][b], pl[a], b0, b1);
            if (b + 1 < DW) {
              mma_bf16(o[a][b + 1 < DW ? b + 1 : b], ph[a], b2, b3);
              mma_bf16(o[a][b + 1 < DW ? b + 1 : b], pl[a], b2, b3);
            }
          }
        }
      }
    }
  }
  cp_async_wait<0>();
  // row sums (and reference maxima, for the merge) to every warp
  __syncthreads();
  if (lane == 0) {
#pragma unroll
    for (int r = 0; r < RW; ++r) {
      l_s[warp * RW + r] = l_r[r];
      alpha_s[warp * RW + r] = m_r[r];
    }
  }
  __syncthreads();
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int row = a * 16 + half * 8 + (lane >> 2), head = hg * ROWS + row;
      if (head >= p.heads) continue;
      const float l = l_s[row], inv = l > 0.f ? 1.f / l : 0.f;
      const int c0 = warp * DW * 8 + (lane & 3) * 2;
      if (p.splits == 1) {
        __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(tok) * p.ld_out +
                             static_cast<long long>(head) * D;
#pragma unroll
        for (int b = 0; b < DW; ++b)
          *reinterpret_cast<uint32_t*>(dst + c0 + b * 8) = pack_bf16x2(o[a][b][2 * half] * inv, o[a][b][2 * half + 1] * inv);
      } else {
        float* ws = p.workspace + ((static_cast<long long>(ti) * p.splits + split) * p.heads + head) * (D + 2);
#pragma unroll
        for (int b = 0; b < DW; ++b)
          *reinterpret_cast<float2*>(ws + c0 + b * 8) = make_float2(o[a][b][2 * half], o[a][b][2 * half + 1]);
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
  for (int s = 0; s < p.splits; ++s) l += ws[s * step + D + 1] * exp2f(ws[s * step + D] - ms);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  const int tok = p.tokens[ti];
  __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(tok) * p.ld_out +
                       static_cast<long long>(head) * D;
  for (int c = threadIdx.x * 2; c < D; c += 256) {
    float x = 0.f, y = 0.f;
    for (int s = 0; s < p.splits; ++s) {
      const float w = exp2f(ws[s * step + D] - ms);
      const float2 v = *reinterpret_cast<const float2*>(ws + s * step + c);
      x += v.x * w;
      y += v.y * w;
    }
    *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16x2(x * inv, y * inv);
  }
}

template <int DW, int MT>
int launch_latent(const nfk_latent_attn_params& p, cudaStream_t stream) {
  using Cfg = LCfg<DW, MT>;
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    if (cudaFuncSetAttribute(latent_attn_mma_kernel<DW, MT>, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM) !=
        cudaSuccess)
      return NF_ERR_CUDA;
    attr = true;
  }
  const int hgroups = (p.heads + Cfg::ROWS - 1) / Cfg::ROWS;
  const long long grid = static_cast<long long>(p.n_tokens) * p.splits * hgroups;
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  latent_attn_mma_kernel<DW, MT><<<static_cast<int>(grid), kLThreads, Cfg::SMEM, stream>>>(p);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  if (p.splits > 1) {
    latent_attn_merge_kernel<<<p.n_tokens * p.heads, 128, 0, stream>>>(p);
    if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  }
  return NF_OK;
}
template <int DW>
int launch_latent_mt(const nfk_latent_attn_params& p, cudaStream_t stream) {
  return p.heads <= 16 ? launch_latent<DW, 1>(p, stream) : launch_latent<DW, 2>(p, stream);
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
