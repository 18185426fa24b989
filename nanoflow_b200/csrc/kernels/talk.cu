// Attention whose heads share their softmax weights: after the softmax (sliding window, a sink per head in the
// denominator) the weights of all heads are mixed by a matrix before they meet the values (Shazeer et al., "Talking-Heads
// Attention"; see kernels.h). Scores, weights, mixing and the turn of the outputs are fp32.
//
// The mixing needs every head's normalised weights, so maxima and sums come first, then weights, mixing and values.
//
// nfk_talk_attn          any sizes, bf16 or fp32: one CTA per token, all heads, two passes over the keys.
// nfk_talk_attn_decode   one token per request (bf16): a cluster of CTAs shares the token's keys. Scores stay in shared
//                        memory, keys and values are read once, straight into registers (a product with the mixing
//                        matrix on tensor cores lies between); maxima, sums and the partial outputs are exchanged through distributed shared memory.
// nfk_talk_attn_prefill  portions (bf16): a cluster takes 16 tokens, each of its CTAs 16 heads, one per warp. First loop
//                        over the keys: maxima and sums; second loop: every CTA's weights go to all CTAs of the cluster,
//                        each mixes them for its own heads (a product with the mixing matrix on tensor cores) and applies
//                        them to the values. Weights enter the products as bf16 pairs (high and low part, about 16 bits).
#include <cooperative_groups.h>

#include "attn_mma.cuh"
#include "elem_io.cuh"

namespace cg = cooperative_groups;

namespace nf {
namespace {

constexpr int kTsThreads = 256, kTsTile = 32;

__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// Element offsets of a tile's key rows (KV head 0), -1 for keys that are not there.
__device__ __forceinline__ void tile_rows(long long* row_s, const nfk_talk_attn_params& p, int j0, int n, int req) {
  if (threadIdx.x < kTsTile) {
    long long r = -1;
    if (static_cast<int>(threadIdx.x) < n) {
      const int j = j0 + threadIdx.x;
      const int page = page_of(j, req, p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages, p.status);
      if (page >= 0) r = (static_cast<long long>(page) * 2 * p.kv_heads * p.page_size + j % p.page_size) * p.hd;
    }
    row_s[threadIdx.x] = r;
  }
}

template <class T>
__global__ void __launch_bounds__(kTsThreads)
talk_attn_kernel(nfk_talk_attn_params p) {
  extern __shared__ float tsm[];                 // q [H][hd] | out [H][hd] | weights [H][32] | mixed [H][32] | max [H] | sum [H]
  __shared__ long long row_s[kTsTile];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = p.heads, hd = p.hd, group = H / p.kv_heads;
  float *q_s = tsm, *o_s = q_s + H * hd, *w_s = o_s + H * hd, *x_s = w_s + H * kTsTile, *m_s = x_s + H * kTsTile, *l_s = m_s + H;
  const int tok = p.token_begin + blockIdx.x;
  const int pos = p.positions[tok], req = p.token_req[tok];
  const T* pool = reinterpret_cast<const T*>(p.pool);
  const long long head_step = static_cast<long long>(p.page_size) * hd, v_step = p.kv_heads * head_step;
  const T* q = reinterpret_cast<const T*>(p.q) + static_cast<long long>(tok) * H * hd;
  for (int c = threadIdx.x; c < H * hd; c += kTsThreads) {
    q_s[c] = to_f32(q[c]);
    o_s[c] = 0.f;
  }
  for (int h = threadIdx.x; h < H; h += kTsThreads) {
    m_s[h] = p.sinks != nullptr ? p.sinks[h] : -INFINITY;
    l_s[h] = p.sinks != nullptr ? 1.f : 0.f;
  }
  auto score = [&](int h) {                      // of this lane's key
    if (row_s[lane] < 0) return -INFINITY;
    const T* k = pool + row_s[lane] + (h / group) * head_step;
    const float* qh = q_s + h * hd;
    float d = 0.f;
    for (int i = 0; i < hd; i += 4) {
      const float4 a = load4(k + i), b = load4(qh + i);
      d += (a.x * b.x + a.y * b.y) + (a.z * b.z + a.w * b.w);
    }
    return d * p.scale;
  };
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  for (int j0 = lo; j0 <= pos; j0 += kTsTile) {
    __syncthreads();
    tile_rows(row_s, p, j0, min(kTsTile, pos + 1 - j0), req);
    __syncthreads();
    for (int h = warp; h < H; h += kTsThreads / 32) {
      const float s = score(h), old = m_s[h], mx = fmaxf(old, warp_max(s));
      const float e = warp_sum(s == -INFINITY ? 0.f : expf(s - mx));
      __syncwarp();
      if (lane == 0 && mx != -INFINITY) {
        l_s[h] = l_s[h] * expf(old - mx) + e;
        m_s[h] = mx;
      }
      __syncwarp();
    }
  }
  for (int j0 = lo; j0 <= pos; j0 += kTsTile) {
    const int n = min(kTsTile, pos + 1 - j0);
    __syncthreads();
    tile_rows(row_s, p, j0, n, req);
    __syncthreads();
    for (int h = warp; h < H; h += kTsThreads / 32) {
      const float s = score(h);
      w_s[h * kTsTile + lane] = s == -INFINITY ? 0.f : expf(s - m_s[h]) / l_s[h];
    }
    __syncthreads();
    for (int h = warp; h < H; h += kTsThreads / 32) {
      float x = 0.f;
      for (int g = 0; g < H; ++g) x += p.talk[h * H + g] * w_s[g * kTsTile + lane];
      x_s[h * kTsTile + lane] = x;
    }
    __syncthreads();
    for (int c = threadIdx.x; c < H * hd; c += kTsThreads) {
      const int h = c / hd;
      const T* v = pool + v_step + (h / group) * head_step + (c - h * hd);
      float o = o_s[c];
      for (int k = 0; k < n; ++k)
        if (row_s[k] >= 0) o += x_s[h * kTsTile + k] * to_f32(v[row_s[k]]);
      o_s[c] = o;
    }
  }
  __syncthreads();
  T* out = reinterpret_cast<T*>(p.out) + static_cast<long long>(tok) * H * hd;
  const float* rot = p.v_rot != nullptr ? p.v_rot + static_cast<long long>(tok) * p.v_ld * 2 : nullptr;
  for (int c = threadIdx.x * 2; c < H * hd; c += kTsThreads * 2) {
    const int i = (c % hd) / 2;
    float a = o_s[c], b = o_s[c + 1];
    if (rot != nullptr && i < p.v_pairs) {
      const float cs = rot[2 * i], sn = rot[2 * i + 1], x = a;
      a = x * cs + b * sn;
      b = b * cs - x * sn;
    }
    put(out + c, a);
    put(out + c + 1, b);
  }
}

// ---- decode ---------------------------------------------------------------------------------------------------
constexpr int kTdThreads = 256, kTdWarps = kTdThreads / 32, kTdKeys = 32;      // keys of a warp's work item
constexpr int kTdMaxCluster = 8, kTpMaxHeads = 64;

// Shared memory: rows [keys] | scores, then weights [H][s_ld] | mixed weights [keys][w_ld] | mixing matrix in fragments |
// (max, sum) [H] | partial outputs [H][hd]. Row strides that spread the fragments' accesses over the banks.
struct TalkDecodeLayout {
  int keys, s_ld, w_ld, scores, mixed, talk, stat, out, bytes;
};
__host__ __device__ inline TalkDecodeLayout talk_decode_layout(int heads, int hd, int keys) {
  TalkDecodeLayout l;
  const int hp = (heads + 15) / 16;
  l.keys = (keys + kTdKeys - 1) / kTdKeys * kTdKeys;
  l.s_ld = l.keys + 4;
  l.w_ld = hp * 16 + 4;
  l.scores = l.keys * 4;
  l.mixed = l.scores + hp * 16 * l.s_ld * 4;
  l.talk = l.mixed + l.keys * l.w_ld * 4;
  l.stat = l.talk + hp * hp * 512;
  l.out = l.stat + (heads * 8 + 15) / 16 * 16;
  l.bytes = l.out + heads * hd * 4;
  return l;
}

__device__ __forceinline__ void split_bf16x2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}
// Two fp32 products and sums at once.
__device__ __forceinline__ uint64_t pair_f32(float x, float y) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(x), "f"(y));
  return r;
}
__device__ __forceinline__ void fma2(uint64_t& acc, uint64_t a, uint64_t b) {
  asm("fma.rn.f32x2 %0, %1, %2, %0;" : "+l"(acc) : "l"(a), "l"(b));
}
__device__ __forceinline__ float2 unpair_f32(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
// Fragments of the mixing matrix (16 x 16 tiles, bf16): piece i of [row tile][column tile][lane].
__device__ __forceinline__ uint4 talk_fragment(const nfk_talk_attn_params& p, int row0, int col0, int lane) {
  const int h = row0 + (lane >> 2), g = col0 + (lane & 3) * 2;
  auto two = [&](int hh, int gg) {
    return pack_bf16x2(hh < p.heads && gg < p.heads ? p.talk[hh * p.heads + gg] : 0.f,
                       hh < p.heads && gg + 1 < p.heads ? p.talk[hh * p.heads + gg + 1] : 0.f);
  };
  return make_uint4(two(h, g), two(h + 8, g), two(h, g + 8), two(h + 8, g + 8));
}

// GV: a thread's heads per pass over the values (heads of one KV head).
template <int HD, int GV>
__global__ void __launch_bounds__(kTdThreads, 2)
talk_decode_kernel(nfk_talk_attn_params p, TalkDecodeLayout lay) {
  extern __shared__ __align__(16) uint8_t tds[];
  int* row_s = reinterpret_cast<int*>(tds);
  float* s_s = reinterpret_cast<float*>(tds + lay.scores);
  float* w_s = reinterpret_cast<float*>(tds + lay.mixed);
  uint4* t_s = reinterpret_cast<uint4*>(tds + lay.talk);
  float2* stat_s = reinterpret_cast<float2*>(tds + lay.stat);
  float* o_s = reinterpret_cast<float*>(tds + lay.out);
  cg::cluster_group cluster = cg::this_cluster();
  const int C = static_cast<int>(cluster.num_blocks()), rank = static_cast<int>(cluster.block_rank());
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = p.heads, G = p.kv_heads, group = H / G;
  const int tok = p.token_begin + blockIdx.x / C;
  const int pos = p.positions[tok], req = p.token_req[tok];
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int total = pos + 1 - lo, per = ((total + C - 1) / C + kTdKeys - 1) / kTdKeys * kTdKeys;
  const int k0 = lo + rank * per;
  int n = min(per, pos + 1 - k0);
  n = n < 0 ? 0 : n;
  if (n > lay.keys) {                            // more keys than the launcher was told
    if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    n = lay.keys;
  }
  const __nv_bfloat16* pool = reinterpret_cast<const __nv_bfloat16*>(p.pool);
  const long long head_step = static_cast<long long>(p.page_size) * HD, v_step = G * head_step;
  // rows of the keys; past the last one its row again, with no weight
  for (int k = threadIdx.x; k < lay.keys; k += kTdThreads) {
    int r = 0;
    if (n > 0) {
      const int j = k0 + min(k, n - 1), page = page_of(j, req, p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages, p.status);
      if (page >= 0) r = page * 2 * G * p.page_size + j % p.page_size;
    }
    row_s[k] = r;
  }
  const int hp = (H + 15) / 16;
  for (int i = threadIdx.x; i < hp * hp * 32; i += kTdThreads) t_s[i] = talk_fragment(p, i / (hp * 32) * 16, i / 32 % hp * 16, i & 31);
  for (int i = threadIdx.x; i < (hp * 16 - H) * lay.s_ld; i += kTdThreads) s_s[H * lay.s_ld + i] = 0.f;      // heads that are not there
  __syncthreads();
  // ---- scores: a warp takes 32 keys of a KV head. Rows of the tiles: the KV head's query heads, 16 at a time ----
  const int blocks = (n + kTdKeys - 1) / kTdKeys;
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(tok) * H * HD;
  for (int item = warp; item < blocks * G; item += kTdWarps) {
    const int kvh = item / blocks, kb = (item - kvh * blocks) * kTdKeys;
    // a lane brings eight neighbouring columns of a key at a time, for two steps of the product: the columns of a step
    // are those {c, c + 1, c + 2, c + 3} of every lane's eight, in queries and keys alike
    uint4 kr[kTdKeys / 8][HD / 32];
#pragma unroll
    for (int t = 0; t < kTdKeys / 8; ++t) {
      const int r = row_s[kb + t * 8 + (lane >> 2)];
      const __nv_bfloat16* src = pool + static_cast<long long>(r) * HD + kvh * head_step + (lane & 3) * 8;
#pragma unroll
      for (int b = 0; b < HD / 32; ++b) kr[t][b] = *reinterpret_cast<const uint4*>(src + b * 32);
    }
    for (int m0 = 0; m0 < group; m0 += 16) {
      float acc[kTdKeys / 8][4];
#pragma unroll
      for (int t = 0; t < kTdKeys / 8; ++t) acc[t][0] = acc[t][1] = acc[t][2] = acc[t][3] = 0.f;
      const int r0 = m0 + (lane >> 2), r1 = r0 + 8;
      const __nv_bfloat16* q0 = q + (kvh * group + r0) * HD + (lane & 3) * 8;
#pragma unroll
      for (int b = 0; b < HD / 32; ++b) {
        const uint4 x0 = r0 < group ? *reinterpret_cast<const uint4*>(q0 + b * 32) : make_uint4(0, 0, 0, 0);
        const uint4 x1 = r1 < group ? *reinterpret_cast<const uint4*>(q0 + 8 * HD + b * 32) : make_uint4(0, 0, 0, 0);
        const uint32_t a0[4] = {x0.x, x1.x, x0.y, x1.y}, a1[4] = {x0.z, x1.z, x0.w, x1.w};
#pragma unroll
        for (int t = 0; t < kTdKeys / 8; ++t) {
          mma_bf16(acc[t], a0, kr[t][b].x, kr[t][b].y);
          mma_bf16(acc[t], a1, kr[t][b].z, kr[t][b].w);
        }
      }
#pragma unroll
      for (int t = 0; t < kTdKeys / 8; ++t) {
        const int k = kb + t * 8 + (lane & 3) * 2;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const bool ok = k + e < n;
          if (r0 < group) s_s[(kvh * group + r0) * lay.s_ld + k + e] = ok ? acc[t][e] * p.scale : -INFINITY;
          if (r1 < group) s_s[(kvh * group + r1) * lay.s_ld + k + e] = ok ? acc[t][2 + e] * p.scale : -INFINITY;
        }
      }
    }
  }
  __syncthreads();
  // ---- maxima and sums, of this CTA's keys and then of the token's ----
  const int nk = blocks * kTdKeys;
  for (int h = warp; h < H; h += kTdWarps) {
    const float* s = s_s + h * lay.s_ld;
    float m = -INFINITY, l = 0.f;
    for (int k = lane; k < nk; k += 32) m = fmaxf(m, s[k]);
    m = warp_max(m);
    if (m != -INFINITY)
      for (int k = lane; k < nk; k += 32) l += expf(s[k] - m);
    l = warp_sum(l);
    if (lane == 0) stat_s[h] = make_float2(m, l);
  }
  cluster.sync();
  for (int h = warp; h < H; h += kTdWarps) {
    const float2 st = lane < C ? *cluster.map_shared_rank(stat_s + h, lane) : make_float2(-INFINITY, 0.f);
    const float sink = p.sinks != nullptr ? p.sinks[h] : -INFINITY;
    const float m = fmaxf(warp_max(st.x), sink);
    float l = st.x == -INFINITY ? 0.f : st.y * expf(st.x - m);
    l = warp_sum(l) + (sink == -INFINITY ? 0.f : expf(sink - m));
    const float inv = l > 0.f ? 1.f / l : 0.f;
    float* s = s_s + h * lay.s_ld;
    for (int k = lane; k < nk; k += 32) s[k] = s[k] == -INFINITY ? 0.f : expf(s[k] - m) * inv;
  }
  __syncthreads();
  // ---- mixing: [H x H] times [H x keys] on tensor cores, eight keys per warp and step, weights as bf16 pairs; the result
  // lies key by key ----
  for (int kb = warp * 8; kb < nk; kb += kTdWarps * 8) {
    constexpr int kTiles = kTpMaxHeads / 16;
    uint32_t bh[kTiles][2], bl[kTiles][2];
#pragma unroll
    for (int g = 0; g < kTiles; ++g)
      if (g < hp) {
        const float* w = s_s + (g * 16 + (lane & 3) * 2) * lay.s_ld + kb + (lane >> 2);
#pragma unroll
        for (int e = 0; e < 2; ++e) split_bf16x2(w[e * 8 * lay.s_ld], w[(e * 8 + 1) * lay.s_ld], bh[g][e], bl[g][e]);
      }
    for (int h = 0; h < hp; ++h) {
      float x[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int g = 0; g < kTiles; ++g)
        if (g < hp) {
          const uint4 tf = t_s[(h * hp + g) * 32 + lane];
          const uint32_t a[4] = {tf.x, tf.y, tf.z, tf.w};
          mma_bf16(x, a, bh[g][0], bh[g][1]);
          mma_bf16(x, a, bl[g][0], bl[g][1]);
        }
      float* dst = w_s + (kb + (lane & 3) * 2) * lay.w_ld + h * 16 + (lane >> 2);
      dst[0] = x[0];
      dst[lay.w_ld] = x[1];
      dst[8] = x[2];
      dst[lay.w_ld + 8] = x[3];
    }
  }
  for (int c = threadIdx.x; c < H * HD; c += kTdThreads) o_s[c] = 0.f;
  __syncthreads();
  // ---- values: a thread takes four columns of a KV head for up to GV of its query heads; what threads are left over
  // split the keys. The next keys' values are on their way while these are worked on ----
  const int quads = G * (HD / 4), parts = max(1, kTdThreads / quads);
  for (int unit = threadIdx.x; unit < quads * parts; unit += kTdThreads) {
    const int part = unit / quads, qd = unit - part * quads, kvh = qd / (HD / 4), col = (qd - kvh * (HD / 4)) * 4;
    const __nv_bfloat16* v = pool + v_step + kvh * head_step + col;
    constexpr int U = 8;
    auto fetch = [&](uint2 (&x)[U], int kb) {
#pragma unroll
      for (int j = 0; j < U; j += 4) {
        const int4 r = *reinterpret_cast<const int4*>(row_s + min(kb, nk - U) + j);      // past the end: not used
        const int rr[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) x[j + i] = *reinterpret_cast<const uint2*>(v + static_cast<long long>(rr[i]) * HD);
      }
    };
    for (int m0 = 0; m0 < group; m0 += GV) {
      const int nh = min(GV, group - m0), h0 = kvh * group + m0;
      uint64_t acc[GV][2];
#pragma unroll
      for (int i = 0; i < GV; ++i) acc[i][0] = acc[i][1] = 0;
      auto add = [&](const uint2 (&x)[U], int kb) {
        const float* w = w_s + kb * lay.w_ld + h0;
#pragma unroll
        for (int j = 0; j < U; ++j, w += lay.w_ld) {
          const float2 a = unpack_bf16x2(x[j].x), b = unpack_bf16x2(x[j].y);
          const uint64_t ab = pair_f32(a.x, a.y), cd = pair_f32(b.x, b.y);
          float f[GV];
          if (GV == 4 && (h0 & 3) == 0 && nh == 4) {
            const float4 q4 = *reinterpret_cast<const float4*>(w);
            f[0] = q4.x; f[GV > 1 ? 1 : 0] = q4.y; f[GV > 2 ? 2 : 0] = q4.z; f[GV > 3 ? 3 : 0] = q4.w;
          } else {
#pragma unroll
            for (int i = 0; i < GV; ++i) f[i] = i < nh ? w[i] : 0.f;
          }
#pragma unroll
          for (int i = 0; i < GV; ++i) {
            const uint64_t ff = pair_f32(f[i], f[i]);
            fma2(acc[i][0], ff, ab);
            fma2(acc[i][1], ff, cd);
          }
        }
      };
      uint2 x[U], y[U];
      const int step = parts * U;
      if (part * U < nk) fetch(x, part * U);
      for (int kb = part * U; kb < nk; kb += 2 * step) {
        fetch(y, kb + step);
        add(x, kb);
        if (kb + step < nk) {
          fetch(x, kb + 2 * step);
          add(y, kb + step);
        }
      }
#pragma unroll
      for (int i = 0; i < GV; ++i)
        if (i < nh) {
          const float2 a = unpair_f32(acc[i][0]), b = unpair_f32(acc[i][1]);
          float* o = o_s + (h0 + i) * HD + col;
          if (parts == 1) {
            store4(o, make_float4(a.x, a.y, b.x, b.y));
          } else {
            atomicAdd(o, a.x); atomicAdd(o + 1, a.y); atomicAdd(o + 2, b.x); atomicAdd(o + 3, b.y);
          }
        }
    }
  }
  cluster.sync();
  // ---- outputs: the CTAs of the cluster share the pairs of columns ----
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out) + static_cast<long long>(tok) * H * HD;
  const float* rot = p.v_rot != nullptr ? p.v_rot + static_cast<long long>(tok) * p.v_ld * 2 : nullptr;
  for (int c = (rank * kTdThreads + threadIdx.x) * 2; c < H * HD; c += C * kTdThreads * 2) {
    float a = 0.f, b = 0.f;
    for (int r = 0; r < C; ++r) {
      const float2 x = *reinterpret_cast<const float2*>(cluster.map_shared_rank(o_s + c, r));
      a += x.x;
      b += x.y;
    }
    const int i = (c % HD) / 2;
    if (rot != nullptr && i < p.v_pairs) {
      const float cs = rot[2 * i], sn = rot[2 * i + 1], x = a;
      a = x * cs + b * sn;
      b = b * cs - x * sn;
    }
    *reinterpret_cast<uint32_t*>(out + c) = pack_bf16x2(a, b);
  }
  cluster.sync();                                // nobody leaves while its shared memory is read
}

template <int HD>
int launch_talk_decode(const nfk_talk_attn_params& p, cudaStream_t stream) {
  // few tokens: more CTAs per token; many keys: enough CTAs for their scores to fit, two CTAs per SM if they can
  const int sms = device_sm_count();
  int C = 1;
  while (C < kTdMaxCluster && (p.n_tokens * C * 2 <= 2 * sms || talk_decode_layout(p.heads, HD, (p.max_keys + C - 1) / C).bytes > 110 * 1024)) C *= 2;
  while (C > 1 && (p.max_keys + C - 1) / C < kTdKeys) C /= 2;
  const TalkDecodeLayout lay = talk_decode_layout(p.heads, HD, (p.max_keys + C - 1) / C);
  if (lay.bytes > 220 * 1024) return NF_ERR_UNSUPPORTED;
  const int group = p.heads / p.kv_heads;
  auto kernel = group == 1 ? talk_decode_kernel<HD, 1> : group == 2 ? talk_decode_kernel<HD, 2> : talk_decode_kernel<HD, 4>;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024) != cudaSuccess) return NF_ERR_CUDA;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(static_cast<unsigned>(p.n_tokens) * C);
  cfg.blockDim = dim3(kTdThreads);
  cfg.dynamicSmemBytes = lay.bytes;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = C;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, p, lay) == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

// ---- prefill --------------------------------------------------------------------------------------------------
constexpr int kTpQ = 16, kTpHeads = 16, kTpThreads = kTpHeads * 32;
constexpr int kTpPages = 1024;             // pages that the keys of a work item may lie in

template <int HD, int KT>
struct TalkCfg {
  static constexpr int XLD = KT + 8;                     // mixed weights [head][query][key]; strides without bank conflicts
  static constexpr int XHD = kTpQ * XLD + 8;             // ... from head to head
  static constexpr int PLD = kTpQ * KT + 8;              // weights [head][query * KT + key], see p_col
  static constexpr int BOX = kPage * 128;                // 64 columns of a page's keys or values, 128-byte swizzle
  static constexpr int PAGE_BYTES = HD / 64 * BOX;
  static constexpr int ROWS = KT / kPage * PAGE_BYTES;   // keys or values of a KV head
  static constexpr int X_BYTES = kTpHeads * XHD * 2;
  __host__ __device__ static constexpr int p_bytes(int hp) { return hp * PLD * 2; }
  // keys | values | weights (pair) | mixed weights (pair, two buffers) | mixing matrix in fragments | page ids | barriers
  __host__ __device__ static constexpr int smem(int hp, int kvs) {
    return 1024 + 2 * kvs * ROWS + 2 * p_bytes(hp) + 4 * X_BYTES + hp / 16 * 512 + kTpPages * 4 + 16;
  }
};
// Column of a query's block of eight keys: neighbouring queries' blocks lie in different banks.
template <int KT>
__device__ __forceinline__ int p_col(int q, int block) {
  return KT == 32 ? q * 32 + ((block ^ (q >> 1)) & 3) * 8 : q * 16 + ((block ^ (q >> 2)) & 1) * 8;
}

__device__ __forceinline__ void stsm_x4(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3)
               : "memory");
}

// x ^ bits, computed where it stands (kept in registers across a loop, the variants of an address cost spills).
__device__ __forceinline__ uint32_t flip(uint32_t x, uint32_t bits) {
  uint32_t r;
  asm volatile("xor.b32 %0, %1, %2;" : "=r"(r) : "r"(x), "r"(bits));
  return r;
}
// The cluster's barrier in two halves, so that work fits in between.
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }

// hp: heads padded to a multiple of 16; kvs: KV heads that 16 query heads can touch.
template <int HD, int KT>
__global__ void __launch_bounds__(kTpThreads, 1)
talk_prefill_kernel(const __grid_constant__ CUtensorMap tm, nfk_talk_attn_params p, int hp, int kvs) {
  using Cfg = TalkCfg<HD, KT>;
  constexpr int NT = KT / 8;                             // key blocks of a tile
  extern __shared__ __align__(16) uint8_t tps_raw[];
  uint8_t* tps = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(tps_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint8_t *k_s = tps, *v_s = tps + kvs * Cfg::ROWS;
  __nv_bfloat16* p_s = reinterpret_cast<__nv_bfloat16*>(tps + 2 * kvs * Cfg::ROWS);          // high parts, then low parts
  __nv_bfloat16* x_s = reinterpret_cast<__nv_bfloat16*>(tps + 2 * kvs * Cfg::ROWS + 2 * Cfg::p_bytes(hp));
  uint4* t_s = reinterpret_cast<uint4*>(tps + 2 * kvs * Cfg::ROWS + 2 * Cfg::p_bytes(hp) + 4 * Cfg::X_BYTES);
  int* page_s = reinterpret_cast<int*>(t_s + hp / 16 * 32);
  uint64_t* bar = reinterpret_cast<uint64_t*>(page_s + kTpPages);            // copies into k_s and v_s
  cg::cluster_group cluster = cg::this_cluster();
  const int C = hp / kTpHeads, rank = static_cast<int>(cluster.block_rank());
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int H = p.heads, G = p.kv_heads, group = H / G;
  // the last items of a portion see most keys: they start first
  const int* item = p.items + (p.num_items - 1 - static_cast<int>(blockIdx.x) / C) * 3;
  const int req = item[0], tok0 = item[1], cnt = min(item[2], kTpQ);
  const int pos0 = p.positions[tok0];
  const int head0 = rank * kTpHeads, head = head0 + warp;
  const bool live = head < H;
  const int kv0 = head0 / group, kvn = (min(H, head0 + kTpHeads) - 1) / group - kv0 + 1;
  const int kvl = live ? head / group - kv0 : 0;         // this warp's KV head among the CTA's
  const int first = p.window > 0 ? max(0, pos0 - p.window + 1) : 0, last = pos0 + cnt - 1;
  const int lo = first / KT * KT, tiles = (last - lo) / KT + 1;
  const int slot0 = first / kPage, slot1 = last / kPage;
  if (threadIdx.x == 0) {
    mbar_init(&bar[0], 1);
    mbar_init(&bar[1], 1);
    mbar_fence_init();
    tma_prefetch_desc(&tm);
  }
  if (slot1 - slot0 >= kTpPages && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
  for (int i = threadIdx.x; i < kTpPages && slot0 + i <= slot1; i += kTpThreads)
    page_s[i] = max(page_of((slot0 + i) * kPage, req, kPage, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages, p.status), 0) * 2 * G * kPage;
  for (int i = threadIdx.x; i < hp / 16 * 32; i += kTpThreads) t_s[i] = talk_fragment(p, head0, i / 32 * 16, i & 31);
  __syncthreads();

  // Copies of a tile's pages, the CTA's KV heads one after the other, by the first warp. kind: 0 keys, 1 values. Past the
  // first and last page that one again: all keys outside the range get no weight.
  const int pages = min(slot1 - slot0, kTpPages - 1), page0 = lo / kPage - slot0;
  auto fetch = [&](int buf, int t, int kind) {
    if (warp != 0) return;
    if (lane == 0) mbar_expect_tx(&bar[buf], kvn * Cfg::ROWS);
    __syncwarp();
    constexpr int HB = HD / 64, PG = KT / kPage;
    const int row0 = (kind * G + kv0) * kPage;
#pragma unroll 1
    for (int i = lane; i < kvn * PG * HB; i += 32) {
      const int half = i % HB, pg = i / HB % PG, kv = i / (HB * PG);
      const int page = page_s[min(max(page0 + t * PG + pg, 0), pages)];
      tma_load_2d((buf == 0 ? k_s : v_s) + kv * Cfg::ROWS + pg * Cfg::PAGE_BYTES + half * Cfg::BOX, &tm, &bar[buf], half * 64,
                  page + row0 + kv * kPage);
    }
  };
  // a wait that runs out is reported at the end; the warps go on in step, so that they meet at their barriers
  bool late = false;
  auto arrived = [&](int buf, int n) { late |= !mbar_wait(&bar[buf], n & 1); };      // the n-th copy into a buffer

  uint32_t qa[HD / 16][4];
  {
    const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(p.q) + static_cast<long long>(tok0) * H * HD + head * HD;
    load_q_frags<HD>(qa, [&](int r) -> const __nv_bfloat16* { return live && r < cnt ? q + static_cast<long long>(r) * H * HD : nullptr; });
  }
  const int mm = lane >> 3, rr = lane & 7;
  const float scale = p.scale * kLog2e;
  const int i0 = pos0 + (lane >> 2), i1 = i0 + 8;        // positions of this lane's two queries
  // 16-byte pieces of a row lie at their number xor the row's: this lane's row and first piece, later ones by an xor
  const uint32_t k_lane = ((mm >> 1) * 8 + rr) * 128 + (((mm & 1) ^ rr) << 4), v_lane = ((mm & 1) * 8 + rr) * 128 + (((mm >> 1) ^ rr) << 4);
  const uint32_t vb = smem_u32(v_s) + kvl * Cfg::ROWS + v_lane;
  auto seen = [&](int i, int j) { return j <= i && j >= 0 && (p.window <= 0 || i - j < p.window); };
  // scores of this warp's head, -inf where the query does not see the key
  auto scores = [&](float (&s)[NT][4], const uint8_t* keys, int t) {
    const uint32_t kb = smem_u32(keys) + kvl * Cfg::ROWS + k_lane;
#pragma unroll
    for (int b = 0; b < NT; ++b) s[b][0] = s[b][1] = s[b][2] = s[b][3] = 0.f;
#pragma unroll
    for (int ks = 0; ks < HD / 16; ++ks)
#pragma unroll
      for (int b = 0; b < NT; b += 2) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4(flip(kb, (ks & 3) << 5) + b / 2 * Cfg::PAGE_BYTES + ks / 4 * Cfg::BOX, b0, b1, b2, b3);
        mma_bf16(s[b], qa[ks], b0, b1);
        mma_bf16(s[b + 1], qa[ks], b2, b3);
      }
    const int j0 = lo + t * KT;
    if (j0 + KT - 1 > pos0 || (p.window > 0 && pos0 + kTpQ - 1 - j0 >= p.window)) {      // not seen by all 16 queries
#pragma unroll
      for (int b = 0; b < NT; ++b)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = j0 + b * 8 + (lane & 3) * 2 + e;
          if (!seen(i0, j)) s[b][e] = -INFINITY;
          if (!seen(i1, j)) s[b][2 + e] = -INFINITY;
        }
    }
  };

  // ---- first loop: maxima and sums, keys in the two buffers by turns ----
  const float sink = p.sinks != nullptr && live ? p.sinks[head] * kLog2e : -INFINITY;
  float m0 = sink, m1 = sink, l0 = 0.f, l1 = 0.f;        // of scores times log2 e; sums of this lane's keys
  fetch(0, 0, 0);
  for (int t = 0; t < tiles; ++t) {
    arrived(t & 1, t >> 1);
    __syncthreads();                                     // everyone is done with the other buffer
    if (t + 1 < tiles) fetch((t + 1) & 1, t + 1, 0);
    float s[NT][4];
    scores(s, (t & 1) != 0 ? v_s : k_s, t);
    float x0 = s[0][0], x1 = s[0][2];
#pragma unroll
    for (int b = 0; b < NT; ++b) {
      x0 = fmaxf(x0, fmaxf(s[b][0], s[b][1]));
      x1 = fmaxf(x1, fmaxf(s[b][2], s[b][3]));
    }
    x0 = fmaxf(m0, quad_max(x0) * scale);
    x1 = fmaxf(m1, quad_max(x1) * scale);
    const float z0 = x0 == -INFINITY ? 0.f : x0, z1 = x1 == -INFINITY ? 0.f : x1;
    l0 *= fast_exp2(m0 - z0);
    l1 *= fast_exp2(m1 - z1);
    m0 = x0;
    m1 = x1;
#pragma unroll
    for (int b = 0; b < NT; ++b) {
      l0 += fast_exp2(fmaf(s[b][0], scale, -z0)) + fast_exp2(fmaf(s[b][1], scale, -z0));
      l1 += fast_exp2(fmaf(s[b][2], scale, -z1)) + fast_exp2(fmaf(s[b][3], scale, -z1));
    }
  }
  __syncthreads();
  fetch(0, 0, 0);
  // weight = 2^(score - m - log2(sum)); rows of the tile that are no queries get none
  l0 = quad_sum(l0);
  l1 = quad_sum(l1);
  m0 = m0 == -INFINITY ? 0.f : m0;
  m1 = m1 == -INFINITY ? 0.f : m1;
  l0 += sink == -INFINITY ? 0.f : fast_exp2(sink - m0);
  l1 += sink == -INFINITY ? 0.f : fast_exp2(sink - m1);
  m0 = live && (lane >> 2) < cnt && l0 > 0.f ? m0 + log2f(l0) : INFINITY;
  m1 = live && (lane >> 2) + 8 < cnt && l1 > 0.f ? m1 + log2f(l1) : INFINITY;

  // ---- second loop: weights, mixing, values ----
  float acc[HD / 8][4];
#pragma unroll
  for (int b = 0; b < HD / 8; ++b) acc[b][0] = acc[b][1] = acc[b][2] = acc[b][3] = 0.f;
  const uint32_t pb = smem_u32(p_s), xb = smem_u32(x_s);
  const uint32_t p_lo = static_cast<uint32_t>(Cfg::p_bytes(hp)), x_lo = Cfg::X_BYTES;
  // mixed weights of tile t times its values
  auto values = [&](int t) {
    const uint32_t base = xb + ((t & 1) != 0 ? 2 * x_lo : 0);
#pragma unroll 1
    for (int ks = 0; ks < KT / 16; ++ks) {               // (registers: what unrolling would hoist has no room)
      uint32_t ah[4], al[4];
      const uint32_t o = (warp * Cfg::XHD + (lane & 15) * Cfg::XLD + ks * 16 + (lane >> 4) * 8) * 2;
      ldsm_x4(base + o, ah[0], ah[1], ah[2], ah[3]);
      ldsm_x4(base + x_lo + o, al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int b = 0; b < HD / 8; b += 2) {
        uint32_t b0, b1, b2, b3;
        ldsm_x4_trans(flip(vb, (b / 2 & 3) << 5) + ks * Cfg::PAGE_BYTES + b / 8 * Cfg::BOX, b0, b1, b2, b3);
        mma_bf16(acc[b], ah, b0, b1);
        mma_bf16(acc[b + 1], ah, b2, b3);
        mma_bf16(acc[b], al, b0, b1);
        mma_bf16(acc[b + 1], al, b2, b3);
      }
    }
  };
  // Products with values lag by one tile: they run while the weights travel to the other CTAs.
  if (C > 1) cluster_arrive();
  for (int t = 0; t < tiles; ++t) {
    {
      float s[NT][4];
      arrived(0, (tiles + 1) / 2 + t);
      scores(s, k_s, t);
      uint32_t hi[NT][2], lw[NT][2];
#pragma unroll
      for (int b = 0; b < NT; ++b) {
        split_bf16x2(fast_exp2(fmaf(s[b][0], scale, -m0)), fast_exp2(fmaf(s[b][1], scale, -m0)), hi[b][0], lw[b][0]);
        split_bf16x2(fast_exp2(fmaf(s[b][2], scale, -m1)), fast_exp2(fmaf(s[b][3], scale, -m1)), hi[b][1], lw[b][1]);
      }
      if (C > 1) cluster_wait();                         // all have started, and mixed the last weights
#pragma unroll
      for (int b = 0; b < NT; b += 2) {
        // matrices: queries 0-7 and 8-15 of key blocks b and b + 1
        const uint32_t o = (head * Cfg::PLD + p_col<KT>((mm & 1) * 8 + rr, b + (mm >> 1))) * 2;
        stsm_x4(pb + o, hi[b][0], hi[b][1], hi[b + 1][0], hi[b + 1][1]);
        stsm_x4(pb + p_lo + o, lw[b][0], lw[b][1], lw[b + 1][0], lw[b + 1][1]);
      }
      if (C > 1) {                                       // the head's weights to the other CTAs of the cluster
        __syncwarp();
        constexpr int N16 = kTpQ * KT / 8;               // 16-byte pieces of a part
        const uint4* src = reinterpret_cast<const uint4*>(p_s + head * Cfg::PLD);
        const int part = static_cast<int>(p_lo / 16);
#pragma unroll 1
        for (int r = 1; r < C; ++r) {
          uint4* dst = cluster.map_shared_rank(const_cast<uint4*>(src), rank + r < C ? rank + r : rank + r - C);
#pragma unroll
          for (int i = 0; i < N16 / 32; ++i) {
            dst[i * 32 + lane] = src[i * 32 + lane];
            dst[part + i * 32 + lane] = src[part + i * 32 + lane];
          }
        }
      }
    }
    if (C > 1) cluster_arrive();
    else __syncthreads();                                // the weights are there
    if (t > 0) {
      arrived(1, tiles / 2 + t - 1);
      values(t - 1);
    }
    if (C > 1) cluster_wait();
    if (t + 1 < tiles) fetch(0, t + 1, 0);               // everyone is done with these keys
    // mixed weights of the CTA's 16 heads: [16 x H] times [H x (query, key)], columns over the warps: one query per warp
    {
      float x[NT][4];
#pragma unroll
      for (int b = 0; b < NT; ++b) x[b][0] = x[b][1] = x[b][2] = x[b][3] = 0.f;
#pragma unroll 1
      for (int g = 0; g < hp; g += 16) {
        const uint4 tf = t_s[g * 2 + lane];
        const uint32_t a[4] = {tf.x, tf.y, tf.z, tf.w};
        const uint32_t row = (g + (mm & 1) * 8 + rr) * Cfg::PLD;
#pragma unroll
        for (int b = 0; b < NT; b += 2) {
          const uint32_t o = (row + p_col<KT>(warp, b + (mm >> 1))) * 2;
          uint32_t b0, b1, b2, b3, c0, c1, c2, c3;
          ldsm_x4_trans(pb + o, b0, b1, b2, b3);
          ldsm_x4_trans(pb + p_lo + o, c0, c1, c2, c3);
          mma_bf16(x[b], a, b0, b1);
          mma_bf16(x[b + 1], a, b2, b3);
          mma_bf16(x[b], a, c0, c1);
          mma_bf16(x[b + 1], a, c2, c3);
        }
      }
      if (C > 1 && t + 1 < tiles) cluster_arrive();
      const uint32_t base = xb + ((t & 1) != 0 ? 2 * x_lo : 0);
#pragma unroll
      for (int b = 0; b < NT; b += 2) {
        uint32_t hi[4], lw[4];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          split_bf16x2(x[b + e][0], x[b + e][1], hi[e * 2], lw[e * 2]);
          split_bf16x2(x[b + e][2], x[b + e][3], hi[e * 2 + 1], lw[e * 2 + 1]);
        }
        // matrices: heads 0-7 and 8-15 of key blocks b and b + 1
        const uint32_t o = (((mm & 1) * 8 + rr) * Cfg::XHD + warp * Cfg::XLD + (b + (mm >> 1)) * 8) * 2;
        stsm_x4(base + o, hi[0], hi[1], hi[2], hi[3]);
        stsm_x4(base + x_lo + o, lw[0], lw[1], lw[2], lw[3]);
      }
    }
    __syncthreads();                                     // mixed weights are there, the last values are read
    fetch(1, t, 1);
  }
  arrived(1, tiles / 2 + tiles - 1);
  values(tiles - 1);
  if (late) report_status(p.status, NF_ST_TIMEOUT_SMEM_FULL);
  // ---- outputs turn back by their query's angles ----
  if (live) {
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.out);
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = (lane >> 2) + h * 8;
      if (r >= cnt) continue;
      const long long tok = tok0 + r;
      const float2* rot = p.v_rot != nullptr ? reinterpret_cast<const float2*>(p.v_rot) + tok * p.v_ld : nullptr;
#pragma unroll
      for (int b = 0; b < HD / 8; ++b) {
        const int i = b * 4 + (lane & 3);
        float x = acc[b][2 * h], y = acc[b][2 * h + 1];
        if (rot != nullptr && i < p.v_pairs) {
          const float2 a = rot[i];
          const float z = x;
          x = z * a.x + y * a.y;
          y = y * a.x - z * a.y;
        }
        *reinterpret_cast<uint32_t*>(out + tok * H * HD + head * HD + i * 2) = pack_bf16x2(x, y);
      }
    }
  }
  // a CTA may only leave when nobody writes to its shared memory any more: every write comes before the last cluster
  // barrier, which all have passed
}

template <int HD, int KT>
int launch_talk_prefill(const nfk_talk_attn_params& p, int hp, int kvs, cudaStream_t stream) {
  const int C = hp / kTpHeads, sm = TalkCfg<HD, KT>::smem(hp, kvs);
  auto kernel = talk_prefill_kernel<HD, KT>;
  CUtensorMap tm;
  const int rc = make_tmap_bf16_2d(&tm, p.pool, static_cast<uint64_t>(p.num_pages) * 2 * p.kv_heads * kPage, HD, HD, kPage, 64);
  if (rc != NF_OK) return rc;
  if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, sm) != cudaSuccess) return NF_ERR_CUDA;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(static_cast<unsigned>(p.num_items) * C);
  cfg.blockDim = dim3(kTpThreads);
  cfg.dynamicSmemBytes = sm;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = C;
  attr[0].val.clusterDim.y = attr[0].val.clusterDim.z = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 1;
  return cudaLaunchKernelEx(&cfg, kernel, tm, p, hp, kvs) == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

// KV heads that 16 neighbouring query heads (from a multiple of 16) can touch.
int kv_heads_of_16(int heads, int group) {
  int most = 1;
  for (int h0 = 0; h0 < heads; h0 += kTpHeads) {
    const int last = (heads < h0 + kTpHeads ? heads : h0 + kTpHeads) - 1, n = last / group - h0 / group + 1;
    if (n > most) most = n;
  }
  return most;
}

int check_talk(const nfk_talk_attn_params* p) {
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (!p->q || !p->pool || !p->out || !p->positions || !p->token_req || !p->kv_indptr || !p->kv_indices || !p->talk ||
      p->n_tokens < 0 || p->token_begin < 0 || p->heads <= 0 || p->kv_heads <= 0 || p->heads % p->kv_heads != 0 || p->hd <= 0 ||
      p->hd % 8 != 0 || p->page_size <= 0 || p->num_pages <= 0 || p->window < 0)
    return NF_ERR_BAD_ARG;
  if (p->v_rot && (p->v_pairs < 0 || p->v_pairs > p->hd / 2 || p->v_ld < p->v_pairs)) return NF_ERR_BAD_ARG;
  return NF_OK;
}

template <class T>
int launch_talk_simple(const nfk_talk_attn_params& p, cudaStream_t stream) {
  const size_t sm = static_cast<size_t>(p.heads) * (2 * p.hd + 2 * kTsTile + 2) * 4;
  if (sm > 220 * 1024) return NF_ERR_UNSUPPORTED;
  if (sm > 48 * 1024 && cudaFuncSetAttribute(talk_attn_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             static_cast<int>(sm)) != cudaSuccess)
    return NF_ERR_CUDA;
  talk_attn_kernel<T><<<p.n_tokens, kTsThreads, sm, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_talk_attn(const nfk_talk_attn_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_talk(p);
  if (rc != NF_OK || p->n_tokens == 0) return rc;
  return p->dtype == NFK_F32 ? launch_talk_simple<float>(*p, stream) : launch_talk_simple<__nv_bfloat16>(*p, stream);
}

extern "C" int nfk_talk_attn_decode(const nfk_talk_attn_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_talk(p);
  if (rc != NF_OK || p->n_tokens == 0) return rc;
  if (p->dtype != NFK_BF16 || (p->hd != 64 && p->hd != 128) || p->heads > kTpMaxHeads) return NF_ERR_UNSUPPORTED;
  if (p->max_keys <= 0 || static_cast<long long>(p->num_pages) * 2 * p->kv_heads * p->page_size > 0x7fffffffll) return NF_ERR_BAD_ARG;
  return p->hd == 64 ? launch_talk_decode<64>(*p, stream) : launch_talk_decode<128>(*p, stream);
}

extern "C" int nfk_talk_attn_prefill(const nfk_talk_attn_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_talk(p);
  if (rc != NF_OK || p->num_items == 0) return rc;
  if (p->num_items < 0 || !p->items) return NF_ERR_BAD_ARG;
  if (p->dtype != NFK_BF16 || (p->hd != 64 && p->hd != 128) || p->heads > kTpMaxHeads || p->page_size != kPage)
    return NF_ERR_UNSUPPORTED;
  const int hp = (p->heads + kTpHeads - 1) / kTpHeads * kTpHeads, kvs = kv_heads_of_16(p->heads, p->heads / p->kv_heads);
  constexpr int kMost = 227 * 1024;
  if (p->hd == 64) {
    if (TalkCfg<64, 32>::smem(hp, kvs) <= kMost) return launch_talk_prefill<64, 32>(*p, hp, kvs, stream);
    if (TalkCfg<64, 16>::smem(hp, kvs) <= kMost) return launch_talk_prefill<64, 16>(*p, hp, kvs, stream);
  } else {
    if (TalkCfg<128, 32>::smem(hp, kvs) <= kMost) return launch_talk_prefill<128, 32>(*p, hp, kvs, stream);
    if (TalkCfg<128, 16>::smem(hp, kvs) <= kMost) return launch_talk_prefill<128, 16>(*p, hp, kvs, stream);
  }
  return NF_ERR_UNSUPPORTED;
}

extern "C" int nfk_talk_attn_fits(int heads, int kv_heads, int hd, int max_keys) {
  using namespace nf;
  if (heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || heads > kTpMaxHeads || (hd != 64 && hd != 128) || max_keys <= 0) return 0;
  const int hp = (heads + kTpHeads - 1) / kTpHeads * kTpHeads, kvs = kv_heads_of_16(heads, heads / kv_heads);
  const int pre = hd == 64 ? TalkCfg<64, 16>::smem(hp, kvs) : TalkCfg<128, 16>::smem(hp, kvs);
  const int dec = talk_decode_layout(heads, hd, (max_keys + kTdMaxCluster - 1) / kTdMaxCluster).bytes;
  return (pre <= 227 * 1024 && max_keys <= (kTpPages - 3) * kPage ? 1 : 0) + (dec <= 220 * 1024 ? 2 : 0);
}
