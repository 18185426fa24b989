// WKV recurrence: a matrix state per head with a decay per key channel and token, and a bonus for the current
// token (Peng et al., "Eagle and Finch: RWKV with Matrix-Valued States and Dynamic Recurrence"; see kernels.h for the
// equations). State, decays and everything derived from them are fp32.
//
// nfk_token_shift   every stream's mix of a token's row with the previous token's row; the last row of a request
//                   is kept for its next step.
// nfk_wkv_decode    one token per request: a CTA per request and head streams S through registers (read out,
//                   update, write back in one pass), then head norm, weight and gate. Bound by the state traffic.
// nfk_wkv_prefill   token by token (any size, bf16 or fp32), S in shared memory; or in chunks of 64 tokens on
//                   tensor cores (bf16), three passes that are parallel over chunks, elements of S, and chunks:
//                   1. what each chunk adds to a zero state, and the chunk's total decay;
//                   2. a scan over the chunks, which leaves the state each chunk starts from (and the final one);
//                   3. the outputs: read-out of the incoming state, plus A V with A_ti the decayed score of token
//                      t and an earlier token i of the chunk.
//                   A chunk is cut into four runs of 16 tokens. Sums of log decays are kept within a run, and the
//                   weight of a (query, key) pair factors at the end of the key's run: the key's factor is the
//                   exponential of a non-positive sum, and so is the query's if it is in a later run. Inside a run the
//                   query's factor grows, at most to 2^110: a run in which some channel decays by more than that
//                   forms its weights pair by pair instead. Weighted rows, scores and the state enter the tensor-core
//                   products as bf16 pairs (high and low part), about 16 bits.
#include "attn_mma.cuh"
#include "elem_io.cuh"

namespace nf {
namespace {

// Largest |log2 of a decay|: beyond it the decayed value is zero in fp32 anyway, and sums of 16 stay exact enough.
constexpr float kMaxDecayLog2 = 150.f;
__device__ __forceinline__ float decay_log2(float x) { return -fminf(expf(x) * kLog2e, kMaxDecayLog2); }

// ---- token shift ------------------------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(256)
token_shift_kernel(nfk_token_shift_params p) {
  const int ld = static_cast<int>(p.ld_h);
  for (int t = blockIdx.x; t < p.T; t += gridDim.x) {
    const int req = p.token_req[t];
    const int t0 = p.qo_indptr[req], t1 = p.qo_indptr[req + 1];
    const int ref = p.state_slot[req], slot = ref >> 1, half = ref & 1;
    const bool ok = ref >= 0 && slot < p.num_slots;
    if (!ok && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    const T* h = reinterpret_cast<const T*>(p.h) + static_cast<long long>(t) * ld;
    T* st = reinterpret_cast<T*>(p.state) + static_cast<long long>(ok ? slot : 0) * 2 * ld;
    const T* before = nullptr;
    if (t > t0) before = h - ld;
    else if (p.positions[t] > 0 && ok) before = st + static_cast<long long>(half) * ld;
    T* keep = (t + 1 == t1 && ok) ? st + static_cast<long long>(half ^ 1) * ld : nullptr;
    T* out = reinterpret_cast<T*>(p.out) + static_cast<long long>(t) * p.n_mix * ld;
    for (int c = threadIdx.x * 4; c < ld; c += 256 * 4) {
      const float4 x = load4(h + c);
      const float4 b = before != nullptr ? load4(before + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      for (int s = 0; s < p.n_mix; ++s) {
        const float4 m = load4(p.mu + static_cast<long long>(s) * ld + c);
        store4(out + static_cast<long long>(s) * ld + c,
               make_float4(x.x + (b.x - x.x) * m.x, x.y + (b.y - x.y) * m.y, x.z + (b.z - x.z) * m.z, x.w + (b.w - x.w) * m.w));
      }
      if (keep != nullptr) store4(keep + c, x);
    }
  }
}

// ---- decode -------------------------------------------------------------------------------------------------
struct WkvState {
  float* S;
  bool ok, fresh;
};
__device__ __forceinline__ WkvState wkv_state(const nfk_wkv_params& p, int req, int head) {
  WkvState s;
  const int ref = p.state_slot[req];
  s.ok = ref >= 0 && (ref >> 1) < p.num_slots;
  s.fresh = p.positions[p.qo_indptr[req]] == 0;
  s.S = p.S + (static_cast<long long>(s.ok ? ref >> 1 : 0) * p.heads + head) * p.dim * p.dim;
  if (!s.ok && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
  return s;
}

__device__ __forceinline__ float wkv_sum256(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < 8 ? red[lane] : 0.f);
}
__device__ __forceinline__ float silu_f(float g) { return g / (1.f + expf(-g)); }
__device__ __forceinline__ float silu_fast(float g) { return __fdividef(g, 1.f + __expf(-g)); }   // for bf16 results

// LC lanes share a row of S (four columns each, 4 * LC columns at a time), 256 / LC rows are in work at once. NR > 0: the
// head fits into one pass of NR rows per thread, which are fetched before anything else.
template <class T, int LC, int NR>
__global__ void __launch_bounds__(256)
wkv_decode_kernel(nfk_wkv_params p) {
  constexpr int R = 256 / LC;
  extern __shared__ float dsm[];                 // r | k | decay | o, [dim] each
  __shared__ float red[8];
  __shared__ float4 part[8][LC];
  float *r_s = dsm, *k_s = r_s + p.dim, *w_s = k_s + p.dim, *o_s = w_s + p.dim;
  const int head = blockIdx.x % p.heads, req = p.req_begin + blockIdx.x / p.heads;
  const int lc = threadIdx.x % LC, lr = threadIdx.x / LC;
  const WkvState st = wkv_state(p, req, head);
  if (!st.ok) return;
  const long long tok = p.qo_indptr[req];
  const int hc = head * p.dim;
  const T* row = reinterpret_cast<const T*>(p.rkvg) + tok * p.ld + hc;
  float4 pre[NR > 0 ? NR : 1];
  if (NR > 0) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = lr + i * R;
      pre[i] = (st.fresh || d >= p.dim || lc * 4 >= p.dim) ? make_float4(0.f, 0.f, 0.f, 0.f)
                                                           : load4(st.S + static_cast<long long>(d) * p.dim + lc * 4);
    }
  }
  float bonus = 0.f;
  for (int d = threadIdx.x; d < p.dim; d += 256) {
    const float r = to_f32(row[p.r_off + d]), k = to_f32(row[p.k_off + d]);
    r_s[d] = r;
    k_s[d] = k;
    w_s[d] = expf(-expf(p.x[tok * p.ld_x + hc + d]));
    bonus += r * p.u[hc + d] * k;
  }
  bonus = wkv_sum256(bonus, red);                // also orders r_s, k_s, w_s
  auto update = [&](float4 s, int d, float4 v, float4& acc, float* dst) {
    const float rd = r_s[d], kd = k_s[d], wd = w_s[d];
    acc.x += s.x * rd; acc.y += s.y * rd; acc.z += s.z * rd; acc.w += s.w * rd;
    store4(dst, make_float4(wd * s.x + kd * v.x, wd * s.y + kd * v.y, wd * s.z + kd * v.z, wd * s.w + kd * v.w));
  };
  for (int c0 = 0; c0 < p.dim; c0 += LC * 4) {
    const int col = c0 + lc * 4;
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f), v = acc;
    if (col < p.dim) {
      v = load4(row + p.v_off + col);
      float* S = st.S + col;
      if (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const int d = lr + i * R;
          if (d < p.dim) update(pre[i], d, v, acc, S + static_cast<long long>(d) * p.dim);
        }
      } else {
#pragma unroll 8
        for (int d = lr; d < p.dim; d += R) {
          float* sp = S + static_cast<long long>(d) * p.dim;
          update(st.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(sp), d, v, acc, sp);
        }
      }
    }
    // rows that share a warp are added up by shuffles, warps through shared memory
#pragma unroll
    for (int o = LC; o < 32; o <<= 1) {
      acc.x += __shfl_xor_sync(0xffffffffu, acc.x, o);
      acc.y += __shfl_xor_sync(0xffffffffu, acc.y, o);
      acc.z += __shfl_xor_sync(0xffffffffu, acc.z, o);
      acc.w += __shfl_xor_sync(0xffffffffu, acc.w, o);
    }
    const int warp = threadIdx.x >> 5;
    if ((threadIdx.x & 31) < LC) part[warp][lc] = acc;
    __syncthreads();
    if (lr == 0 && col < p.dim) {
#pragma unroll
      for (int w = 1; w < 8; ++w) {
        const float4 o = part[w][lc];
        acc.x += o.x; acc.y += o.y; acc.z += o.z; acc.w += o.w;
      }
      store4(o_s + col, make_float4(acc.x + bonus * v.x, acc.y + bonus * v.y, acc.z + bonus * v.z, acc.w + bonus * v.w));
    }
    __syncthreads();
  }
  float ss = 0.f;
  for (int d = threadIdx.x; d < p.dim; d += 256) ss += o_s[d] * o_s[d];      // padding columns are zero
  const float inv = rsqrtf(wkv_sum256(ss, red) / static_cast<float>(p.dim_real) + p.eps);
  T* y = reinterpret_cast<T*>(p.y) + tok * p.ld_y + hc;
  for (int d = threadIdx.x; d < p.dim; d += 256)
    put(y + d, o_s[d] * inv * p.norm[hc + d] * silu_f(to_f32(row[p.g_off + d])));
}

// ---- prefill, token by token ----------------------------------------------------------------------------------
constexpr int kSeqCols = 32;

template <class T>
__global__ void __launch_bounds__(256)
wkv_seq_kernel(nfk_wkv_params p, int v_slices) {
  extern __shared__ float dsm[];                 // S[dim][32] | r | k | decay
  __shared__ float red[8];
  __shared__ float part[8][32];
  float* S_s = dsm;
  float *r_s = S_s + p.dim * kSeqCols, *k_s = r_s + p.dim, *w_s = k_s + p.dim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vs = blockIdx.x % v_slices;
  const int head = (blockIdx.x / v_slices) % p.heads;
  const int req = p.seq_reqs[blockIdx.x / (v_slices * p.heads)];
  const WkvState st = wkv_state(p, req, head);
  if (!st.ok) return;
  const int t0 = p.qo_indptr[req], t1 = p.qo_indptr[req + 1], hc = head * p.dim;
  const int col = vs * kSeqCols + lane;
  const bool col_ok = col < p.dim;
  float* S = st.S + col;
  for (int d = warp; d < p.dim; d += 8)
    S_s[d * kSeqCols + lane] = (st.fresh || !col_ok) ? 0.f : S[static_cast<long long>(d) * p.dim];
  for (int t = t0; t < t1; ++t) {
    const T* row = reinterpret_cast<const T*>(p.rkvg) + static_cast<long long>(t) * p.ld + hc;
    __syncthreads();                             // the previous token's reads are done
    float bonus = 0.f;
    for (int d = threadIdx.x; d < p.dim; d += 256) {
      const float r = to_f32(row[p.r_off + d]), k = to_f32(row[p.k_off + d]);
      r_s[d] = r;
      k_s[d] = k;
      w_s[d] = expf(-expf(p.x[static_cast<long long>(t) * p.ld_x + hc + d]));
      bonus += r * p.u[hc + d] * k;
    }
    bonus = wkv_sum256(bonus, red);
    const float v = col_ok ? to_f32(row[p.v_off + col]) : 0.f;
    float acc = 0.f;
    for (int d = warp; d < p.dim; d += 8) {
      const float s = S_s[d * kSeqCols + lane];
      acc += s * r_s[d];
      S_s[d * kSeqCols + lane] = w_s[d] * s + k_s[d] * v;
    }
    part[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && col_ok) {
      for (int w = 1; w < 8; ++w) acc += part[w][lane];
      p.o[static_cast<long long>(t) * p.heads * p.dim + hc + col] = acc + bonus * v;
    }
  }
  __syncthreads();
  for (int d = warp; d < p.dim; d += 8)
    if (col_ok) S[static_cast<long long>(d) * p.dim] = S_s[d * kSeqCols + lane];
}

// Head norm, weight and gate of the rows that wkv_seq_kernel left in p.o: one warp per (token, head).
template <class T>
__global__ void __launch_bounds__(256)
wkv_seq_norm_kernel(nfk_wkv_params p) {
  const int lane = threadIdx.x & 31;
  const int req = p.seq_reqs[blockIdx.y];
  const int t0 = p.qo_indptr[req];
  const long long total = static_cast<long long>(p.qo_indptr[req + 1] - t0) * p.heads;
  for (long long i = blockIdx.x * 8ll + (threadIdx.x >> 5); i < total; i += gridDim.x * 8ll) {
    const long long t = t0 + i / p.heads;
    const int hc = static_cast<int>(i % p.heads) * p.dim;
    const float* o = p.o + t * p.heads * p.dim + hc;
    float ss = 0.f;
    for (int c = lane * 4; c < p.dim; c += 128) {
      const float4 v = load4(o + c);
      ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(p.dim_real) + p.eps);
    const T* g = reinterpret_cast<const T*>(p.rkvg) + t * p.ld + p.g_off + hc;
    T* y = reinterpret_cast<T*>(p.y) + t * p.ld_y + hc;
    for (int c = lane * 4; c < p.dim; c += 128) {
      const float4 v = load4(o + c), w = load4(p.norm + hc + c), gg = load4(g + c);
      store4(y + c, make_float4(v.x * inv * w.x * silu_f(gg.x), v.y * inv * w.y * silu_f(gg.y),
                                v.z * inv * w.z * silu_f(gg.z), v.w * inv * w.w * silu_f(gg.w)));
    }
  }
}

// ---- prefill, chunks of 64 tokens -------------------------------------------------------------------------------
constexpr int kChunk = 64, kRun = 16, kRuns = kChunk / kRun;
constexpr float kMaxRunLog2 = 110.f;       // largest decay of a run (log2) whose weights are factored inside the run

__host__ __device__ __forceinline__ long long wkv_item_floats(int dim) { return static_cast<long long>(dim) * dim + dim; }

template <int DP>
struct WkvCfg {
  static constexpr int BLD = DP + 8;                     // bf16 row stride: conflict-free ldmatrix
  static constexpr int FLD = DP + 4;                     // fp32 row stride
  static constexpr int ALD = kChunk + 8;
  static constexpr int ROWS_BYTES = kChunk * BLD * 2;    // r, k or v
  static constexpr int CE_BYTES = kChunk * FLD * 4;
  static constexpr int TOT_BYTES = kRuns * DP * 4;
  static constexpr int S_BYTES = DP * BLD * 2;           // one part
  static constexpr int A_BYTES = kChunk * ALD * 2;       // one part
  static constexpr int STATE_SMEM = 2 * ROWS_BYTES + CE_BYTES + TOT_BYTES;
  static constexpr int OUT_SMEM = 5 * ROWS_BYTES + CE_BYTES + TOT_BYTES + 2 * S_BYTES + 2 * A_BYTES + DP * 4 + 3 * kChunk * 4 + 16;
};

// A chunk's operands are all requested before any of them is waited for: rows of r, k, v by asynchronous copies, logs
// of the decays (and the incoming state) into registers.
__device__ __forceinline__ void cp_async16_or_zero(void* smem_dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem_dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
// 64 rows of a head's columns of rkvg into [64][BLD]; rows past `n` and columns past the head's are zero.
template <int DP>
__device__ __forceinline__ void load_rows(__nv_bfloat16* dst, const nfk_wkv_params& p, long long tok0, int n, int col0) {
  constexpr int CH = DP / 8;
  const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.rkvg);
#pragma unroll
  for (int j = 0; j < kChunk * CH / 256; ++j) {
    const int i = threadIdx.x + j * 256, r = i / CH, c = (i % CH) * 8;
    const bool ok = r < n && c < p.dim;
    cp_async16_or_zero(dst + r * WkvCfg<DP>::BLD + c, src + (ok ? (tok0 + r) * p.ld + col0 + c : 0), ok);
  }
}
template <int DP>
struct DecayRegs {
  static constexpr int N = kChunk * (DP / 4) / 256;
  float4 v[N];
  __device__ __forceinline__ void fetch(const nfk_wkv_params& p, long long tok0, int n, int hc) {
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const int i = threadIdx.x + j * 256, r = i / (DP / 4), c = (i % (DP / 4)) * 4;
      // no decay past the last token: the chunk's total is that of its tokens
      v[j] = (r < n && c < p.dim) ? load4(p.x + (tok0 + r) * p.ld_x + hc + c) : make_float4(-INFINITY, -INFINITY, -INFINITY, -INFINITY);
    }
  }
  // ce[t][d]: sum of the log2 decays of the tokens of t's run before t; tot[run][d]: sum over the run. Also waits for the
  // rows.
  __device__ __forceinline__ void finish(float* ce, float* tot, int* slow) const {
    constexpr int FLD = WkvCfg<DP>::FLD;
#pragma unroll
    for (int j = 0; j < N; ++j) {
      const int i = threadIdx.x + j * 256, r = i / (DP / 4), c = (i % (DP / 4)) * 4;
      store4(ce + r * FLD + c, make_float4(decay_log2(v[j].x), decay_log2(v[j].y), decay_log2(v[j].z), decay_log2(v[j].w)));
    }
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    for (int i = threadIdx.x; i < kRuns * DP; i += 256) {
      const int run = i / DP, d = i % DP;
      float l[kRun], s = 0.f;
#pragma unroll
      for (int j = 0; j < kRun; ++j) l[j] = ce[(run * kRun + j) * FLD + d];
#pragma unroll
      for (int j = 0; j < kRun; ++j) {
        ce[(run * kRun + j) * FLD + d] = s;
        s += l[j];
      }
      tot[i] = s;
      if (slow != nullptr && s < -kMaxRunLog2) slow[run] = 1;
    }
    __syncthreads();
  }
};
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}

// Pass 1: sum over the chunk's tokens of (decayed key) x value, [dim][dim], and the chunk's decay.
template <int DP>
__global__ void __launch_bounds__(256)
wkv_chunk_state_kernel(nfk_wkv_params p) {
  using C = WkvCfg<DP>;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(smem + C::ROWS_BYTES);
  float* ce = reinterpret_cast<float*>(smem + 2 * C::ROWS_BYTES);
  float* tot = reinterpret_cast<float*>(smem + 2 * C::ROWS_BYTES + C::CE_BYTES);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x % p.heads, item = blockIdx.x / p.heads;
  const int n = p.items[item * 4 + 2], hc = head * p.dim;
  const long long tok0 = p.items[item * 4 + 1];
  load_rows<DP>(k_s, p, tok0, n, p.k_off + hc);
  load_rows<DP>(v_s, p, tok0, n, p.v_off + hc);
  DecayRegs<DP> dec;
  dec.fetch(p, tok0, n, hc);
  dec.finish(ce, tot, nullptr);
  float* L = p.scratch + (static_cast<long long>(item) * p.heads + head) * wkv_item_floats(p.dim);
  for (int d = threadIdx.x; d < p.dim; d += 256)
    L[p.dim * p.dim + d] = fast_exp2((tot[d] + tot[DP + d]) + (tot[2 * DP + d] + tot[3 * DP + d]));
  // warps over 16-row tiles of the key channels and, for the small size, halves of the columns
  constexpr int MT = DP / 16, WN = 8 / MT, NT = DP / 8 / WN;
  const int m0 = (warp % MT) * 16, n0 = (warp / MT) * NT;
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
  const int mm = lane >> 3, rr = lane & 7;
  const uint32_t vb = smem_u32(v_s);
  const int d0 = m0 + (lane >> 2), d1 = d0 + 8;
#pragma unroll
  for (int run = 0; run < kRuns; ++run) {
    // what decays a key after its token: the rest of its run, then the later runs
    float after0 = 0.f, after1 = 0.f;
#pragma unroll
    for (int j = run; j < kRuns; ++j) {
      after0 += tot[j * DP + d0];
      after1 += tot[j * DP + d1];
    }
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int j = half * 8 + (lane & 3) * 2;           // token of the run
      float x0[2], x1[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = run * kRun + j + e;
        const bool last = j + e == kRun - 1;
        const float c0 = last ? tot[run * DP + d0] : ce[(t + 1) * C::FLD + d0];
        const float c1 = last ? tot[run * DP + d1] : ce[(t + 1) * C::FLD + d1];
        x0[e] = to_f32(k_s[t * C::BLD + d0]) * fast_exp2(after0 - c0);
        x1[e] = to_f32(k_s[t * C::BLD + d1]) * fast_exp2(after1 - c1);
      }
      split_pair(x0[0], x0[1], hi[half * 2], lo[half * 2]);
      split_pair(x1[0], x1[1], hi[half * 2 + 1], lo[half * 2 + 1]);
    }
#pragma unroll
    for (int i = 0; i < NT; i += 2) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4_trans(vb + ((run * kRun + (mm & 1) * 8 + rr) * C::BLD + (n0 + i + (mm >> 1)) * 8) * 2, b0, b1, b2, b3);
      mma_bf16(acc[i], hi, b0, b1);
      mma_bf16(acc[i + 1], hi, b2, b3);
      mma_bf16(acc[i], lo, b0, b1);
      mma_bf16(acc[i + 1], lo, b2, b3);
    }
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    const int v = (n0 + i) * 8 + (lane & 3) * 2;
    if (v >= p.dim) continue;
    if (d0 < p.dim) *reinterpret_cast<float2*>(L + d0 * p.dim + v) = make_float2(acc[i][0], acc[i][1]);
    if (d1 < p.dim) *reinterpret_cast<float2*>(L + d1 * p.dim + v) = make_float2(acc[i][2], acc[i][3]);
  }
}

// Pass 2: chunk contributions -> incoming states, in place; the final state goes to the request's slot. One thread
// per four elements of S.
__global__ void __launch_bounds__(256)
wkv_scan_kernel(nfk_wkv_params p, int e_blocks) {
  const int eb = blockIdx.x % e_blocks;
  const int head = (blockIdx.x / e_blocks) % p.heads;
  const int item0 = blockIdx.x / (e_blocks * p.heads);
  if (p.items[item0 * 4 + 3] != 0) return;                 // not the first chunk of a portion
  const int req = p.items[item0 * 4];
  const WkvState st = wkv_state(p, req, head);
  if (!st.ok) return;
  const int e = (eb * 256 + threadIdx.x) * 4;
  if (e >= p.dim * p.dim) return;
  const int d = e / p.dim;
  const int n = (p.qo_indptr[req + 1] - p.qo_indptr[req] + kChunk - 1) / kChunk;
  const long long step = static_cast<long long>(p.heads) * wkv_item_floats(p.dim);
  float* sc = p.scratch + (static_cast<long long>(item0) * p.heads + head) * wkv_item_floats(p.dim);
  float4 R = st.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(st.S + e);
  constexpr int B = 8;
  for (int c0 = 0; c0 < n; c0 += B) {
    float4 L[B];
    float w[B];
#pragma unroll
    for (int i = 0; i < B; ++i)
      if (c0 + i < n && item0 + c0 + i < p.num_items) {
        L[i] = load4(sc + (c0 + i) * step + e);
        w[i] = sc[(c0 + i) * step + p.dim * p.dim + d];
      }
#pragma unroll
    for (int i = 0; i < B; ++i)
      if (c0 + i < n && item0 + c0 + i < p.num_items) {
        store4(sc + (c0 + i) * step + e, R);
        R.x = w[i] * R.x + L[i].x;
        R.y = w[i] * R.y + L[i].y;
        R.z = w[i] * R.z + L[i].z;
        R.w = w[i] * R.w + L[i].w;
      }
  }
  store4(st.S + e, R);
}

// Pass 3: outputs of a chunk, normed, weighted and gated.
template <int DP>
__global__ void __launch_bounds__(256)
wkv_chunk_out_kernel(nfk_wkv_params p) {
  using C = WkvCfg<DP>;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* r_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem + C::ROWS_BYTES);
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(smem + 2 * C::ROWS_BYTES);
  __nv_bfloat16* kh_s = reinterpret_cast<__nv_bfloat16*>(smem + 3 * C::ROWS_BYTES);      // decayed keys, two parts
  __nv_bfloat16* kl_s = reinterpret_cast<__nv_bfloat16*>(smem + 4 * C::ROWS_BYTES);
  float* ce = reinterpret_cast<float*>(smem + 5 * C::ROWS_BYTES);
  float* tot = reinterpret_cast<float*>(smem + 5 * C::ROWS_BYTES + C::CE_BYTES);
  __nv_bfloat16* sh_s = reinterpret_cast<__nv_bfloat16*>(tot + kRuns * DP);              // incoming state, two parts
  __nv_bfloat16* sl_s = sh_s + DP * C::BLD;
  __nv_bfloat16* ah_s = sl_s + DP * C::BLD;                                             // scores, two parts
  __nv_bfloat16* al_s = ah_s + kChunk * C::ALD;
  float* u_s = reinterpret_cast<float*>(al_s + kChunk * C::ALD);
  float* bonus_s = u_s + DP;                               // [64]
  float* ss_s = bonus_s + kChunk;                          // [2][64]
  int* slow_s = reinterpret_cast<int*>(ss_s + 2 * kChunk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x % p.heads, item = blockIdx.x / p.heads;
  const int n = p.items[item * 4 + 2], hc = head * p.dim;
  const long long tok0 = p.items[item * 4 + 1];
  load_rows<DP>(r_s, p, tok0, n, p.r_off + hc);
  load_rows<DP>(k_s, p, tok0, n, p.k_off + hc);
  load_rows<DP>(v_s, p, tok0, n, p.v_off + hc);
  DecayRegs<DP> dec;
  dec.fetch(p, tok0, n, hc);
  const float* S = p.scratch + (static_cast<long long>(item) * p.heads + head) * wkv_item_floats(p.dim);
  constexpr int SN = DP * (DP / 4) / 256;
  float4 s_in[SN];
#pragma unroll
  for (int j = 0; j < SN; ++j) {
    const int i = threadIdx.x + j * 256, d = i / (DP / 4), c = (i % (DP / 4)) * 4;
    s_in[j] = (d < p.dim && c < p.dim) ? load4(S + d * p.dim + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  for (int d = threadIdx.x; d < DP; d += 256) u_s[d] = d < p.dim ? p.u[hc + d] : 0.f;
  if (threadIdx.x < kRuns) slow_s[threadIdx.x] = 0;
#pragma unroll
  for (int j = 0; j < SN; ++j) {
    const int i = threadIdx.x + j * 256, d = i / (DP / 4), c = (i % (DP / 4)) * 4;
    uint2 hi, lo;
    split_pair(s_in[j].x, s_in[j].y, hi.x, lo.x);
    split_pair(s_in[j].z, s_in[j].w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(sh_s + d * C::BLD + c) = hi;
    *reinterpret_cast<uint2*>(sl_s + d * C::BLD + c) = lo;
  }
  dec.finish(ce, tot, slow_s);

  // ---- keys decayed to the end of their run, and every token's own score ----
  for (int i = threadIdx.x; i < kChunk * (DP / 2); i += 256) {
    const int t = i / (DP / 2), d = (i % (DP / 2)) * 2;
    const float2 k = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_s + t * C::BLD + d));
    const float2 e = *reinterpret_cast<const float2*>(tot + (t / kRun) * DP + d);
    const float2 c = (t & (kRun - 1)) == kRun - 1 ? e : *reinterpret_cast<const float2*>(ce + (t + 1) * C::FLD + d);
    uint32_t hi, lo;
    split_pair(k.x * fast_exp2(e.x - c.x), k.y * fast_exp2(e.y - c.y), hi, lo);
    *reinterpret_cast<uint32_t*>(kh_s + t * C::BLD + d) = hi;
    *reinterpret_cast<uint32_t*>(kl_s + t * C::BLD + d) = lo;
  }
  {
    const int t = threadIdx.x >> 2;
    float b = 0.f;
#pragma unroll
    for (int d = (threadIdx.x & 3) * 2; d < DP; d += 8) {
      const float2 r = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r_s + t * C::BLD + d));
      const float2 k = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_s + t * C::BLD + d));
      b += r.x * k.x * u_s[d] + r.y * k.y * u_s[d + 1];
    }
    b = quad_sum(b);
    if ((threadIdx.x & 3) == 0) bonus_s[t] = b;
  }
  __syncthreads();

  // ---- scores and read-out of the incoming state. A warp takes a run `a` of queries; one of the run's two warps has
  // the key runs 0 and 2 and the first half of the columns, the other one key runs 1 and 3 and the second half ----
  constexpr int NT = DP / 16;
  const int half = warp >> 2, a = half == 0 ? warp & 3 : 3 - (warp & 3), n0 = half * NT;
  const int t0 = a * kRun + (lane >> 2);
  const int mm = lane >> 3, rr = lane & 7;
  const uint32_t khb = smem_u32(kh_s), klb = smem_u32(kl_s), shb = smem_u32(sh_s), slb = smem_u32(sl_s);
  float acc[NT][4], sc[2][2][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 2; ++j) sc[i][j][0] = sc[i][j][1] = sc[i][j][2] = sc[i][j][3] = 0.f;
  const bool has[2] = {half <= a && !(half == a && slow_s[a] != 0), half + 2 <= a && !(half + 2 == a && slow_s[a] != 0)};
#pragma unroll 1
  for (int ks = 0; ks < DP / 16; ++ks) {
    // queries decayed to the start of their run
    float2 f[2][2], pre[2], own[2], cum[2][2];
#pragma unroll
    for (int dh = 0; dh < 2; ++dh) {
      const int d = ks * 16 + dh * 8 + (lane & 3) * 2;
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float2 r = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r_s + (t0 + h * 8) * C::BLD + d));
        const float2 c = *reinterpret_cast<const float2*>(ce + (t0 + h * 8) * C::FLD + d);
        f[dh][h] = make_float2(r.x * fast_exp2(c.x), r.y * fast_exp2(c.y));
      }
      // log decays of the runs before `a`, and of those between each of this warp's key runs and `a` (within a run: what
      // takes the query back from the run's end)
      pre[dh] = make_float2(0.f, 0.f);
      cum[0][dh] = cum[1][dh] = make_float2(0.f, 0.f);
#pragma unroll
      for (int j = 0; j < kRuns; ++j) {
        const float2 x = *reinterpret_cast<const float2*>(tot + j * DP + d);
        if (j == a) own[dh] = x;
        if (j < a) {
          pre[dh].x += x.x;
          pre[dh].y += x.y;
          if (j > half) {
            cum[0][dh].x += x.x;
            cum[0][dh].y += x.y;
          }
          if (j > half + 2) {
            cum[1][dh].x += x.x;
            cum[1][dh].y += x.y;
          }
        }
      }
#pragma unroll
      for (int s = 0; s < 2; ++s)
        if (half + 2 * s == a) cum[s][dh] = make_float2(-own[dh].x, -own[dh].y);
    }
    uint32_t qh[4], ql[4];
    auto weighted = [&](const float2 (&e)[2]) {
#pragma unroll
      for (int dh = 0; dh < 2; ++dh) {
        const float ex = fast_exp2(e[dh].x), ey = fast_exp2(e[dh].y);
#pragma unroll
        for (int h = 0; h < 2; ++h) split_pair(f[dh][h].x * ex, f[dh][h].y * ey, qh[dh * 2 + h], ql[dh * 2 + h]);
      }
    };
#pragma unroll
    for (int s = 0; s < 2; ++s) {
      if (!has[s]) continue;
      weighted(cum[s]);
      const uint32_t o = (((half + 2 * s) * kRun + (mm >> 1) * 8 + rr) * C::BLD + (2 * ks + (mm & 1)) * 8) * 2;
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm_x4(khb + o, h0, h1, h2, h3);
      ldsm_x4(klb + o, l0, l1, l2, l3);
      mma_bf16(sc[s][0], qh, h0, h1);
      mma_bf16(sc[s][1], qh, h2, h3);
      mma_bf16(sc[s][0], qh, l0, l1);
      mma_bf16(sc[s][1], qh, l2, l3);
      mma_bf16(sc[s][0], ql, h0, h1);
      mma_bf16(sc[s][1], ql, h2, h3);
    }
    weighted(pre);
#pragma unroll
    for (int i = 0; i < NT; i += 2) {
      const uint32_t o = ((ks * 16 + (mm & 1) * 8 + rr) * C::BLD + (n0 + i + (mm >> 1)) * 8) * 2;
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm_x4_trans(shb + o, h0, h1, h2, h3);
      ldsm_x4_trans(slb + o, l0, l1, l2, l3);
      mma_bf16(acc[i], qh, h0, h1);
      mma_bf16(acc[i + 1], qh, h2, h3);
      mma_bf16(acc[i], qh, l0, l1);
      mma_bf16(acc[i + 1], qh, l2, l3);
      mma_bf16(acc[i], ql, h0, h1);
      mma_bf16(acc[i + 1], ql, h2, h3);
    }
  }
#pragma unroll
  for (int s = 0; s < 2; ++s) {
    if (!has[s]) continue;
    const int b = half + 2 * s;
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = t0 + h * 8, i = b * kRun + j * 8 + (lane & 3) * 2;
        float x = sc[s][j][2 * h], y = sc[s][j][2 * h + 1];
        if (b == a) {                       // the token itself with its bonus, later ones not at all
          x = i < t ? x : i == t ? bonus_s[t] : 0.f;
          y = i + 1 < t ? y : i + 1 == t ? bonus_s[t] : 0.f;
        }
        uint32_t hi, lo;
        split_pair(x, y, hi, lo);
        *reinterpret_cast<uint32_t*>(ah_s + t * C::ALD + i) = hi;
        *reinterpret_cast<uint32_t*>(al_s + t * C::ALD + i) = lo;
      }
  }
  // ---- runs that decay too much for factored weights: 64 threads per run, 2 x 2 (query, key) pairs each ----
  if (slow_s[threadIdx.x >> 6] != 0) {
    const int run = threadIdx.x >> 6, ti = (threadIdx.x >> 3) & 7, ii = threadIdx.x & 7;
    const int t = run * kRun + ti * 2, i = run * kRun + ii * 2;
    float a00 = 0.f, a10 = 0.f, a11 = 0.f, a01 = 0.f;      // a[query][key]
    if (ii < ti) {
#pragma unroll 2
      for (int d = 0; d < DP; d += 2) {
        const float2 r0 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r_s + t * C::BLD + d));
        const float2 r1 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r_s + (t + 1) * C::BLD + d));
        const float2 k0 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_s + i * C::BLD + d));
        const float2 k1 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_s + (i + 1) * C::BLD + d));
        const float2 q0 = *reinterpret_cast<const float2*>(ce + t * C::FLD + d);
        const float2 q1 = *reinterpret_cast<const float2*>(ce + (t + 1) * C::FLD + d);
        const float2 c0 = *reinterpret_cast<const float2*>(ce + (i + 1) * C::FLD + d);   // through key i
        const float2 c1 = *reinterpret_cast<const float2*>(ce + (i + 2) * C::FLD + d);   // through key i + 1 <= t - 1
        a00 += r0.x * k0.x * fast_exp2(q0.x - c0.x) + r0.y * k0.y * fast_exp2(q0.y - c0.y);
        a01 += r0.x * k1.x * fast_exp2(q0.x - c1.x) + r0.y * k1.y * fast_exp2(q0.y - c1.y);
        a10 += r1.x * k0.x * fast_exp2(q1.x - c0.x) + r1.y * k0.y * fast_exp2(q1.y - c0.y);
        a11 += r1.x * k1.x * fast_exp2(q1.x - c1.x) + r1.y * k1.y * fast_exp2(q1.y - c1.y);
      }
    } else if (ii == ti) {
      a00 = bonus_s[t];
      a11 = bonus_s[t + 1];
      for (int d = 0; d < DP; d += 2) {                    // the token right before: not decayed yet
        const float2 r1 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(r_s + (t + 1) * C::BLD + d));
        const float2 k0 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_s + i * C::BLD + d));
        a10 += r1.x * k0.x + r1.y * k0.y;
      }
    }
    uint32_t hi, lo;
    split_pair(a00, a01, hi, lo);
    *reinterpret_cast<uint32_t*>(ah_s + t * C::ALD + i) = hi;
    *reinterpret_cast<uint32_t*>(al_s + t * C::ALD + i) = lo;
    split_pair(a10, a11, hi, lo);
    *reinterpret_cast<uint32_t*>(ah_s + (t + 1) * C::ALD + i) = hi;
    *reinterpret_cast<uint32_t*>(al_s + (t + 1) * C::ALD + i) = lo;
  }
  __syncthreads();

  // ---- scores times values ----
  const uint32_t vb = smem_u32(v_s), ahb = smem_u32(ah_s), alb = smem_u32(al_s);
#pragma unroll
  for (int ks = 0; ks < kRuns; ++ks) {
    if (ks > a) continue;
    uint32_t ph[4], pl[4];
    const uint32_t ao = ((a * kRun + (lane & 15)) * C::ALD + ks * 16 + (lane >> 4) * 8) * 2;
    ldsm_x4(ahb + ao, ph[0], ph[1], ph[2], ph[3]);
    ldsm_x4(alb + ao, pl[0], pl[1], pl[2], pl[3]);
#pragma unroll
    for (int i = 0; i < NT; i += 2) {
      uint32_t b0, b1, b2, b3;
      ldsm_x4_trans(vb + ((ks * 16 + (mm & 1) * 8 + rr) * C::BLD + (n0 + i + (mm >> 1)) * 8) * 2, b0, b1, b2, b3);
      mma_bf16(acc[i], ph, b0, b1);
      mma_bf16(acc[i + 1], ph, b2, b3);
      mma_bf16(acc[i], pl, b0, b1);
      mma_bf16(acc[i + 1], pl, b2, b3);
    }
  }
  // ---- head norm over both column halves, weight, gate ----
  const __nv_bfloat16* rkvg = reinterpret_cast<const __nv_bfloat16*>(p.rkvg);
  uint32_t gate[2][NT];
#pragma unroll
  for (int h = 0; h < 2; ++h)
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int t = t0 + h * 8, v = (n0 + i) * 8 + (lane & 3) * 2;
      gate[h][i] = (t < n && v < p.dim) ? *reinterpret_cast<const uint32_t*>(rkvg + (tok0 + t) * p.ld + p.g_off + hc + v) : 0u;
    }
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NT; ++i) ss += acc[i][2 * h] * acc[i][2 * h] + acc[i][2 * h + 1] * acc[i][2 * h + 1];
    ss = quad_sum(ss);
    if ((lane & 3) == 0) ss_s[half * kChunk + t0 + h * 8] = ss;
  }
  __syncthreads();
  __nv_bfloat16* y = reinterpret_cast<__nv_bfloat16*>(p.y);
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    const int t = t0 + h * 8;
    if (t >= n) continue;
    const float inv = rsqrtf((ss_s[t] + ss_s[kChunk + t]) / static_cast<float>(p.dim_real) + p.eps);
    __nv_bfloat16* dst = y + (tok0 + t) * p.ld_y + hc;
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int v = (n0 + i) * 8 + (lane & 3) * 2;
      if (v >= p.dim) continue;
      const float2 gg = unpack_bf16x2(gate[h][i]);
      const float2 w = *reinterpret_cast<const float2*>(p.norm + hc + v);
      *reinterpret_cast<uint32_t*>(dst + v) =
          pack_bf16x2(acc[i][2 * h] * inv * w.x * silu_fast(gg.x), acc[i][2 * h + 1] * inv * w.y * silu_fast(gg.y));
    }
  }
}

template <class K>
int set_smem(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return NF_ERR_UNSUPPORTED;
  if (bytes > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)) != cudaSuccess)
    return NF_ERR_CUDA;
  return NF_OK;
}

int check_wkv(const nfk_wkv_params* p) {
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (!p->rkvg || !p->x || !p->u || !p->norm || !p->S || !p->y || !p->positions || !p->qo_indptr || !p->state_slot)
    return NF_ERR_BAD_ARG;
  if (p->heads <= 0 || p->dim <= 0 || p->dim % 8 != 0 || p->dim_real <= 0 || p->dim_real > p->dim || p->num_slots <= 0)
    return NF_ERR_BAD_ARG;
  if (p->ld % 8 != 0 || p->r_off % 8 != 0 || p->k_off % 8 != 0 || p->v_off % 8 != 0 || p->g_off % 8 != 0 ||
      p->ld_x % 4 != 0 || p->ld_y % 8 != 0 || (reinterpret_cast<uintptr_t>(p->rkvg) & 15) != 0)
    return NF_ERR_BAD_ARG;
  return NF_OK;
}

template <int DP>
int launch_wkv_chunks(const nfk_wkv_params& p, cudaStream_t stream) {
  using C = WkvCfg<DP>;
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    int rc = set_smem(wkv_chunk_state_kernel<DP>, C::STATE_SMEM);
    if (rc == NF_OK) rc = set_smem(wkv_chunk_out_kernel<DP>, C::OUT_SMEM);
    if (rc != NF_OK) return rc;
    attr = true;
  }
  const int grid = p.num_items * p.heads;
  wkv_chunk_state_kernel<DP><<<grid, 256, C::STATE_SMEM, stream>>>(p);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  const int e_blocks = (p.dim * p.dim + 1023) / 1024;
  wkv_scan_kernel<<<grid * e_blocks, 256, 0, stream>>>(p, e_blocks);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  wkv_chunk_out_kernel<DP><<<grid, 256, C::OUT_SMEM, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

template <class T>
int launch_wkv_seq(const nfk_wkv_params& p, cudaStream_t stream) {
  const int v_slices = (p.dim + kSeqCols - 1) / kSeqCols;
  const size_t sm = static_cast<size_t>(p.dim) * (kSeqCols + 3) * 4;
  const long long grid = static_cast<long long>(p.num_seq) * p.heads * v_slices;
  if (grid > 0x7fffffffll || p.num_seq > 65535) return NF_ERR_BAD_ARG;
  const int rc = set_smem(wkv_seq_kernel<T>, sm);
  if (rc != NF_OK) return rc;
  wkv_seq_kernel<T><<<static_cast<int>(grid), 256, sm, stream>>>(p, v_slices);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  wkv_seq_norm_kernel<T><<<dim3(64, p.num_seq), 256, 0, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

template <class T>
int launch_wkv_decode(const nfk_wkv_params& p, cudaStream_t stream) {
  const long long grid = static_cast<long long>(p.req_count) * p.heads;
  const size_t sm = static_cast<size_t>(p.dim) * 16;
  if (grid > 0x7fffffffll || sm > 40 * 1024) return NF_ERR_BAD_ARG;
  const int g = static_cast<int>(grid);
  if (p.dim <= 32) wkv_decode_kernel<T, 8, 1><<<g, 256, sm, stream>>>(p);
  else if (p.dim <= 64) wkv_decode_kernel<T, 16, 4><<<g, 256, sm, stream>>>(p);
  else if (p.dim <= 128) wkv_decode_kernel<T, 32, 16><<<g, 256, sm, stream>>>(p);
  else wkv_decode_kernel<T, 32, 0><<<g, 256, sm, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_token_shift(const nfk_token_shift_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == 0) return NF_OK;
  if (!p->h || !p->out || !p->mu || !p->state || !p->state_slot || !p->positions || !p->token_req || !p->qo_indptr ||
      p->T < 0 || p->n_mix <= 0 || p->num_slots <= 0 || p->ld_h <= 0 || p->ld_h % 4 != 0)
    return NF_ERR_BAD_ARG;
  int grid = 8 * device_sm_count();
  if (grid > p->T) grid = p->T;
  if (p->dtype == NFK_F32) token_shift_kernel<float><<<grid, 256, 0, stream>>>(*p);
  else token_shift_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_wkv_decode(const nfk_wkv_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_wkv(p);
  if (rc != NF_OK) return rc;
  if (p->req_count == 0) return NF_OK;
  if (p->req_count < 0 || p->req_begin < 0) return NF_ERR_BAD_ARG;
  return p->dtype == NFK_F32 ? launch_wkv_decode<float>(*p, stream) : launch_wkv_decode<__nv_bfloat16>(*p, stream);
}

extern "C" int nfk_wkv_prefill(const nfk_wkv_params* p, cudaStream_t stream) {
  using namespace nf;
  int rc = check_wkv(p);
  if (rc != NF_OK) return rc;
  if (p->num_seq < 0 || p->num_items < 0 || (p->num_seq > 0 && (!p->seq_reqs || !p->o)) || (p->num_items > 0 && !p->items))
    return NF_ERR_BAD_ARG;
  if (p->num_items > 0) {
    if (p->dtype != NFK_BF16 || p->dim > 128) return NF_ERR_UNSUPPORTED;
    if (p->scratch == nullptr || (reinterpret_cast<uintptr_t>(p->scratch) & 15) != 0 ||
        p->num_items * static_cast<long long>(p->heads) * wkv_item_floats(p->dim) > p->scratch_floats)
      return NF_ERR_BAD_ARG;
    rc = p->dim <= 64 ? launch_wkv_chunks<64>(*p, stream) : launch_wkv_chunks<128>(*p, stream);
    if (rc != NF_OK) return rc;
  }
  if (p->num_seq == 0) return NF_OK;
  return p->dtype == NFK_F32 ? launch_wkv_seq<float>(*p, stream) : launch_wkv_seq<__nv_bfloat16>(*p, stream);
}
