// Delta-rule recurrence with a decay per key channel and token (Yang et al., "Gated Delta Networks: Improving Mamba2 with
// Delta Rule", with a vector of decays in place of one per head; see kernels.h for the equations). State, unit vectors,
// decays, step sizes and everything derived from them are fp32.
//
// nfk_delta_decode   one token per request: a CTA per request and head streams S through registers (recall, read-out and
//                    update in one pass: o = S'^T q = (diag(w) S)^T q + (q . k) u), then head norm, weight and gate.
// nfk_delta_prefill  token by token (any size, bf16 or fp32), S in shared memory; or in chunks of 64 tokens on tensor cores
//                    (bf16). With c_t the sum of log decays from the chunk's start through token t, the values written are
//                        u_t = beta_t (v_t - S0^T (e^c_t k_t) - sum_{s<t} <k_t, k_s>_ts u_s),  <x, y>_ts = sum_d x y e^(c_t - c_s),
//                    a lower-triangular system with the same matrix for all columns. Three kernels:
//                    1. per chunk: the decayed scores <k, k> and <q, k>, the inverse M = (1 + diag(beta) <k, k>)^-1 diag(beta)
//                       (forward substitution in fp32, by blocks of 16), then M V and W = M (e^c k);
//                    2. along the chunks, 32 columns of S per CTA, S in registers: u = M V - W S0, the outputs
//                       (e^c q) S0 + <q, k> u, and S = e^c_end S0 + (e^(c_end - c) k)^T u;
//                    3. head norm, weight and gate.
//                    Decayed rows, scores, W, u and S enter the products as bf16 pairs (high and low part, about 16 bits).
//                    Weights of scores factor at the ends of runs of 16 tokens: the key's factor is the exponential of a
//                    non-positive sum, and so is the query's in a later run; inside a run the query's factor grows, at most to
//                    2^110, and a run in which some channel decays by more forms its scores pair by pair.
#include "attn_mma.cuh"
#include "elem_io.cuh"

namespace nf {
namespace {

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float delta_decay(float x, float bias, float rate) { return expf(-rate * softplus_f(x + bias)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
// With the special-function unit's exponential and logarithm; small values by their series, which keeps them exact to a
// few units in the last place.
__device__ __forceinline__ float softplus_fast(float x) {
  const float e = __expf(x);
  return x > 20.f ? x : e < 0.015625f ? e * (1.f - e * (0.5f - e * (0.33333333f - 0.25f * e))) : __logf(1.f + e);
}
__device__ __forceinline__ float sigmoid_fast(float z) { return __fdividef(1.f, 1.f + __expf(-z)); }

struct DeltaState {
  float* S;
  bool ok, fresh;
};
__device__ __forceinline__ DeltaState delta_state(const nfk_delta_params& p, int req, int head) {
  DeltaState s;
  const int ref = p.state_slot[req];
  s.ok = ref >= 0 && (ref >> 1) < p.num_slots;
  s.fresh = p.positions[p.qo_indptr[req]] == 0;
  s.S = p.S + (static_cast<long long>(s.ok ? ref >> 1 : 0) * p.heads + head) * p.dim * p.vdim;
  if (!s.ok && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
  return s;
}

// Sums over the CTA of three values per thread; every thread gets them. The leading barrier also orders what was written
// to shared memory before the call.
__device__ __forceinline__ float3 cta_sum3(float3 v, float (*red)[8]) {
  v = make_float3(warp_sum(v.x), warp_sum(v.y), warp_sum(v.z));
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) {
    red[0][warp] = v.x;
    red[1][warp] = v.y;
    red[2][warp] = v.z;
  }
  __syncthreads();
  return make_float3(warp_sum(lane < 8 ? red[0][lane] : 0.f), warp_sum(lane < 8 ? red[1][lane] : 0.f),
                     warp_sum(lane < 8 ? red[2][lane] : 0.f));
}

// The head's query and key as they are, decays, and (returned) the factors that make them unit vectors and their product.
template <class T>
__device__ __forceinline__ float3 load_qk(const nfk_delta_params& p, long long tok, int head, float* q_s, float* k_s, float* w_s,
                                          float (*red)[8]) {
  const int kvh = head / (p.heads / p.kv_heads);
  const T* q = reinterpret_cast<const T*>(p.qkv) + tok * p.ld + p.q_off + kvh * p.dim;
  const T* k = reinterpret_cast<const T*>(p.qkv) + tok * p.ld + p.k_off + kvh * p.dim;
  const float rate = p.rate[head];
  float3 s = make_float3(0.f, 0.f, 0.f);
  for (int d = threadIdx.x; d < p.dim; d += 256) {
    const float qd = to_f32(q[d]), kd = to_f32(k[d]);
    q_s[d] = qd;
    k_s[d] = kd;
    w_s[d] = delta_decay(p.x[tok * p.ld_x + head * p.dim + d], p.dt_bias[head * p.dim + d], rate);
    s.x += qd * qd;
    s.y += kd * kd;
    s.z += qd * kd;
  }
  s = cta_sum3(s, red);
  const float qn = rsqrtf(s.x + p.unit_eps) * p.q_scale, kn = rsqrtf(s.y + p.unit_eps);
  return make_float3(qn, kn, s.z * qn * kn);
}

__device__ __forceinline__ void fma4(float4& a, float f, float4 b) {
  a.x += f * b.x; a.y += f * b.y; a.z += f * b.z; a.w += f * b.w;
}

// LC lanes share a row of S (four columns each, 4 * LC columns at a time), 256 / LC rows are in work at once. NR > 0: the
// head fits into one pass of NR rows per thread, which are fetched before anything else and stay in registers.
template <class T, int LC, int NR>
__global__ void __launch_bounds__(256)
delta_decode_kernel(nfk_delta_params p) {
  constexpr int R = 256 / LC;
  extern __shared__ float dsm[];                 // q | k | decay [dim] each | o [vdim]
  __shared__ float red[3][8];
  __shared__ float4 part[2][8][LC];
  float *q_s = dsm, *k_s = q_s + p.dim, *w_s = k_s + p.dim, *o_s = w_s + p.dim;
  const int head = blockIdx.x % p.heads, req = p.req_begin + blockIdx.x / p.heads;
  const int lc = threadIdx.x % LC, lr = threadIdx.x / LC;
  const DeltaState st = delta_state(p, req, head);
  if (!st.ok) return;
  const long long tok = p.qo_indptr[req];
  auto row_of = [&](int d, int col) {
    return st.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : load4(st.S + static_cast<long long>(d) * p.vdim + col);
  };
  float4 pre[NR > 0 ? NR : 1];
  if (NR > 0) {
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = lr + i * R;
      pre[i] = (d < p.dim && lc * 4 < p.vdim) ? row_of(d, lc * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  const float beta = sigmoid_f(p.beta[tok * p.ld_b + head]);
  const float3 f = load_qk<T>(p, tok, head, q_s, k_s, w_s, red);
  const T* v_row = reinterpret_cast<const T*>(p.qkv) + tok * p.ld + p.v_off + head * p.vdim;
  for (int c0 = 0; c0 < p.vdim; c0 += LC * 4) {
    const int col = c0 + lc * 4;
    const bool ok = col < p.vdim;
    float4 recall = make_float4(0.f, 0.f, 0.f, 0.f), read = recall;
    if (ok) {
      if (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const int d = lr + i * R;
          if (d < p.dim) {
            const float w = w_s[d];
            pre[i] = make_float4(w * pre[i].x, w * pre[i].y, w * pre[i].z, w * pre[i].w);
            fma4(recall, k_s[d], pre[i]);
            fma4(read, q_s[d], pre[i]);
          }
        }
      } else {
#pragma unroll 4
        for (int d = lr; d < p.dim; d += R) {
          const float4 s = row_of(d, col);
          fma4(recall, k_s[d] * w_s[d], s);
          fma4(read, q_s[d] * w_s[d], s);
        }
      }
    }
    // rows that share a warp are added up by shuffles, warps through shared memory
#pragma unroll
    for (int o = LC; o < 32; o <<= 1) {
      recall.x += __shfl_xor_sync(0xffffffffu, recall.x, o); recall.y += __shfl_xor_sync(0xffffffffu, recall.y, o);
      recall.z += __shfl_xor_sync(0xffffffffu, recall.z, o); recall.w += __shfl_xor_sync(0xffffffffu, recall.w, o);
      read.x += __shfl_xor_sync(0xffffffffu, read.x, o); read.y += __shfl_xor_sync(0xffffffffu, read.y, o);
      read.z += __shfl_xor_sync(0xffffffffu, read.z, o); read.w += __shfl_xor_sync(0xffffffffu, read.w, o);
    }
    if ((threadIdx.x & 31) < LC) {
      part[0][threadIdx.x >> 5][lc] = recall;
      part[1][threadIdx.x >> 5][lc] = read;
    }
    __syncthreads();
    recall = read = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      fma4(recall, f.y, part[0][w][lc]);
      fma4(read, f.x, part[1][w][lc]);
    }
    if (ok) {
      const float4 v = load4(v_row + col);
      const float4 u = make_float4(beta * (v.x - recall.x), beta * (v.y - recall.y), beta * (v.z - recall.z), beta * (v.w - recall.w));
      if (lr == 0) {
        fma4(read, f.z, u);
        store4(o_s + col, read);
      }
      float* S = st.S + col;
      if (NR > 0) {
#pragma unroll
        for (int i = 0; i < NR; ++i) {
          const int d = lr + i * R;
          if (d < p.dim) {
            fma4(pre[i], k_s[d] * f.y, u);
            store4(S + static_cast<long long>(d) * p.vdim, pre[i]);
          }
        }
      } else {
#pragma unroll 4
        for (int d = lr; d < p.dim; d += R) {
          const float w = w_s[d];
          float4 s = row_of(d, col);
          s = make_float4(w * s.x, w * s.y, w * s.z, w * s.w);
          fma4(s, k_s[d] * f.y, u);
          store4(S + static_cast<long long>(d) * p.vdim, s);
        }
      }
    }
    __syncthreads();
  }
  float ss = 0.f;
  for (int d = threadIdx.x; d < p.vdim; d += 256) ss += o_s[d] * o_s[d];      // padding columns are zero
  const float inv = rsqrtf(cta_sum3(make_float3(ss, 0.f, 0.f), red).x / static_cast<float>(p.vdim_real) + p.eps);
  const T* g = reinterpret_cast<const T*>(p.g) + tok * p.ld_g + head * p.vdim;
  T* y = reinterpret_cast<T*>(p.y) + tok * p.ld_y + head * p.vdim;
  for (int d = threadIdx.x; d < p.vdim; d += 256) put(y + d, o_s[d] * inv * p.norm[d] * sigmoid_f(to_f32(g[d])));
}

// ---- prefill, token by token ----------------------------------------------------------------------------------
constexpr int kSeqCols = 32;

template <class T>
__global__ void __launch_bounds__(256)
delta_seq_kernel(nfk_delta_params p, int v_slices) {
  extern __shared__ float dsm[];                 // S[dim][32] | q | k | decay
  __shared__ float red[3][8];
  __shared__ float part[2][8][32];
  float* S_s = dsm;
  float *q_s = S_s + p.dim * kSeqCols, *k_s = q_s + p.dim, *w_s = k_s + p.dim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vs = blockIdx.x % v_slices;
  const int head = (blockIdx.x / v_slices) % p.heads;
  const int req = p.seq_reqs[blockIdx.x / (v_slices * p.heads)];
  const DeltaState st = delta_state(p, req, head);
  if (!st.ok) return;
  const int t0 = p.qo_indptr[req], t1 = p.qo_indptr[req + 1];
  const int col = vs * kSeqCols + lane;
  const bool col_ok = col < p.vdim;
  float* S = st.S + col;
  for (int d = warp; d < p.dim; d += 8)
    S_s[d * kSeqCols + lane] = (st.fresh || !col_ok) ? 0.f : S[static_cast<long long>(d) * p.vdim];
  for (int t = t0; t < t1; ++t) {
    __syncthreads();                             // the previous token's reads are done
    const float3 f = load_qk<T>(p, t, head, q_s, k_s, w_s, red);
    float recall = 0.f, read = 0.f;
    for (int d = warp; d < p.dim; d += 8) {
      const float s = w_s[d] * S_s[d * kSeqCols + lane];
      S_s[d * kSeqCols + lane] = s;
      recall += k_s[d] * s;
      read += q_s[d] * s;
    }
    part[0][warp][lane] = recall;
    part[1][warp][lane] = read;
    __syncthreads();
    recall = read = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      recall += part[0][w][lane];
      read += part[1][w][lane];
    }
    const float v = col_ok ? to_f32(reinterpret_cast<const T*>(p.qkv)[t * p.ld + p.v_off + head * p.vdim + col]) : 0.f;
    const float u = sigmoid_f(p.beta[t * p.ld_b + head]) * (v - f.y * recall);
    for (int d = warp; d < p.dim; d += 8) S_s[d * kSeqCols + lane] += k_s[d] * f.y * u;
    if (warp == 0 && col_ok) p.o[(static_cast<long long>(t) * p.heads + head) * p.vdim + col] = f.x * read + f.z * u;
  }
  __syncthreads();
  for (int d = warp; d < p.dim; d += 8)
    if (col_ok) S[static_cast<long long>(d) * p.vdim] = S_s[d * kSeqCols + lane];
}

// Head norm, weight and gate of the rows that delta_seq_kernel left in p.o: one warp per (token, head).
template <class T>
__global__ void __launch_bounds__(256)
delta_seq_norm_kernel(nfk_delta_params p) {
  const int lane = threadIdx.x & 31;
  const int req = p.seq_reqs[blockIdx.y], t0 = p.qo_indptr[req];
  const unsigned total = static_cast<unsigned>(p.qo_indptr[req + 1] - t0) * p.heads;
  for (unsigned i = blockIdx.x * 8u + (threadIdx.x >> 5); i < total; i += gridDim.x * 8u) {
    const unsigned row = i / static_cast<unsigned>(p.heads);
    const long long t = t0 + static_cast<long long>(row);
    const int head = static_cast<int>(i - row * p.heads);
    const float* o = p.o + (t * p.heads + head) * p.vdim;
    float ss = 0.f;
    for (int c = lane * 4; c < p.vdim; c += 128) {
      const float4 v = load4(o + c);
      ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(p.vdim_real) + p.eps);
    const T* g = reinterpret_cast<const T*>(p.g) + t * p.ld_g + head * p.vdim;
    T* y = reinterpret_cast<T*>(p.y) + t * p.ld_y + head * p.vdim;
    for (int c = lane * 4; c < p.vdim; c += 128) {
      const float4 v = load4(o + c), w = load4(p.norm + c), gg = load4(g + c);
      store4(y + c, make_float4(v.x * inv * w.x * sigmoid_f(gg.x), v.y * inv * w.y * sigmoid_f(gg.y),
                                v.z * inv * w.z * sigmoid_f(gg.z), v.w * inv * w.w * sigmoid_f(gg.w)));
    }
  }
}

// ---- prefill, chunks of 64 tokens -------------------------------------------------------------------------------
constexpr int kChunk = 64, kRun = 16, kRuns = kChunk / kRun, kDcThreads = 1024, kDsThreads = 512, kDsGroup = kDsThreads / 2;
constexpr int kDcWarps = kDcThreads / 32;
constexpr int kSlice = 32;                 // columns of S per CTA of the second kernel
constexpr float kMaxRunLog2 = 110.f;       // largest decay of a run (log2) whose weights are factored inside the run
constexpr float kMaxDecayLog2 = 150.f;     // a stronger decay is zero in fp32 anyway

// Scratch of a chunk and head, laid out as the second kernel keeps it in shared memory (padded rows), so that a few bulk
// copies bring it in: W [2 parts][64][P + 8] | decayed keys alike | the chunk's decay [P] fp32 | decayed queries as W | scores
// [2][64][72] | M V [P / 32 slices][64][36] fp32. P: the head's size rounded up to 64 or 128, columns past it are zero.
template <int P>
struct DeltaItem {
  static constexpr int BLD = P + 8, MLD = kChunk + 8, ULD = kSlice + 4;
  static constexpr int PAIR = 2 * kChunk * BLD * 2, A = 2 * kChunk * MLD * 2, U = kChunk * ULD * 4;      // bytes
  static constexpr int KEYS = PAIR + P * 4, READ = PAIR + A;             // what S is updated with, what outputs need
  static constexpr int BYTES = PAIR + KEYS + READ + P / kSlice * U;
  __nv_bfloat16 *w, *k, *q, *a;
  float *decay, *u;
  __device__ __forceinline__ DeltaItem(const nfk_delta_params& p, int item, int head) {
    char* b = reinterpret_cast<char*>(p.scratch) + (static_cast<long long>(item) * p.heads + head) * BYTES;
    w = reinterpret_cast<__nv_bfloat16*>(b);
    k = reinterpret_cast<__nv_bfloat16*>(b + PAIR);
    decay = reinterpret_cast<float*>(b + 2 * PAIR);
    q = reinterpret_cast<__nv_bfloat16*>(b + PAIR + KEYS);
    a = reinterpret_cast<__nv_bfloat16*>(b + 2 * PAIR + KEYS);
    u = reinterpret_cast<float*>(b + PAIR + KEYS + READ);
  }
};
__host__ __device__ __forceinline__ long long delta_item_floats(int dim, int vdim) {
  return (dim <= 64 && vdim <= 64 ? DeltaItem<64>::BYTES : DeltaItem<128>::BYTES) / 4;
}
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  const float2 h = unpack_bf16x2(hi);
  lo = pack_bf16x2(x - h.x, y - h.y);
}
// Untiled bulk copy global -> shared, counted by an mbarrier.
__device__ __forceinline__ void bulk_load(void* smem_dst, const void* src, int bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(smem_dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}
__device__ __forceinline__ void cp_async16_or_zero(void* smem_dst, const void* src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem_dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}

template <int P>
struct DeltaChunkCfg {
  static constexpr int BLD = P + 8;                      // bf16 row stride: conflict-free ldmatrix
  static constexpr int FLD = P + 4;                      // fp32 row stride
  static constexpr int MLD = kChunk + 8, XLD = kChunk + 4;
  static constexpr int ROWS = kChunk * BLD * 2;
  static constexpr int CE = kChunk * FLD * 4, TOT = kRuns * P * 4, M = kChunk * MLD * 2, X = kChunk * XLD * 4;
  // q | k | v | decayed keys (pair) | log decays | sums of runs, of those before, of those after | N | X | Y | M (pair) | factors
  static constexpr int SMEM = 5 * ROWS + CE + 3 * TOT + 2 * X + 16 * kChunk * 4 + 2 * M + 3 * kChunk * 4 + 16;
};

template <int P>
__global__ void __launch_bounds__(kDcThreads, 1)
delta_chunk_kernel(nfk_delta_params p) {
  using C = DeltaChunkCfg<P>;
  extern __shared__ __align__(16) uint8_t smem[];
  __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* k_s = q_s + kChunk * C::BLD;
  __nv_bfloat16* v_s = k_s + kChunk * C::BLD;
  __nv_bfloat16* kh_s = v_s + kChunk * C::BLD;
  __nv_bfloat16* kl_s = kh_s + kChunk * C::BLD;
  float* ce = reinterpret_cast<float*>(kl_s + kChunk * C::BLD);     // log2 decays through a token, from its run's start
  float* tot = ce + kChunk * C::FLD;                                 // ... of whole runs
  float* pre = tot + kRuns * P;                                      // ... of the runs before, and of those after
  float* post = pre + kRuns * P;
  float* n_s = post + kRuns * P;                                     // diag(beta) <k, k>, strictly lower
  float* x_s = n_s + kChunk * C::XLD;                                // its (1 + N)^-1
  float* y_s = x_s + kChunk * C::XLD;                                // [16][64]
  __nv_bfloat16* mh_s = reinterpret_cast<__nv_bfloat16*>(y_s + 16 * kChunk);
  __nv_bfloat16* ml_s = mh_s + kChunk * C::MLD;
  float* qn_s = reinterpret_cast<float*>(ml_s + kChunk * C::MLD);    // factors that make queries and keys unit vectors
  float* kn_s = qn_s + kChunk;
  float* beta_s = kn_s + kChunk;
  int* slow_s = reinterpret_cast<int*>(beta_s + kChunk);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.x % p.heads, item = blockIdx.x / p.heads, kvh = head / (p.heads / p.kv_heads);
  const int n = p.items[item * 4 + 2];
  const long long tok0 = p.items[item * 4 + 1];
  const DeltaItem<P> out(p, item, head);

  // ---- operands: all requested before any of them is waited for ----
  {
    const __nv_bfloat16* src = reinterpret_cast<const __nv_bfloat16*>(p.qkv);
    constexpr int CH = P / 8;
    const int off[3] = {p.q_off + kvh * p.dim, p.k_off + kvh * p.dim, p.v_off + head * p.vdim};
#pragma unroll
    for (int a = 0; a < 3; ++a)
#pragma unroll
      for (int i = threadIdx.x; i < kChunk * CH; i += kDcThreads) {
        const int r = i / CH, c = (i % CH) * 8;
        const bool ok = r < n && c < (a == 2 ? p.vdim : p.dim);
        cp_async16_or_zero(q_s + a * kChunk * C::BLD + r * C::BLD + c, src + (ok ? (tok0 + r) * p.ld + off[a] + c : 0), ok);
      }
    cp_async_commit();
  }
  const float rate = p.rate[head] * kLog2e;
  for (int i = threadIdx.x; i < kChunk * (P / 4); i += kDcThreads) {
    const int r = i / (P / 4), c = (i % (P / 4)) * 4;
    float4 l = make_float4(0.f, 0.f, 0.f, 0.f);           // no decay past the last token: the chunk's is that of its tokens
    if (r < n && c < p.dim) {
      const float4 x = load4(p.x + (tok0 + r) * p.ld_x + head * p.dim + c), b = load4(p.dt_bias + head * p.dim + c);
      l = make_float4(-fminf(rate * softplus_fast(x.x + b.x), kMaxDecayLog2), -fminf(rate * softplus_fast(x.y + b.y), kMaxDecayLog2),
                      -fminf(rate * softplus_fast(x.z + b.z), kMaxDecayLog2), -fminf(rate * softplus_fast(x.w + b.w), kMaxDecayLog2));
    }
    store4(ce + r * C::FLD + c, l);
  }
  if (threadIdx.x < kRuns) slow_s[threadIdx.x] = 0;
  cp_async_wait<0>();
  __syncthreads();

  // ---- sums of log decays, norms, step sizes ----
  for (int i = threadIdx.x; i < kRuns * P; i += kDcThreads) {
    const int run = i / P, d = i % P;
    float s = 0.f;
#pragma unroll
    for (int j = 0; j < kRun; ++j) {
      s += ce[(run * kRun + j) * C::FLD + d];
      ce[(run * kRun + j) * C::FLD + d] = s;
    }
    tot[i] = s;
    if (s < -kMaxRunLog2) slow_s[run] = 1;
  }
#pragma unroll
  for (int j = 0; j < kChunk / kDcWarps; ++j) {
    const int t = warp * (kChunk / kDcWarps) + j;
    float sq = 0.f, sk = 0.f;
    for (int d = lane * 2; d < P; d += 64) {
      const float2 a = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(q_s + t * C::BLD + d));
      const float2 b = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(k_s + t * C::BLD + d));
      sq += a.x * a.x + a.y * a.y;
      sk += b.x * b.x + b.y * b.y;
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      qn_s[t] = rsqrtf(sq + p.unit_eps) * p.q_scale;
      kn_s[t] = rsqrtf(sk + p.unit_eps);
      beta_s[t] = t < n ? sigmoid_f(p.beta[(tok0 + t) * p.ld_b + head]) : 0.f;
    }
  }
  __syncthreads();

  // ---- keys decayed to the end of their run; sums over runs ----
  for (int i = threadIdx.x; i < kChunk * (P / 4); i += kDcThreads) {
    const int t = i / (P / 4), d = (i % (P / 4)) * 4;
    const float4 k = load4(k_s + t * C::BLD + d), e = load4(tot + (t / kRun) * P + d), c = load4(ce + t * C::FLD + d);
    const float f = kn_s[t];
    uint2 hi, lo;
    split_pair(k.x * f * fast_exp2(e.x - c.x), k.y * f * fast_exp2(e.y - c.y), hi.x, lo.x);
    split_pair(k.z * f * fast_exp2(e.z - c.z), k.w * f * fast_exp2(e.w - c.w), hi.y, lo.y);
    *reinterpret_cast<uint2*>(kh_s + t * C::BLD + d) = hi;
    *reinterpret_cast<uint2*>(kl_s + t * C::BLD + d) = lo;
  }
  if (threadIdx.x < P) {
    const int d = threadIdx.x;
    float x = 0.f, y = 0.f;
#pragma unroll
    for (int j = 0; j < kRuns; ++j) {
      pre[j * P + d] = x;
      x += tot[j * P + d];
      post[(kRuns - 1 - j) * P + d] = y;
      y += tot[(kRuns - 1 - j) * P + d];
    }
    out.decay[d] = fast_exp2(x);
  }
  __syncthreads();

  // ---- scores of (row run a, key run b <= a), rows of queries and rows of keys with the same weights. Two warps share a
  // pair of runs, half of the key channels each ----
  const int mm = lane >> 3, rr = lane & 7;
  const uint32_t khb = smem_u32(kh_s), klb = smem_u32(kl_s);
  if (warp < kRuns * (kRuns + 1)) {
    const int half = warp & 1;
    int b = warp >> 1, a = 0;                              // the pair's number -> (a, b)
    while (b > a) {
      ++a;
      b -= a;
    }
    const int t0 = a * kRun + (lane >> 2), t1 = t0 + 8;
    const float q0 = qn_s[t0], q1 = qn_s[t1], f0 = kn_s[t0], f1 = kn_s[t1];
    float sc[2][2][4];                                     // [queries, keys][block of keys]
#pragma unroll
    for (int r = 0; r < 2; ++r)
#pragma unroll
      for (int j = 0; j < 2; ++j) sc[r][j][0] = sc[r][j][1] = sc[r][j][2] = sc[r][j][3] = 0.f;
    if (a == b && slow_s[a] != 0) {
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int t = e < 2 ? t0 : t1, s = b * kRun + j * 8 + (lane & 3) * 2 + (e & 1);
          if (s > t) continue;
          float x = 0.f, y = 0.f;
          for (int d = half * (P / 2); d < (half + 1) * (P / 2); ++d) {
            const float w = to_f32(k_s[s * C::BLD + d]) * fast_exp2(ce[t * C::FLD + d] - ce[s * C::FLD + d]);
            x += to_f32(q_s[t * C::BLD + d]) * w;
            y += to_f32(k_s[t * C::BLD + d]) * w;
          }
          sc[0][j][e] = x * (e < 2 ? q0 : q1) * kn_s[s];
          sc[1][j][e] = y * (e < 2 ? f0 : f1) * kn_s[s];
        }
    } else {
#pragma unroll 2
      for (int ks = half * (P / 32); ks < (half + 1) * (P / 32); ++ks) {
        uint32_t rh[2][4], rl[2][4];
#pragma unroll
        for (int dh = 0; dh < 2; ++dh) {
          const int d = ks * 16 + dh * 8 + (lane & 3) * 2;
          // log decays of the runs between; within a run: what takes the row back from the run's end
          float2 cum = make_float2(0.f, 0.f);
          if (a == b) {
            const float2 x = *reinterpret_cast<const float2*>(tot + a * P + d);
            cum = make_float2(-x.x, -x.y);
          }
          for (int j = b + 1; j < a; ++j) {
            const float2 x = *reinterpret_cast<const float2*>(tot + j * P + d);
            cum.x += x.x;
            cum.y += x.y;
          }
          const float2 c0 = *reinterpret_cast<const float2*>(ce + t0 * C::FLD + d);
          const float2 c1 = *reinterpret_cast<const float2*>(ce + t1 * C::FLD + d);
          const float2 w0 = make_float2(fast_exp2(c0.x + cum.x), fast_exp2(c0.y + cum.y));
          const float2 w1 = make_float2(fast_exp2(c1.x + cum.x), fast_exp2(c1.y + cum.y));
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const __nv_bfloat16* rows = r == 0 ? q_s : k_s;
            const float g0 = r == 0 ? q0 : f0, g1 = r == 0 ? q1 : f1;
            const float2 r0 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(rows + t0 * C::BLD + d));
            const float2 r1 = unpack_bf16x2(*reinterpret_cast<const uint32_t*>(rows + t1 * C::BLD + d));
            split_pair(r0.x * g0 * w0.x, r0.y * g0 * w0.y, rh[r][dh * 2], rl[r][dh * 2]);
            split_pair(r1.x * g1 * w1.x, r1.y * g1 * w1.y, rh[r][dh * 2 + 1], rl[r][dh * 2 + 1]);
          }
        }
        const uint32_t o = ((b * kRun + (mm >> 1) * 8 + rr) * C::BLD + (2 * ks + (mm & 1)) * 8) * 2;
        uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
        ldsm_x4(khb + o, h0, h1, h2, h3);
        ldsm_x4(klb + o, l0, l1, l2, l3);
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          mma_bf16(sc[r][0], rh[r], h0, h1);
          mma_bf16(sc[r][1], rh[r], h2, h3);
          mma_bf16(sc[r][0], rh[r], l0, l1);
          mma_bf16(sc[r][1], rh[r], l2, l3);
          mma_bf16(sc[r][0], rl[r], h0, h1);
          mma_bf16(sc[r][1], rl[r], h2, h3);
        }
      }
    }
    // each warp of the pair finishes one kind of rows: it gives the other kind's sums away (through the place of Y and M)
    float4* swap = reinterpret_cast<float4*>(y_s) + (warp >> 1) * 128 + half * 64 + lane;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float(&g)[4] = half == 0 ? sc[1][j] : sc[0][j];
      swap[j * 32] = make_float4(g[0], g[1], g[2], g[3]);
    }
    asm volatile("bar.sync %0, 64;" ::"r"((warp >> 1) + 1) : "memory");
    swap += half == 0 ? 64 : -64;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float4 other = swap[j * 32];
      const float z[4] = {other.x, other.y, other.z, other.w};
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = h == 0 ? t0 : t1, s = b * kRun + j * 8 + (lane & 3) * 2;
        const float x = (half == 0 ? sc[0][j][2 * h] : sc[1][j][2 * h]) + z[2 * h];
        const float y = (half == 0 ? sc[0][j][2 * h + 1] : sc[1][j][2 * h + 1]) + z[2 * h + 1];
        if (half == 1) {
          const float bt = beta_s[t];
          *reinterpret_cast<float2*>(n_s + t * C::XLD + s) = make_float2(s < t ? bt * x : 0.f, s + 1 < t ? bt * y : 0.f);
        } else {
          uint32_t hi, lo;
          split_pair(s <= t ? x : 0.f, s + 1 <= t ? y : 0.f, hi, lo);
          *reinterpret_cast<uint32_t*>(out.a + t * C::MLD + s) = hi;
          *reinterpret_cast<uint32_t*>(out.a + kChunk * C::MLD + t * C::MLD + s) = lo;
        }
      }
    }
  }
  __syncthreads();

  // ---- X = (1 + N)^-1: blocks on the diagonal column by column, then the rows of blocks below ----
  if (threadIdx.x < kChunk) {
    const int b0 = (threadIdx.x / kRun) * kRun, c = threadIdx.x % kRun;
    float x[kRun];
#pragma unroll
    for (int i = 0; i < kRun; ++i) {
      float s = i == c ? 1.f : 0.f;
#pragma unroll
      for (int j = 0; j < i; ++j) s -= n_s[(b0 + i) * C::XLD + b0 + j] * x[j];
      x[i] = i < c ? 0.f : s;
      x_s[(b0 + i) * C::XLD + b0 + c] = x[i];
    }
  }
  __syncthreads();
  for (int a = 1; a < kRuns; ++a) {
    const int w = a * kRun, groups = w / 4;                // four columns per thread
    const int r = threadIdx.x / groups, c = (threadIdx.x % groups) * 4;
    if (r < kRun) {
      float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int j = c / kRun * kRun; j < w; ++j) fma4(y, n_s[(w + r) * C::XLD + j], load4(x_s + j * C::XLD + c));
      store4(y_s + r * kChunk + c, y);
    }
    __syncthreads();
    if (r < kRun) {
      float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int j = 0; j <= r; ++j) fma4(x, -x_s[(w + r) * C::XLD + w + j], load4(y_s + j * kChunk + c));
      store4(x_s + (w + r) * C::XLD + c, x);
    }
    __syncthreads();
  }

  // ---- M, and what the second kernel reads: keys decayed to the chunk's end, queries decayed from its start; keys
  // decayed from its start take the place of those above ----
  for (int i = threadIdx.x; i < kChunk * kChunk / 4; i += kDcThreads) {
    const int t = i / (kChunk / 4), s = (i % (kChunk / 4)) * 4;
    const bool low = s <= t;                               // (blocks above the diagonal were never written)
    const float4 x = load4(x_s + t * C::XLD + s), bt = load4(beta_s + s);
    uint2 hi, lo;
    split_pair(low ? x.x * bt.x : 0.f, s + 1 <= t ? x.y * bt.y : 0.f, hi.x, lo.x);
    split_pair(s + 2 <= t ? x.z * bt.z : 0.f, s + 3 <= t ? x.w * bt.w : 0.f, hi.y, lo.y);
    *reinterpret_cast<uint2*>(mh_s + t * C::MLD + s) = hi;
    *reinterpret_cast<uint2*>(ml_s + t * C::MLD + s) = lo;
  }
  for (int i = threadIdx.x; i < kChunk * (P / 4); i += kDcThreads) {
    const int t = i / (P / 4), d = (i % (P / 4)) * 4, run = t / kRun;
    const float4 k = load4(k_s + t * C::BLD + d), q = load4(q_s + t * C::BLD + d), c = load4(ce + t * C::FLD + d);
    const float4 from = load4(pre + run * P + d), to = load4(post + run * P + d), own = load4(tot + run * P + d);
    const float kf = kn_s[t], qf = qn_s[t];
    const float4 e = make_float4(fast_exp2(from.x + c.x), fast_exp2(from.y + c.y), fast_exp2(from.z + c.z), fast_exp2(from.w + c.w));
    const float4 kk = make_float4(k.x * kf, k.y * kf, k.z * kf, k.w * kf);
    const int o = t * C::BLD + d, low = kChunk * C::BLD;
    uint2 hi, lo;
    split_pair(kk.x * e.x, kk.y * e.y, hi.x, lo.x);
    split_pair(kk.z * e.z, kk.w * e.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(kh_s + o) = hi;
    *reinterpret_cast<uint2*>(kl_s + o) = lo;
    split_pair(q.x * qf * e.x, q.y * qf * e.y, hi.x, lo.x);
    split_pair(q.z * qf * e.z, q.w * qf * e.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(out.q + o) = hi;
    *reinterpret_cast<uint2*>(out.q + low + o) = lo;
    split_pair(kk.x * fast_exp2((own.x - c.x) + to.x), kk.y * fast_exp2((own.y - c.y) + to.y), hi.x, lo.x);
    split_pair(kk.z * fast_exp2((own.z - c.z) + to.z), kk.w * fast_exp2((own.w - c.w) + to.w), hi.y, lo.y);
    *reinterpret_cast<uint2*>(out.k + o) = hi;
    *reinterpret_cast<uint2*>(out.k + low + o) = lo;
  }
  __syncthreads();

  // ---- M V and W = M (decayed keys): a warp takes a run of rows and an eighth of the columns ----
  constexpr int NT = P / 8 / (kDcWarps / 4);
  const int a = warp & 3, n0 = (warp >> 2) * NT;
  float u[NT][4], w[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    u[i][0] = u[i][1] = u[i][2] = u[i][3] = 0.f;
    w[i][0] = w[i][1] = w[i][2] = w[i][3] = 0.f;
  }
  const uint32_t vb = smem_u32(v_s), mhb = smem_u32(mh_s), mlb = smem_u32(ml_s);
  for (int ks = 0; ks <= a; ++ks) {
    uint32_t mh[4], ml[4];
    const uint32_t mo = ((a * kRun + (lane & 15)) * C::MLD + ks * 16 + (lane >> 4) * 8) * 2;
    ldsm_x4(mhb + mo, mh[0], mh[1], mh[2], mh[3]);
    ldsm_x4(mlb + mo, ml[0], ml[1], ml[2], ml[3]);
    // two blocks of columns per load; a warp with one block (the small size) loads its neighbour's too
#pragma unroll
    for (int i = 0; i < NT; i += 2) {
      const uint32_t o = ((ks * 16 + (mm & 1) * 8 + rr) * C::BLD + (NT == 1 ? n0 : n0 + i + (mm >> 1)) * 8) * 2;
      uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
      ldsm_x4_trans(vb + o, h0, h1, h2, h3);
      mma_bf16(u[i], mh, h0, h1);
      mma_bf16(u[i], ml, h0, h1);
      if (NT > 1) {
        mma_bf16(u[i + 1 < NT ? i + 1 : i], mh, h2, h3);
        mma_bf16(u[i + 1 < NT ? i + 1 : i], ml, h2, h3);
      }
      ldsm_x4_trans(khb + o, h0, h1, h2, h3);
      ldsm_x4_trans(klb + o, l0, l1, l2, l3);
      mma_bf16(w[i], mh, h0, h1);
      mma_bf16(w[i], mh, l0, l1);
      mma_bf16(w[i], ml, h0, h1);
      if (NT > 1) {
        mma_bf16(w[i + 1 < NT ? i + 1 : i], mh, h2, h3);
        mma_bf16(w[i + 1 < NT ? i + 1 : i], mh, l2, l3);
        mma_bf16(w[i + 1 < NT ? i + 1 : i], ml, h2, h3);
      }
    }
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int t = a * kRun + (lane >> 2) + h * 8, c = (n0 + i) * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(out.u + c / kSlice * (DeltaItem<P>::U / 4) + t * DeltaItem<P>::ULD + c % kSlice) =
          make_float2(u[i][2 * h], u[i][2 * h + 1]);
      uint32_t hi, lo;
      split_pair(w[i][2 * h], w[i][2 * h + 1], hi, lo);
      *reinterpret_cast<uint32_t*>(out.w + t * C::BLD + c) = hi;
      *reinterpret_cast<uint32_t*>(out.w + kChunk * C::BLD + t * C::BLD + c) = lo;
    }
}

template <int P>
struct DeltaScanCfg {
  using I = DeltaItem<P>;
  static constexpr int BLD = I::BLD, MLD = I::MLD, SLD = kSlice + 8, ULD = I::ULD;
  static constexpr int S = 2 * P * SLD * 2, U = 2 * kChunk * SLD * 2;    // pairs
  // W | M V | keys, decay | queries, scores | S (two buffers) | u (two buffers) | barriers
  static constexpr int SMEM = I::PAIR + I::U + I::KEYS + I::READ + 2 * S + 2 * U + 64;
};
__device__ __forceinline__ void named_sync(int id, int threads) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory"); }
__device__ __forceinline__ void named_arrive(int id, int threads) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(threads) : "memory"); }

// Two groups of eight warps. The first follows the chain from chunk to chunk (values written, next state); the second forms
// the outputs of a chunk from the state and the values that the first one left for it, one chunk behind at most.
template <int P>
__global__ void __launch_bounds__(kDsThreads, 1)
delta_scan_kernel(nfk_delta_params p, int slices) {
  using C = DeltaScanCfg<P>;
  using I = DeltaItem<P>;
  enum { kBarChain = 1, kBarOut = 2, kBarFull = 3, kBarFree = 5 };       // the last two: one per buffer
  extern __shared__ __align__(16) uint8_t smem[];
  uint8_t *w_b = smem, *mv_b = w_b + I::PAIR, *keys_b = mv_b + I::U, *read_b = keys_b + I::KEYS;
  float* mv_s = reinterpret_cast<float*>(mv_b);
  float* decay_s = reinterpret_cast<float*>(keys_b + I::PAIR);
  uint8_t *s_b = read_b + I::READ, *u_b = s_b + 2 * C::S;
  uint64_t* bar = reinterpret_cast<uint64_t*>(u_b + 2 * C::U);           // W and M V, keys, queries
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int v0 = (blockIdx.x % slices) * kSlice, head = (blockIdx.x / slices) % p.heads, portion = blockIdx.x / (slices * p.heads);
  int item0 = -1;                                          // first chunk of the portion
  for (int base = 0, before = 0; base < p.num_items; base += 32) {
    const unsigned firsts = __ballot_sync(0xffffffffu, base + lane < p.num_items && p.items[(base + lane) * 4 + 3] == 0);
    if (portion < before + __popc(firsts)) {
      item0 = base + static_cast<int>(__fns(firsts, 0, portion - before + 1));
      break;
    }
    before += __popc(firsts);
  }
  if (item0 < 0) return;
  const int req = p.items[item0 * 4];
  const DeltaState st = delta_state(p, req, head);
  if (!st.ok) return;
  const int n_tok = p.qo_indptr[req + 1] - p.qo_indptr[req];
  const int chunks = min((n_tok + kChunk - 1) / kChunk, p.num_items - item0);
  const long long tok0 = p.qo_indptr[req];

  auto fetch_w = [&](int c) {                              // one thread
    const I d(p, item0 + c, head);
    mbar_expect_tx(&bar[0], I::PAIR + I::U);
    bulk_load(w_b, d.w, I::PAIR, &bar[0]);
    bulk_load(mv_b, d.u + v0 / kSlice * (I::U / 4), I::U, &bar[0]);
  };
  auto fetch_keys = [&](int c) {
    const I d(p, item0 + c, head);
    mbar_expect_tx(&bar[1], I::KEYS);
    bulk_load(keys_b, d.k, I::KEYS, &bar[1]);
  };
  auto fetch_read = [&](int c) {
    const I d(p, item0 + c, head);
    mbar_expect_tx(&bar[2], I::READ);
    bulk_load(read_b, d.q, I::READ, &bar[2]);
  };
  if (threadIdx.x == 0) {
    for (int i = 0; i < 3; ++i) mbar_init(&bar[i], 1);
    mbar_fence_init();
    fetch_w(0);
    fetch_keys(0);
    fetch_read(0);
  }
  __syncthreads();
  // a wait that runs out is reported; the warps go on in step, so that they meet at their barriers
  auto arrived = [&](int i, int c) {
    if (!mbar_wait(&bar[i], c & 1)) report_status(p.status, NF_ST_TIMEOUT_SMEM_FULL);
  };
  const int mm = lane >> 3, rr = lane & 7;
  const int a = warp & 3, c0 = ((warp >> 2) & 1) * 16;     // a warp's run of rows and its columns
  const int t0 = a * kRun + (lane >> 2);
  const uint32_t wb = smem_u32(w_b), kb = smem_u32(keys_b), qb = smem_u32(read_b), ab = qb + I::PAIR;
  constexpr uint32_t R_LO = I::PAIR / 2, A_LO = I::A / 2, S_LO = C::S / 2, U_LO = C::U / 2;
  // acc += rows (pair, of this warp's run) x S (pair, this warp's columns)
  auto rows_times_s = [&](float (&acc)[2][4], uint32_t base, uint32_t sb) {
#pragma unroll
    for (int ks = 0; ks < P / 16; ++ks) {
      uint32_t rh[4], rl[4], h0, h1, h2, h3, l0, l1, l2, l3;
      const uint32_t ro = ((a * kRun + (lane & 15)) * C::BLD + ks * 16 + (lane >> 4) * 8) * 2;
      ldsm_x4(base + ro, rh[0], rh[1], rh[2], rh[3]);
      ldsm_x4(base + R_LO + ro, rl[0], rl[1], rl[2], rl[3]);
      const uint32_t so = ((ks * 16 + (mm & 1) * 8 + rr) * C::SLD + c0 + (mm >> 1) * 8) * 2;
      ldsm_x4_trans(sb + so, h0, h1, h2, h3);
      ldsm_x4_trans(sb + S_LO + so, l0, l1, l2, l3);
      mma_bf16(acc[0], rh, h0, h1);
      mma_bf16(acc[1], rh, h2, h3);
      mma_bf16(acc[0], rh, l0, l1);
      mma_bf16(acc[1], rh, l2, l3);
      mma_bf16(acc[0], rl, h0, h1);
      mma_bf16(acc[1], rl, h2, h3);
    }
  };

  if (warp >= kDsGroup / 32) {
    // ---- outputs ----
    for (int c = 0; c < chunks; ++c) {
      named_sync(kBarFull + (c & 1), kDsThreads);
      arrived(2, c);
      const uint32_t sb = smem_u32(s_b + (c & 1) * C::S), ub = smem_u32(u_b + (c & 1) * C::U);
      float acc[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
      rows_times_s(acc, qb, sb);
#pragma unroll
      for (int ks = 0; ks < kRuns; ++ks) {
        if (ks > a) continue;
        uint32_t ah[4], al[4], h0, h1, h2, h3, l0, l1, l2, l3;
        const uint32_t ao = ((a * kRun + (lane & 15)) * C::MLD + ks * 16 + (lane >> 4) * 8) * 2;
        ldsm_x4(ab + ao, ah[0], ah[1], ah[2], ah[3]);
        ldsm_x4(ab + A_LO + ao, al[0], al[1], al[2], al[3]);
        const uint32_t uo = ((ks * 16 + (mm & 1) * 8 + rr) * C::SLD + c0 + (mm >> 1) * 8) * 2;
        ldsm_x4_trans(ub + uo, h0, h1, h2, h3);
        ldsm_x4_trans(ub + U_LO + uo, l0, l1, l2, l3);
        mma_bf16(acc[0], ah, h0, h1);
        mma_bf16(acc[1], ah, h2, h3);
        mma_bf16(acc[0], ah, l0, l1);
        mma_bf16(acc[1], ah, l2, l3);
        mma_bf16(acc[0], al, h0, h1);
        mma_bf16(acc[1], al, h2, h3);
      }
      named_sync(kBarOut, kDsGroup);                       // queries and scores are read
      if (threadIdx.x == kDsGroup && c + 1 < chunks) fetch_read(c + 1);
      if (c + 2 < chunks) named_arrive(kBarFree + (c & 1), kDsThreads);      // (waited for when chunk c + 2 gets its state)
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int t = c * kChunk + t0 + h * 8, col = v0 + c0 + i * 8 + (lane & 3) * 2;
          if (t < n_tok && col < p.vdim)
            *reinterpret_cast<float2*>(p.o + ((tok0 + t) * p.heads + head) * p.vdim + col) = make_float2(acc[i][2 * h], acc[i][2 * h + 1]);
        }
    }
    return;
  }

  // ---- S: warps over 16-row tiles of the key channels and parts of the columns ----
  constexpr int MT = P / 16, SN = kSlice / 8 * MT / (kDsGroup / 32);     // row tiles; column blocks per warp
  const int sm0 = (warp % MT) * 16, sn0 = (warp / MT) * SN;
  const int d0 = sm0 + (lane >> 2), d1 = d0 + 8;
  float S[SN][4];
#pragma unroll
  for (int i = 0; i < SN; ++i) {
    const int c = (sn0 + i) * 8 + (lane & 3) * 2;
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int d = h == 0 ? d0 : d1;
      const bool ok = !st.fresh && d < p.dim && v0 + c < p.vdim;
      const float2 x = ok ? *reinterpret_cast<const float2*>(st.S + static_cast<long long>(d) * p.vdim + v0 + c) : make_float2(0.f, 0.f);
      S[i][2 * h] = x.x;
      S[i][2 * h + 1] = x.y;
    }
  }
  auto publish = [&](int buf) {
    __nv_bfloat16* dst = reinterpret_cast<__nv_bfloat16*>(s_b + buf * C::S);
#pragma unroll
    for (int i = 0; i < SN; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int o = (h == 0 ? d0 : d1) * C::SLD + (sn0 + i) * 8 + (lane & 3) * 2;
        uint32_t hi, lo;
        split_pair(S[i][2 * h], S[i][2 * h + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(dst + o) = hi;
        *reinterpret_cast<uint32_t*>(dst + P * C::SLD + o) = lo;
      }
  };
  publish(0);
  named_sync(kBarChain, kDsGroup);
  for (int c = 0; c < chunks; ++c) {
    // ---- values written: u = M V - W S ----
    arrived(0, c);
    float acc[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    rows_times_s(acc, wb, smem_u32(s_b + (c & 1) * C::S));
    __nv_bfloat16* u_s = reinterpret_cast<__nv_bfloat16*>(u_b + (c & 1) * C::U);       // the outputs are done with it
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int t = t0 + h * 8, col = c0 + i * 8 + (lane & 3) * 2;
        const float2 m = *reinterpret_cast<const float2*>(mv_s + t * C::ULD + col);
        uint32_t hi, lo;
        split_pair(m.x - acc[i][2 * h], m.y - acc[i][2 * h + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(u_s + t * C::SLD + col) = hi;
        *reinterpret_cast<uint32_t*>(u_s + kChunk * C::SLD + t * C::SLD + col) = lo;
      }
    named_sync(kBarChain, kDsGroup);                       // u is written, W and M V are read
    if (threadIdx.x == 0 && c + 1 < chunks) fetch_w(c + 1);
    named_arrive(kBarFull + (c & 1), kDsThreads);
    // ---- the next state ----
    arrived(1, c);
    const uint32_t ub = smem_u32(u_s);
    const float e0 = decay_s[d0], e1 = decay_s[d1];
#pragma unroll
    for (int i = 0; i < SN; ++i) {
      S[i][0] *= e0;
      S[i][1] *= e0;
      S[i][2] *= e1;
      S[i][3] *= e1;
    }
#pragma unroll
    for (int ks = 0; ks < kRuns; ++ks) {
      uint32_t kh[4], kl[4];                               // transposed: rows are key channels
      const uint32_t ko = ((ks * 16 + (mm >> 1) * 8 + rr) * C::BLD + sm0 + (mm & 1) * 8) * 2;
      ldsm_x4_trans(kb + ko, kh[0], kh[1], kh[2], kh[3]);
      ldsm_x4_trans(kb + R_LO + ko, kl[0], kl[1], kl[2], kl[3]);
#pragma unroll
      for (int i = 0; i < SN; i += 2) {
        uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
        const uint32_t uo = ((ks * 16 + (mm & 1) * 8 + rr) * C::SLD + (sn0 + i + (mm >> 1)) * 8) * 2;
        ldsm_x4_trans(ub + uo, h0, h1, h2, h3);
        ldsm_x4_trans(ub + U_LO + uo, l0, l1, l2, l3);
        mma_bf16(S[i], kh, h0, h1);
        mma_bf16(S[i + 1], kh, h2, h3);
        mma_bf16(S[i], kh, l0, l1);
        mma_bf16(S[i + 1], kh, l2, l3);
        mma_bf16(S[i], kl, h0, h1);
        mma_bf16(S[i + 1], kl, h2, h3);
      }
    }
    if (c + 1 == chunks) break;
    if (c > 0) named_sync(kBarFree + ((c - 1) & 1), kDsThreads);         // the outputs are done with the other buffers
    publish((c + 1) & 1);
    named_sync(kBarChain, kDsGroup);                       // the state is published, keys are read
    if (threadIdx.x == 0) fetch_keys(c + 1);
  }
#pragma unroll
  for (int i = 0; i < SN; ++i) {
    const int c = v0 + (sn0 + i) * 8 + (lane & 3) * 2;
    if (c >= p.vdim) continue;
    if (d0 < p.dim) *reinterpret_cast<float2*>(st.S + static_cast<long long>(d0) * p.vdim + c) = make_float2(S[i][0], S[i][1]);
    if (d1 < p.dim) *reinterpret_cast<float2*>(st.S + static_cast<long long>(d1) * p.vdim + c) = make_float2(S[i][2], S[i][3]);
  }
}

// Head norm, weight and gate of a chunk (row y of the grid): a block takes a head, its warps a token each in turn. At most
// 128 values per head, four per lane.
__global__ void __launch_bounds__(256)
delta_chunk_norm_kernel(nfk_delta_params p) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, head = blockIdx.x, c = lane * 4;
  const int n = p.items[blockIdx.y * 4 + 2];
  const long long t0 = p.items[blockIdx.y * 4 + 1];
  const bool ok = c < p.vdim;
  const int col = head * p.vdim + (ok ? c : 0);
  const float* o = p.o + t0 * p.heads * p.vdim + col;
  const __nv_bfloat16* g = reinterpret_cast<const __nv_bfloat16*>(p.g) + t0 * p.ld_g + col;
  __nv_bfloat16* y = reinterpret_cast<__nv_bfloat16*>(p.y) + t0 * p.ld_y + col;
  const float4 w = load4(p.norm + (ok ? c : 0));
  const float inv_n = 1.f / static_cast<float>(p.vdim_real);
#pragma unroll 4
  for (int t = warp; t < n; t += 8) {
    const float4 gg = load4(g + t * p.ld_g);
    float4 v = load4(o + static_cast<long long>(t) * p.heads * p.vdim);
    if (!ok) v = make_float4(0.f, 0.f, 0.f, 0.f);
    const float inv = rsqrtf(warp_sum((v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w)) * inv_n + p.eps);
    if (ok)
      store4(y + t * p.ld_y, make_float4(v.x * inv * w.x * sigmoid_fast(gg.x), v.y * inv * w.y * sigmoid_fast(gg.y),
                                         v.z * inv * w.z * sigmoid_fast(gg.z), v.w * inv * w.w * sigmoid_fast(gg.w)));
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

int check_delta(const nfk_delta_params* p) {
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (!p->qkv || !p->x || !p->beta || !p->g || !p->rate || !p->dt_bias || !p->norm || !p->S || !p->y || !p->positions ||
      !p->qo_indptr || !p->state_slot)
    return NF_ERR_BAD_ARG;
  if (p->heads <= 0 || p->kv_heads <= 0 || p->heads % p->kv_heads != 0 || p->dim <= 0 || p->dim % 8 != 0 || p->vdim <= 0 ||
      p->vdim % 8 != 0 || p->vdim_real <= 0 || p->vdim_real > p->vdim || p->num_slots <= 0)
    return NF_ERR_BAD_ARG;
  if (p->ld % 8 != 0 || p->q_off % 8 != 0 || p->k_off % 8 != 0 || p->v_off % 8 != 0 || p->ld_g % 8 != 0 || p->ld_x % 4 != 0 ||
      p->ld_y % 8 != 0 || (reinterpret_cast<uintptr_t>(p->qkv) & 15) != 0 || (reinterpret_cast<uintptr_t>(p->g) & 15) != 0)
    return NF_ERR_BAD_ARG;
  return NF_OK;
}

template <class T>
int launch_delta_seq(const nfk_delta_params& p, cudaStream_t stream) {
  const int v_slices = (p.vdim + kSeqCols - 1) / kSeqCols;
  const size_t sm = static_cast<size_t>(p.dim) * (kSeqCols + 3) * 4;
  const long long grid = static_cast<long long>(p.num_seq) * p.heads * v_slices;
  if (grid > 0x7fffffffll || p.num_seq > 65535) return NF_ERR_BAD_ARG;
  const int rc = set_smem(delta_seq_kernel<T>, sm);
  if (rc != NF_OK) return rc;
  delta_seq_kernel<T><<<static_cast<int>(grid), 256, sm, stream>>>(p, v_slices);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  delta_seq_norm_kernel<T><<<dim3(64, p.num_seq), 256, 0, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

template <int P>
int launch_delta_chunks(const nfk_delta_params& p, cudaStream_t stream) {
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    int rc = set_smem(delta_chunk_kernel<P>, DeltaChunkCfg<P>::SMEM);
    if (rc == NF_OK) rc = set_smem(delta_scan_kernel<P>, DeltaScanCfg<P>::SMEM);
    if (rc != NF_OK) return rc;
    attr = true;
  }
  const int grid = p.num_items * p.heads, slices = (p.vdim + kSlice - 1) / kSlice;
  const int portions = p.num_portions > 0 && p.num_portions < p.num_items ? p.num_portions : p.num_items;
  delta_chunk_kernel<P><<<grid, kDcThreads, DeltaChunkCfg<P>::SMEM, stream>>>(p);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  delta_scan_kernel<P><<<portions * p.heads * slices, kDsThreads, DeltaScanCfg<P>::SMEM, stream>>>(p, slices);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  delta_chunk_norm_kernel<<<dim3(p.heads, p.num_items), 256, 0, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

template <class T>
int launch_delta_decode(const nfk_delta_params& p, cudaStream_t stream) {
  const long long grid = static_cast<long long>(p.req_count) * p.heads;
  const size_t sm = (static_cast<size_t>(p.dim) * 3 + p.vdim) * 4;
  if (grid > 0x7fffffffll || sm > 36 * 1024) return NF_ERR_BAD_ARG;
  const int g = static_cast<int>(grid);
  if (p.dim <= 32 && p.vdim <= 32) delta_decode_kernel<T, 8, 1><<<g, 256, sm, stream>>>(p);
  else if (p.dim <= 64 && p.vdim <= 64) delta_decode_kernel<T, 16, 4><<<g, 256, sm, stream>>>(p);
  else if (p.dim <= 128 && p.vdim <= 128) delta_decode_kernel<T, 32, 16><<<g, 256, sm, stream>>>(p);
  else delta_decode_kernel<T, 32, 0><<<g, 256, sm, stream>>>(p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_delta_decode(const nfk_delta_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_delta(p);
  if (rc != NF_OK || p->req_count == 0) return rc;
  if (p->req_count < 0 || p->req_begin < 0) return NF_ERR_BAD_ARG;
  return p->dtype == NFK_F32 ? launch_delta_decode<float>(*p, stream) : launch_delta_decode<__nv_bfloat16>(*p, stream);
}

extern "C" int nfk_delta_prefill(const nfk_delta_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_delta(p);
  if (rc != NF_OK) return rc;
  if (p->num_seq < 0 || p->num_items < 0 || p->num_items > 65535 || (p->num_seq > 0 && !p->seq_reqs) ||
      (p->num_items > 0 && !p->items) || (p->num_seq + p->num_items > 0 && !p->o))
    return NF_ERR_BAD_ARG;
  if (p->num_items > 0) {
    if (p->dtype != NFK_BF16 || p->dim > 128 || p->vdim > 128) return NF_ERR_UNSUPPORTED;
    if (p->scratch == nullptr || (reinterpret_cast<uintptr_t>(p->scratch) & 15) != 0 ||
        p->num_items * static_cast<long long>(p->heads) * delta_item_floats(p->dim, p->vdim) > p->scratch_floats)
      return NF_ERR_BAD_ARG;
    const int rc2 = p->dim <= 64 && p->vdim <= 64 ? launch_delta_chunks<64>(*p, stream) : launch_delta_chunks<128>(*p, stream);
    if (rc2 != NF_OK) return rc2;
  }
  if (p->num_seq == 0) return NF_OK;
  return p->dtype == NFK_F32 ? launch_delta_seq<float>(*p, stream) : launch_delta_seq<__nv_bfloat16>(*p, stream);
}

extern "C" long long nfk_delta_item_floats(int dim, int vdim) { return nf::delta_item_floats(dim, vdim); }
