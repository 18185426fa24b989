// mLSTM: a recurrent mixer with a matrix memory per head, exponential input gate and sigmoid forget gate,
// stabilised by a running maximum m (Beck et al., "xLSTM: Extended Long Short-Term Memory"):
//
//   m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' = e^(f + m - m') n + e^(i - m') k
//   out = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6)
//
// with i = cap tanh((x_i + b_i) / cap) and f = logsigmoid(cap tanh((x_f + b_f) / cap)). State, gates and
// everything derived from them are fp32 (see kernels.h for where the state of a request lives).
//
// nfk_mlstm_decode   one token per request: a CTA streams 128 columns of one head's S through registers
//                    (update, read out, write back in one pass). Bound by the state traffic.
// nfk_mlstm_prefill  impl 1: token by token with 32 columns of S in shared memory; any size, bf16 or fp32.
//                    impl 2 (bf16): chunks of 64 tokens on tensor cores. With F the running sum of f inside the
//                    chunk, a_j = i_j - F_j and M_t = max(m_in, max_{j<=t} a_j), every weight of the chunk is
//                    an exponential of a non-positive number (a small kernel computes a, its running maximum and F
//                    of all chunks first): token j enters output t with e^(a_j - M_t), the
//                    incoming state with e^(m_in - M_t), and m_t = F_t + M_t. Weights, weighted values and the
//                    state enter the products as bf16 pairs (high and low part), so they keep about 16 bits.
//                    Long prompts are cut into segments: their own contributions are computed side by side from
//                    zero, a scan turns them into the state each segment starts from, and the outputs of all
//                    segments are then computed side by side.
// nfk_head_norm_gate RMS norm of each head's output, weight, output gate.
#include "attn_mma.cuh"
#include "elem_io.cuh"

namespace nf {
namespace {

__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ void gate_values(const nfk_mlstm_params& p, long long tok, int head, float& li, float& lf) {
  const float* g = p.gates + tok * p.ld_gates;
  li = soft_cap(g[head] + p.i_bias[head], p.gate_cap);
  lf = log_sigmoid(soft_cap(g[p.heads + head] + p.f_bias[head], p.gate_cap));
}

// Where a request's state is: slot index and which half of n / m to read (the other half is written).
struct StateRef {
  int slot, half;
  bool ok, fresh;
};
__device__ __forceinline__ StateRef state_ref(const nfk_mlstm_params& p, int req) {
  StateRef r;
  const int v = p.state_slot[req];
  r.slot = v >> 1;
  r.half = v & 1;
  r.ok = v >= 0 && r.slot < p.num_slots;
  r.fresh = p.positions[p.qo_indptr[req]] == 0;
  if (!r.ok) report_status(p.status, NF_ST_BAD_INDEX);
  return r;
}

__device__ __forceinline__ float cta_sum256(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < 8 ? red[lane] : 0.f);
}

// ---- decode -----------------------------------------------------------------------------------------
constexpr int kDecCols = 128;

template <class T>
__global__ void __launch_bounds__(256)
mlstm_decode_kernel(nfk_mlstm_params p, int v_slices) {
  extern __shared__ float dsm[];                 // k[dim] | q[dim]
  __shared__ float red[8];
  __shared__ float4 part[8][32];
  float* k_s = dsm;
  float* q_s = dsm + p.dim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vs = blockIdx.x % v_slices;
  const int head = (blockIdx.x / v_slices) % p.heads;
  const int req = p.req_begin + blockIdx.x / (v_slices * p.heads);
  const StateRef st = state_ref(p, req);
  if (!st.ok) return;
  const long long tok = p.qo_indptr[req];
  const long long sh = static_cast<long long>(st.slot) * p.heads + head;
  const float* n_old = p.n + (sh * 2 + st.half) * p.dim;
  float* n_new = p.n + (sh * 2 + (st.half ^ 1)) * p.dim;
  float li, lf;
  gate_values(p, tok, head, li, lf);
  const float m_old = st.fresh ? 0.f : p.m[sh * 2 + st.half];
  const float m_new = fmaxf(lf + m_old, li);
  const float keep = expf(lf + m_old - m_new), write = expf(li - m_new);
  const T* row = reinterpret_cast<const T*>(p.qkv) + tok * p.ld_qkv;
  float nq = 0.f;
  for (int d = threadIdx.x; d < p.dim; d += 256) {
    const float k = to_f32(row[p.k_off + head * p.dim + d]), q = to_f32(row[p.q_off + head * p.dim + d]) * p.q_scale;
    k_s[d] = k * write;
    q_s[d] = q;
    const float n = (st.fresh ? 0.f : keep * n_old[d]) + write * k;
    if (vs == 0) n_new[d] = n;
    nq += n * q;
  }
  nq = cta_sum256(nq, red);                      // also orders k_s / q_s
  if (vs == 0 && threadIdx.x == 0) p.m[sh * 2 + (st.half ^ 1)] = m_new;
  const float inv = 1.f / (fmaxf(fabsf(nq), expf(-m_new)) + 1e-6f);
  const int col = vs * kDecCols + lane * 4;
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (col < p.vdim) {
    const float4 v = load4(row + p.v_off + head * p.vdim + col);
    float* S = p.S + sh * p.dim * p.vdim + col;
#pragma unroll 8
    for (int d = warp; d < p.dim; d += 8) {
      float4* sp = reinterpret_cast<float4*>(S + static_cast<long long>(d) * p.vdim);
      float4 s = st.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *sp;
      const float kd = k_s[d], qd = q_s[d];
      s.x = keep * s.x + kd * v.x;
      s.y = keep * s.y + kd * v.y;
      s.z = keep * s.z + kd * v.z;
      s.w = keep * s.w + kd * v.w;
      *sp = s;
      acc.x += s.x * qd; acc.y += s.y * qd; acc.z += s.z * qd; acc.w += s.w * qd;
    }
  }
  part[warp][lane] = acc;
  __syncthreads();
  if (warp == 0 && col < p.vdim) {
#pragma unroll
    for (int w = 1; w < 8; ++w) {
      const float4 o = part[w][lane];
      acc.x += o.x; acc.y += o.y; acc.z += o.z; acc.w += o.w;
    }
    acc.x *= inv; acc.y *= inv; acc.z *= inv; acc.w *= inv;
    store4(p.out + tok * p.ld_out + head * p.vdim + col, acc);
  }
}

// ---- prefill, token by token ---------------------------------------------------------------------------
constexpr int kSeqCols = 32;

template <class T>
__global__ void __launch_bounds__(256)
mlstm_seq_kernel(nfk_mlstm_params p, int v_slices) {
  extern __shared__ float dsm[];                 // S[dim][32] | k[dim] | q[dim] | n[dim]
  __shared__ float red[8];
  __shared__ float part[8][32];
  float* S_s = dsm;
  float* k_s = S_s + p.dim * kSeqCols;
  float* q_s = k_s + p.dim;
  float* n_s = q_s + p.dim;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int vs = blockIdx.x % v_slices;
  const int head = (blockIdx.x / v_slices) % p.heads;
  const int req = p.req_begin + blockIdx.x / (v_slices * p.heads);
  const StateRef st = state_ref(p, req);
  if (!st.ok) return;
  const int t0 = p.qo_indptr[req], t1 = p.qo_indptr[req + 1];
  const long long sh = static_cast<long long>(st.slot) * p.heads + head;
  const int col = vs * kSeqCols + lane;
  const bool col_ok = col < p.vdim;
  float* S = p.S + sh * p.dim * p.vdim + col;
  for (int d = warp; d < p.dim; d += 8)
    S_s[d * kSeqCols + lane] = (st.fresh || !col_ok) ? 0.f : S[static_cast<long long>(d) * p.vdim];
  for (int d = threadIdx.x; d < p.dim; d += 256) n_s[d] = st.fresh ? 0.f : p.n[(sh * 2 + st.half) * p.dim + d];
  float m = st.fresh ? 0.f : p.m[sh * 2 + st.half];
  for (int t = t0; t < t1; ++t) {
    float li, lf;
    gate_values(p, t, head, li, lf);
    const float m_new = fmaxf(lf + m, li);
    const float keep = expf(lf + m - m_new), write = expf(li - m_new);
    m = m_new;
    const T* row = reinterpret_cast<const T*>(p.qkv) + static_cast<long long>(t) * p.ld_qkv;
    __syncthreads();                             // the previous token's reads of k_s / q_s are done
    float nq = 0.f;
    for (int d = threadIdx.x; d < p.dim; d += 256) {
      const float k = to_f32(row[p.k_off + head * p.dim + d]), q = to_f32(row[p.q_off + head * p.dim + d]) * p.q_scale;
      k_s[d] = k * write;
      q_s[d] = q;
      const float n = keep * n_s[d] + write * k;
      n_s[d] = n;
      nq += n * q;
    }
    nq = cta_sum256(nq, red);
    const float v = col_ok ? to_f32(row[p.v_off + head * p.vdim + col]) : 0.f;
    float acc = 0.f;
    for (int d = warp; d < p.dim; d += 8) {
      const float s = keep * S_s[d * kSeqCols + lane] + k_s[d] * v;
      S_s[d * kSeqCols + lane] = s;
      acc += s * q_s[d];
    }
    part[warp][lane] = acc;
    __syncthreads();
    if (warp == 0 && col_ok) {
      for (int w = 1; w < 8; ++w) acc += part[w][lane];
      p.out[static_cast<long long>(t) * p.ld_out + head * p.vdim + col] =
          acc / (fmaxf(fabsf(nq), expf(-m)) + 1e-6f);
    }
  }
  __syncthreads();
  for (int d = warp; d < p.dim; d += 8)
    if (col_ok) S[static_cast<long long>(d) * p.vdim] = S_s[d * kSeqCols + lane];
  if (vs == 0) {
    for (int d = threadIdx.x; d < p.dim; d += 256) p.n[(sh * 2 + (st.half ^ 1)) * p.dim + d] = n_s[d];
    if (threadIdx.x == 0) p.m[sh * 2 + (st.half ^ 1)] = m;
  }
}

// ---- prefill, chunks of 64 tokens on tensor cores ----------------------------------------------------------
constexpr int kChunk = 64, kVs = 64, kGroup = 256, kChThreads = 2 * kGroup;   // output warps, state warps

template <int DP>
struct ChCfg {
  static constexpr int QK_BYTES = kChunk * DP * 2;        // [DP / 64][64 tokens][64 columns], 128-byte swizzle
  static constexpr int V_BYTES = kChunk * kVs * 2;
  static constexpr int S_BYTES = DP * kVs * 2;
  static constexpr int P_BYTES = kChunk * kChunk * 2;
  static constexpr int Q_OFF = 0;
  static constexpr int K_OFF = Q_OFF + QK_BYTES;          // two buffers
  static constexpr int V_OFF = K_OFF + 2 * QK_BYTES;      // two buffers
  static constexpr int SH_OFF = V_OFF + 2 * V_BYTES;      // state, high part
  static constexpr int SL_OFF = SH_OFF + S_BYTES;         // low part
  static constexpr int PH_OFF = SL_OFF + S_BYTES;
  static constexpr int PL_OFF = PH_OFF + P_BYTES;
  static constexpr int WH_OFF = PL_OFF + P_BYTES;         // weighted values, high / low part
  static constexpr int WL_OFF = WH_OFF + V_BYTES;
  static constexpr int N_OFF = WL_OFF + V_BYTES;          // n as a ninth column tile of the state, [DP][8]: columns
                                                          // 0-2 are three bf16 parts that add up to it
  static constexpr int U_OFF = N_OFF + DP * 16;           // its weighted values: the weights in three parts, [64][8]
  static constexpr int F_OFF = U_OFF + kChunk * 16;       // fp32 arrays
  static constexpr int N_F32 = 12 * kChunk;
  static constexpr int BAR_OFF = F_OFF + N_F32 * 4;
  static constexpr int SMEM = BAR_OFF + 64 + 1024;
  static constexpr int WM = DP / 16 < 8 ? DP / 16 : 8;    // warps along dim in the state update
  static constexpr int WN = 8 / WM;                       // ... and along the columns
  static constexpr int MTS = DP / 16 / WM;                // 16-row tiles of S per warp
  static constexpr int NTS = 8 / WN;                      // 8-column tiles of S per warp
};

// Byte offset of 16-byte chunk `ch` of row `row`: 128-byte rows, and blocks of 64 columns of 64-row tiles.
__device__ __forceinline__ uint32_t swz(int row, int ch) {
  return static_cast<uint32_t>(row * 128 + ((ch ^ (row & 7)) << 4));
}
__device__ __forceinline__ uint32_t swz_blk(int row, int ch) {
  return static_cast<uint32_t>((ch >> 3) * (kChunk * 128) + row * 128 + (((ch ^ row) & 7) << 4));
}
__device__ __forceinline__ void ldsm_x2_trans(uint32_t addr, uint32_t& r0, uint32_t& r1) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
// Three bf16 values that add up to v, in the first three places of a row.
__device__ __forceinline__ void store_parts(uint8_t* row, float v) {
  const __nv_bfloat16 a = __float2bfloat16(v);
  const float r = v - __bfloat162float(a);
  const __nv_bfloat16 b = __float2bfloat16(r);
  __nv_bfloat16* p = reinterpret_cast<__nv_bfloat16*>(row);
  p[0] = a;
  p[1] = b;
  p[2] = __float2bfloat16(r - __bfloat162float(b));
}
__device__ __forceinline__ void tma_load_3d(void* smem_dst, const CUtensorMap* tm, uint64_t* bar, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes"
      " [%0], [%1, {%3, %4, %5}], [%2];" ::"r"(smem_u32(smem_dst)),
      "l"(reinterpret_cast<uint64_t>(tm)), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z)
      : "memory");
}

// Floats of scratch per (item, head): S [dim][vdim], n [dim], then m and the sum of f of the segment's own
// contribution and m of the state it starts from.
__host__ __device__ __forceinline__ long long seg_floats(int dim, int vdim) {
  return static_cast<long long>(dim) * vdim + dim + 8;
}
// Gate values of all chunks: [chunk][head][a | running maximum of a | F][64]. A chunk's index is its distance from
// the launch's first token in chunks plus the number of its item, which no two chunks share.
__host__ __device__ __forceinline__ long long gate_floats(int tokens, int items, int heads) {
  return static_cast<long long>(tokens / kChunk + items + 1) * heads * (3 * kChunk);
}
__device__ __forceinline__ float* chunk_gates(const nfk_mlstm_params& p, int item, int tok0, int c, int head) {
  return p.scratch + (static_cast<long long>(tok0 / kChunk + item + c) * p.heads + head) * (3 * kChunk);
}

// a_j = i_j - F_j, its running maximum and F_j inside every chunk: one warp per (item, head, chunk), two tokens per
// lane. Tokens past the item's last one get a = -inf.
__global__ void __launch_bounds__(256)
mlstm_gates_kernel(nfk_mlstm_params p) {
  const int lane = threadIdx.x & 31;
  const int head = blockIdx.x % p.heads, item = blockIdx.x / p.heads;
  const int tok0 = p.items[item * 4 + 1], ntok = p.items[item * 4 + 2];
  for (int c = threadIdx.x >> 5; c * kChunk < ntok; c += 8) {
    float gi[2], gf[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = c * kChunk + lane * 2 + e;
      gi[e] = -INFINITY;
      gf[e] = 0.f;
      if (t < ntok) gate_values(p, tok0 + t, head, gi[e], gf[e]);
    }
    float s = gf[0] + gf[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += up;
    }
    const float F1 = s, F0 = s - gf[1];
    const float a0 = gi[0] - F0, a1 = gi[1] - F1;
    float mx = fmaxf(a0, a1);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, mx, o);
      if (lane >= o) mx = fmaxf(mx, up);
    }
    const float before = __shfl_up_sync(0xffffffffu, mx, 1);
    float2* dst = reinterpret_cast<float2*>(chunk_gates(p, item, tok0, c, head)) + lane;
    dst[0] = make_float2(a0, a1);
    dst[32] = make_float2(lane == 0 ? a0 : fmaxf(before, a0), mx);
    dst[64] = make_float2(F0, F1);
  }
}

// Named barriers: one per group, and two that hand the state's bf16 pair back and forth between the groups.
enum : int { kBarOut = 1, kBarState = 2, kBarPublished = 3, kBarRead = 4 };
__device__ __forceinline__ void bar_sync(int id, int n) { asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(n) : "memory"); }
__device__ __forceinline__ void bar_arrive(int id, int n) { asm volatile("bar.arrive %0, %1;" ::"r"(id), "r"(n) : "memory"); }

// STATE_ONLY: the segment's own contribution to the state, from zero, into scratch. Otherwise: outputs, from the
// request's state (first segment) or from scratch; the last segment leaves the state in the request's slot.
// Tiles of q, k, v come by TMA (columns past a head's are filled with zeros; rows past the segment's last token
// are other tokens' and get zero weights). Two groups of eight warps work side by side. The state warps keep S in
// registers (16-row tiles), update it chunk by chunk and publish its bf16 pair in shared memory once the output
// warps have read the previous one. The output warps compute scores and the read-out of the published state by
// (32 tokens, 16 keys or columns), then the outputs by (32 tokens, 16 columns). n rides along as one more column
// of S (its values are all ones), in three bf16 parts: the products n . q and K^T w come out of the same
// instructions in full fp32 accuracy.
template <int DP, bool STATE_ONLY>
__global__ void __launch_bounds__(kChThreads, 1)
mlstm_chunk_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                   const __grid_constant__ CUtensorMap tmV, nfk_mlstm_params p, int v_slices, long long seg_off) {
  using C = ChCfg<DP>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  const uint32_t sb = smem_u32(smem);
  float* a_s = reinterpret_cast<float*>(smem + C::F_OFF);   // a_j log2(e)
  float* mx_s = a_s + kChunk;         // M_t log2(e) - log2(q_scale)
  float* int_s = mx_s + kChunk;       // q_scale e^(m_in - M_t)
  float* em_s = int_s + kChunk;       // e^(-m_t)
  float* rs_s = em_s + kChunk;        // [4][64] row sums of the weighted scores
  float* nq_s = rs_s + 4 * kChunk;    // [4][64] parts of n . q_t
  uint64_t* q_full = reinterpret_cast<uint64_t*>(smem + C::BAR_OFF);
  uint64_t* kv_full = q_full + 1;     // two
  volatile int* abort_flag = reinterpret_cast<volatile int*>(q_full + 3);

  const int warp = (threadIdx.x >> 5) & 7, lane = threadIdx.x & 31, tid = threadIdx.x % kGroup;
  const bool state_warp = threadIdx.x >= kGroup;
  const int vs = blockIdx.x % v_slices;
  const int head = (blockIdx.x / v_slices) % p.heads;
  const int item = blockIdx.x / (v_slices * p.heads);
  const int req = p.items[item * 4], tok0 = p.items[item * 4 + 1], ntok = p.items[item * 4 + 2], seg = p.items[item * 4 + 3];
  const bool has_next = item + 1 < p.num_items && p.items[(item + 1) * 4] == req;
  if (STATE_ONLY && !has_next) return;
  const StateRef st = state_ref(p, req);
  if (!st.ok || ntok <= 0) return;
  const long long sh = static_cast<long long>(st.slot) * p.heads + head;
  const int v0 = vs * kVs;
  float* sc_S = p.scratch + seg_off + (static_cast<long long>(item) * p.heads + head) * seg_floats(p.dim, p.vdim);
  float* sc_n = sc_S + static_cast<long long>(p.dim) * p.vdim;
  const int n_chunks = (ntok + kChunk - 1) / kChunk;
  const int mm = lane >> 3, rr = lane & 7;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(kv_full, 1);
    mbar_init(kv_full + 1, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  for (int i = threadIdx.x; i < (C::F_OFF - C::N_OFF) / 16; i += kChThreads)
    *reinterpret_cast<uint4*>(smem + C::N_OFF + i * 16) = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  auto load_kv = [&](int c) {        // one thread
    uint64_t* bar = kv_full + (c & 1);
    mbar_expect_tx(bar, C::QK_BYTES + C::V_BYTES);
#pragma unroll
    for (int b = 0; b < DP / 64; ++b)
      tma_load_3d(smem + C::K_OFF + (c & 1) * C::QK_BYTES + b * (kChunk * 128), &tmK, bar, b * 64, head, tok0 + c * kChunk);
    tma_load_3d(smem + C::V_OFF + (c & 1) * C::V_BYTES, &tmV, bar, v0, head, tok0 + c * kChunk);
  };
  auto load_q = [&](int c) {
    mbar_expect_tx(q_full, C::QK_BYTES);
#pragma unroll
    for (int b = 0; b < DP / 64; ++b)
      tma_load_3d(smem + C::Q_OFF + b * (kChunk * 128), &tmQ, q_full, b * 64, head, tok0 + c * kChunk);
  };
  // A wait that runs out is reported; the warps go on in step, so that they meet at their barriers.
  auto wait_tile = [&](uint64_t* bar, int parity) {
    if (*abort_flag == 0 && !mbar_wait(bar, parity)) {
      if (lane == 0) report_status(p.status, NF_ST_TIMEOUT_SMEM_FULL);
      *abort_flag = 1;
    }
  };
  if (threadIdx.x == 0) {
    load_kv(0);
    if (!STATE_ONLY) load_q(0);
  }
  const bool from_zero = STATE_ONLY || (seg == 0 && st.fresh);
  float m_in = STATE_ONLY ? -INFINITY : (seg == 0 ? (st.fresh ? 0.f : p.m[sh * 2 + st.half]) : sc_n[p.dim + 2]);
  auto gates_of = [&](int c) { return chunk_gates(p, item, tok0, c < n_chunks ? c : n_chunks - 1, head); };

  if (state_warp) {
    // ------------------------------------------------------------------ state
    const float* S_in = seg == 0 ? p.S + sh * p.dim * p.vdim : sc_S;
    const float* n_in = seg == 0 ? p.n + (sh * 2 + st.half) * p.dim : sc_n;
    const int wm = warp % C::WM, wn = warp / C::WM;
    float S[C::MTS][C::NTS][4];
#pragma unroll
    for (int a = 0; a < C::MTS; ++a)
#pragma unroll
      for (int b = 0; b < C::NTS; ++b)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int d = (wm * C::MTS + a) * 16 + (lane >> 2) + h * 8;
          const int v = v0 + (wn * C::NTS + b) * 8 + (lane & 3) * 2;
          float2 x = make_float2(0.f, 0.f);
          if (!from_zero && d < p.dim && v < p.vdim) x = *reinterpret_cast<const float2*>(S_in + static_cast<long long>(d) * p.vdim + v);
          S[a][b][2 * h] = x.x;
          S[a][b][2 * h + 1] = x.y;
        }
    // n is the sum of columns 0-2 of the ninth tile, the others stay zero
    float Sn[C::MTS][4];
#pragma unroll
    for (int a = 0; a < C::MTS; ++a)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int d = (wm * C::MTS + a) * 16 + (lane >> 2) + (e >> 1) * 8;
        Sn[a][e] = (from_zero || d >= p.dim || (lane & 3) != 0 || (e & 1) != 0) ? 0.f : n_in[d];
      }
    auto n_of = [&](int a, int h) {   // n of row (lane >> 2) + 8 h of row tile a, in every lane of its quad
      const float x = (lane & 3) == 0 ? Sn[a][2 * h] + Sn[a][2 * h + 1] : (lane & 3) == 1 ? Sn[a][2 * h] : 0.f;
      return quad_sum(x);
    };
    auto publish_state = [&]() {      // the state's bf16 pair, B operand of the next chunk's read-out
#pragma unroll
      for (int a = 0; a < C::MTS; ++a)
#pragma unroll
        for (int b = 0; b < C::NTS; ++b)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int d = (wm * C::MTS + a) * 16 + (lane >> 2) + h * 8;
            const uint32_t off = swz(d, wn * C::NTS + b) + (lane & 3) * 4;
            const uint32_t hi = pack_bf16x2(S[a][b][2 * h], S[a][b][2 * h + 1]);
            const float2 hf = unpack_bf16x2(hi);
            *reinterpret_cast<uint32_t*>(smem + C::SH_OFF + off) = hi;
            *reinterpret_cast<uint32_t*>(smem + C::SL_OFF + off) = pack_bf16x2(S[a][b][2 * h] - hf.x, S[a][b][2 * h + 1] - hf.y);
          }
      if (wn == 0) {
#pragma unroll
        for (int a = 0; a < C::MTS; ++a)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const float n = n_of(a, h);
            if ((lane & 3) == 0)
              store_parts(smem + C::N_OFF + ((wm * C::MTS + a) * 16 + (lane >> 2) + h * 8) * 16, n);
          }
      }
    };
    if (!STATE_ONLY) {
      publish_state();
      bar_arrive(kBarPublished, kChThreads);
    }
    // gates of a chunk, fetched one chunk ahead: of the token rows this thread weights, and the chunk's last ones
    float ga[2], gm_last, gF_last, F_total = 0.f;
    auto fetch_gates = [&](int c) {
      const float* g = gates_of(c);
      ga[0] = g[tid >> 3];
      ga[1] = g[32 + (tid >> 3)];
      gm_last = g[2 * kChunk - 1];
      gF_last = g[3 * kChunk - 1];
    };
    fetch_gates(0);
    for (int c = 0; c < n_chunks; ++c) {
      const float M_last = fmaxf(m_in, gm_last);
      const float decay = expf(m_in - M_last);
      m_in = gF_last + M_last;
      F_total += gF_last;
      const float w[2] = {expf(ga[0] - M_last), expf(ga[1] - M_last)};
      fetch_gates(c + 1);
      const uint32_t kb = sb + C::K_OFF + (c & 1) * C::QK_BYTES;
      wait_tile(kv_full + (c & 1), (c >> 1) & 1);
      // values weighted by e^(a_j - M_last), as a bf16 pair, and the weights as values of n
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = i * 32 + (tid >> 3);
        const uint32_t off = swz(r, tid & 7);
        const uint4 v = *reinterpret_cast<const uint4*>(smem + C::V_OFF + (c & 1) * C::V_BYTES + off);
        const uint32_t vw[4] = {v.x, v.y, v.z, v.w};
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float2 f = unpack_bf16x2(vw[j]);
          f.x *= w[i];
          f.y *= w[i];
          hi[j] = pack_bf16x2(f.x, f.y);
          const float2 hf = unpack_bf16x2(hi[j]);
          lo[j] = pack_bf16x2(f.x - hf.x, f.y - hf.y);
        }
        *reinterpret_cast<uint4*>(smem + C::WH_OFF + off) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
        *reinterpret_cast<uint4*>(smem + C::WL_OFF + off) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        if ((tid & 7) == 0) store_parts(smem + C::U_OFF + r * 16, w[i]);
      }
      bar_sync(kBarState, kGroup);
      if (STATE_ONLY && tid == 0 && c + 1 < n_chunks) load_kv(c + 1);
      // S = decay S + K^T (w V), n = decay n + K^T w
#pragma unroll
      for (int a = 0; a < C::MTS; ++a) {
#pragma unroll
        for (int b = 0; b < C::NTS; ++b)
#pragma unroll
          for (int e = 0; e < 4; ++e) S[a][b][e] *= decay;
#pragma unroll
        for (int e = 0; e < 4; ++e) Sn[a][e] *= decay;
      }
#pragma unroll
      for (int ks = 0; ks < kChunk / 16; ++ks) {
        uint32_t ak[C::MTS][4];
#pragma unroll
        for (int a = 0; a < C::MTS; ++a)
          ldsm_x4_trans(kb + swz_blk(ks * 16 + (mm >> 1) * 8 + rr, (wm * C::MTS + a) * 2 + (mm & 1)), ak[a][0], ak[a][1],
                        ak[a][2], ak[a][3]);
        if (wn == 0) {
          uint32_t u0, u1;
          ldsm_x2_trans(sb + C::U_OFF + (ks * 16 + (lane & 15)) * 16, u0, u1);
#pragma unroll
          for (int a = 0; a < C::MTS; ++a) mma_bf16(Sn[a], ak[a], u0, u1);
        }
#pragma unroll
        for (int b = 0; b < C::NTS; b += 2) {
          const uint32_t off = swz(ks * 16 + (mm & 1) * 8 + rr, wn * C::NTS + b + (mm >> 1));
          uint32_t h0, h1, h2, h3, l0, l1, l2, l3;
          ldsm_x4_trans(sb + C::WH_OFF + off, h0, h1, h2, h3);
          ldsm_x4_trans(sb + C::WL_OFF + off, l0, l1, l2, l3);
#pragma unroll
          for (int a = 0; a < C::MTS; ++a) {
            mma_bf16(S[a][b], ak[a], h0, h1);
            mma_bf16(S[a][b + 1], ak[a], h2, h3);
          }
#pragma unroll
          for (int a = 0; a < C::MTS; ++a) {
            mma_bf16(S[a][b], ak[a], l0, l1);
            mma_bf16(S[a][b + 1], ak[a], l2, l3);
          }
        }
      }
      if (!STATE_ONLY && c + 1 < n_chunks) {
        bar_sync(kBarRead, kChThreads);        // the output warps have read the previous state
        publish_state();
        bar_arrive(kBarPublished, kChThreads);
      } else {
        bar_sync(kBarState, kGroup);           // weighted values are free for the next chunk
      }
    }
    // ---- state out ----
    if (STATE_ONLY || !has_next) {
      float* S_out = STATE_ONLY ? sc_S : p.S + sh * p.dim * p.vdim;
      float* n_out = STATE_ONLY ? sc_n : p.n + (sh * 2 + (st.half ^ 1)) * p.dim;
#pragma unroll
      for (int a = 0; a < C::MTS; ++a)
#pragma unroll
        for (int b = 0; b < C::NTS; ++b)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int d = (wm * C::MTS + a) * 16 + (lane >> 2) + h * 8;
            const int v = v0 + (wn * C::NTS + b) * 8 + (lane & 3) * 2;
            if (d < p.dim && v < p.vdim)
              *reinterpret_cast<float2*>(S_out + static_cast<long long>(d) * p.vdim + v) = make_float2(S[a][b][2 * h], S[a][b][2 * h + 1]);
          }
      if (vs == 0) {
        if (wn == 0) {
#pragma unroll
          for (int a = 0; a < C::MTS; ++a)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
              const int d = (wm * C::MTS + a) * 16 + (lane >> 2) + h * 8;
              const float n = n_of(a, h);
              if ((lane & 3) == 0 && d < p.dim) n_out[d] = n;
            }
        }
        if (tid == 0) {
          if (STATE_ONLY) {
            sc_n[p.dim] = m_in;
            sc_n[p.dim + 1] = F_total;
          } else {
            p.m[sh * 2 + (st.half ^ 1)] = m_in;
          }
        }
      }
    }
  } else if (!STATE_ONLY) {
    // ------------------------------------------------------------------ outputs
    const int th = warp & 1, cq = warp >> 1;              // 32 tokens, 16 keys / columns
    const float log2_qs = log2f(p.q_scale);
    float ga, gm, gF, gm_last, gF_last;
    auto fetch_gates = [&](int c) {
      const float* g = gates_of(c);
      const int t = tid & 63;
      ga = g[t];
      gm = g[kChunk + t];
      gF = g[2 * kChunk + t];
      gm_last = g[2 * kChunk - 1];
      gF_last = g[3 * kChunk - 1];
    };
    fetch_gates(0);
    for (int c = 0; c < n_chunks; ++c) {
      if (tid < kChunk) {
        const float M = fmaxf(m_in, gm);
        a_s[tid] = ga * kLog2e;
        mx_s[tid] = M * kLog2e - log2_qs;
        int_s[tid] = p.q_scale * expf(m_in - M);
        em_s[tid] = expf(-(gF + M));
      }
      m_in = gF_last + fmaxf(m_in, gm_last);
      fetch_gates(c + 1);
      wait_tile(q_full, c & 1);
      wait_tile(kv_full + (c & 1), (c >> 1) & 1);
      // chunk c's gates and the state before it are in shared memory; chunk c - 1's k and v have been used up
      bar_sync(kBarPublished, kChThreads);
      if (tid == 0 && c + 1 < n_chunks) load_kv(c + 1);
      const uint32_t kb = sb + C::K_OFF + (c & 1) * C::QK_BYTES;
      const uint32_t vb = sb + C::V_OFF + (c & 1) * C::V_BYTES;
      // ---- scores Q K^T (16 keys) and read-out Q S (16 columns) of this warp's 32 tokens ----
      float sc[2][2][4], qs[2][2][4], nq[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) sc[i][j][e] = qs[i][j][e] = nq[i][e] = 0.f;
      const bool keys_seen = cq * 16 <= th * 32 + 31;          // some of these keys are not in the future
#pragma unroll 2
      for (int ks = 0; ks < DP / 16; ++ks) {
        uint32_t a[2][4], b0, b1, b2, b3, h0, h1, h2, h3, l0, l1, l2, l3;
#pragma unroll
        for (int i = 0; i < 2; ++i)
          ldsm_x4(sb + C::Q_OFF + swz_blk(th * 32 + i * 16 + (lane & 15), 2 * ks + (lane >> 4)), a[i][0], a[i][1], a[i][2], a[i][3]);
        const uint32_t off = swz(ks * 16 + (mm & 1) * 8 + rr, cq * 2 + (mm >> 1));
        ldsm_x4_trans(sb + C::SH_OFF + off, h0, h1, h2, h3);
        ldsm_x4_trans(sb + C::SL_OFF + off, l0, l1, l2, l3);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_bf16(qs[i][0], a[i], h0, h1);
          mma_bf16(qs[i][1], a[i], h2, h3);
        }
        if (keys_seen) {
          ldsm_x4(kb + swz_blk(cq * 16 + (mm >> 1) * 8 + rr, 2 * ks + (mm & 1)), b0, b1, b2, b3);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma_bf16(sc[i][0], a[i], b0, b1);
            mma_bf16(sc[i][1], a[i], b2, b3);
          }
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_bf16(qs[i][0], a[i], l0, l1);
          mma_bf16(qs[i][1], a[i], l2, l3);
        }
        if ((ks & 3) == cq) {              // n . q: every fourth step of the columns per warp
          ldsm_x2_trans(sb + C::N_OFF + (ks * 16 + (lane & 15)) * 16, b0, b1);
#pragma unroll
          for (int i = 0; i < 2; ++i) mma_bf16(nq[i], a[i], b0, b1);
        }
      }
      if (c + 1 < n_chunks) bar_arrive(kBarRead, kChThreads);
      // ---- weights, row sums, bf16 pair of the weighted scores ----
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int r = th * 32 + i * 16 + h * 8 + (lane >> 2);
          const float M = mx_s[r];
          float sum = 0.f;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int col = cq * 16 + j * 8 + (lane & 3) * 2;
            const float2 ac = *reinterpret_cast<const float2*>(a_s + col);
            const float x0 = col <= r ? sc[i][j][2 * h] * fast_exp2(ac.x - M) : 0.f;
            const float x1 = col + 1 <= r ? sc[i][j][2 * h + 1] * fast_exp2(ac.y - M) : 0.f;
            sum += x0 + x1;
            const uint32_t hi = pack_bf16x2(x0, x1);
            const float2 hf = unpack_bf16x2(hi);
            const uint32_t o = swz(r, cq * 2 + j) + (lane & 3) * 4;
            *reinterpret_cast<uint32_t*>(smem + C::PH_OFF + o) = hi;
            *reinterpret_cast<uint32_t*>(smem + C::PL_OFF + o) = pack_bf16x2(x0 - hf.x, x1 - hf.y);
          }
          sum = quad_sum(sum);
          const float nqr = quad_sum((lane & 3) == 0 ? nq[i][2 * h] + nq[i][2 * h + 1] : (lane & 3) == 1 ? nq[i][2 * h] : 0.f);
          if ((lane & 3) == 0) {
            rs_s[cq * kChunk + r] = sum;
            nq_s[cq * kChunk + r] = nqr;
          }
        }
      bar_sync(kBarOut, kGroup);         // weighted scores are in shared memory, Q is free
      if (tid == 0 && c + 1 < n_chunks) load_q(c + 1);
      // ---- P V, then the outputs of these 32 tokens x 16 columns ----
      float pv[2][2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) pv[i][j][0] = pv[i][j][1] = pv[i][j][2] = pv[i][j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks * 16 > th * 32 + 31) continue;
        uint32_t ph[2][4], pl[2][4], b0, b1, b2, b3;
        ldsm_x4_trans(vb + swz(ks * 16 + (mm & 1) * 8 + rr, cq * 2 + (mm >> 1)), b0, b1, b2, b3);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const uint32_t ao = swz(th * 32 + i * 16 + (lane & 15), 2 * ks + (lane >> 4));
          ldsm_x4(sb + C::PH_OFF + ao, ph[i][0], ph[i][1], ph[i][2], ph[i][3]);
          ldsm_x4(sb + C::PL_OFF + ao, pl[i][0], pl[i][1], pl[i][2], pl[i][3]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_bf16(pv[i][0], ph[i], b0, b1);
          mma_bf16(pv[i][1], ph[i], b2, b3);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma_bf16(pv[i][0], pl[i], b0, b1);
          mma_bf16(pv[i][1], pl[i], b2, b3);
        }
      }
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int h = 0; h < 2; ++h) {
          const int r = th * 32 + i * 16 + h * 8 + (lane >> 2), t = c * kChunk + r;
          if (t >= ntok) continue;
          const float inter = int_s[r];
          const float den = (rs_s[r] + rs_s[kChunk + r]) + (rs_s[2 * kChunk + r] + rs_s[3 * kChunk + r]) +
                            inter * ((nq_s[r] + nq_s[kChunk + r]) + (nq_s[2 * kChunk + r] + nq_s[3 * kChunk + r]));
          const float inv = 1.f / (fmaxf(fabsf(den), em_s[r]) + 1e-6f);
          float* dst = p.out + static_cast<long long>(tok0 + t) * p.ld_out + head * p.vdim;
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            const int v = v0 + cq * 16 + j * 8 + (lane & 3) * 2;
            if (v < p.vdim)
              *reinterpret_cast<float2*>(dst + v) = make_float2((inter * qs[i][j][2 * h] + pv[i][j][2 * h]) * inv,
                                                                (inter * qs[i][j][2 * h + 1] + pv[i][j][2 * h + 1]) * inv);
          }
        }
      bar_sync(kBarOut, kGroup);         // gate arrays, sums and weighted scores are free for the next chunk
    }
    if (*abort_flag != 0 && tid == 0) (void)mbar_wait(q_full, (n_chunks - 1) & 1);
  }
  if (*abort_flag != 0 && state_warp && tid == 0) {
    // a wait ran out: give copies still in flight a bounded chance to land before the CTA ends
    for (int c = n_chunks > 1 ? n_chunks - 2 : 0; c < n_chunks; ++c) (void)mbar_wait(kv_full + (c & 1), (c >> 1) & 1);
  }
}

// Segment contributions -> incoming states, in place, for requests with more than one segment. One thread per
// four elements of (S, n) of a head; all threads follow the same m.
__global__ void __launch_bounds__(256)
mlstm_scan_kernel(nfk_mlstm_params p, int e_blocks, long long seg_off) {
  const int eb = blockIdx.x % e_blocks;
  const int head = (blockIdx.x / e_blocks) % p.heads;
  const int item0 = blockIdx.x / (e_blocks * p.heads);
  const int req = p.items[item0 * 4];
  if (p.items[item0 * 4 + 3] != 0) return;                                   // not a request's first segment
  if (item0 + 1 >= p.num_items || p.items[(item0 + 1) * 4] != req) return;   // its only segment
  const StateRef st = state_ref(p, req);
  if (!st.ok) return;
  const long long sh = static_cast<long long>(st.slot) * p.heads + head;
  const long long ns = static_cast<long long>(p.dim) * p.vdim, total = ns + p.dim;
  const long long e = (static_cast<long long>(eb) * 256 + threadIdx.x) * 4;
  const bool in = e < total;
  float4 R = make_float4(0.f, 0.f, 0.f, 0.f);
  float m = 0.f;
  if (!st.fresh) {
    m = p.m[sh * 2 + st.half];
    if (in) R = e < ns ? load4(p.S + sh * ns + e) : load4(p.n + (sh * 2 + st.half) * p.dim + (e - ns));
  }
  for (int it = item0; it < p.num_items && p.items[it * 4] == req; ++it) {
    float* sc = p.scratch + seg_off + (static_cast<long long>(it) * p.heads + head) * seg_floats(p.dim, p.vdim);
    const bool last = it + 1 >= p.num_items || p.items[(it + 1) * 4] != req;
    float m_loc = 0.f, F = 0.f;
    float4 L = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!last) {
      m_loc = sc[total];
      F = sc[total + 1];
      if (in) L = load4(sc + e);
    }
    if (it != item0) {
      if (in) store4(sc + e, R);
      // m of the incoming state goes to a word of its own: the contribution's m and F are still being read
      if (eb == 0 && threadIdx.x == 0) sc[total + 2] = m;
    }
    if (last) break;
    const float m_new = fmaxf(F + m, m_loc);
    const float ka = expf(F + m - m_new), kb = expf(m_loc - m_new);
    R.x = ka * R.x + kb * L.x;
    R.y = ka * R.y + kb * L.y;
    R.z = ka * R.z + kb * L.z;
    R.w = ka * R.w + kb * L.w;
    m = m_new;
  }
}

// ---- head norm + output gate ---------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(256)
head_norm_gate_kernel(nfk_head_norm_gate_params p) {
  const int lane = threadIdx.x & 31;
  const long long total = static_cast<long long>(p.T) * p.heads;
  for (long long i = blockIdx.x * 8ll + (threadIdx.x >> 5); i < total; i += gridDim.x * 8ll) {
    const long long t = i / p.heads;
    const int c0 = static_cast<int>(i % p.heads) * p.vdim_p;
    const float* o = p.o + t * p.ld_o + c0;
    float ss = 0.f;
    for (int c = lane * 4; c < p.vdim_p; c += 128) {       // padding columns are zero
      const float4 v = load4(o + c);
      ss += (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    }
    const float inv = rsqrtf(warp_sum(ss) / static_cast<float>(p.vdim) + p.eps);
    const T* g = reinterpret_cast<const T*>(p.g) + t * p.ld_g + c0;
    T* dst = reinterpret_cast<T*>(p.out) + t * p.ld_out + c0;
    for (int c = lane * 4; c < p.vdim_p; c += 128) {
      float4 v = load4(o + c);
      const float4 w = load4(p.w + c0 + c), gg = load4(g + c);
      v.x = v.x * inv * w.x / (1.f + expf(-gg.x));
      v.y = v.y * inv * w.y / (1.f + expf(-gg.y));
      v.z = v.z * inv * w.z / (1.f + expf(-gg.z));
      v.w = v.w * inv * w.w / (1.f + expf(-gg.w));
      store4(dst + c, v);
    }
  }
}

int check_mlstm(const nfk_mlstm_params* p) {
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (!p->qkv || !p->gates || !p->i_bias || !p->f_bias || !p->S || !p->n || !p->m || !p->out || !p->positions ||
      !p->qo_indptr || !p->state_slot)
    return NF_ERR_BAD_ARG;
  if (p->heads <= 0 || p->dim <= 0 || p->vdim <= 0 || p->dim % 8 != 0 || p->vdim % 8 != 0 || p->num_slots <= 0 ||
      p->req_begin < 0 || p->req_count < 0 || !(p->gate_cap > 0.f))
    return NF_ERR_BAD_ARG;
  if (p->ld_qkv % 8 != 0 || p->q_off % 8 != 0 || p->k_off % 8 != 0 || p->v_off % 8 != 0 || p->ld_out % 4 != 0)
    return NF_ERR_BAD_ARG;
  return NF_OK;
}

template <class K>
int set_smem(K kernel, size_t bytes) {
  if (bytes > 227 * 1024) return NF_ERR_UNSUPPORTED;
  if (bytes > 48 * 1024 &&
      cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(bytes)) != cudaSuccess)
    return NF_ERR_CUDA;
  return NF_OK;
}

// [num_tokens][heads][cols] view of a column block of qkv; box: 64 tokens of one head, 64 columns.
int head_tmap(CUtensorMap* out, const nfk_mlstm_params& p, int col0, int cols) {
  nf_encode_tiled_fn enc = get_encode_tiled();
  if (enc == nullptr) return NF_ERR_CUDA;
  cuuint64_t dim[3] = {static_cast<cuuint64_t>(cols), static_cast<cuuint64_t>(p.heads), static_cast<cuuint64_t>(p.num_tokens)};
  cuuint64_t stride[2] = {static_cast<cuuint64_t>(cols) * 2, static_cast<cuuint64_t>(p.ld_qkv) * 2};
  cuuint32_t box[3] = {64, 1, kChunk}, estr[3] = {1, 1, 1};
  const __nv_bfloat16* base = reinterpret_cast<const __nv_bfloat16*>(p.qkv) + col0;
  return enc(out, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<__nv_bfloat16*>(base), dim, stride, box, estr,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS
             ? NF_OK : NF_ERR_CUDA;
}

template <int DP>
int launch_chunk(const nfk_mlstm_params& p, cudaStream_t stream) {
  using C = ChCfg<DP>;
  static bool attr_dev[kMaxDevices] = {false};
  bool& attr = attr_dev[device_slot()];
  if (!attr) {
    int rc = set_smem(mlstm_chunk_kernel<DP, false>, C::SMEM);
    if (rc == NF_OK) rc = set_smem(mlstm_chunk_kernel<DP, true>, C::SMEM);
    if (rc != NF_OK) return rc;
    attr = true;
  }
  CUtensorMap tq, tk, tv;
  int rc = head_tmap(&tq, p, p.q_off, p.dim);
  if (rc == NF_OK) rc = head_tmap(&tk, p, p.k_off, p.dim);
  if (rc == NF_OK) rc = head_tmap(&tv, p, p.v_off, p.vdim);
  if (rc != NF_OK) return rc;
  const int v_slices = (p.vdim + kVs - 1) / kVs;
  const int grid = p.num_items * p.heads * v_slices;
  const long long seg_off = gate_floats(p.num_tokens, p.num_items, p.heads);
  mlstm_gates_kernel<<<p.num_items * p.heads, 256, 0, stream>>>(p);
  if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  if (p.num_items > p.req_count) {       // some request has several segments
    mlstm_chunk_kernel<DP, true><<<grid, kChThreads, C::SMEM, stream>>>(tq, tk, tv, p, v_slices, seg_off);
    if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
    const int e_blocks = (p.dim * p.vdim + p.dim + 1023) / 1024;
    mlstm_scan_kernel<<<p.num_items * p.heads * e_blocks, 256, 0, stream>>>(p, e_blocks, seg_off);
    if (cudaGetLastError() != cudaSuccess) return NF_ERR_CUDA;
  }
  mlstm_chunk_kernel<DP, false><<<grid, kChThreads, C::SMEM, stream>>>(tq, tk, tv, p, v_slices, seg_off);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_mlstm_decode(const nfk_mlstm_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_mlstm(p);
  if (rc != NF_OK) return rc;
  if (p->req_count == 0) return NF_OK;
  const int v_slices = (p->vdim + kDecCols - 1) / kDecCols;
  const long long grid = static_cast<long long>(p->req_count) * p->heads * v_slices;
  const size_t sm = static_cast<size_t>(p->dim) * 8;
  if (grid > 0x7fffffffll || sm > 40 * 1024) return NF_ERR_BAD_ARG;
  if (p->dtype == NFK_F32) mlstm_decode_kernel<float><<<static_cast<int>(grid), 256, sm, stream>>>(*p, v_slices);
  else mlstm_decode_kernel<__nv_bfloat16><<<static_cast<int>(grid), 256, sm, stream>>>(*p, v_slices);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_mlstm_prefill(const nfk_mlstm_params* p, cudaStream_t stream) {
  using namespace nf;
  int rc = check_mlstm(p);
  if (rc != NF_OK) return rc;
  if (p->req_count == 0) return NF_OK;
  const bool chunk_ok =
      p->dtype == NFK_BF16 && p->dim <= 256 && p->items != nullptr && p->num_items >= p->req_count && p->num_tokens > 0 && p->q_scale > 0.f &&
      (reinterpret_cast<uintptr_t>(p->qkv) & 15) == 0 && p->scratch != nullptr &&
      (reinterpret_cast<uintptr_t>(p->scratch) & 15) == 0 &&
      gate_floats(p->num_tokens, p->num_items, p->heads) +
              (p->num_items > p->req_count ? p->num_items * p->heads * seg_floats(p->dim, p->vdim) : 0ll) <= p->scratch_floats;
  if (p->impl == 2 && !chunk_ok) return NF_ERR_UNSUPPORTED;
  if (p->impl != 1 && chunk_ok) {
    if (p->dim <= 64) return launch_chunk<64>(*p, stream);
    if (p->dim <= 128) return launch_chunk<128>(*p, stream);
    return launch_chunk<256>(*p, stream);
  }
  const int v_slices = (p->vdim + kSeqCols - 1) / kSeqCols;
  const size_t sm = static_cast<size_t>(p->dim) * (kSeqCols + 3) * 4;
  const long long grid = static_cast<long long>(p->req_count) * p->heads * v_slices;
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  if (p->dtype == NFK_F32) {
    rc = set_smem(mlstm_seq_kernel<float>, sm);
    if (rc == NF_OK) mlstm_seq_kernel<float><<<static_cast<int>(grid), 256, sm, stream>>>(*p, v_slices);
  } else {
    rc = set_smem(mlstm_seq_kernel<__nv_bfloat16>, sm);
    if (rc == NF_OK) mlstm_seq_kernel<__nv_bfloat16><<<static_cast<int>(grid), 256, sm, stream>>>(*p, v_slices);
  }
  if (rc != NF_OK) return rc;
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_head_norm_gate(const nfk_head_norm_gate_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == 0) return NF_OK;
  if (!p->o || !p->g || !p->w || !p->out || p->T < 0 || p->heads <= 0 || p->vdim <= 0 || p->vdim_p < p->vdim ||
      p->vdim_p % 4 != 0 || p->ld_o % 4 != 0 || p->ld_g % 4 != 0 || p->ld_out % 4 != 0)
    return NF_ERR_BAD_ARG;
  long long grid = (static_cast<long long>(p->T) * p->heads + 7) / 8;
  if (grid > 16ll * device_sm_count()) grid = 16ll * device_sm_count();
  if (p->dtype == NFK_F32) head_norm_gate_kernel<float><<<static_cast<int>(grid), 256, 0, stream>>>(*p);
  else head_norm_gate_kernel<__nv_bfloat16><<<static_cast<int>(grid), 256, 0, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}
