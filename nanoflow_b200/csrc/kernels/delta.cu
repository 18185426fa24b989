// Delta-rule recurrence with a decay per key channel and token (Yang et al., "Gated Delta Networks: Improving Mamba2 with
// Delta Rule", with a vector of decays in place of one per head; see kernels.h for the equations). State, unit vectors,
// decays, step sizes and everything derived from them are fp32.
//
// nfk_delta_decode   one token per request: a CTA per request and head streams S through registers (recall, read-out and
//                    update in one pass: o = S'^T q = (diag(w) S)^T q + (q . k) u), then head norm, weight and gate.
// nfk_delta_prefill  token by token (any size, bf16 or fp32), S in shared memory.
#include "elem_io.cuh"

namespace nf {
namespace {

__device__ __forceinline__ float softplus_f(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float delta_decay(float x, float bias, float rate) { return expf(-rate * softplus_f(x + bias)); }
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

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
  const int req = p.seq_reqs[blockIdx.y];
  const int t0 = p.qo_indptr[req];
  const long long total = static_cast<long long>(p.qo_indptr[req + 1] - t0) * p.heads;
  for (long long i = blockIdx.x * 8ll + (threadIdx.x >> 5); i < total; i += gridDim.x * 8ll) {
    const long long t = t0 + i / p.heads;
    const int head = static_cast<int>(i % p.heads);
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
  if (p->num_seq < 0 || (p->num_seq > 0 && (!p->seq_reqs || !p->o))) return NF_ERR_BAD_ARG;
  if (p->num_seq == 0) return NF_OK;
  return p->dtype == NFK_F32 ? launch_delta_seq<float>(*p, stream) : launch_delta_seq<__nv_bfloat16>(*p, stream);
}
