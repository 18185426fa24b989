// Grouped-query attention with options (see kernels.h for the pool layout).
//
// nfk_gqa_append   per token: RMS norm over the whole query row and the whole key row (all heads at once), rotation,
//                  keys and values to their page slot, values optionally mixed with those of an earlier layer.
// nfk_gqa_attn     attention for any head size, bf16 or fp32, with window, chunks, distance bias, sink and capped
//                  scores: one CTA per token and query head. 32-bit engines use it for everything, bf16 engines for heads that the tensor-core
//                  kernels (nfk_attn_decode, nfk_attn_prefill_ws) are not built for.
#include "elem_io.cuh"

namespace nf {
namespace {

constexpr int kApThreads = 256;

__device__ __forceinline__ float ap_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < (kApThreads >> 5) ? red[lane] : 0.f);
}

// Two neighbouring pairs from column `col` of a head, turned by the token's angles.
__device__ __forceinline__ float4 turn4(float4 x, int col, const float* table, int pairs) {
  const int i = col >> 1;
  if (i >= pairs) return x;
  const float2 a = *reinterpret_cast<const float2*>(table + 2 * i);
  const float2 b = i + 1 < pairs ? *reinterpret_cast<const float2*>(table + 2 * i + 2) : make_float2(1.f, 0.f);
  return make_float4(x.x * a.x - x.y * a.y, x.y * a.x + x.x * a.y, x.z * b.x - x.w * b.y, x.w * b.x + x.z * b.y);
}

template <class T>
__global__ void __launch_bounds__(kApThreads)
gqa_append_kernel(nfk_gqa_append_params p) {
  __shared__ float red[kApThreads / 32];
  const int nq = p.heads * p.hd, nkv = p.kv_heads * p.hd;
  for (int t = blockIdx.x; t < p.T; t += gridDim.x) {
    const T* row = reinterpret_cast<const T*>(p.src) + static_cast<long long>(t) * p.ld_src;
    const T* q = row + p.q_off;
    const T* k = row + p.k_off;
    const T* v = row + p.v_off;
    const int pos = p.positions[t];
    const int page = page_of(pos, p.token_req[t], p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages,
                             threadIdx.x == 0 ? p.status : nullptr);
    float qi = 1.f, ki = 1.f;
    if (p.q_w != nullptr) {
      float sq = 0.f, sk = 0.f;
      for (int c = threadIdx.x * 4; c < nq; c += kApThreads * 4) {       // padding columns are zero
        const float4 x = load4(q + c);
        sq += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
      }
      for (int c = threadIdx.x * 4; c < nkv; c += kApThreads * 4) {
        const float4 x = load4(k + c);
        sk += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
      }
      qi = rsqrtf(ap_sum(sq, red) / static_cast<float>(p.heads * p.dim) + p.eps);
      ki = rsqrtf(ap_sum(sk, red) / static_cast<float>(p.kv_heads * p.dim) + p.eps);
    }
    const float* rot = p.rot != nullptr ? p.rot + static_cast<long long>(t) * p.rot_ld * 2 : nullptr;
    const float* v_rot = p.v_rot != nullptr ? p.v_rot + static_cast<long long>(t) * p.v_ld * 2 : nullptr;
    T* qo = p.q_out != nullptr ? reinterpret_cast<T*>(p.q_out) + static_cast<long long>(t) * nq : nullptr;
    for (int c = threadIdx.x * 4; c < nq && qo != nullptr; c += kApThreads * 4) {
      float4 x = load4(q + c);
      if (p.q_w != nullptr) {
        const float4 w = load4(p.q_w + c);
        x = make_float4(x.x * qi * w.x, x.y * qi * w.y, x.z * qi * w.z, x.w * qi * w.w);
      }
      if (rot != nullptr) x = turn4(x, c % p.hd, rot, p.rot_pairs);
      store4(qo + c, x);
    }
    T* vf = p.v_mode != 0 ? reinterpret_cast<T*>(p.v_first) + static_cast<long long>(t) * nkv : nullptr;
    T* pool = reinterpret_cast<T*>(p.pool);
    for (int c = threadIdx.x * 4; c < nkv; c += kApThreads * 4) {
      float4 x = load4(k + c), y = load4(v + c);
      if (p.q_w != nullptr) {
        const float4 w = load4(p.k_w + c);
        x = make_float4(x.x * ki * w.x, x.y * ki * w.y, x.z * ki * w.z, x.w * ki * w.w);
      }
      if (p.v_mode == 1) {
        store4(vf + c, y);
      } else if (p.v_mode == 2) {
        const float4 f = load4(vf + c);
        const float a = 1.f - p.v_lambda, b = p.v_lambda;
        y = make_float4(a * y.x + b * f.x, a * y.y + b * f.y, a * y.z + b * f.z, a * y.w + b * f.w);
      }
      if (page < 0) continue;
      const int head = c / p.hd, col = c - head * p.hd;
      if (rot != nullptr) x = turn4(x, col, rot, p.rot_pairs);
      if (v_rot != nullptr) y = turn4(y, col, v_rot, p.v_pairs);
      T* kp = pool + ((static_cast<long long>(page) * 2 * p.kv_heads + head) * p.page_size + pos % p.page_size) * p.hd + col;
      store4(kp, x);
      store4(kp + static_cast<long long>(p.kv_heads) * p.page_size * p.hd, y);
    }
  }
}

// ---- attention, any size -------------------------------------------------------------------------------
constexpr int kGaThreads = 128, kGaTile = 64, kGaCols = 8;     // up to 1024 columns per head

template <class T>
__global__ void __launch_bounds__(kGaThreads)
gqa_attn_kernel(nfk_gqa_attn_params p) {
  extern __shared__ float q_s[];                      // [hd]
  __shared__ float s_s[kGaTile];
  __shared__ long long row_s[kGaTile];                // element offset of the key row, or -1
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int hd = p.hd, head = blockIdx.x % p.heads, kvh = head / (p.heads / p.kv_heads);
  const int tok = p.token_begin + blockIdx.x / p.heads;
  const int pos = p.positions[tok], req = p.token_req[tok];
  const T* pool = reinterpret_cast<const T*>(p.pool);
  const long long v_step = static_cast<long long>(p.kv_heads) * p.page_size * hd;
  const T* q = reinterpret_cast<const T*>(p.q) + static_cast<long long>(tok) * (p.ld_q > 0 ? p.ld_q : p.heads * hd) + head * hd;
  const float far_a = p.dist != nullptr ? p.dist[2 * head] : 0.f, far_b = p.dist != nullptr ? p.dist[2 * head + 1] : 0.f;
  for (int c = threadIdx.x; c < hd; c += kGaThreads) q_s[c] = to_f32(q[c]);
  float acc[kGaCols];
#pragma unroll
  for (int i = 0; i < kGaCols; ++i) acc[i] = 0.f;
  float m = p.sinks != nullptr ? p.sinks[head] : -INFINITY, l = p.sinks != nullptr ? 1.f : 0.f;
  const int lo = max(p.window > 0 ? max(0, pos - p.window + 1) : 0, p.chunk > 0 ? pos / p.chunk * p.chunk : 0);
  for (int j0 = lo; j0 <= pos; j0 += kGaTile) {
    const int n = min(kGaTile, pos + 1 - j0);
    __syncthreads();
    if (threadIdx.x < n) {
      const int j = j0 + threadIdx.x;
      const int page = page_of(j, req, p.page_size, p.kv_indptr, p.kv_indices, p.kv_first, p.num_pages, p.status);
      row_s[threadIdx.x] = page < 0 ? -1 : ((static_cast<long long>(page) * 2 * p.kv_heads + kvh) * p.page_size + j % p.page_size) * hd;
    }
    __syncthreads();
    for (int k = warp; k < n; k += kGaThreads / 32) {
      float d = 0.f;
      if (row_s[k] >= 0) {
        const T* kr = pool + row_s[k];
        for (int i = lane * 4; i < hd; i += 128) {
          const float4 x = load4(kr + i), y = load4(q_s + i);
          d += (x.x * y.x + x.y * y.y) + (x.z * y.z + x.w * y.w);
        }
      }
      d = warp_sum(d) * p.scale;
      if (p.softcap > 0.f) d = p.softcap * tanhf(d / p.softcap);
      if (p.dist != nullptr) d -= far_a * logf(fmaf(far_b, static_cast<float>(pos - j0 - k), 1.f));
      if (lane == 0) s_s[k] = row_s[k] >= 0 ? d : -INFINITY;
    }
    __syncthreads();
    float mx = m;
    for (int k = 0; k < n; ++k) mx = fmaxf(mx, s_s[k]);
    if (mx == -INFINITY) continue;
    const float alpha = expf(m - mx);
    m = mx;
    l *= alpha;
#pragma unroll
    for (int i = 0; i < kGaCols; ++i) acc[i] *= alpha;
    for (int k = 0; k < n; ++k) {
      if (row_s[k] < 0) continue;
      const float w = expf(s_s[k] - m);
      l += w;
      const T* vr = pool + row_s[k] + v_step;
#pragma unroll
      for (int i = 0; i < kGaCols; ++i) {
        const int col = threadIdx.x + i * kGaThreads;
        if (col < hd) acc[i] += w * to_f32(vr[col]);
      }
    }
  }
  const float inv = l > 0.f ? 1.f / l : 0.f;
  T* out = reinterpret_cast<T*>(p.out) + (static_cast<long long>(tok) * p.heads + head) * hd;
#pragma unroll
  for (int i = 0; i < kGaCols; ++i) {
    const int col = threadIdx.x + i * kGaThreads;
    if (col < hd) put(out + col, acc[i] * inv);
  }
}

}  // namespace
}  // namespace nf

extern "C" int nfk_gqa_append(const nfk_gqa_append_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == 0) return NF_OK;
  if (!p->src || !p->pool || !p->positions || !p->token_req || !p->kv_indptr || !p->kv_indices || p->T < 0 ||
      p->heads <= 0 || p->kv_heads <= 0 || p->hd <= 0 || p->hd % 8 != 0 || p->dim <= 0 || p->dim > p->hd ||
      p->page_size <= 0 || p->num_pages <= 0)
    return NF_ERR_BAD_ARG;
  if (p->ld_src % 8 != 0 || p->q_off % 8 != 0 || p->k_off % 8 != 0 || p->v_off % 8 != 0) return NF_ERR_BAD_ARG;
  if (!p->q_out && (p->q_w || p->rot)) return NF_ERR_BAD_ARG;
  if ((p->q_w == nullptr) != (p->k_w == nullptr) || p->v_mode < 0 || p->v_mode > 2 || (p->v_mode != 0 && !p->v_first))
    return NF_ERR_BAD_ARG;
  if ((p->rot && (p->rot_pairs < 0 || p->rot_pairs > p->hd / 2 || p->rot_ld < p->rot_pairs || p->rot_ld % 2 != 0)) ||
      (p->v_rot && (p->v_pairs < 0 || p->v_pairs > p->hd / 2 || p->v_ld < p->v_pairs || p->v_ld % 2 != 0)))
    return NF_ERR_BAD_ARG;
  int grid = 8 * device_sm_count();
  if (grid > p->T) grid = p->T;
  if (p->dtype == NFK_F32) gqa_append_kernel<float><<<grid, kApThreads, 0, stream>>>(*p);
  else gqa_append_kernel<__nv_bfloat16><<<grid, kApThreads, 0, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_gqa_attn(const nfk_gqa_attn_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->n_tokens == 0) return NF_OK;
  if (!p->q || !p->pool || !p->out || !p->positions || !p->token_req || !p->kv_indptr || !p->kv_indices || p->n_tokens < 0 ||
      p->token_begin < 0 || p->heads <= 0 || p->kv_heads <= 0 || p->heads % p->kv_heads != 0 || p->hd <= 0 || p->hd % 8 != 0 ||
      p->page_size <= 0 || p->num_pages <= 0 || p->window < 0 || p->chunk < 0 ||
      (p->ld_q > 0 && (p->ld_q % 4 != 0 || p->ld_q < p->heads * p->hd)))
    return NF_ERR_BAD_ARG;
  if (p->hd > kGaThreads * kGaCols) return NF_ERR_UNSUPPORTED;
  const long long grid = static_cast<long long>(p->n_tokens) * p->heads;
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  const size_t sm = static_cast<size_t>(p->hd) * 4;
  if (p->dtype == NFK_F32) gqa_attn_kernel<float><<<static_cast<int>(grid), kGaThreads, sm, stream>>>(*p);
  else gqa_attn_kernel<__nv_bfloat16><<<static_cast<int>(grid), kGaThreads, sm, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}
