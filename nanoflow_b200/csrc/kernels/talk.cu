// Attention whose heads share their softmax weights: after the softmax (sliding window, a sink per head in the
// denominator) the weights of all heads are mixed by a matrix before they meet the values (Shazeer et al., "Talking-Heads
// Attention"; see kernels.h). Scores, weights, mixing and the turn of the outputs are fp32.
//
// nfk_talk_attn   any sizes, bf16 or fp32: one CTA per token, all heads. Two passes over the keys, because the mixing
//                 needs every head's normalised weights: maxima and sums first, then weights, mixing and values.
#include "elem_io.cuh"

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
