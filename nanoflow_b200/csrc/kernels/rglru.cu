// Real-gated linear recurrent unit (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient
// Language Models"; see kernels.h for the equations). State, gates, decays and their logarithms are fp32.
//
// nfk_rglru_decode   one token per request: a thread per channel.
// nfk_rglru_prefill  a CTA takes 32 channels of a request and walks its tokens 256 at a time: each of 32 warps reduces
//                    eight tokens to (decay, end state from zero), one warp chains those, and every warp then runs its
//                    tokens again from the state it starts with, out of registers. Inputs are read once.
#include "elem_io.cuh"

namespace nf {
namespace {

struct RgStep {
  float a, b;      // S <- a S + b
};
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ RgStep rg_step(float r, float i, float u, float r_b, float i_b, float log_a) {
  const float la = log_a * sigmoid_f(r + r_b);
  RgStep s;
  s.a = expf(la);
  s.b = sqrtf(-expm1f(2.f * la)) * sigmoid_f(i + i_b) * u;
  return s;
}
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}
// Column of a channel's recurrence gate; its input gate is `block` columns on.
__device__ __forceinline__ int gate_col(int c, int block) { return c / block * 2 * block + c % block; }

template <class T>
__global__ void __launch_bounds__(256)
rglru_decode_kernel(nfk_rglru_params p) {
  const int c = blockIdx.x * 256 + threadIdx.x;
  const int req = p.req_begin + blockIdx.y;
  const int ref = p.state_slot[req];
  if (ref < 0 || (ref >> 1) >= p.num_slots) {
    if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    return;
  }
  if (c >= p.cols) return;
  const long long t = p.qo_indptr[req];
  float* S = p.S + static_cast<long long>(ref >> 1) * p.cols + c;
  const float* g = p.gates + t * p.ld_g + gate_col(c, p.block);
  const RgStep s = rg_step(g[0], g[p.block], to_f32(reinterpret_cast<const T*>(p.u)[t * p.ld_u + c]), p.r_b[c], p.i_b[c], p.log_a[c]);
  const float x = s.a * (p.positions[t] == 0 ? 0.f : *S) + s.b;
  *S = x;
  put(reinterpret_cast<T*>(p.out) + t * p.ld_out + c, x * gelu_tanh_f(to_f32(reinterpret_cast<const T*>(p.y)[t * p.ld_y + c])));
}

constexpr int kRgWarps = 32, kRgRun = 8;

template <class T>
__global__ void __launch_bounds__(kRgWarps * 32)
rglru_prefill_kernel(nfk_rglru_params p) {
  __shared__ float a_s[kRgWarps][32], b_s[kRgWarps][32], carry_s[32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int c = blockIdx.x * 32 + lane;
  const int req = p.req_begin + blockIdx.y;
  const int ref = p.state_slot[req];
  if (ref < 0 || (ref >> 1) >= p.num_slots) {
    if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    return;
  }
  const bool ok = c < p.cols;
  const int t0 = p.qo_indptr[req], t1 = p.qo_indptr[req + 1];
  float* S = p.S + static_cast<long long>(ref >> 1) * p.cols + c;
  const int gc = ok ? gate_col(c, p.block) : 0;
  const float r_b = ok ? p.r_b[c] : 0.f, i_b = ok ? p.i_b[c] : 0.f, log_a = ok ? p.log_a[c] : 0.f;
  if (warp == 0) carry_s[lane] = (ok && p.positions[t0] != 0) ? *S : 0.f;
  const T* u = reinterpret_cast<const T*>(p.u) + c;
  const T* y = reinterpret_cast<const T*>(p.y) + c;
  T* out = reinterpret_cast<T*>(p.out) + c;
  for (int base = t0; base < t1; base += kRgWarps * kRgRun) {
    const int begin = base + warp * kRgRun;
    RgStep s[kRgRun];
    float yy[kRgRun];
    float a = 1.f, b = 0.f;
#pragma unroll
    for (int j = 0; j < kRgRun; ++j) {
      const long long t = begin + j;
      s[j].a = 1.f;
      s[j].b = yy[j] = 0.f;
      if (t < t1 && ok) {
        const float* g = p.gates + t * p.ld_g + gc;
        s[j] = rg_step(g[0], g[p.block], to_f32(u[t * p.ld_u]), r_b, i_b, log_a);
        yy[j] = to_f32(y[t * p.ld_y]);
      }
      a *= s[j].a;
      b = s[j].a * b + s[j].b;
    }
    a_s[warp][lane] = a;
    b_s[warp][lane] = b;
    __syncthreads();
    if (warp == 0) {
      float x = carry_s[lane];
#pragma unroll
      for (int k = 0; k < kRgWarps; ++k) {
        const float next = a_s[k][lane] * x + b_s[k][lane];
        b_s[k][lane] = x;                        // what warp k starts from
        x = next;
      }
      carry_s[lane] = x;
    }
    __syncthreads();
    float x = b_s[warp][lane];
#pragma unroll
    for (int j = 0; j < kRgRun; ++j) {
      const long long t = begin + j;
      x = s[j].a * x + s[j].b;
      if (t < t1 && ok) put(out + t * p.ld_out, x * gelu_tanh_f(yy[j]));
    }
    __syncthreads();
  }
  if (warp == 0 && ok) *S = carry_s[lane];
}

int check_rglru(const nfk_rglru_params* p) {
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (!p->u || !p->y || !p->gates || !p->r_b || !p->i_b || !p->log_a || !p->S || !p->out || !p->positions || !p->qo_indptr ||
      !p->state_slot || p->req_begin < 0 || p->req_count < 0 || p->req_count > 65535 || p->cols <= 0 || p->block <= 0 ||
      p->cols % p->block != 0 || p->num_slots <= 0)
    return NF_ERR_BAD_ARG;
  return NF_OK;
}

}  // namespace
}  // namespace nf

extern "C" int nfk_rglru_decode(const nfk_rglru_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_rglru(p);
  if (rc != NF_OK || p->req_count == 0) return rc;
  const dim3 grid((p->cols + 255) / 256, p->req_count);
  if (p->dtype == NFK_F32) rglru_decode_kernel<float><<<grid, 256, 0, stream>>>(*p);
  else rglru_decode_kernel<__nv_bfloat16><<<grid, 256, 0, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

extern "C" int nfk_rglru_prefill(const nfk_rglru_params* p, cudaStream_t stream) {
  using namespace nf;
  const int rc = check_rglru(p);
  if (rc != NF_OK || p->req_count == 0) return rc;
  const dim3 grid((p->cols + 31) / 32, p->req_count);
  if (p->dtype == NFK_F32) rglru_prefill_kernel<float><<<grid, kRgWarps * 32, 0, stream>>>(*p);
  else rglru_prefill_kernel<__nv_bfloat16><<<grid, kRgWarps * 32, 0, stream>>>(*p);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}
