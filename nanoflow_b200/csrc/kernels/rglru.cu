// Real-gated linear recurrent unit (De et al., "Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient
// Language Models"; see kernels.h for the equations). State, gates, decays and their logarithms are fp32.
//
// nfk_rglru_decode   one token per request: a thread per channel.
// nfk_rglru_prefill  a CTA takes 32 (or 16) channels of a request and walks its tokens 128 (256) at a time, in runs of eight:
//                    each run is reduced to (decay, end state from zero), all chain those, and every run then goes through
//                    its tokens again from the state it starts with, out of registers. Inputs are read once, a step ahead.
#include "elem_io.cuh"

namespace nf {
namespace {

struct RgStep {
  float a, b;      // S <- a S + b
};
// FAST (bf16 results): exponentials, reciprocals and square roots of the special-function unit, a few units in the last
// place of fp32; 1 - a^2 of slow decays by the exponential's series, so that it does not cancel.
template <bool FAST>
__device__ __forceinline__ float sigmoid_f(float z) {
  return FAST ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z));
}
template <bool FAST>
__device__ __forceinline__ RgStep rg_step(float r, float i, float u, float r_b, float i_b, float log_a) {
  const float la = log_a * sigmoid_f<FAST>(r + r_b);
  RgStep s;
  float rest;      // sqrt(1 - a^2)
  if (FAST) {
    const float x = -2.f * la;
    s.a = __expf(la);
    const float d = x < 0.03125f ? x * (1.f - x * (0.5f - x * (0.16666667f - x * 0.041666667f))) : 1.f - s.a * s.a;
    asm("sqrt.approx.f32 %0, %1;" : "=f"(rest) : "f"(d));
  } else {
    s.a = expf(la);
    rest = sqrtf(-expm1f(2.f * la));
  }
  s.b = rest * sigmoid_f<FAST>(i + i_b) * u;
  return s;
}
template <bool FAST>
__device__ __forceinline__ float gelu_tanh_f(float z) {
  const float w = 0.7978845608028654f * (z + 0.044715f * z * z * z);
  return FAST ? z * sigmoid_f<true>(2.f * w) : 0.5f * z * (1.f + tanhf(w));
}
template <class T>
constexpr bool kFast = sizeof(T) == 2;
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
  const RgStep s = rg_step<kFast<T>>(g[0], g[p.block], to_f32(reinterpret_cast<const T*>(p.u)[t * p.ld_u + c]), p.r_b[c], p.i_b[c], p.log_a[c]);
  const float x = s.a * (p.positions[t] == 0 ? 0.f : *S) + s.b;
  *S = x;
  put(reinterpret_cast<T*>(p.out) + t * p.ld_out + c, x * gelu_tanh_f<kFast<T>>(to_f32(reinterpret_cast<const T*>(p.y)[t * p.ld_y + c])));
}

constexpr int kRgWarps = 16, kRgRun = 8;

// What a thread reads of its run of tokens.
template <class T>
struct RgInputs {
  float r[kRgRun], i[kRgRun];
  T u[kRgRun], y[kRgRun];
};

// CW: channels per CTA, 32 or (when there are few CTAs) 16; 32 / CW runs of tokens share a warp.
template <class T, int CW>
__global__ void __launch_bounds__(kRgWarps * 32)
rglru_prefill_kernel(nfk_rglru_params p) {
  constexpr int kRuns = kRgWarps * 32 / CW, kBlock = kRuns * kRgRun;
  __shared__ float a_s[2][kRuns][CW], b_s[2][kRuns][CW];
  const int run = threadIdx.x / CW, lane = threadIdx.x % CW;
  const int c = blockIdx.x * CW + lane;
  const int req = p.req_begin + blockIdx.y;
  const int ref = p.state_slot[req];
  if (ref < 0 || (ref >> 1) >= p.num_slots) {
    if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
    return;
  }
  const bool ok = c < p.cols;
  const int t0 = p.qo_indptr[req], t1 = p.qo_indptr[req + 1];
  float* S = p.S + static_cast<long long>(ref >> 1) * p.cols + c;
  const float r_b = ok ? p.r_b[c] : 0.f, i_b = ok ? p.i_b[c] : 0.f, log_a = ok ? p.log_a[c] : 0.f;
  const T* u = reinterpret_cast<const T*>(p.u) + (ok ? c : 0);
  const T* y = reinterpret_cast<const T*>(p.y) + (ok ? c : 0);
  const float* g = p.gates + (ok ? gate_col(c, p.block) : 0);
  T* out = reinterpret_cast<T*>(p.out) + c;
  auto fetch = [&](RgInputs<T>& in, int begin) {
#pragma unroll
    for (int j = 0; j < kRgRun; ++j) {
      const long long t = begin + j < t1 ? begin + j : t1 - 1;       // past the end: not used
      in.r[j] = g[t * p.ld_g];
      in.i[j] = g[t * p.ld_g + p.block];
      in.u[j] = u[t * p.ld_u];
      in.y[j] = y[t * p.ld_y];
    }
  };
  float carry = (ok && p.positions[t0] != 0) ? *S : 0.f;             // every run keeps it
  RgInputs<T> in;
  fetch(in, t0 + run * kRgRun);
  int buf = 0;
  for (int base = t0; base < t1; base += kBlock, buf ^= 1) {
    const int begin = base + run * kRgRun;
    RgStep s[kRgRun];
    float yy[kRgRun], a = 1.f, b = 0.f;
#pragma unroll
    for (int j = 0; j < kRgRun; ++j) {
      s[j].a = 1.f;
      s[j].b = yy[j] = 0.f;
      if (begin + j < t1) {
        s[j] = rg_step<kFast<T>>(in.r[j], in.i[j], to_f32(in.u[j]), r_b, i_b, log_a);
        yy[j] = gelu_tanh_f<kFast<T>>(to_f32(in.y[j]));
      }
      a *= s[j].a;
      b = s[j].a * b + s[j].b;
    }
    if (base + kBlock < t1) fetch(in, begin + kBlock);               // while the warps wait for one another
    a_s[buf][run][lane] = a;
    b_s[buf][run][lane] = b;
    __syncthreads();
    float x = carry;
#pragma unroll
    for (int k = 0; k < kRuns; ++k) {
      if (k == run) x = carry;                                       // what this run starts from
      carry = a_s[buf][k][lane] * carry + b_s[buf][k][lane];
    }
#pragma unroll
    for (int j = 0; j < kRgRun; ++j) {
      x = s[j].a * x + s[j].b;
      if (begin + j < t1 && ok) put(out + static_cast<long long>(begin + j) * p.ld_out, x * yy[j]);
    }
  }
  if (run == 0 && ok) *S = carry;
}

template <class T>
void launch_rglru_prefill(const nfk_rglru_params& p, cudaStream_t stream) {
  const int wide = (p.cols + 31) / 32;
  if (wide * p.req_count < device_sm_count())
    rglru_prefill_kernel<T, 16><<<dim3((p.cols + 15) / 16, p.req_count), kRgWarps * 32, 0, stream>>>(p);
  else
    rglru_prefill_kernel<T, 32><<<dim3(wide, p.req_count), kRgWarps * 32, 0, stream>>>(p);
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
  if (p->dtype == NFK_F32) launch_rglru_prefill<float>(*p, stream);
  else launch_rglru_prefill<__nv_bfloat16>(*p, stream);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}
