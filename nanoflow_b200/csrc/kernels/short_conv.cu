// Short causal convolution over time, one filter per channel, with the last inputs of every request kept in its state
// (see kernels.h). A thread takes four channels of a run of tokens and keeps the filter's window in registers, so that
// every input is read once; where a request starts inside the run, the window is loaded again: from the request's own
// rows, its state, or zeros.
#include "elem_io.cuh"

namespace nf {
namespace {

constexpr int kScRun = 8, kScThreads = 128;

__device__ __forceinline__ uint2 load_raw(const __nv_bfloat16* p) { return *reinterpret_cast<const uint2*>(p); }
__device__ __forceinline__ float4 load_raw(const float* p) { return load4(p); }
__device__ __forceinline__ float4 as_f32(float4 v) { return v; }
__device__ __forceinline__ float4 as_f32(uint2 u) {
  const float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y);
  return make_float4(a.x, a.y, b.x, b.y);
}
template <bool FAST>
__device__ __forceinline__ float silu_f(float y) { return FAST ? __fdividef(y, 1.f + __expf(-y)) : y / (1.f + expf(-y)); }

// RUN: tokens per thread.
template <class T, int TAPS, int RUN>
__global__ void __launch_bounds__(kScThreads)
short_conv_kernel(nfk_short_conv_params p, int groups) {
  constexpr int H = TAPS - 1;                    // inputs before the current one
  constexpr bool FAST = sizeof(T) == 2;
  using Raw = decltype(load_raw(static_cast<const T*>(nullptr)));
  const unsigned id = blockIdx.x * kScThreads + threadIdx.x;
  const unsigned run = id / static_cast<unsigned>(groups);
  const int c = static_cast<int>(id - run * groups) * 4;
  const int begin = p.row_begin + static_cast<int>(run) * RUN, end = min(begin + RUN, p.T);
  if (begin >= end) return;
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  Raw raw[RUN];                                  // all rows are requested before any of them is used
#pragma unroll
  for (int i = 0; i < RUN; ++i)
    if (begin + i < end) raw[i] = load_raw(x + (begin + i) * p.ld_x);
  float4 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = load4(p.w + static_cast<long long>(j) * p.cols + c);
  const float4 b = p.bias != nullptr ? load4(p.bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  T* out = reinterpret_cast<T*>(p.out) + c;
  T* state = reinterpret_cast<T*>(p.state) + c;
  float4 hist[H > 0 ? H : 1];
  int t1 = begin;                                // end of the current request
  int ref = -1;
#pragma unroll
  for (int i = 0; i < RUN; ++i) {
    const int t = begin + i;
    if (t >= end) break;
    if (t == t1 || i == 0) {
      const int req = p.token_req[t];
      const int t0 = p.qo_indptr[req];
      t1 = p.qo_indptr[req + 1];
      ref = p.state_slot[req];
      if (ref < 0 || (ref >> 1) >= p.num_slots) {
        if (c == 0) report_status(p.status, NF_ST_BAD_INDEX);
        ref = -1;
      }
      const bool older = ref >= 0 && t - H < t0 && p.positions[t0] > 0;
      const T* st = state + static_cast<long long>(ref >= 0 ? ref : 0) * (H > 0 ? H : 1) * p.cols;
#pragma unroll
      for (int j = 0; j < H; ++j) {
        const int s = t - H + j;                 // token whose input this is
        hist[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s >= t0) hist[j] = load4(x + s * p.ld_x);
        else if (older) hist[j] = load4(st + static_cast<long long>(s - t0 + H) * p.cols);
      }
    }
    const float4 v = as_f32(raw[i]);
    float4 y = b;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float4 s = j < H ? hist[j < H ? j : 0] : v;
      y.x += w[j].x * s.x; y.y += w[j].y * s.y; y.z += w[j].z * s.z; y.w += w[j].w * s.w;
    }
    if (p.act == NFK_CONV_SILU) y = make_float4(silu_f<FAST>(y.x), silu_f<FAST>(y.y), silu_f<FAST>(y.z), silu_f<FAST>(y.w));
    if (p.residual != 0) {
      y.x += v.x; y.y += v.y; y.z += v.z; y.w += v.w;
    }
    store4(out + t * p.ld_out, y);
#pragma unroll
    for (int j = 0; j + 1 < H; ++j) hist[j] = hist[j + 1];
    if (H > 0) hist[H > 0 ? H - 1 : 0] = v;
    if (H > 0 && t + 1 == t1 && ref >= 0) {      // the other half; the one read above stays as it is in this launch
      T* keep = state + static_cast<long long>(ref ^ 1) * H * p.cols;
#pragma unroll
      for (int j = 0; j < H; ++j) store4(keep + static_cast<long long>(j) * p.cols, hist[j]);
    }
  }
}

template <class T, int TAPS>
int launch_taps(const nfk_short_conv_params& p, cudaStream_t stream) {
  const int groups = p.cols / 4, rows = p.T - p.row_begin;
  const int run = rows <= 1024 ? 1 : kScRun;     // few rows: one thread each, also for single tokens of many requests
  const long long threads = static_cast<long long>((rows + run - 1) / run) * groups;
  if (threads > 0x7fffffffll) return NF_ERR_BAD_ARG;
  const int g = static_cast<int>((threads + kScThreads - 1) / kScThreads);
  if (run == 1) short_conv_kernel<T, TAPS, 1><<<g, kScThreads, 0, stream>>>(p, groups);
  else short_conv_kernel<T, TAPS, kScRun><<<g, kScThreads, 0, stream>>>(p, groups);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

template <class T>
int launch_short_conv(const nfk_short_conv_params& p, cudaStream_t stream) {
  switch (p.taps) {
    case 1: return launch_taps<T, 1>(p, stream);
    case 2: return launch_taps<T, 2>(p, stream);
    case 3: return launch_taps<T, 3>(p, stream);
    case 4: return launch_taps<T, 4>(p, stream);
    case 5: return launch_taps<T, 5>(p, stream);
    case 6: return launch_taps<T, 6>(p, stream);
    case 7: return launch_taps<T, 7>(p, stream);
    case 8: return launch_taps<T, 8>(p, stream);
    default: return NF_ERR_UNSUPPORTED;
  }
}

}  // namespace
}  // namespace nf

extern "C" int nfk_short_conv(const nfk_short_conv_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->T == p->row_begin) return NF_OK;
  if (!p->x || !p->out || p->x == p->out || !p->w || !p->state || !p->state_slot || !p->positions || !p->token_req ||
      !p->qo_indptr || p->row_begin < 0 || p->T < p->row_begin || p->cols <= 0 || p->cols % 4 != 0 || p->taps <= 0 ||
      p->num_slots <= 0 || p->ld_x % 4 != 0 || p->ld_out % 4 != 0 || p->act < NFK_CONV_NONE || p->act > NFK_CONV_SILU)
    return NF_ERR_BAD_ARG;
  return p->dtype == NFK_F32 ? launch_short_conv<float>(*p, stream) : launch_short_conv<__nv_bfloat16>(*p, stream);
}
