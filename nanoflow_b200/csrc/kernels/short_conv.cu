// Short causal convolution over time, one filter per channel, with the last inputs of every request kept in its state
// (see kernels.h). A thread takes four channels of a run of tokens and keeps the filter's window in registers, so that
// every input is read once; where a request starts inside the run, the window is loaded again: from the request's own
// rows, its state, or zeros.
#include "elem_io.cuh"

namespace nf {
namespace {

constexpr int kScRun = 8, kScThreads = 128;

template <class T, int TAPS>
__global__ void __launch_bounds__(kScThreads)
short_conv_kernel(nfk_short_conv_params p, int groups) {
  constexpr int H = TAPS - 1;                    // inputs before the current one
  const long long id = blockIdx.x * static_cast<long long>(kScThreads) + threadIdx.x;
  const int c = static_cast<int>(id % groups) * 4;
  const int begin = p.row_begin + static_cast<int>(id / groups) * kScRun, end = min(begin + kScRun, p.T);
  if (begin >= end) return;
  float4 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) w[j] = load4(p.w + static_cast<long long>(j) * p.cols + c);
  const float4 b = p.bias != nullptr ? load4(p.bias + c) : make_float4(0.f, 0.f, 0.f, 0.f);
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  T* out = reinterpret_cast<T*>(p.out) + c;
  T* state = reinterpret_cast<T*>(p.state) + c;
  float4 hist[H > 0 ? H : 1];
  int t1 = begin;                                // end of the current request
  int ref = -1;
  for (int t = begin; t < end; ++t) {
    if (t == t1 || t == begin) {
      const int req = p.token_req[t];
      const int t0 = p.qo_indptr[req];
      t1 = p.qo_indptr[req + 1];
      ref = p.state_slot[req];
      if (ref < 0 || (ref >> 1) >= p.num_slots) {
        if (c == 0) report_status(p.status, NF_ST_BAD_INDEX);
        ref = -1;
      }
      const bool older = ref >= 0 && p.positions[t0] > 0;
      const T* st = state + static_cast<long long>(ref >= 0 ? ref : 0) * (H > 0 ? H : 1) * p.cols;
#pragma unroll
      for (int j = 0; j < H; ++j) {
        const int s = t - H + j;                 // token whose input this is
        hist[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (s >= t0) hist[j] = load4(x + s * p.ld_x);
        else if (older) hist[j] = load4(st + static_cast<long long>(s - t0 + H) * p.cols);
      }
    }
    const float4 v = load4(x + t * p.ld_x);
    float4 y = b;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      const float4 s = j < H ? hist[j < H ? j : 0] : v;
      y.x += w[j].x * s.x; y.y += w[j].y * s.y; y.z += w[j].z * s.z; y.w += w[j].w * s.w;
    }
    if (p.act == NFK_CONV_SILU) {
      y.x = y.x / (1.f + expf(-y.x)); y.y = y.y / (1.f + expf(-y.y));
      y.z = y.z / (1.f + expf(-y.z)); y.w = y.w / (1.f + expf(-y.w));
    }
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

template <class T>
int launch_short_conv(const nfk_short_conv_params& p, cudaStream_t stream) {
  const int groups = p.cols / 4;
  const long long threads = static_cast<long long>((p.T - p.row_begin + kScRun - 1) / kScRun) * groups;
  const long long grid = (threads + kScThreads - 1) / kScThreads;
  if (grid > 0x7fffffffll) return NF_ERR_BAD_ARG;
  const int g = static_cast<int>(grid);
  switch (p.taps) {
    case 1: short_conv_kernel<T, 1><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 2: short_conv_kernel<T, 2><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 3: short_conv_kernel<T, 3><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 4: short_conv_kernel<T, 4><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 5: short_conv_kernel<T, 5><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 6: short_conv_kernel<T, 6><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 7: short_conv_kernel<T, 7><<<g, kScThreads, 0, stream>>>(p, groups); break;
    case 8: short_conv_kernel<T, 8><<<g, kScThreads, 0, stream>>>(p, groups); break;
    default: return NF_ERR_UNSUPPORTED;
  }
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
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
