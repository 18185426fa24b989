// The step between two sublayers in one pass over the row: norm of the sublayer's output, residual sum in
// fp32, an optional vector added to the stream, and the norm that the next sublayer reads.
//
//   x <- (table ? 0 : x) + norm_in(src) (+ second output) (+ weighted expert outputs) (+ add);   h = norm_out(x)
//
// The norm can also be taken of the whole sum, the source can be the mean of two normed outputs, and the embedding row
// can join a stream that goes on (see kernels.h). A position vector can join the embedding row, the "norm" of the source can
// be a mere scale per column, and what goes on can be a weighted sum of the result and of earlier results. Where the next sublayer reads its input through a convolution over time,
// rows that are the only token of their request get it here, from the request's state.
// `src` is the sublayer's output row, or the embedding row of the token (ids as in nfk_embedding, with the
// previous iteration's tokens fed back on the device). Norms are RMS or layer norms with fp32 weights. The
// stream x is fp32; src and h are bf16 or fp32. One CTA per row, the row stays in registers.
#include "elem_io.cuh"

namespace nf {
namespace {

constexpr int kRnThreads = 256;

// Sum over the CTA of one value per thread; every thread gets the result.
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  __syncthreads();                       // readers of the previous sum are done with `red`
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < (kRnThreads >> 5) ? red[lane] : 0.f);
}

__device__ __forceinline__ void fma4(float4& a, float f, float4 b) {
  a.x += f * b.x; a.y += f * b.y; a.z += f * b.z; a.w += f * b.w;
}

// In-place norm of the row held in v (elements at or past `cols` are zero and stay zero).
template <int NV>
__device__ __forceinline__ void norm_row(float4 (&v)[NV], int kind, const float* w, const float* b, int cols, int nvec,
                                         float eps, float* red) {
  if (kind == NFK_NORM_NONE) return;
  if (kind == NFK_NORM_SCALE) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      if (vi >= nvec) continue;
      const float4 ww = load4(w + vi * 4);            // zero past `cols`
      v[i] = make_float4(v[i].x * ww.x, v[i].y * ww.y, v[i].z * ww.z, v[i].w * ww.w);
    }
    return;
  }
  const float inv_n = 1.f / static_cast<float>(cols);
  float mean = 0.f;
  if (kind == NFK_NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
    mean = cta_sum(s, red) * inv_n;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int c = (threadIdx.x + i * kRnThreads) * 4;
    float* e = reinterpret_cast<float*>(&v[i]);
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (c + j < cols) {
        e[j] -= mean;
        ss += e[j] * e[j];
      }
  }
  const float inv = rsqrtf(cta_sum(ss, red) * inv_n + eps);
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int vi = threadIdx.x + i * kRnThreads;
    if (vi < nvec) {
      const float4 ww = load4(w + vi * 4);            // zero past `cols`
      const float4 bb = b != nullptr ? load4(b + vi * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      v[i].x = v[i].x * inv * ww.x + bb.x;
      v[i].y = v[i].y * inv * ww.y + bb.y;
      v[i].z = v[i].z * inv * ww.z + bb.z;
      v[i].w = v[i].w * inv * ww.w + bb.w;
    }
  }
}

__device__ __forceinline__ float4 rounded(float4 v, float) { return v; }
__device__ __forceinline__ float4 rounded(float4 v, __nv_bfloat16) {
  const float2 a = unpack_bf16x2(pack_bf16x2(v.x, v.y)), b = unpack_bf16x2(pack_bf16x2(v.z, v.w));
  return make_float4(a.x, a.y, b.x, b.y);
}
// The normed row v of a request's only token plus its convolution with the inputs kept in the request's state.
template <class T, int NV>
__device__ __forceinline__ void input_conv(const float4 (&v)[NV], const nfk_residual_norm_params& p, int row, int nvec) {
  const int ref = p.state_slot[row], before = p.conv_taps - 1;
  const bool ok = ref >= 0 && (ref >> 1) < p.num_slots, older = ok && p.positions[row] > 0;
  if (!ok && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
  const long long half = static_cast<long long>(before > 0 ? before : 1) * p.conv_ld;
  const T* st = reinterpret_cast<const T*>(p.conv_state) + (ok ? ref : 0) * half;
  T* keep = reinterpret_cast<T*>(p.conv_state) + (ok ? ref ^ 1 : 0) * half;
  T* out = reinterpret_cast<T*>(p.conv_out) + static_cast<long long>(row) * p.conv_ld;
  if (NV <= 8 && before == 1) {                          // two taps: everything is requested before anything is stored
    float4 s[NV], f[NV], w[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      if (vi >= nvec) continue;
      s[i] = older ? load4(st + vi * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      f[i] = load4(p.conv_w + vi * 4);
      w[i] = load4(p.conv_w + p.conv_ld + vi * 4);
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      if (vi >= nvec) continue;
      const float4 x = rounded(v[i], T(0.f));
      if (ok) store4(keep + vi * 4, x);
      store4(out + vi * 4, make_float4(x.x + w[i].x * x.x + f[i].x * s[i].x, x.y + w[i].y * x.y + f[i].y * s[i].y,
                                       x.z + w[i].z * x.z + f[i].z * s[i].z, x.w + w[i].w * x.w + f[i].w * s[i].w));
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < NV; ++i) {
    const int vi = threadIdx.x + i * kRnThreads;
    if (vi >= nvec) continue;
    const float4 x = rounded(v[i], T(0.f)), w = load4(p.conv_w + static_cast<long long>(before) * p.conv_ld + vi * 4);
    float4 y = make_float4(x.x + w.x * x.x, x.y + w.y * x.y, x.z + w.z * x.z, x.w + w.w * x.w);
    for (int j0 = 0; j0 < before; j0 += 3) {             // three taps are requested at once
      float4 s[3], f[3];
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        const int j = j0 + k < before ? j0 + k : 0;
        s[k] = older ? load4(st + static_cast<long long>(j) * p.conv_ld + vi * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
        f[k] = load4(p.conv_w + static_cast<long long>(j) * p.conv_ld + vi * 4);
      }
#pragma unroll
      for (int k = 0; k < 3; ++k) {
        const int j = j0 + k;
        if (j >= before) break;
        y.x += f[k].x * s[k].x; y.y += f[k].y * s[k].y; y.z += f[k].z * s[k].z; y.w += f[k].w * s[k].w;
        if (ok && j > 0) store4(keep + static_cast<long long>(j - 1) * p.conv_ld + vi * 4, s[k]);
      }
    }
    if (ok && before > 0) store4(keep + static_cast<long long>(before - 1) * p.conv_ld + vi * 4, x);
    store4(out + vi * 4, y);
  }
}

// sin and cos of pos * (hi + lo), the rounding of the product included.
__device__ __forceinline__ float2 sin_cos(float pos, float2 f) {
  const float a = pos * f.x, e = fmaf(pos, f.x, -a) + pos * f.y;
  float s, c;
  sincosf(a, &s, &c);
  const float h = 0.5f * e * e;
  return make_float2(fmaf(-h, s, fmaf(e, c, s)), fmaf(-h, c, fmaf(-e, s, c)));
}

// v (the sum of the row) is kept as a result of its own, and replaced by the weighted sum of all results so far.
template <int NV>
__device__ __forceinline__ void depth_average(float4 (&v)[NV], const nfk_residual_norm_params& p, long long row_off, int nvec) {
  if (p.hist_out != nullptr) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      if (vi < nvec) store4(p.hist_out + row_off + vi * 4, v[i]);
    }
  }
  if (p.hist_w == nullptr) return;
  const float own = p.hist_w[p.hist_n];
#pragma unroll
  for (int i = 0; i < NV; ++i) v[i] = make_float4(own * v[i].x, own * v[i].y, own * v[i].z, own * v[i].w);
  const float* src = p.hist + row_off;
#pragma unroll 4
  for (int j = 0; j < p.hist_n; ++j, src += p.hist_stride) {
    const float f = p.hist_w[j];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      if (vi < nvec) fma4(v[i], f, load4(src + vi * 4));
    }
  }
}

// CONV: some rows go through the input convolution. DEEP: position vectors and earlier results.
template <class T, int NV, bool CONV, bool DEEP>
__global__ void __launch_bounds__(kRnThreads)
residual_norm_kernel(nfk_residual_norm_params p) {
  __shared__ float red[kRnThreads / 32];
  const int nvec = (p.cols + 3) >> 2;
  for (int row = blockIdx.x; row < p.rows; row += gridDim.x) {
    int src_row = row;
    if (p.rows_idx != nullptr) {
      src_row = p.rows_idx[row];
      if (src_row < 0 || src_row >= p.in_rows) {
        if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
        src_row = 0;
      }
    }
    const T *src = nullptr, *again = nullptr;
    if (p.table != nullptr) {
      int id = p.host_ids != nullptr ? p.host_ids[row] : 0;
      if (p.feedback_src != nullptr && p.prev_tokens != nullptr) {
        const int f = p.feedback_src[row];
        if (f >= 0) id = p.prev_tokens[f];
      }
      if (id < 0 || id >= p.vocab) {
        if (threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
        id = 0;
      }
      (p.table_add != 0 ? again : src) = reinterpret_cast<const T*>(p.table) + static_cast<long long>(id) * p.ld_table;
    }
    if (p.y != nullptr && (p.table == nullptr || p.table_add != 0)) {
      src = reinterpret_cast<const T*>(p.y) + static_cast<long long>(src_row) * p.ld_y;
    }
    float* xr = p.x + static_cast<long long>(src_row) * p.ld_x;
    float4 v[NV];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      v[i] = (src != nullptr && vi < nvec) ? load4(src + vi * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    if (src != nullptr && again == nullptr && p.src_scale != 0.f) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        v[i].x *= p.src_scale; v[i].y *= p.src_scale; v[i].z *= p.src_scale; v[i].w *= p.src_scale;
      }
    }
    if (DEEP && p.pos_freq != nullptr) {
      const float pos = static_cast<float>(p.positions[row]);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int vi = threadIdx.x + i * kRnThreads;
        if (vi >= nvec) continue;
        const int c = vi * 4;
        const float2* f = reinterpret_cast<const float2*>(p.pos_freq) + vi * 2;
        const float2 a = sin_cos(pos, f[0]), b = c + 2 < p.cols ? sin_cos(pos, f[1]) : make_float2(0.f, 0.f);
        v[i].x += a.x; v[i].z += b.x;
        if (c + 1 < p.cols) v[i].y += a.y;
        if (c + 3 < p.cols) v[i].w += b.y;
      }
    }
    if (p.pair_w != nullptr) {
      const T* y2 = reinterpret_cast<const T*>(p.y2) + static_cast<long long>(src_row) * p.ld_y2;
      float4 o[NV];
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int vi = threadIdx.x + i * kRnThreads;
        o[i] = vi < nvec ? load4(y2 + vi * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
      norm_row<NV>(v, NFK_NORM_RMS, p.pair_w, nullptr, p.cols, nvec, p.eps, red);
      norm_row<NV>(o, NFK_NORM_RMS, p.pair_w2, nullptr, p.cols, nvec, p.eps, red);
#pragma unroll
      for (int i = 0; i < NV; ++i)
        v[i] = make_float4(0.5f * (v[i].x + o[i].x), 0.5f * (v[i].y + o[i].y), 0.5f * (v[i].z + o[i].z), 0.5f * (v[i].w + o[i].w));
    }
    if (src != nullptr && p.norm_sum == 0) norm_row<NV>(v, p.in_kind, p.in_w, p.in_b, p.cols, nvec, p.eps, red);
    if (p.y2 != nullptr && p.pair_w == nullptr) {
      const float f = p.y2_gate != nullptr ? p.y2_gate[src_row] : 1.f;
      const T* y2 = reinterpret_cast<const T*>(p.y2) + static_cast<long long>(src_row) * p.ld_y2;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int vi = threadIdx.x + i * kRnThreads;
        if (vi < nvec) fma4(v[i], f, load4(y2 + vi * 4));
      }
    }
    if (p.e_out != nullptr) {
      for (int k = 0; k < p.e_top; ++k) {
        const int slot = p.e_slot[static_cast<long long>(src_row) * p.e_top + k];
        const float f = p.e_weight[static_cast<long long>(src_row) * p.e_top + k];
        if (slot < 0 || slot >= p.e_rows) {
          if (slot != -1 && threadIdx.x == 0) report_status(p.status, NF_ST_BAD_INDEX);
          continue;
        }
        const T* e = reinterpret_cast<const T*>(p.e_out) + static_cast<long long>(slot) * p.ld_e;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
          const int vi = threadIdx.x + i * kRnThreads;
          if (vi < nvec) fma4(v[i], f, load4(e + vi * 4));
        }
      }
    }
    if (p.norm_sum != 0) norm_row<NV>(v, p.in_kind, p.in_w, p.in_b, p.cols, nvec, p.eps, red);
    if (again != nullptr) {
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int vi = threadIdx.x + i * kRnThreads;
        if (vi < nvec) fma4(v[i], p.src_scale != 0.f ? p.src_scale : 1.f, load4(again + vi * 4));
      }
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int vi = threadIdx.x + i * kRnThreads;
      if (vi < nvec) {
        if (p.table == nullptr || p.table_add != 0) {
          const float4 x = load4(xr + vi * 4);
          v[i].x += x.x; v[i].y += x.y; v[i].z += x.z; v[i].w += x.w;
        }
        if (p.add != nullptr) {
          const float4 a = load4(p.add + vi * 4);
          v[i].x += a.x; v[i].y += a.y; v[i].z += a.z; v[i].w += a.w;
        }
        if (!DEEP && p.rows_idx == nullptr) store4(xr + vi * 4, v[i]);
      }
    }
    if (DEEP) {
      depth_average<NV>(v, p, static_cast<long long>(src_row) * p.ld_x, nvec);
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int vi = threadIdx.x + i * kRnThreads;
        if (vi < nvec && p.rows_idx == nullptr) store4(xr + vi * 4, v[i]);
      }
    }
    if (p.h != nullptr) {
      norm_row<NV>(v, p.out_kind, p.out_w, p.out_b, p.cols, nvec, p.eps, red);
      if (CONV && row < p.conv_rows) {
        input_conv<T, NV>(v, p, row, nvec);
        continue;
      }
      T* hr = reinterpret_cast<T*>(p.h) + static_cast<long long>(row) * p.ld_h;
#pragma unroll
      for (int i = 0; i < NV; ++i) {
        const int vi = threadIdx.x + i * kRnThreads;
        if (vi < nvec) store4(hr + vi * 4, v[i]);
      }
    }
  }
}

template <class T, bool CONV, bool DEEP>
int launch_rn(const nfk_residual_norm_params& p, cudaStream_t stream) {
  const int nvec = (p.cols + 3) / 4, per = (nvec + kRnThreads - 1) / kRnThreads;
  const int cap = device_sm_count() * 16;
  const int grid = p.rows < cap ? p.rows : cap;
  if (per <= 1) residual_norm_kernel<T, 1, CONV, DEEP><<<grid, kRnThreads, 0, stream>>>(p);
  else if (per <= 2) residual_norm_kernel<T, 2, CONV, DEEP><<<grid, kRnThreads, 0, stream>>>(p);
  else if (per <= 4) residual_norm_kernel<T, 4, CONV, DEEP><<<grid, kRnThreads, 0, stream>>>(p);
  else if (per <= 8) residual_norm_kernel<T, 8, CONV, DEEP><<<grid, kRnThreads, 0, stream>>>(p);
  else if (per <= 16) residual_norm_kernel<T, 16, CONV, DEEP><<<grid, kRnThreads, 0, stream>>>(p);
  else return NF_ERR_UNSUPPORTED;
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}

template <class T>
int launch_rn_form(const nfk_residual_norm_params& p, cudaStream_t stream) {
  const bool deep = p.pos_freq != nullptr || p.hist_w != nullptr || p.hist_out != nullptr;
  if (p.conv_w != nullptr && p.conv_rows > 0) return deep ? launch_rn<T, true, true>(p, stream) : launch_rn<T, true, false>(p, stream);
  return deep ? launch_rn<T, false, true>(p, stream) : launch_rn<T, false, false>(p, stream);
}

}  // namespace
}  // namespace nf

extern "C" int nfk_residual_norm(const nfk_residual_norm_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->rows == 0) return NF_OK;
  if (!p->x || p->rows < 0 || p->cols <= 0 || p->ld_x % 4 != 0 || p->ld_x < p->cols) return NF_ERR_BAD_ARG;
  if (p->table && (p->rows_idx || p->vocab <= 0 || p->ld_table % 4 != 0)) return NF_ERR_BAD_ARG;
  if (p->table && !p->host_ids && !(p->feedback_src && p->prev_tokens)) return NF_ERR_BAD_ARG;
  if ((p->y && p->ld_y % 4 != 0) || (p->h && p->ld_h % 4 != 0)) return NF_ERR_BAD_ARG;
  if (p->rows_idx && (p->in_rows <= 0 || !p->h)) return NF_ERR_BAD_ARG;
  if (p->y2 && p->ld_y2 % 4 != 0) return NF_ERR_BAD_ARG;
  if (p->e_out && (!p->e_slot || !p->e_weight || p->e_top <= 0 || p->e_rows <= 0 || p->ld_e % 4 != 0)) return NF_ERR_BAD_ARG;
  if (p->conv_w && (!p->conv_out || !p->conv_state || !p->state_slot || !p->positions || !p->h || p->conv_taps <= 0 ||
                    p->conv_rows < 0 || p->conv_ld < p->cols || p->conv_ld % 4 != 0 || p->num_slots <= 0 || p->rows_idx))
    return NF_ERR_BAD_ARG;
  if (p->pair_w && (!p->pair_w2 || !p->y || !p->y2)) return NF_ERR_BAD_ARG;
  if (p->norm_sum && p->in_kind != NFK_NORM_NONE && !p->in_w) return NF_ERR_BAD_ARG;
  for (int kind : {p->in_kind, p->out_kind})
    if (kind < NFK_NORM_NONE || kind > NFK_NORM_SCALE) return NF_ERR_BAD_ARG;
  if ((p->table || p->y) && p->in_kind != NFK_NORM_NONE && !p->in_w) return NF_ERR_BAD_ARG;
  if (p->h && p->out_kind != NFK_NORM_NONE && !p->out_w) return NF_ERR_BAD_ARG;
  if (p->pos_freq && (!p->table || p->table_add || !p->positions)) return NF_ERR_BAD_ARG;
  if (p->hist_w && (p->hist_n < 0 || (p->hist_n > 0 && !p->hist))) return NF_ERR_BAD_ARG;
  if (p->hist_out && p->rows_idx) return NF_ERR_BAD_ARG;
  return p->dtype == NFK_F32 ? launch_rn_form<float>(*p, stream) : launch_rn_form<__nv_bfloat16>(*p, stream);
}
