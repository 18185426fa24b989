// GEMM in plain fp32 FMA arithmetic (no reduced-precision matrix mode), for engines that run in 32-bit:
// the same products, epilogues and block-diagonal form as gemm.cu on fp32 operands. A 64 x 64 output tile
// per 256-thread CTA, 4 x 4 outputs per thread, operands staged 16 k at a time in shared memory.
#include "common.cuh"
#include "gated_act.cuh"
#include "kernels.h"

namespace nf {
namespace {

constexpr int kT = 64, kKb = 16, kThr = 256;

template <bool GATED>
__global__ void __launch_bounds__(kThr)
gemm_f32_kernel(nfk_gemm_params p, int groups, int group_n) {
  __shared__ float sa[kKb][kT + 4], sb[kKb][kT + 4], sc[GATED ? kKb : 1][kT + 4];
  const int per = (group_n + kT - 1) / kT;
  const int g = blockIdx.x / per;
  const int col0 = g * group_n + (blockIdx.x - g * per) * kT;     // first output column = first row of B
  const int col_end = min((g + 1) * group_n, col0 + kT);
  const int row0 = blockIdx.y * kT;
  const float* A = reinterpret_cast<const float*>(p.A) + static_cast<long long>(g) * p.group_k;
  const float* B = reinterpret_cast<const float*>(p.B);
  const float* B2 = reinterpret_cast<const float*>(p.B2);
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {}, up[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += kKb) {
    for (int i = threadIdx.x; i < kT * kKb; i += kThr) {
      const int r = i / kKb, k = i % kKb;
      const bool kin = k0 + k < p.K;
      sa[k][r] = (kin && row0 + r < p.M) ? A[static_cast<long long>(row0 + r) * p.lda + k0 + k] : 0.f;
      const bool in = kin && col0 + r < col_end;
      const long long bo = static_cast<long long>(col0 + r) * p.ldb + k0 + k;
      sb[k][r] = in ? B[bo] : 0.f;
      if (GATED) sc[k][r] = in ? B2[bo] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kKb; ++k) {
      float a[4], b[4], c[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        a[i] = sa[k][ty * 4 + i];
        b[i] = sb[k][tx * 4 + i];
        if (GATED) c[i] = sc[k][tx * 4 + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
          if (GATED) up[i][j] = fmaf(a[i], c[j], up[i][j]);
        }
    }
    __syncthreads();
  }
  float* D = reinterpret_cast<float*>(p.D);
  float* D32 = reinterpret_cast<float*>(p.D32);
  const float* C = reinterpret_cast<const float*>(p.C);
  const float* bias = reinterpret_cast<const float*>(p.bias);
  const float* bias2 = reinterpret_cast<const float*>(p.bias2);
  const GatedAct act{p.act, p.act_limit, p.act_alpha, p.act_shift};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int row = row0 + ty * 4 + i;
    if (row >= p.M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = col0 + tx * 4 + j;
      if (col >= col_end) continue;
      float v = acc[i][j];
      if (GATED) {
        const float u = up[i][j];
        v = bias != nullptr ? gated_act_of<true>(v + bias[col], u + bias2[col], act) : gated_act_of<true>(v, u, act);
      } else {
        if (bias != nullptr) v += bias[col];
        if (C != nullptr) v += p.beta * C[static_cast<long long>(row) * p.ldc + col];
      }
      if (!GATED) v = lin_act_of(v, p.lin_act);
      if (D32 != nullptr && col >= p.f32_col0) D32[static_cast<long long>(row) * p.ld32 + col - p.f32_col0] = v;
      else D[static_cast<long long>(row) * p.ldd + col] = v;
    }
  }
}

}  // namespace
}  // namespace nf

extern "C" int nfk_gemm_f32(const nfk_gemm_params* p, cudaStream_t stream) {
  using namespace nf;
  if (p == nullptr) return NF_ERR_BAD_ARG;
  if (p->M == 0 || p->N == 0) return NF_OK;
  const int groups = p->groups > 1 ? p->groups : 1;
  if (!p->A || !p->B || p->M < 0 || p->N < 0 || p->K <= 0 || p->N % groups != 0 || p->group_k < 0) return NF_ERR_BAD_ARG;
  if (!p->D && !(p->D32 && p->f32_col0 == 0)) return NF_ERR_BAD_ARG;
  if (p->epilogue == NFK_EPI_SWIGLU && (!p->B2 || groups > 1 || p->D32 || (p->bias == nullptr) != (p->bias2 == nullptr))) return NF_ERR_BAD_ARG;
  if (p->epilogue != NFK_EPI_LINEAR && p->epilogue != NFK_EPI_SWIGLU) return NF_ERR_UNSUPPORTED;
  if (p->norm_w || p->gate_flags) return NF_ERR_UNSUPPORTED;
  const int group_n = p->N / groups;
  const int m_tiles = (p->M + kT - 1) / kT;
  if (m_tiles > 65535) return NF_ERR_BAD_ARG;
  const dim3 grid(groups * ((group_n + kT - 1) / kT), m_tiles);
  if (p->epilogue == NFK_EPI_SWIGLU) gemm_f32_kernel<true><<<grid, kThr, 0, stream>>>(*p, groups, group_n);
  else gemm_f32_kernel<false><<<grid, kThr, 0, stream>>>(*p, groups, group_n);
  return cudaGetLastError() == cudaSuccess ? NF_OK : NF_ERR_CUDA;
}
