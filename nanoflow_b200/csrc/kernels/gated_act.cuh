// Activations of the GEMM epilogues (NFK_ACT_*, NFK_LIN_*), shared by the dense and the grouped products.
#pragma once
#include "kernels.h"

namespace nf {

struct GatedAct {
  int kind;
  float limit, alpha, shift;
};

template <bool PRECISE>
__device__ __forceinline__ float gated_act_of(float g, float u, const GatedAct& a) {
  if (a.kind == NFK_ACT_RELU) return fmaxf(g, 0.f) * u;
  if (a.kind == NFK_ACT_GELU_TANH) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
  if (a.kind == NFK_ACT_CAPPED) {
    g = fminf(g, a.limit);
    u = fminf(fmaxf(u, -a.limit), a.limit);
    const float z = -a.alpha * g;
    return g / (1.f + (PRECISE ? expf(z) : __expf(z))) * (u + a.shift);
  }
  return g / (1.f + (PRECISE ? expf(-g) : __expf(-g))) * u;
}
__device__ __forceinline__ float gated_act(float g, float u, const GatedAct& a) { return gated_act_of<false>(g, u, a); }

__device__ __forceinline__ float lin_act_of(float v, int kind) {
  if (kind == NFK_LIN_TANH) return tanhf(v);
  if (kind == NFK_LIN_GELU) return 0.5f * v * (1.f + erff(v * 0.7071067811865476f));
  if (kind == NFK_LIN_RELU2) {
    const float r = fmaxf(v, 0.f);
    return r * r;
  }
  return v;
}

}  // namespace nf
