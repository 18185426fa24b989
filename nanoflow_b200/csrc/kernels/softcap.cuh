// Capped attention scores, cap tanh(score / cap), shared by the attention kernels.
#pragma once
#include "common.cuh"

namespace nf {

// tanh x = 1 - 2 / (e^(2x) + 1): within a few 1e-7 absolute everywhere, and +-1 at the far ends.
NF_DEVICE float tanh_by_exp(float x) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * 2.8853900817779268f));   // 2 log2(e)
  return 1.f - __fdividef(2.f, e + 1.f);
}
// The same for |x| <= kTanhSmall without the special function unit: odd polynomial of degree 9, fitted to tanh by
// reweighted least squares on that interval (within 8e-8 in fp32).
constexpr float kTanhSmall = 0.6f;
NF_DEVICE float tanh_small(float x) {
  const float u = x * x;
  float p = 0.01497695975f;
  p = fmaf(p, u, -0.05169674269f);
  p = fmaf(p, u, 0.1329921021f);
  p = fmaf(p, u, -0.3333120859f);
  p = fmaf(p, u, 0.9999996274f);
  return p * x;
}

}  // namespace nf
