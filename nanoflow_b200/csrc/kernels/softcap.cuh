// Forms of attention scores shared by the attention kernels: capped scores, cap tanh(score / cap), and distance biases.
#pragma once
#include "common.cuh"

namespace nf {

// tanh x = 1 - 2 / (e^(2x) + 1): within a few 1e-7 absolute everywhere, and +-1 at the far ends.
NF_DEVICE float tanh_by_exp(float x) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(x * 2.8853900817779268f));   // 2 log2(e)
  return 1.f - __fdividef(2.f, e + 1.f);
}

// What a score (in units of log2) loses at a distance: a log2(1 + b distance). The argument is 1 or more.
NF_DEVICE float distance_loss(float2 ab, float distance) {
  float l;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(fmaf(ab.y, distance, 1.f)));
  return ab.x * l;
}

}  // namespace nf
