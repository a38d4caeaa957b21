// Attention scores on their way into a base-2 softmax: scaled, and optionally squashed into (-softcap, softcap) by
// softcap * tanh(score / softcap).
#pragma once
#include <cuda_runtime.h>

#include "ptx_sm100.cuh"

namespace artb {

// tanh(u) = 1 - 2 / (1 + e^(2u)) on the special-function units; the error is a few 1e-7 absolute, which is what a softmax
// over softcap * tanh(u) sees of it, times softcap
__device__ __forceinline__ float tanh_from_exp(float u) {
  float e;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(u * 2.885390081777927f));
  return fmaf(-2.f, rcp_approx(1.f + e), 1.f);
}

struct ScoreScale {
  float in;            // score / softcap = in * (q . k); 0: not squashed
  float scale_log2;    // factor behind it, log2(e) included

  static ScoreScale of(float scale, float softcap) {
    constexpr float LOG2E = 1.4426950408889634f;
    return softcap > 0.f ? ScoreScale{scale / softcap, softcap * LOG2E} : ScoreScale{0.f, scale * LOG2E};
  }
  __host__ __device__ __forceinline__ bool capped() const { return in != 0.f; }
  __device__ __forceinline__ float squash(float qk) const { return tanh_from_exp(qk * in); }
  // the exponent (base 2) of a product q . k
  __device__ __forceinline__ float operator()(float qk) const { return (capped() ? squash(qk) : qk) * scale_log2; }
};

}  // namespace artb
