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

// of two numbers with one reciprocal: 1 / a = b / (a b).  From |u| = 20 on tanh is 1 in fp32; the product stays finite.
__device__ __forceinline__ void tanh_pair(float& u, float& v) {
  float e, f;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(fminf(u, 20.f) * 2.885390081777927f));
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(f) : "f"(fminf(v, 20.f) * 2.885390081777927f));
  e += 1.f;
  f += 1.f;
  const float r = -2.f * rcp_approx(e * f);
  u = fmaf(r, f, 1.f);
  v = fmaf(r, e, 1.f);
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
  __device__ __forceinline__ void squash(float& a, float& b) const {
    a *= in;
    b *= in;
    tanh_pair(a, b);
  }
  // the exponents of two products
  __device__ __forceinline__ void operator()(float& a, float& b) const {
    if (capped()) squash(a, b);
    a *= scale_log2;
    b *= scale_log2;
  }
  // the exponent (base 2) of a product q . k
  __device__ __forceinline__ float operator()(float qk) const { return (capped() ? squash(qk) : qk) * scale_log2; }
};

}  // namespace artb
