// What an attention kernel makes of a score besides an ordinary softmax:
//
//   distance bias    a number per head and distance (query position - key position) added to the scaled score, constant from
//                    the table's last distance on; the table also carries whatever else is constant for a head
//   sigmoid weights  a key weighs sigmoid(score): nothing is divided by the weights' sum, so that tiles and splits simply add
//   sink             a term exp(sink_h) of the softmax's denominator without a key: the running maximum starts at it with a
//                    sum of one
//   column gate      the result is multiplied, column by column, by the sigmoid of a projection of the layer's input
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "ptx_sm100.cuh"
#include "row_io.cuh"

namespace artb {

constexpr float KW_LOG2E = 1.4426950408889634f;

// fp32 [heads][PAD + n + PAD], in base-2 units.  Entry PAD + t belongs to distance t; the padding in front (keys behind the
// query, masked elsewhere) and behind (a copy of the last entry) lets tile kernels index a whole tile without clamping.
struct DistanceBias {
  static constexpr int PAD = 256;
  const float* tab;
  int n;
  __device__ __forceinline__ const float* head(int h) const { return tab + static_cast<size_t>(h) * (n + 2 * PAD) + PAD; }
  __device__ __forceinline__ float at(const float* row, int dist) const { return __ldg(row + min(dist, n - 1)); }
  __device__ __forceinline__ float last(const float* row) const { return __ldg(row + n - 1); }
  // every key from position `k_last` down lies beyond the table for queries from position `q` on
  __device__ __forceinline__ bool beyond(int q, int k_last) const { return q - k_last >= n - 1; }
};

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// sigmoid(x ln 2), the weight of a key whose score is x in base-2 units, of two keys with one reciprocal (1 / a = b / (a b));
// weights below 2^-60 count as that, so that the product stays finite
__device__ __forceinline__ void sigmoid_pair(float& x, float& y) {
  const float a = 1.f + exp2_approx(fminf(-x, 60.f)), b = 1.f + exp2_approx(fminf(-y, 60.f)), r = rcp_approx(a * b);
  x = r * b;
  y = r * a;
}

// Gate logits of type T, row m and head h at g + m * ld + h * pitch; null: no gate
template <typename T>
struct ColumnGate {
  const T* g;
  int ld, pitch, vdim;
  bool vec;      // eight columns may be loaded at once

  __host__ __device__ static ColumnGate of(const void* p, int ld, int pitch, int vdim) {
    const T* g = reinterpret_cast<const T*>(p);
    return {g, ld, pitch, vdim, p && !((ld | pitch) & 7) && !(reinterpret_cast<uintptr_t>(p) & 15)};
  }
  __device__ __forceinline__ const T* row(int m, int h) const { return g + static_cast<size_t>(m) * ld + static_cast<size_t>(h) * pitch; }
  __device__ __forceinline__ void prefetch(int m, int h, int d) const { asm volatile("prefetch.global.L2 [%0];" ::"l"(row(m, h) + d)); }
  // factor of column d (1 for padding columns)
  __device__ __forceinline__ float operator()(int m, int h, int d) const { return g && d < vdim ? logistic_f(ld1(row(m, h) + d)) : 1.f; }
  // logits of columns d .. d + 7 (bf16), and what they make of those columns
  __device__ __forceinline__ uint4 load8(int m, int h, int d) const {
    if (vec && d + 8 <= vdim) return *reinterpret_cast<const uint4*>(row(m, h) + d);
    __align__(16) T z[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) z[i] = d + i < vdim ? row(m, h)[d + i] : T(0.f);
    return *reinterpret_cast<const uint4*>(z);
  }
  static __device__ __forceinline__ void apply8(const uint4& q, float (&x)[8]) {
    const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&q);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      float2 z = __bfloat1622float2(b[i]);
      z.x *= KW_LOG2E;
      z.y *= KW_LOG2E;
      sigmoid_pair(z.x, z.y);
      x[2 * i] *= z.x;
      x[2 * i + 1] *= z.y;
    }
  }
};

}  // namespace artb
