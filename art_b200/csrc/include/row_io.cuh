// Element access shared by the row kernels of the hybrid decoder: four elements at a time from bf16 or fp32 rows, block
// sums, and the three kinds of input such a kernel may finish (the bf16 output of a GEMM, an fp32 output, or the fp32
// workspace of a split-K GEMM, which has to be left zero).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace artb {

enum RowKind : int { ROW_BF16 = 0, ROW_F32 = 1, ROW_F32_TAKE = 2 };

__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 ld4(const __nv_bfloat16* p) {
  const uint2 r = *reinterpret_cast<const uint2*>(p);
  const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.x));
  const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&r.y));
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, float4 v) {
  uint2 r;
  *reinterpret_cast<__nv_bfloat162*>(&r.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&r.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = r;
}
__device__ __forceinline__ void st1(float* p, float v) { *p = v; }
__device__ __forceinline__ void st1(__nv_bfloat16* p, float v) { *p = __float2bfloat16(v); }

// four elements at element offset `off` of an input of kind `kind` (16-byte aligned for fp32, 8-byte for bf16)
__device__ __forceinline__ float4 take4(void* p, size_t off, int kind) {
  if (kind == ROW_BF16) return ld4(reinterpret_cast<const __nv_bfloat16*>(p) + off);
  float* f = reinterpret_cast<float*>(p) + off;
  const float4 v = ld4(f);
  if (kind == ROW_F32_TAKE) st4(f, make_float4(0.f, 0.f, 0.f, 0.f));
  return v;
}
__device__ __forceinline__ float take1(void* p, size_t off, int kind) {
  if (kind == ROW_BF16) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[off]);
  float* f = reinterpret_cast<float*>(p) + off;
  const float v = *f;
  if (kind == ROW_F32_TAKE) *f = 0.f;
  return v;
}

__device__ __forceinline__ float lane_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// Sum over the CTA (up to 1024 threads, whole warps); `red` holds 32 floats.  Every thread gets the sum.
__device__ __forceinline__ float cta_sum(float v, float* red) {
  v = lane_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  __syncthreads();                 // the previous use of `red` is over
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = lane < nw ? red[lane] : 0.f;
  return lane_sum(t);
}

__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

}  // namespace artb
