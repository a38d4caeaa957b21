// Element access shared by the row kernels of the hybrid decoder: four elements at a time from bf16 or fp32 rows, block
// sums, and the three kinds of input such a kernel may finish (the bf16 output of a GEMM, an fp32 output, or the fp32
// workspace of a split-K GEMM, which has to be left zero).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace artb {

enum RowAct : int { ACT_SILU = 0, ACT_RELU = 1, ACT_RELU2 = 2 };      // ACT_RELU2: the square of relu
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
__device__ __forceinline__ float ld1(const float* p) { return *p; }
__device__ __forceinline__ float ld1(const __nv_bfloat16* p) { return __bfloat162float(*p); }
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
// The two halves of take4 / take1: where several loads are in flight, the workspace is cleared once they have arrived (a store
// behind a load of the same line that is still under way holds up the loads behind it).
__device__ __forceinline__ int peek_kind(int kind) { return kind == ROW_BF16 ? ROW_BF16 : ROW_F32; }
__device__ __forceinline__ void clear4(void* p, size_t off, int kind) {
  if (kind == ROW_F32_TAKE) st4(reinterpret_cast<float*>(p) + off, make_float4(0.f, 0.f, 0.f, 0.f));
}
__device__ __forceinline__ void clear1(void* p, size_t off, int kind) {
  if (kind == ROW_F32_TAKE) reinterpret_cast<float*>(p)[off] = 0.f;
}
__device__ __forceinline__ void clear8(void* p, size_t off, int kind) {
  clear4(p, off, kind);
  clear4(p, off + 4, kind);
}
// eight elements (16-byte aligned)
__device__ __forceinline__ void take8(void* p, size_t off, int kind, float (&f)[8]) {
  if (kind == ROW_BF16) {
    const uint4 r = *reinterpret_cast<const uint4*>(reinterpret_cast<const __nv_bfloat16*>(p) + off);
    const __nv_bfloat162* b = reinterpret_cast<const __nv_bfloat162*>(&r);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 v = __bfloat1622float2(b[i]);
      f[2 * i] = v.x;
      f[2 * i + 1] = v.y;
    }
    return;
  }
  const float4 a = take4(p, off, kind), c = take4(p, off + 4, kind);
  f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w, f[4] = c.x, f[5] = c.y, f[6] = c.z, f[7] = c.w;
}
__device__ __forceinline__ void put8(float* p, const float (&f)[8]) {
  st4(p, make_float4(f[0], f[1], f[2], f[3]));
  st4(p + 4, make_float4(f[4], f[5], f[6], f[7]));
}
__device__ __forceinline__ void put8(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 r;
  __nv_bfloat162* b = reinterpret_cast<__nv_bfloat162*>(&r);
#pragma unroll
  for (int i = 0; i < 4; ++i) b[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
  *reinterpret_cast<uint4*>(p) = r;
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

// sine and cosine of pos * freq; the angle is reduced in double so that far positions lose nothing
__device__ __forceinline__ float2 position_pair(int pos, double freq) {
  constexpr double TWO_PI = 6.283185307179586476925;
  const double ang = pos * freq;
  float2 r;
  sincosf(static_cast<float>(ang - rint(ang * (1.0 / TWO_PI)) * TWO_PI), &r.x, &r.y);
  return r;
}

__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float logistic_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return z / (1.f + expf(-z)); }

}  // namespace artb
