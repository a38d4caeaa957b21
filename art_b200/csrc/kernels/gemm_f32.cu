// fp32 GEMM  C_b[m, n] = A_b[m, :] . B_b[n, :]  (+ batch strides), fp32 multiply-adds in K order.
//
// With `tile_expert` the rows of A and C are sorted by expert in segments of 128-row tiles and expert e's matrix is the e-th
// batch member of B; tiles of expert -1 are left alone.
//
// The 32-bit mode of the hybrid decoder: a reference for the bf16 kernels on the device, not a fast path, so a plain
// 64 x 64 register-tiled kernel.  The reduction order of an element depends on nothing but K.
#include <cuda_runtime.h>
#include <stdint.h>

#include "host_utils.h"

namespace artb {

constexpr int GF_T = 64, GF_K = 16;

__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, int lda, long sa, const float* __restrict__ B, int ldb, long sb, float* __restrict__ C,
                int ldc, long sc, int M, int N, int K, const int* __restrict__ tile_expert) {
  __shared__ float As[GF_K][GF_T + 4], Bs[GF_K][GF_T + 4];
  if (tile_expert) {
    const int e = tile_expert[blockIdx.y * GF_T / 128];
    if (e < 0) return;
    B += e * sb;
  }
  A += blockIdx.z * sa;
  B += blockIdx.z * sb;
  C += blockIdx.z * sc;
  const int m0 = blockIdx.y * GF_T, n0 = blockIdx.x * GF_T, tid = threadIdx.x;
  const int tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += GF_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256, r = e >> 4, k = e & 15;
      As[k][r] = (m0 + r < M && k0 + k < K) ? A[static_cast<size_t>(m0 + r) * lda + k0 + k] : 0.f;
      Bs[k][r] = (n0 + r < N && k0 + k < K) ? B[static_cast<size_t>(n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GF_K; ++k) {
      float a[4], b[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = As[k][ty * 4 + i], b[i] = Bs[k][tx * 4 + i];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + ty * 4 + i, n = n0 + tx * 4 + j;
      if (m < M && n < N) C[static_cast<size_t>(m) * ldc + n] = acc[i][j];
    }
}

}  // namespace artb

using namespace artb;

ARTB_EXPORT int artb_gemm_f32_tn(const float* A, int lda, long sa, const float* B, int ldb, long sb, float* C, int ldc, long sc,
                                 int batch, int M, int N, int K, cudaStream_t stream) {
  if (batch <= 0 || batch > 65535 || M <= 0 || N <= 0 || K <= 0) return ERR_BAD_SHAPE;
  if ((M + GF_T - 1) / GF_T > 65535) return ERR_TOO_LARGE;
  gemm_f32_kernel<<<dim3((N + GF_T - 1) / GF_T, (M + GF_T - 1) / GF_T, batch), 256, 0, stream>>>(A, lda, sa, B, ldb, sb, C, ldc, sc,
                                                                                              M, N, K, nullptr);
  return static_cast<int>(cudaGetLastError());
}

// A [m_tiles * 128, K], B [experts * N, K], C [m_tiles * 128, N]; tile_expert int32 [m_tiles]
ARTB_EXPORT int artb_gemm_f32_grouped_tn(const float* A, int lda, const float* B, int ldb, float* C, int ldc, const int* tile_expert,
                                         int m_tiles, int N, int K, cudaStream_t stream) {
  if (m_tiles <= 0 || N <= 0 || K <= 0 || !tile_expert) return ERR_BAD_SHAPE;
  if (m_tiles * (128 / GF_T) > 65535) return ERR_TOO_LARGE;
  gemm_f32_kernel<<<dim3((N + GF_T - 1) / GF_T, m_tiles * (128 / GF_T), 1), 256, 0, stream>>>(
      A, lda, 0, B, ldb, static_cast<long>(N) * ldb, C, ldc, 0, m_tiles * 128, N, K, tile_expert);
  return static_cast<int>(cudaGetLastError());
}
