// Gated linear recurrent unit behind a short convolution (the recurrent branch of a Griffin-style mixer), per channel c of
// block b:
//
//   u_t = sum_j w_j x_{t - taps + 1 + j} + bias                      causal convolution, zeros before the sequence
//   r, i = sigmoid(gate products of u's block + bias)                one batched GEMM over the blocks
//   log a = -8 r softplus(lam),  S_t = a S_{t-1} + sqrt(1 - a^2) i u_t,  out = S_t gelu_tanh(y_t)
//
// Convolution inputs, gates, recurrence and state are fp32.  u reaches the gate product as a bf16 pair (high part, remainder)
// against the same matrix twice, so that the product loses nothing to the 16-bit operand; the 32-bit mode takes fp32.
//
//   short_conv_kernel    u of every new token; with one token per sequence it also advances the stored inputs
//   conv_state_kernel    portions: the last taps - 1 inputs of every sequence
//   rglru_scan_kernel    portions: a CTA owns 32 channels of a sequence; its warps take 16 tokens each, scan them from zero,
//                        exchange (decay product, end state) and add what came before
//   rglru_step_kernel    one token per sequence
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "row_io.cuh"

namespace artb {

struct ShortConv {
  void* x;                  // [M, ldx] of kind `kind` (not ROW_F32_TAKE unless every sequence brings one token)
  int ldx, kind;
  const float* x_bias;      // [n] added to every input
  const float* w;           // [n, taps]
  const float* bias;        // [n]
  int taps;
  float* state;             // [slots, taps - 1, n]: the last inputs, oldest first
  long num_slots;
  const int *row_seq, *cu_q, *ctx, *state_slot;
  void* u;                  // T [blocks][pitch][ldu]: bf16: high parts, remainders (bp columns each); fp32: bp columns
  int pitch, ldu;
  int n, bs, bp;            // channels, channels per block, padded
  int M, single;
  int* status;
};

template <typename T>
__device__ __forceinline__ void store_u(const ShortConv& a, int m, int c, float v) {
  const int b = c / a.bs, j = c - b * a.bs;
  T* u = reinterpret_cast<T*>(a.u) + (static_cast<size_t>(b) * a.pitch + m) * a.ldu + j;
  st1(u, v);
  if (sizeof(T) == 2) st1(u + a.bp, v - __bfloat162float(__float2bfloat16(v)));
}

template <typename T>
__global__ void __launch_bounds__(256) short_conv_kernel(const ShortConv a) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;
  if (c >= a.n) return;
  const int seq = a.row_seq[m], r0 = a.cu_q[seq], len = a.cu_q[seq + 1] - r0, t = m - r0, hist = a.taps - 1;
  int slot = a.state_slot[seq];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const bool old = slot >= 0 && a.ctx[seq] != len;        // the sequence has earlier tokens
  float* st = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * hist * a.n + c;
  const float* w = a.w + static_cast<size_t>(c) * a.taps;
  const float xb = a.x_bias[c];
  float acc = a.bias[c];
  const float now = take1(a.x, static_cast<size_t>(m) * a.ldx + c, a.kind) + xb;
  for (int j = 0; j < hist; ++j) {
    const int i = t - hist + j;                            // token of the portion; before it: the stored inputs
    float x = 0.f;
    if (i >= 0) x = take1(a.x, static_cast<size_t>(r0 + i) * a.ldx + c, a.kind) + xb;
    else if (old) x = st[static_cast<size_t>(hist + i) * a.n];
    acc = fmaf(w[j], x, acc);
    if (a.single && slot >= 0 && j > 0) st[static_cast<size_t>(j - 1) * a.n] = x;
  }
  store_u<T>(a, m, c, fmaf(w[hist], now, acc));
  if (a.single && slot >= 0 && hist > 0) st[static_cast<size_t>(hist - 1) * a.n] = now;
}

__global__ void __launch_bounds__(256) conv_state_kernel(const ShortConv a) {
  const int seq = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.n) return;
  const int r0 = a.cu_q[seq], len = a.cu_q[seq + 1] - r0, hist = a.taps - 1, slot = a.state_slot[seq];
  if (len <= 0 || slot < 0 || !index_ok(slot, a.num_slots, a.status)) return;
  const bool old = a.ctx[seq] != len;
  float* st = a.state + static_cast<size_t>(slot) * hist * a.n + c;
  for (int j = 0; j < hist; ++j) {                         // an old input moves towards the front: in place
    const int i = len - hist + j;
    st[static_cast<size_t>(j) * a.n] = i >= 0 ? take1(a.x, static_cast<size_t>(r0 + i) * a.ldx + c, a.kind) + a.x_bias[c]
                                              : (old ? st[static_cast<size_t>(hist + i) * a.n] : 0.f);
  }
}

struct Rglru {
  const void* u;            // as ShortConv::u
  int pitch, ldu;
  const float* z;           // [M, ldz]: gate products, per block bp columns of r, then bp of i
  int ldz;
  const float *r_bias, *i_bias, *decay;      // [n]; decay = 8 softplus(lam)
  void* y;                  // [M, ldy] of kind `kind`
  int ldy, kind;
  const float* y_bias;
  float* state;             // [slots, n]
  long num_slots;
  const int *cu_q, *ctx, *state_slot;
  void* o;                  // T [M, ldo]
  int ldo;
  float out_scale;
  int n, bs, bp, rows;
  int* status;
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }
__device__ __forceinline__ float gelu_tanh_f(float z) {
  constexpr float C = 0.7978845608028654f;      // sqrt(2 / pi)
  return 0.5f * z * (1.f + tanhf(C * (z + 0.044715f * z * z * z)));
}

// decay factor and input term of one token
template <typename T>
__device__ __forceinline__ void rglru_terms(const Rglru& a, int m, int b, int j, float rb, float ib, float dec, float& av, float& bv) {
  const T* up = reinterpret_cast<const T*>(a.u) + (static_cast<size_t>(b) * a.pitch + m) * a.ldu + j;
  const float u = sizeof(T) == 2 ? ld1(up) + ld1(up + a.bp) : ld1(up);
  const float* z = a.z + static_cast<size_t>(m) * a.ldz + b * 2 * a.bp + j;
  const float la = -sigmoid_f(z[0] + rb) * dec;
  av = expf(la);
  bv = sqrtf(-expm1f(2.f * la)) * sigmoid_f(z[a.bp] + ib) * u;
}

constexpr int RG_T = 16;      // tokens per warp and pass

template <typename T, int WARPS>
__global__ void __launch_bounds__(32 * WARPS) rglru_scan_kernel(const Rglru a) {
  __shared__ float sA[WARPS][32], sB[WARPS][32];
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = blockIdx.x * 32 + lane;
  const int r0 = a.cu_q[seq], len = a.cu_q[seq + 1] - r0;
  if (len <= 0) return;
  if (r0 < 0 || len > a.rows - r0) {      // not a portion of this batch
    if (threadIdx.x == 0) atomicMax(a.status, ST_BAD_ARGS);
    return;
  }
  int slot = a.state_slot[seq];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const bool live = c < a.n;
  const int cc = live ? c : 0, b = cc / a.bs, j = cc - b * a.bs;
  const float rb = a.r_bias[cc], ib = a.i_bias[cc], dec = a.decay[cc], yb = a.y_bias[cc];
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.n + cc;
  float carry = slot >= 0 && a.ctx[seq] != len ? *sp : 0.f;      // state before the pass, the same in every warp
  for (int t0 = 0; t0 < len; t0 += WARPS * RG_T) {
    const int w0 = t0 + warp * RG_T, nt = min(RG_T, len - w0);
    float A[RG_T], S[RG_T];
    float prod = 1.f, s = 0.f;
#pragma unroll
    for (int t = 0; t < RG_T; ++t) {
      A[t] = 1.f;
      S[t] = 0.f;
      if (t < nt) rglru_terms<T>(a, r0 + w0 + t, b, j, rb, ib, dec, A[t], S[t]);
    }
#pragma unroll
    for (int t = 0; t < RG_T; ++t) {       // tokens past the portion: factor 1, term 0
      prod *= A[t];
      s = fmaf(A[t], s, S[t]);
      A[t] = prod;
      S[t] = s;
    }
    sA[warp][lane] = prod;
    sB[warp][lane] = s;
    __syncthreads();
    float before = carry;
    for (int w = 0; w < WARPS; ++w) {
      if (w == warp) before = carry;
      carry = fmaf(sA[w][lane], carry, sB[w][lane]);
    }
    __syncthreads();
    if (live) {
#pragma unroll
      for (int t = 0; t < RG_T; ++t)
        if (t < nt) {
          const size_t m = r0 + w0 + t;
          const float y = gelu_tanh_f(take1(a.y, m * a.ldy + c, a.kind) + yb);
          st1(reinterpret_cast<T*>(a.o) + m * a.ldo + c, fmaf(A[t], before, S[t]) * y * a.out_scale);
        }
    }
  }
  if (live && warp == 0 && slot >= 0) *sp = carry;
}

template <typename T>
__global__ void __launch_bounds__(256) rglru_step_kernel(const Rglru a) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, c = blockIdx.y * 256 + threadIdx.x;      // row m holds sequence m's one token
  if (c >= a.n) return;
  int slot = a.state_slot[m];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const int b = c / a.bs, j = c - b * a.bs;
  float av, bv;
  rglru_terms<T>(a, m, b, j, a.r_bias[c], a.i_bias[c], a.decay[c], av, bv);
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.n + c;
  const float s = fmaf(av, slot >= 0 && a.ctx[m] != 1 ? *sp : 0.f, bv);
  if (slot >= 0) *sp = s;
  const float y = gelu_tanh_f(take1(a.y, static_cast<size_t>(m) * a.ldy + c, a.kind) + a.y_bias[c]);
  st1(reinterpret_cast<T*>(a.o) + static_cast<size_t>(m) * a.ldo + c, s * y * a.out_scale);
}

}  // namespace artb

using namespace artb;

// single: every sequence brings one token (row m = sequence m).  Otherwise n_seqs portions.  Padding columns of u are left alone.
ARTB_EXPORT int artb_short_conv(int f32, void* x, int ldx, int kind, const float* x_bias, const float* w, const float* bias, int taps,
                                float* state, long num_slots, const int* row_seq, const int* cu_q, const int* ctx,
                                const int* state_slot, int n_seqs, int single, void* u, int pitch, int ldu, int n, int bs, int bp,
                                int M, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (n <= 0 || bs <= 0 || n % bs || bp < bs || taps < 1 || ldx < n || pitch < M || ldu < (f32 ? bp : 2 * bp) || (n + 255) / 256 > 65535 ||
      (!single && kind == ROW_F32_TAKE) || n_seqs <= 0 || n_seqs > 65535)
    return ERR_BAD_SHAPE;
  const ShortConv a{x, ldx, kind, x_bias, w, bias, taps, state, num_slots, row_seq, cu_q, ctx, state_slot, u, pitch, ldu, n, bs, bp, M,
                    single, status};
  const dim3 grid(M, (n + 255) / 256);
  cudaError_t e = f32 ? launch_kernel(short_conv_kernel<float>, grid, dim3(256), 0, st, a)
                      : launch_kernel(short_conv_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a);
  if (e != cudaSuccess || single || taps == 1) return static_cast<int>(e);
  conv_state_kernel<<<dim3((n + 255) / 256, n_seqs), 256, 0, st>>>(a);
  return static_cast<int>(cudaGetLastError());
}

ARTB_EXPORT int artb_rglru(int f32, int single, const void* u, int pitch, int ldu, const float* z, int ldz, const float* r_bias,
                           const float* i_bias, const float* decay, void* y, int ldy, int kind, const float* y_bias, float* state,
                           long num_slots, const int* cu_q, const int* ctx, const int* state_slot, int n_seqs, void* o, int ldo,
                           float out_scale, int n, int bs, int bp, int M, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (n <= 0 || bs <= 0 || n % bs || bp < bs || pitch < M || ldz < n / bs * 2 * bp || ldo < n || ldy < n || n_seqs <= 0 || n_seqs > 65535 ||
      (single && n_seqs != M))
    return ERR_BAD_SHAPE;
  const Rglru a{u, pitch, ldu, z, ldz, r_bias, i_bias, decay, y, ldy, kind, y_bias, state, num_slots, cu_q, ctx, state_slot, o, ldo,
                out_scale, n, bs, bp, M, status};
  if (single) {
    const dim3 grid(M, (n + 255) / 256);
    return static_cast<int>(f32 ? launch_kernel(rglru_step_kernel<float>, grid, dim3(256), 0, st, a)
                                : launch_kernel(rglru_step_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a));
  }
  const dim3 grid((n + 31) / 32, n_seqs);
  return static_cast<int>(f32 ? launch_kernel(rglru_scan_kernel<float, 16>, grid, dim3(512), 0, st, a)
                              : launch_kernel(rglru_scan_kernel<__nv_bfloat16, 16>, grid, dim3(512), 0, st, a));
}
