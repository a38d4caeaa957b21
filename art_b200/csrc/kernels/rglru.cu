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
//   conv_rows_kernel     the same for portions: a thread slides over 16 rows with four channels
//   conv_state_kernel    portions: the last taps - 1 inputs of every sequence
//   rglru_scan_kernel    portions: a CTA owns 64 channels of a sequence; its warps take 8 tokens each, scan them from zero,
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

__device__ __forceinline__ float bf16_part(float v) { return __bfloat162float(__float2bfloat16(v)); }

template <typename T>
__device__ __forceinline__ void store_u(const ShortConv& a, int m, int c, float v) {
  const int b = c / a.bs, j = c - b * a.bs;
  T* u = reinterpret_cast<T*>(a.u) + (static_cast<size_t>(b) * a.pitch + m) * a.ldu + j;
  st1(u, v);
  if (sizeof(T) == 2) st1(u + a.bp, v - bf16_part(v));
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

constexpr int CONV_ROWS = 16;

// Rows of portions, four channels a thread (n, bs, bp and all strides multiples of 4), inputs of the operand type.  The last
// TAPS - 1 inputs slide through registers; at the first row of the run and of every sequence they are fetched anew.
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_rows_kernel(const ShortConv a) {
  constexpr int HIST = TAPS - 1;
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 4, m0 = blockIdx.y * CONV_ROWS, m1 = min(a.M, m0 + CONV_ROWS);
  if (c >= a.n) return;
  float4 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)
    w[j] = make_float4(a.w[c * TAPS + j], a.w[(c + 1) * TAPS + j], a.w[(c + 2) * TAPS + j], a.w[(c + 3) * TAPS + j]);
  const float4 xb = ld4(a.x_bias + c), cb = ld4(a.bias + c);
  const int b = c / a.bs, j0 = c - b * a.bs;
  T* u = reinterpret_cast<T*>(a.u) + static_cast<size_t>(b) * a.pitch * a.ldu + j0;
  const T* xp = reinterpret_cast<const T*>(a.x) + c;
  auto input = [&](int m) {
    const float4 x = ld4(xp + static_cast<size_t>(m) * a.ldx);
    return make_float4(x.x + xb.x, x.y + xb.y, x.z + xb.z, x.w + xb.w);
  };
  float4 h[HIST > 0 ? HIST : 1];
  int seq_end = m0;                            // the first row fetches its history
  float4 x[4], next[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) x[i] = input(min(m0 + i, m1 - 1));
  for (int m4 = m0; m4 < m1; m4 += 4) {
#pragma unroll
    for (int i = 0; i < 4; ++i) next[i] = input(min(m4 + 4 + i, m1 - 1));
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int m = m4 + i;
      if (m >= m1) break;
      if (m == seq_end) {
        const int seq = a.row_seq[m], r0 = a.cu_q[seq];
        seq_end = a.cu_q[seq + 1];
        int slot = a.state_slot[seq];
        if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
        const bool old = slot >= 0 && a.ctx[seq] != seq_end - r0;
#pragma unroll
        for (int j = 0; j < HIST; ++j) {
          const int p = m - HIST + j;
          h[j] = make_float4(0.f, 0.f, 0.f, 0.f);
          if (p >= r0) h[j] = input(p);
          else if (old) h[j] = ld4(a.state + (static_cast<size_t>(slot) * HIST + HIST + p - r0) * a.n + c);
        }
      }
      float4 y = cb;
#pragma unroll
      for (int j = 0; j < TAPS; ++j) {
        const float4 v = j < HIST ? h[j < HIST ? j : 0] : x[i];
        y = make_float4(fmaf(w[j].x, v.x, y.x), fmaf(w[j].y, v.y, y.y), fmaf(w[j].z, v.z, y.z), fmaf(w[j].w, v.w, y.w));
      }
      T* up = u + static_cast<size_t>(m) * a.ldu;
      st4(up, y);
      if (sizeof(T) == 2)
        st4(up + a.bp, make_float4(y.x - bf16_part(y.x), y.y - bf16_part(y.y), y.z - bf16_part(y.z), y.w - bf16_part(y.w)));
#pragma unroll
      for (int j = 0; j + 1 < HIST; ++j) h[j] = h[j + 1];
      if (HIST > 0) h[HIST > 0 ? HIST - 1 : 0] = x[i];
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) x[i] = next[i];
  }
}

template <typename T>
static cudaError_t launch_conv_rows(const ShortConv& a, cudaStream_t st) {
  const dim3 grid((a.n / 4 + 127) / 128, (a.M + CONV_ROWS - 1) / CONV_ROWS);
#define ARTB_CR(N_) \
  case N_: return launch_kernel(conv_rows_kernel<T, N_>, grid, dim3(128), 0, st, a)
  switch (a.taps) {
    ARTB_CR(1);
    ARTB_CR(2);
    ARTB_CR(3);
    ARTB_CR(4);
    ARTB_CR(5);
    ARTB_CR(6);
    ARTB_CR(7);
    default: return launch_kernel(conv_rows_kernel<T, 8>, grid, dim3(128), 0, st, a);
  }
#undef ARTB_CR
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

// FAST (bf16 operands): hardware exponential, division and square root, a few units in the last place of fp32; the 32-bit mode
// takes the library functions
template <bool FAST>
__device__ __forceinline__ float sigmoid_f(float z) {
  return FAST ? __fdividef(1.f, 1.f + __expf(-z)) : 1.f / (1.f + expf(-z));
}
template <bool FAST>
__device__ __forceinline__ float gelu_tanh_f(float z) {      // 0.5 (1 + tanh x) = sigmoid(2 x)
  constexpr float C = 0.7978845608028654f;                   // sqrt(2 / pi)
  return z * sigmoid_f<FAST>(2.f * C * (z + 0.044715f * z * z * z));
}
// sqrt(1 - exp(2 la)), la <= 0
template <bool FAST>
__device__ __forceinline__ float input_gain(float la) {
  const float x = -2.f * la;
  if (!FAST) return sqrtf(-expm1f(-x));
  // near zero the difference cancels: Taylor polynomial of 1 - exp(-x)
  const float p = x * fmaf(x, fmaf(x, fmaf(x, fmaf(x, 1.f / 120.f, -1.f / 24.f), 1.f / 6.f), -0.5f), 1.f);
  const float d = x < 0.0625f ? p : 1.f - __expf(-x);
  return d > 0.f ? d * rsqrtf(d) : 0.f;
}
template <bool FAST>
__device__ __forceinline__ void rglru_terms(float u, float zr, float zi, float dec, float& av, float& bv) {
  const float la = -sigmoid_f<FAST>(zr) * dec;
  av = FAST ? __expf(la) : expf(la);
  bv = input_gain<FAST>(la) * sigmoid_f<FAST>(zi) * u;
}

// decay factor and input term of one token and channel (b, j)
template <typename T>
__device__ __forceinline__ void rglru_token(const Rglru& a, int m, int b, int j, float rb, float ib, float dec, float& av, float& bv) {
  const T* up = reinterpret_cast<const T*>(a.u) + (static_cast<size_t>(b) * a.pitch + m) * a.ldu + j;
  const float u = sizeof(T) == 2 ? ld1(up) + ld1(up + a.bp) : ld1(up);
  const float* z = a.z + static_cast<size_t>(m) * a.ldz + b * 2 * a.bp + j;
  rglru_terms<sizeof(T) == 2>(u, z[0] + rb, z[a.bp] + ib, dec, av, bv);
}

constexpr int RG_T = 8;       // tokens per warp and pass

// V neighbouring channels (1 or 2)
template <int V>
__device__ __forceinline__ void ldv(const float* p, float (&f)[V]) {
  if (V == 2) {
    const float2 v = *reinterpret_cast<const float2*>(p);
    f[0] = v.x, f[V - 1] = v.y;
  } else {
    f[0] = *p;
  }
}
template <int V>
__device__ __forceinline__ void ldv(const __nv_bfloat16* p, float (&f)[V]) {
  if (V == 2) {
    const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
    f[0] = v.x, f[V - 1] = v.y;
  } else {
    f[0] = __bfloat162float(*p);
  }
}
template <int V>
__device__ __forceinline__ void stv(float* p, const float (&f)[V]) {
  if (V == 2) *reinterpret_cast<float2*>(p) = make_float2(f[0], f[V - 1]);
  else *p = f[0];
}
template <int V>
__device__ __forceinline__ void stv(__nv_bfloat16* p, const float (&f)[V]) {
  if (V == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(f[0], f[V - 1]);
  else *p = __float2bfloat16(f[0]);
}

// V channels per lane (2: n, bs, bp and all strides even, both channels of a lane then belong to one block); y of the operand
// type.  Rows past the portion are read as its last row (so that all loads of a pass go out together) and not used.
template <typename T, int WARPS, int V>
__global__ void __launch_bounds__(32 * WARPS, 2) rglru_scan_kernel(const Rglru a) {
  constexpr bool FAST = sizeof(T) == 2;
  __shared__ float sA[WARPS][32 * V], sB[WARPS][32 * V];
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, c = (blockIdx.x * 32 + lane) * V;
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
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.n + cc;
  const T* __restrict__ up = reinterpret_cast<const T*>(a.u) + static_cast<size_t>(b) * a.pitch * a.ldu + j;
  const T* __restrict__ yp = reinterpret_cast<const T*>(a.y) + cc;
  const float* __restrict__ zp = a.z + b * 2 * a.bp + j;
  T* __restrict__ op = reinterpret_cast<T*>(a.o) + cc;
  float rb[V], ib[V], dec[V], yb[V], carry[V];      // carry: state before the pass, the same in every warp
#pragma unroll
  for (int e = 0; e < V; ++e) {
    rb[e] = a.r_bias[cc + e];
    ib[e] = a.i_bias[cc + e];
    dec[e] = a.decay[cc + e];
    yb[e] = a.y_bias[cc + e];
    carry[e] = slot >= 0 && a.ctx[seq] != len ? sp[e] : 0.f;
  }
  for (int t0 = 0; t0 < len; t0 += WARPS * RG_T) {
    const int w0 = t0 + warp * RG_T, nt = min(RG_T, len - w0);
    float A[RG_T][V], S[RG_T][V], y[RG_T][V];
    {
      float u[RG_T][V], lo[RG_T][V], zr[RG_T][V], zi[RG_T][V];
#pragma unroll
      for (int t = 0; t < RG_T; ++t) {
        const size_t m = r0 + min(w0 + t, len - 1);
        ldv<V>(up + m * a.ldu, u[t]);
        if (FAST) ldv<V>(up + m * a.ldu + a.bp, lo[t]);
        ldv<V>(zp + m * a.ldz, zr[t]);
        ldv<V>(zp + m * a.ldz + a.bp, zi[t]);
        ldv<V>(yp + m * a.ldy, y[t]);
      }
#pragma unroll
      for (int t = 0; t < RG_T; ++t)
#pragma unroll
        for (int e = 0; e < V; ++e)
          rglru_terms<FAST>(FAST ? u[t][e] + lo[t][e] : u[t][e], zr[t][e] + rb[e], zi[t][e] + ib[e], dec[e], A[t][e], S[t][e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) {
      float prod = 1.f, s = 0.f;
#pragma unroll
      for (int t = 0; t < RG_T; ++t) {
        if (t < nt) {                        // tokens past the portion: factor 1, term 0
          prod *= A[t][e];
          s = fmaf(A[t][e], s, S[t][e]);
        }
        A[t][e] = prod;
        S[t][e] = s;
      }
      sA[warp][lane * V + e] = prod;
      sB[warp][lane * V + e] = s;
    }
    __syncthreads();
    float before[V];
#pragma unroll
    for (int e = 0; e < V; ++e) {
      before[e] = carry[e];
#pragma unroll
      for (int w = 0; w < WARPS; ++w) {
        if (w == warp) before[e] = carry[e];
        carry[e] = fmaf(sA[w][lane * V + e], carry[e], sB[w][lane * V + e]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int t = 0; t < RG_T; ++t) {
      float o[V];
#pragma unroll
      for (int e = 0; e < V; ++e) o[e] = fmaf(A[t][e], before[e], S[t][e]) * gelu_tanh_f<FAST>(y[t][e] + yb[e]) * a.out_scale;
      if (live && t < nt) stv<V>(op + static_cast<size_t>(r0 + w0 + t) * a.ldo, o);
    }
  }
  if (live && warp == 0 && slot >= 0) {
#pragma unroll
    for (int e = 0; e < V; ++e) sp[e] = carry[e];
  }
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
  rglru_token<T>(a, m, b, j, a.r_bias[c], a.i_bias[c], a.decay[c], av, bv);
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.n + c;
  const float s = fmaf(av, slot >= 0 && a.ctx[m] != 1 ? *sp : 0.f, bv);
  if (slot >= 0) *sp = s;
  const float y = gelu_tanh_f<sizeof(T) == 2>(take1(a.y, static_cast<size_t>(m) * a.ldy + c, a.kind) + a.y_bias[c]);
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
  const bool rows = !single && taps <= 8 && kind == (f32 ? ROW_F32 : ROW_BF16) && !((n | bs | bp | ldx | ldu) & 3) &&
                    !(reinterpret_cast<uintptr_t>(x) & 15) && (M + CONV_ROWS - 1) / CONV_ROWS <= 65535;
  cudaError_t e = rows  ? (f32 ? launch_conv_rows<float>(a, st) : launch_conv_rows<__nv_bfloat16>(a, st))
                  : f32 ? launch_kernel(short_conv_kernel<float>, grid, dim3(256), 0, st, a)
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
      (single ? n_seqs != M : kind != (f32 ? ROW_F32 : ROW_BF16)))
    return ERR_BAD_SHAPE;
  const Rglru a{u, pitch, ldu, z, ldz, r_bias, i_bias, decay, y, ldy, kind, y_bias, state, num_slots, cu_q, ctx, state_slot, o, ldo,
                out_scale, n, bs, bp, M, status};
  if (single) {
    const dim3 grid(M, (n + 255) / 256);
    return static_cast<int>(f32 ? launch_kernel(rglru_step_kernel<float>, grid, dim3(256), 0, st, a)
                                : launch_kernel(rglru_step_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, a));
  }
  const bool two = !((n | bs | bp | ldy | ldo | ldu | ldz) & 1) &&
                   !((reinterpret_cast<uintptr_t>(y) | reinterpret_cast<uintptr_t>(o)) & 7);
  const dim3 grid((n + (two ? 63 : 31)) / (two ? 64 : 32), n_seqs);
  if (two)
    return static_cast<int>(f32 ? launch_kernel(rglru_scan_kernel<float, 8, 2>, grid, dim3(256), 0, st, a)
                                : launch_kernel(rglru_scan_kernel<__nv_bfloat16, 8, 2>, grid, dim3(256), 0, st, a));
  return static_cast<int>(f32 ? launch_kernel(rglru_scan_kernel<float, 8, 1>, grid, dim3(256), 0, st, a)
                              : launch_kernel(rglru_scan_kernel<__nv_bfloat16, 8, 1>, grid, dim3(256), 0, st, a));
}
