// Row kernels of the hybrid decoder: everything between its matrix products that works on one token at a time.
//
//   residual_step      the fp32 residual stream across a sublayer boundary, one pass:
//                        x = x + mult * RMSNorm(y) w_post          (or x = RMSNorm(table[token]) w_post at the input)
//                        without w_post: x = x + mult * y          (or x = mult * table[token] + position vector)
//                        y may have a factor per row, a bias and the weighted rows of a token's experts (or of the
//                        sublayer's input, for experts that are the identity) added to it
//                        and the sum a gate per column, sigmoid(logits + bias)
//                        depth average: x <- sum_j weight[j] X_j over the results X_j of all layers so far
//                        h = RMSNorm(x) w_next, or x               (operand of the next matrix product)
//   stream_step        the same with hyper-connections: the residual stream has several copies x_s, and a boundary mixes them
//                        x_t <- sum_s mix[s][t] x_s + out[t] * y   (all at once from the old ones)
//                        h = RMSNorm(sum_t in[t] x_t) w_next
//   norm_shift_mix     h = RMSNorm(x) w; the inputs h + (h' - h) mu_s of a token-shifted mixer, h' being the h of the
//                      token before (from the sequence's state at the start of a portion)
//   poly_norm          a N(z) + b N(z^2) + c N(z^3) + e, N(v) = v / rms(v)
//   gated_act          act(gate) * up of a gate|up projection, gate and up columns interleaved in blocks of 16
//   plain_act          act(z)
//   split_tanh         tanh(z) as a bf16 pair (high part, remainder), so that a product with it loses no 16-bit digits
//   head_norm          per-head RMSNorm of a mixer's fp32 output, with an optional silu or sigmoid gate
//   row_norm           the same over a whole row of heads
//   gather_norm        RMSNorm of chosen rows (inputs of the LM head)
//
// The residual stream, its history, norms and states are fp32; GEMM operands are written as bf16 (or fp32 in the 32-bit
// mode).  Widths are padded to a multiple of 8 with zero weights, so padding columns stay zero; means divide by the real
// width.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "row_io.cuh"

namespace artb {

enum GateAct : int { GATE_SILU = 0, GATE_SIGMOID = 1 };

struct ResidualArgs {
  const int64_t* tokens;   // embedding lookup instead of y when set
  const void* table;       // T [vocab, ldt]
  int ldt;
  long vocab;
  void* y;                 // sublayer output, kind y_kind
  int ldy, y_kind;
  const float* x_in;
  float* x_out;            // may alias x_in
  int ldx;
  const float* w_post;     // fp32 [dp], or null: y is not normalised
  float mult;
  const float* y_gate;     // fp32 [rows] factor of y (before the bias), or null
  const float* y_bias;     // fp32 [dp] added to y, or null
  const void* ex;          // T [.., ldex] rows of experts: y += sum_s ex_w[row, s] * ex[ex_pos[row, s]], or null
  int ldex, ex_k;
  const int* ex_pos;       // < 0: the identity, row `row` of idn
  const float* ex_w;
  long ex_rows;
  void* idn;               // [rows, ldidn] of idn_kind, or null; may alias x_in, x_out or h
  int ldidn, idn_kind;
  const double* freq;      // sinusoidal position vector added at the input: angle of column pair i is pos * freq[i]
  const int* pos;
  float* hist;             // fp32 [.., rows, ldx] results of the layers, or null
  long hist_stride;
  int hist_n;              // earlier results 0 .. hist_n - 1 are in hist; this one is stored as hist_n
  const float* avg;        // fp32 [hist_n + 1], or null: store without averaging
  const float* w_next;     // fp32 [dp], or null: h is x itself
  void* h;                 // T [rows, ldh], or null
  int ldh;
  int d, dp;
  float eps;
  int* status;
  void* rg;                // logits [rows, ldrg] of rg_kind of a gate on the result's columns, or null
  int ldrg, rg_kind;
  const float* rg_b;       // fp32 [dp] added to them
  // stream_step_kernel alone
  const float* coef;       // mix [n_in][n_out] | out [n_out] | in of the next sublayer [n_out]
  int n_in, n_out;         // copies of the stream before (x_in: rows of n_in * dp columns) and behind the step (x_out)
  int ldxi;
};

// The sublayer's result (or the embedding row) of row `row`, four columns per thread and vector; `y` of columns past the row is
// zero.  Workspaces are cleared by clear_inputs at the end of a kernel.
template <typename T, int MAXV>
__device__ __forceinline__ void sublayer_result(const ResidualArgs& a, int row, int nv, float4 (&y)[MAXV]) {
  long tok = 0;
  if (a.tokens) {
    tok = a.tokens[row];
    if (!index_ok(tok, a.vocab, a.status)) tok = 0;
  }
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    y[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (v < nv) {
      if (a.tokens) y[i] = ld4(reinterpret_cast<const T*>(a.table) + static_cast<size_t>(tok) * a.ldt + v * 4);
      else if (a.y) y[i] = take4(a.y, static_cast<size_t>(row) * a.ldy + v * 4, peek_kind(a.y_kind));
      if (a.y_gate) {
        const float g = __ldg(a.y_gate + row);
        y[i] = make_float4(y[i].x * g, y[i].y * g, y[i].z * g, y[i].w * g);
      }
      if (a.y_bias) {
        const float4 b = ld4(a.y_bias + v * 4);
        y[i] = make_float4(y[i].x + b.x, y[i].y + b.y, y[i].z + b.z, y[i].w + b.w);
      }
    }
  }
  if (a.ex) {
    auto add = [&](float ew, auto&& row4) {
#pragma unroll
      for (int i = 0; i < MAXV; ++i) {
        const int v = threadIdx.x + i * blockDim.x;
        if (v < nv) {
          const float4 e = row4(v * 4);
          y[i] = make_float4(fmaf(ew, e.x, y[i].x), fmaf(ew, e.y, y[i].y), fmaf(ew, e.z, y[i].z), fmaf(ew, e.w, y[i].w));
        }
      }
    };
    for (int s = 0; s < a.ex_k; ++s) {
      const int er = a.ex_pos[static_cast<size_t>(row) * a.ex_k + s];
      const float ew = a.ex_w[static_cast<size_t>(row) * a.ex_k + s];
      if (er < 0 && a.idn) {                                // uniform for the CTA
        add(ew, [&](int c) { return take4(a.idn, static_cast<size_t>(row) * a.ldidn + c, a.idn_kind); });
      } else if (index_ok(er, a.ex_rows, a.status)) {
        const T* ep = reinterpret_cast<const T*>(a.ex) + static_cast<size_t>(er) * a.ldex;
        add(ew, [&](int c) { return ld4(ep + c); });
      }
    }
  }
  if (a.rg) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nv) {
        const float4 z = take4(a.rg, static_cast<size_t>(row) * a.ldrg + v * 4, peek_kind(a.rg_kind)), b = ld4(a.rg_b + v * 4);
        y[i] = make_float4(y[i].x * logistic_f(z.x + b.x), y[i].y * logistic_f(z.y + b.y), y[i].z * logistic_f(z.z + b.z), y[i].w * logistic_f(z.w + b.w));
      }
    }
  }
}

template <int MAXV>
__device__ __forceinline__ void clear_inputs(const ResidualArgs& a, int row, int nv) {
  const bool y = a.y && a.y_kind == ROW_F32_TAKE, rg = a.rg && a.rg_kind == ROW_F32_TAKE;
  if (!y && !rg) return;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nv && y) clear4(a.y, static_cast<size_t>(row) * a.ldy + v * 4, ROW_F32_TAKE);
    if (v < nv && rg) clear4(a.rg, static_cast<size_t>(row) * a.ldrg + v * 4, ROW_F32_TAKE);
  }
}

// h = RMSNorm(x) w_next, or x
template <typename T, int MAXV>
__device__ __forceinline__ void write_operand(const ResidualArgs& a, int row, int nv, const float4 (&x)[MAXV], float ss, float* red) {
  T* h = reinterpret_cast<T*>(a.h) + static_cast<size_t>(row) * a.ldh;
  if (!a.w_next) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int v = threadIdx.x + i * blockDim.x;
      if (v < nv) st4(h + v * 4, x[i]);
    }
    return;
  }
  ss = cta_sum(ss, red);
  const float r = 1.f / sqrtf(ss / a.d + a.eps);
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nv) {
      const float4 w = ld4(a.w_next + v * 4);
      st4(h + v * 4, make_float4(x[i].x * r * w.x, x[i].y * r * w.y, x[i].z * r * w.z, x[i].w * r * w.w));
    }
  }
}

template <typename T, int MAXV>
__global__ void __launch_bounds__(256) residual_step_kernel(const ResidualArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, nv = a.dp >> 2;
  float4 y[MAXV];
  float ss = 0.f;
  sublayer_result<T, MAXV>(a, row, nv, y);
  float r = 1.f;
  if (a.w_post) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) ss += sq4(y[i]);        // columns past the row are zero
    ss = cta_sum(ss, red);
    r = 1.f / sqrtf(ss / a.d + a.eps);
  }
  const size_t xo = static_cast<size_t>(row) * a.ldx;
  ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int v = threadIdx.x + i * blockDim.x;
    if (v < nv) {
      float4 x = y[i];
      if (a.w_post) {
        const float4 w = ld4(a.w_post + v * 4);
        x = make_float4(x.x * r * w.x, x.y * r * w.y, x.z * r * w.z, x.w * r * w.w);
      } else if (a.tokens) {
        x = make_float4(a.mult * x.x, a.mult * x.y, a.mult * x.z, a.mult * x.w);
      }
      if (a.tokens && a.freq) {
        const float2 p0 = position_pair(a.pos[row], a.freq[v * 2]), p1 = position_pair(a.pos[row], a.freq[v * 2 + 1]);
        const int c = v * 4;
        if (c < a.d) x.x += p0.x;
        if (c + 1 < a.d) x.y += p0.y;
        if (c + 2 < a.d) x.z += p1.x;
        if (c + 3 < a.d) x.w += p1.y;
      }
      if (!a.tokens) {
        const float4 x0 = ld4(a.x_in + xo + v * 4);
        x = make_float4(fmaf(a.mult, x.x, x0.x), fmaf(a.mult, x.y, x0.y), fmaf(a.mult, x.z, x0.z), fmaf(a.mult, x.w, x0.w));
      }
      if (a.hist) {
        float* hp = a.hist + xo + v * 4;
        st4(hp + a.hist_n * a.hist_stride, x);
        if (a.avg) {
          const float wl = __ldg(a.avg + a.hist_n);
          float4 s = make_float4(wl * x.x, wl * x.y, wl * x.z, wl * x.w);
#pragma unroll 4
          for (int j = 0; j < a.hist_n; ++j) {
            const float wj = __ldg(a.avg + j);
            const float4 q = ld4(hp + j * a.hist_stride);
            s.x = fmaf(wj, q.x, s.x);
            s.y = fmaf(wj, q.y, s.y);
            s.z = fmaf(wj, q.z, s.z);
            s.w = fmaf(wj, q.w, s.w);
          }
          x = s;
        }
      }
      st4(a.x_out + xo + v * 4, x);
      y[i] = x;
      ss += sq4(x);
    }
  }
  if (a.h) write_operand<T, MAXV>(a, row, nv, y, ss, red);      // uniform for the grid
  clear_inputs<MAXV>(a, row, nv);
}

// Hyper-connections.  NS: the most copies on either side; the copies of a vector are read together, several vectors in flight.
template <typename T, int MAXV, int NS>
__global__ void __launch_bounds__(256) stream_step_kernel(const ResidualArgs a) {
  constexpr int B = MAXV * NS <= 16 ? MAXV : NS >= 16 ? 1 : 16 / NS;
  __shared__ float red[32];
  __shared__ float sc[NS * NS + 2 * NS];     // mix [NS][NS] (zeros where there is no copy) | out | in
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, nv = a.dp >> 2;
  for (int i = threadIdx.x; i < NS * NS + 2 * NS; i += blockDim.x) {
    const int s = i / NS, t = i % NS;
    float c = 0.f;
    if (t < a.n_out) {
      if (s < a.n_in) c = a.coef[s * a.n_out + t];
      else if (s >= NS) c = a.coef[(a.n_in + s - NS) * a.n_out + t];
    }
    sc[i] = c;
  }
  float4 y[MAXV];
  float ss = 0.f;
  sublayer_result<T, MAXV>(a, row, nv, y);
  __syncthreads();
  const float* xi = a.x_in + static_cast<size_t>(row) * a.ldxi;
  float* xo = a.x_out + static_cast<size_t>(row) * a.ldx;
#pragma unroll
  for (int i0 = 0; i0 < MAXV; i0 += B) {
    float4 x[B][NS];
#pragma unroll
    for (int i = 0; i < B; ++i) {
      const int v = threadIdx.x + (i0 + i) * blockDim.x;
#pragma unroll
      for (int s = 0; s < NS; ++s)
        x[i][s] = v < nv && s < a.n_in ? ld4(xi + s * a.dp + v * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int i = 0; i < B; ++i) {
      const int v = threadIdx.x + (i0 + i) * blockDim.x;
      float4 u = make_float4(0.f, 0.f, 0.f, 0.f);
      if (v < nv) {
        const float4 yv = y[i0 + i];
#pragma unroll
        for (int t = 0; t < NS; ++t)
          if (t < a.n_out) {
            const float o = sc[NS * NS + t], in = sc[NS * NS + NS + t];
            float4 n = make_float4(o * yv.x, o * yv.y, o * yv.z, o * yv.w);
#pragma unroll
            for (int s = 0; s < NS; ++s) {
              const float m = sc[s * NS + t];
              n = make_float4(fmaf(m, x[i][s].x, n.x), fmaf(m, x[i][s].y, n.y), fmaf(m, x[i][s].z, n.z), fmaf(m, x[i][s].w, n.w));
            }
            st4(xo + t * a.dp + v * 4, n);
            u = make_float4(fmaf(in, n.x, u.x), fmaf(in, n.y, u.y), fmaf(in, n.z, u.z), fmaf(in, n.w, u.w));
          }
      }
      y[i0 + i] = u;
      ss += sq4(u);
    }
  }
  if (a.h) write_operand<T, MAXV>(a, row, nv, y, ss, red);
  clear_inputs<MAXV>(a, row, nv);
}

// ---------------------------------------------------------------------------------------------- token shift
struct ShiftArgs {
  const float* x;
  int ldx;
  const float* w;            // norm weight [dp]
  const float* mu;           // [n_mix, dp]
  int n_mix;
  void* out;                 // T [n_mix][pitch rows][ldo]
  long out_batch;            // elements between two mixes
  int ldo;
  float* state;              // [slots, dp]: h of the last token seen
  long num_slots;
  const int* row_seq;        // sequence of every row
  const int* cu_q;           // first row of every sequence [n + 1]
  const int* ctx;            // tokens of every sequence after this step
  const int* state_slot;     // < 0: padding row
  int d, dp;
  float eps;
  int* status;
};

// RMSNorm of row `x` (with weight) into v[]; contains block barriers
template <int MAXV>
__device__ __forceinline__ void norm_row(const float* x, const float* w, int nv, int d, float eps, float* red, float4 (&v)[MAXV]) {
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    v[i] = c < nv ? ld4(x + c * 4) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += sq4(v[i]);
  }
  ss = cta_sum(ss, red);
  const float r = 1.f / sqrtf(ss / d + eps);
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < nv) {
      const float4 g = ld4(w + c * 4);
      v[i] = make_float4(v[i].x * r * g.x, v[i].y * r * g.y, v[i].z * r * g.z, v[i].w * r * g.w);
    }
  }
}

template <typename T, int MAXV>
__global__ void __launch_bounds__(256) norm_shift_mix_kernel(const ShiftArgs a) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, nv = a.dp >> 2;
  const int seq = a.row_seq[row];
  const int r0 = a.cu_q[seq], rl = a.cu_q[seq + 1] - 1;
  int slot = a.state_slot[seq];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  float4 h[MAXV], p[MAXV];
  norm_row<MAXV>(a.x + static_cast<size_t>(row) * a.ldx, a.w, nv, a.d, a.eps, red, h);
  const bool first = row == r0;
  const bool start = first && a.ctx[seq] == rl - r0 + 1;      // the portion starts the sequence
  if (first) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      p[i] = (start || slot < 0 || c >= nv) ? make_float4(0.f, 0.f, 0.f, 0.f)
                                            : ld4(a.state + static_cast<size_t>(slot) * a.dp + c * 4);
    }
  } else {
    norm_row<MAXV>(a.x + static_cast<size_t>(row - 1) * a.ldx, a.w, nv, a.d, a.eps, red, p);
  }
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < nv) {
      const float4 dlt = make_float4(p[i].x - h[i].x, p[i].y - h[i].y, p[i].z - h[i].z, p[i].w - h[i].w);
      for (int s = 0; s < a.n_mix; ++s) {
        const float4 m = ld4(a.mu + static_cast<size_t>(s) * a.dp + c * 4);
        st4(reinterpret_cast<T*>(a.out) + s * a.out_batch + static_cast<size_t>(row) * a.ldo + c * 4,
            make_float4(fmaf(dlt.x, m.x, h[i].x), fmaf(dlt.y, m.y, h[i].y), fmaf(dlt.z, m.z, h[i].z), fmaf(dlt.w, m.w, h[i].w)));
      }
    }
  }
  // The CTA of a portion's first row replaces the state: it is the only one that reads it, so no other CTA can see the
  // new value too early.
  if (first && slot >= 0) {
    if (rl != r0) norm_row<MAXV>(a.x + static_cast<size_t>(rl) * a.ldx, a.w, nv, a.d, a.eps, red, h);
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + i * blockDim.x;
      if (c < nv) st4(a.state + static_cast<size_t>(slot) * a.dp + c * 4, h[i]);
    }
  }
}

// ------------------------------------------------------------------------------------------------ PolyNorm
// vectors of eight elements (16 bytes of bf16); np is a multiple of 8
template <typename T, int MAXV>
__global__ void __launch_bounds__(512)
poly_norm_kernel(void* z, int ldz, int kind, const float* __restrict__ act, T* out, int ldo, int n, int np, float eps) {
  __shared__ float red[3][16];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x, nv = np >> 3;
  float v[MAXV][8];
  float s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
#pragma unroll
    for (int j = 0; j < 8; ++j) v[i][j] = 0.f;
    if (c < nv) take8(z, static_cast<size_t>(row) * ldz + c * 8, peek_kind(kind), v[i]);
  }
#pragma unroll
  for (int i = 0; i < MAXV; ++i)
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float q = v[i][j] * v[i][j], q2 = q * q;
      s1 += q;
      s2 += q2;
      s3 = fmaf(q2, q, s3);
    }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  s1 = lane_sum(s1);
  s2 = lane_sum(s2);
  s3 = lane_sum(s3);
  if (lane == 0) red[0][warp] = s1, red[1][warp] = s2, red[2][warp] = s3;
  __syncthreads();
  s1 = lane_sum(lane < nw ? red[0][lane] : 0.f);
  s2 = lane_sum(lane < nw ? red[1][lane] : 0.f);
  s3 = lane_sum(lane < nw ? red[2][lane] : 0.f);
  const float a = act[0] / sqrtf(s1 / n + eps), b = act[1] / sqrtf(s2 / n + eps), c3 = act[2] / sqrtf(s3 / n + eps);
  const float e0 = act[3];
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < nv) {
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        const float x = v[i][j];
        v[i][j] = c * 8 + j < n ? fmaf(fmaf(fmaf(c3, x, b), x, a), x, e0) : 0.f;
      }
      put8(out + static_cast<size_t>(row) * ldo + c * 8, v[i]);
      clear8(z, static_cast<size_t>(row) * ldz + c * 8, kind);
    }
  }
}

// ------------------------------------------------------------------------------------- tanh for a low-rank decay
// bf16: out[row] = [ hi(tanh z) | tanh z - hi ], r_p columns each; fp32: out[row] = tanh z
template <typename T>
__global__ void split_tanh_kernel(void* z, int ldz, int kind, T* out, int ldo, int M, int r, int rp) {
  pdl_wait();
  pdl_launch_dependents();
  const int i = blockIdx.x * blockDim.x + threadIdx.x;
  if (i >= M * rp) return;
  const int m = i / rp, c = i % rp;
  const float t = c < r ? tanhf(take1(z, static_cast<size_t>(m) * ldz + c, kind)) : 0.f;
  T* o = out + static_cast<size_t>(m) * ldo + c;
  st1(o, t);
  if (sizeof(T) == 2) st1(o + rp, t - __bfloat162float(__float2bfloat16(t)));
}

// --------------------------------------------------------------------------------------------- per-head norm
// out[row, h * vp + j] = rms(o[row, h, :])_j * w  (* silu(gate)), padding columns zero.  LPH lanes share a (row, head);
// with V4 a lane handles four neighbouring elements (vdim, vp and all strides multiples of 4).
__device__ __forceinline__ float gate_f(float z, int act) { return act == GATE_SIGMOID ? 1.f / (1.f + expf(-z)) : silu_f(z); }

template <typename T, int LPH, bool V4>
__global__ void __launch_bounds__(256)
head_norm_kernel(const float* __restrict__ o, int ldi, const float* __restrict__ w, int w_per_head, void* gate, int ldg,
                 int gate_kind, int gate_act, T* out, int ldo, int M, int H, int vdim, int vp, float eps) {
  pdl_wait();
  pdl_launch_dependents();
  const int u = static_cast<int>(blockIdx.x * (256u / LPH) + threadIdx.x / LPH);     // M * H < 2^31
  const int lane = threadIdx.x % LPH;
  const bool live = u < M * H;
  const int m = live ? u / H : 0, h = live ? u % H : 0;
  const float* x = o + static_cast<size_t>(m) * ldi + h * vdim;
  float ss = 0.f;
  if (live) {
    if (V4)
      for (int j = lane * 4; j < vdim; j += LPH * 4) ss += sq4(ld4(x + j));
    else
      for (int j = lane; j < vdim; j += LPH) ss += x[j] * x[j];
  }
#pragma unroll
  for (int s = LPH / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!live) return;
  const float r = 1.f / sqrtf(ss / vdim + eps);
  const float* wh = w + (w_per_head ? h * vdim : 0);
  T* y = out + static_cast<size_t>(m) * ldo + h * vp;
  const size_t go = static_cast<size_t>(m) * ldg + h * vdim;
  if (V4) {
    for (int j = lane * 4; j < vp; j += LPH * 4) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (j < vdim) {
        const float4 a = ld4(x + j), b = ld4(wh + j);
        v = make_float4(a.x * r * b.x, a.y * r * b.y, a.z * r * b.z, a.w * r * b.w);
        if (gate) {
          const float4 g = take4(gate, go + j, gate_kind);
          v = make_float4(v.x * gate_f(g.x, gate_act), v.y * gate_f(g.y, gate_act), v.z * gate_f(g.z, gate_act), v.w * gate_f(g.w, gate_act));
        }
      }
      st4(y + j, v);
    }
  } else {
    for (int j = lane; j < vp; j += LPH) {
      float v = 0.f;
      if (j < vdim) {
        v = x[j] * r * wh[j];
        if (gate) v *= gate_f(take1(gate, go + j, gate_kind), gate_act);
      }
      st1(y + j, v);
    }
  }
}

// One norm over the n columns of a row (all heads together); a CTA per row, columns n .. np - 1 of out are zero.
template <typename T, int MAXV>
__global__ void __launch_bounds__(256)
row_norm_kernel(const float* __restrict__ o, int ldi, const float* __restrict__ w, void* gate, int ldg, int gate_kind, int gate_act,
                T* out, int ldo, int n, int np, float eps) {
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int row = blockIdx.x;
  const float* x = o + static_cast<size_t>(row) * ldi;
  float4 v[MAXV];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    v[i] = c < n ? ld4(x + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += sq4(v[i]);
  }
  const float r = 1.f / sqrtf(cta_sum(ss, red) / n + eps);
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = (threadIdx.x + i * blockDim.x) * 4;
    if (c >= np) continue;
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < n) {
      const float4 b = ld4(w + c);
      y = make_float4(v[i].x * r * b.x, v[i].y * r * b.y, v[i].z * r * b.z, v[i].w * r * b.w);
      if (gate) {
        const float4 g = take4(gate, static_cast<size_t>(row) * ldg + c, gate_kind);
        y = make_float4(y.x * gate_f(g.x, gate_act), y.y * gate_f(g.y, gate_act), y.z * gate_f(g.z, gate_act), y.w * gate_f(g.w, gate_act));
      }
    }
    st4(out + static_cast<size_t>(row) * ldo + c, y);
  }
}

// z [M, 2 np]: blocks of 16 gate columns and their 16 up columns in turn -> out [M, np] = act(gate) * up.  Eight columns a thread.
template <typename T>
__global__ void __launch_bounds__(256) gated_act_kernel(void* z, int ldz, int kind, T* out, int ldo, long units, int nv, int act) {
  pdl_wait();
  pdl_launch_dependents();
  const long u = blockIdx.x * 256L + threadIdx.x;
  if (u >= units) return;
  const long m = u / nv;
  const int c = static_cast<int>(u - m * nv) * 8;
  const size_t zo = static_cast<size_t>(m) * ldz + (c >> 4) * 32 + (c & 15);
  float g[8], x[8];
  take8(z, zo, peek_kind(kind), g);
  take8(z, zo + 16, peek_kind(kind), x);
#pragma unroll
  for (int i = 0; i < 8; ++i) x[i] *= act == ACT_RELU ? fmaxf(g[i], 0.f) : silu_f(g[i]);
  put8(out + static_cast<size_t>(m) * ldo + c, x);
  clear8(z, zo, kind);
  clear8(z, zo + 16, kind);
}

// z [M, np] -> out [M, np] = act(z).  Eight columns a thread.
template <typename T>
__global__ void __launch_bounds__(256) plain_act_kernel(void* z, int ldz, int kind, T* out, int ldo, long units, int nv, int act) {
  pdl_wait();
  pdl_launch_dependents();
  const long u = blockIdx.x * 256L + threadIdx.x;
  if (u >= units) return;
  const long m = u / nv;
  const int c = static_cast<int>(u - m * nv) * 8;
  float x[8];
  take8(z, static_cast<size_t>(m) * ldz + c, peek_kind(kind), x);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const float p = fmaxf(x[i], 0.f);
    x[i] = act == ACT_RELU2 ? p * p : act == ACT_RELU ? p : silu_f(x[i]);
  }
  put8(out + static_cast<size_t>(m) * ldo + c, x);
  clear8(z, static_cast<size_t>(m) * ldz + c, kind);
}

template <typename T, int MAXV>
__global__ void __launch_bounds__(256)
gather_norm_kernel(const float* __restrict__ x, int ldx, const int64_t* __restrict__ rows, const float* __restrict__ w, T* h,
                   int ldh, int d, int dp, float eps, long n_rows, int* status) {
  __shared__ float red[32];
  float4 v[MAXV];
  long r = rows[blockIdx.x];
  if (!index_ok(r, n_rows, status)) r = 0;
  norm_row<MAXV>(x + static_cast<size_t>(r) * ldx, w, dp >> 2, d, eps, red, v);
#pragma unroll
  for (int i = 0; i < MAXV; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < (dp >> 2)) st4(h + static_cast<size_t>(blockIdx.x) * ldh + c * 4, v[i]);
  }
}

constexpr int MAX_STREAMS = 8;
static int row_threads(int dp) { return dp <= 512 ? 128 : 256; }
// vectors of four per thread, rounded up to the instantiated counts; 0: too wide
static int row_vecs(int dp, int threads) {
  const int per = (dp / 4 + threads - 1) / threads;
  return per <= 1 ? 1 : per <= 2 ? 2 : per <= 4 ? 4 : per <= 8 ? 8 : per <= 16 ? 16 : 0;
}

}  // namespace artb

using namespace artb;

#define ARTB_BY_VECS(V, CALL) \
  switch (V) {                \
    case 1: CALL(1); break;   \
    case 2: CALL(2); break;   \
    case 4: CALL(4); break;   \
    case 8: CALL(8); break;   \
    case 16: CALL(16); break; \
    default: return ERR_TOO_LARGE; \
  }

#define ARTB_BY_VECS8(V, CALL) \
  switch (V) {                 \
    case 1: CALL(1); break;    \
    case 2: CALL(2); break;    \
    case 4: CALL(4); break;    \
    case 8: CALL(8); break;    \
    default: return ERR_TOO_LARGE; \
  }

// f32: operands (table, h) are fp32 instead of bf16.  See ResidualArgs; y_kind, rg_kind are RowKinds.  coef: a step of hyper-connected
// streams (stream_step_kernel; n_in = 0: the embedding, of which every copy is the same).
ARTB_EXPORT int artb_residual_step(int f32, const int64_t* tokens, const void* table, int ldt, long vocab, void* y, int ldy,
                                   int y_kind, const float* x_in, float* x_out, int ldx, const float* w_post, float mult,
                                   const float* y_gate, const float* y_bias, const void* ex, int ldex, int ex_k, const int* ex_pos,
                                   const float* ex_w, long ex_rows, void* idn, int ldidn, int idn_kind, const double* freq, const int* pos, float* hist, long hist_stride, int hist_n, const float* avg, const float* w_next, void* h,
                                   int ldh, int M, int d, int dp, float eps, int* status, void* rg, int ldrg, int rg_kind, const float* rg_b,
                                   const float* coef, int n_in, int n_out, int ldxi, cudaStream_t st) {
  if (M <= 0) return 0;
  if ((dp & 3) || dp < d || (ldx & 3) || (ldy & 3) || (ldh & 3) || (ldt & 3) || (ldex & 3) || (ldidn & 3) || !x_out || (w_next && !h)) return ERR_BAD_SHAPE;
  if (!tokens && ((!y && !ex) || !x_in)) return ERR_BAD_SHAPE;
  if (rg && ((rg_kind == ROW_BF16 ? 7 : 15) & reinterpret_cast<uintptr_t>(rg))) return ERR_BAD_ALIGN;
  if ((ex && (ex_k <= 0 || !ex_pos || !ex_w)) || (idn && (!ex || idn_kind == ROW_F32_TAKE)) || (freq && (!tokens || !pos))) return ERR_BAD_SHAPE;
  const ResidualArgs a{tokens, table, ldt, vocab, y, ldy, y_kind, x_in, x_out, ldx, w_post, mult, y_gate, y_bias, ex, ldex, ex_k, ex_pos, ex_w,
                       ex_rows, idn, ldidn, idn_kind, freq, pos, hist, hist_stride, hist_n, avg, w_next, h, ldh, d, dp, eps, status, rg, ldrg, rg_kind,
                       rg_b, coef, n_in, n_out, ldxi};
  if (rg && (!rg_b || tokens || w_post || (ldrg & 3))) return ERR_BAD_SHAPE;
  const int th = row_threads(dp);
  cudaError_t e = cudaSuccess;
  if (coef) {
    if (n_in < 0 || n_out < 1 || n_in > MAX_STREAMS || n_out > MAX_STREAMS || (n_in == 0) != (tokens != nullptr) || (tokens && mult != 1.f) || w_post ||
        hist || freq || idn || (ldxi & 3) || ldxi < n_in * dp || ldx < n_out * dp || (n_in != n_out && x_in == x_out))
      return ERR_BAD_SHAPE;
    const int ns = n_in > n_out ? n_in : n_out;
#define ARTB_SS_N(V, N)                                                                                                \
  e = f32 ? launch_kernel(stream_step_kernel<float, V, N>, dim3(M), dim3(th), 0, st, a)                                 \
          : launch_kernel(stream_step_kernel<__nv_bfloat16, V, N>, dim3(M), dim3(th), 0, st, a)
#define ARTB_SS(V)              \
  if (ns <= 1) ARTB_SS_N(V, 1); \
  else if (ns <= 2) ARTB_SS_N(V, 2); \
  else if (ns <= 4) ARTB_SS_N(V, 4); \
  else ARTB_SS_N(V, 8)
    ARTB_BY_VECS(row_vecs(dp, th), ARTB_SS)
#undef ARTB_SS
#undef ARTB_SS_N
    return static_cast<int>(e);
  }
#define ARTB_RS(V)                                                                                                     \
  e = f32 ? launch_kernel(residual_step_kernel<float, V>, dim3(M), dim3(th), 0, st, a)                                  \
          : launch_kernel(residual_step_kernel<__nv_bfloat16, V>, dim3(M), dim3(th), 0, st, a)
  ARTB_BY_VECS(row_vecs(dp, th), ARTB_RS)
#undef ARTB_RS
  return static_cast<int>(e);
}

ARTB_EXPORT int artb_norm_shift_mix(int f32, const float* x, int ldx, const float* w, const float* mu, int n_mix, void* out,
                                    long out_batch, int ldo, float* state, long num_slots, const int* row_seq,
                                    const int* cu_q, const int* ctx, const int* state_slot, int M, int d, int dp, float eps,
                                    int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if ((dp & 3) || dp < d || (ldx & 3) || (ldo & 3) || (out_batch & 3) || n_mix < 1) return ERR_BAD_SHAPE;
  const ShiftArgs a{x, ldx, w, mu, n_mix, out, out_batch, ldo, state, num_slots, row_seq, cu_q, ctx, state_slot, d, dp, eps,
                    status};
  const int th = row_threads(dp);
  cudaError_t e = cudaSuccess;
#define ARTB_SM(V)                                                                                                      \
  e = f32 ? launch_kernel(norm_shift_mix_kernel<float, V>, dim3(M), dim3(th), 0, st, a)                                  \
          : launch_kernel(norm_shift_mix_kernel<__nv_bfloat16, V>, dim3(M), dim3(th), 0, st, a)
  ARTB_BY_VECS(row_vecs(dp, th), ARTB_SM)
#undef ARTB_SM
  return static_cast<int>(e);
}

// act: fp32 {a, b, c, e}; n real width, np padded width (columns n .. np - 1 of out are zero)
ARTB_EXPORT int artb_poly_norm(int f32, void* z, int ldz, int kind, const float* act, void* out, int ldo, int M, int n, int np,
                               float eps, cudaStream_t st) {
  if (M <= 0) return 0;
  if ((np & 7) || np < n || (ldz & 7) || (ldo & 7)) return ERR_BAD_SHAPE;
  const int th = np <= 2048 ? 128 : np <= 8192 ? 256 : 512;
  cudaError_t e = cudaSuccess;
#define ARTB_PN(V)                                                                                                       \
  e = f32 ? launch_kernel(poly_norm_kernel<float, V>, dim3(M), dim3(th), 0, st, z, ldz, kind, act,                        \
                          reinterpret_cast<float*>(out), ldo, n, np, eps)                                                 \
          : launch_kernel(poly_norm_kernel<__nv_bfloat16, V>, dim3(M), dim3(th), 0, st, z, ldz, kind, act,                \
                          reinterpret_cast<__nv_bfloat16*>(out), ldo, n, np, eps)
  ARTB_BY_VECS8(row_vecs(np / 2, th), ARTB_PN)
#undef ARTB_PN
  return static_cast<int>(e);
}

ARTB_EXPORT int artb_split_tanh(int f32, void* z, int ldz, int kind, void* out, int ldo, int M, int r, int rp, cudaStream_t st) {
  if (M <= 0) return 0;
  if (rp < r || ldo < (f32 ? rp : 2 * rp)) return ERR_BAD_SHAPE;
  const dim3 grid((M * rp + 255) / 256);
  return static_cast<int>(f32 ? launch_kernel(split_tanh_kernel<float>, grid, dim3(256), 0, st, z, ldz, kind,
                                              reinterpret_cast<float*>(out), ldo, M, r, rp)
                              : launch_kernel(split_tanh_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, z, ldz, kind,
                                              reinterpret_cast<__nv_bfloat16*>(out), ldo, M, r, rp));
}

// z [M, 2 np] of `kind` in gate|up blocks of 16 columns -> out [M, np] (np a multiple of 16)
ARTB_EXPORT int artb_gated_act(int f32, void* z, int ldz, int kind, void* out, int ldo, int M, int np, int act, cudaStream_t st) {
  if (M <= 0) return 0;
  if ((np & 15) || (ldz & 7) || (ldo & 7) || (act != ACT_SILU && act != ACT_RELU)) return ERR_BAD_SHAPE;
  const long units = static_cast<long>(M) * (np >> 3);
  const dim3 grid(static_cast<unsigned>((units + 255) / 256));
  return static_cast<int>(f32 ? launch_kernel(gated_act_kernel<float>, grid, dim3(256), 0, st, z, ldz, kind, reinterpret_cast<float*>(out),
                                              ldo, units, np >> 3, act)
                              : launch_kernel(gated_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, z, ldz, kind,
                                              reinterpret_cast<__nv_bfloat16*>(out), ldo, units, np >> 3, act));
}

// z [M, np] of `kind` -> out [M, np] = act(z) (np a multiple of 8)
ARTB_EXPORT int artb_plain_act(int f32, void* z, int ldz, int kind, void* out, int ldo, int M, int np, int act, cudaStream_t st) {
  if (M <= 0) return 0;
  if ((np & 7) || (ldz & 7) || (ldo & 7) || (act != ACT_SILU && act != ACT_RELU && act != ACT_RELU2)) return ERR_BAD_SHAPE;
  const long units = static_cast<long>(M) * (np >> 3);
  const dim3 grid(static_cast<unsigned>((units + 255) / 256));
  return static_cast<int>(f32 ? launch_kernel(plain_act_kernel<float>, grid, dim3(256), 0, st, z, ldz, kind, reinterpret_cast<float*>(out),
                                              ldo, units, np >> 3, act)
                              : launch_kernel(plain_act_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, z, ldz, kind,
                                              reinterpret_cast<__nv_bfloat16*>(out), ldo, units, np >> 3, act));
}

// o fp32 [M, H * vdim]; w [vdim] or, with w_per_head, [H * vdim]; gate [M, H * vdim] of kind gate_kind or null
ARTB_EXPORT int artb_head_norm(int f32, const float* o, int ldi, const float* w, int w_per_head, void* gate, int ldg,
                               int gate_kind, int gate_act, void* out, int ldo, int M, int H, int vdim, int vp, float eps,
                               cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || vdim <= 0 || vp < vdim || ldo < H * vp || static_cast<long>(M) * H >= (1L << 31)) return ERR_BAD_SHAPE;
  const bool v4 = !((vdim | vp | ldi | ldo | (gate ? ldg : 0)) & 3) && !(reinterpret_cast<uintptr_t>(gate) & 15);
  if (H == 1 && v4 && vp > 256) {      // one norm per row: a CTA each
    const int th = row_threads(vp);
    cudaError_t e = cudaSuccess;
#define ARTB_RN(V)                                                                                                         \
  e = f32 ? launch_kernel(row_norm_kernel<float, V>, dim3(M), dim3(th), 0, st, o, ldi, w, gate, ldg, gate_kind, gate_act,   \
                          reinterpret_cast<float*>(out), ldo, vdim, vp, eps)                                               \
          : launch_kernel(row_norm_kernel<__nv_bfloat16, V>, dim3(M), dim3(th), 0, st, o, ldi, w, gate, ldg, gate_kind,     \
                          gate_act, reinterpret_cast<__nv_bfloat16*>(out), ldo, vdim, vp, eps)
    ARTB_BY_VECS(row_vecs(vp, th), ARTB_RN)
#undef ARTB_RN
    return static_cast<int>(e);
  }
  const int lph = !v4 ? 32 : vdim <= 16 ? 4 : vdim <= 64 ? 16 : 32;
  const dim3 grid(static_cast<unsigned>((static_cast<long>(M) * H * lph + 255) / 256));
#define ARTB_HN(T_, L_, V_)                                                                                             \
  return static_cast<int>(launch_kernel(head_norm_kernel<T_, L_, V_>, grid, dim3(256), 0, st, o, ldi, w, w_per_head, gate, ldg, \
                                        gate_kind, gate_act, reinterpret_cast<T_*>(out), ldo, M, H, vdim, vp, eps))
  if (f32) {
    if (lph == 4) ARTB_HN(float, 4, true);
    if (lph == 16) ARTB_HN(float, 16, true);
    if (v4) ARTB_HN(float, 32, true);
    ARTB_HN(float, 32, false);
  }
  if (lph == 4) ARTB_HN(__nv_bfloat16, 4, true);
  if (lph == 16) ARTB_HN(__nv_bfloat16, 16, true);
  if (v4) ARTB_HN(__nv_bfloat16, 32, true);
  ARTB_HN(__nv_bfloat16, 32, false);
#undef ARTB_HN
}

ARTB_EXPORT int artb_gather_norm(int f32, const float* x, int ldx, const int64_t* rows, int n, const float* w, void* h, int ldh,
                                 int d, int dp, float eps, long n_rows, int* status, cudaStream_t st) {
  if (n <= 0) return 0;
  if ((dp & 3) || dp < d || (ldx & 3) || (ldh & 3)) return ERR_BAD_SHAPE;
  const int th = row_threads(dp);
#define ARTB_GN(V)                                                                                                        \
  if (f32)                                                                                                                \
    gather_norm_kernel<float, V><<<n, th, 0, st>>>(x, ldx, rows, w, reinterpret_cast<float*>(h), ldh, d, dp, eps, n_rows, status); \
  else                                                                                                                    \
    gather_norm_kernel<__nv_bfloat16, V><<<n, th, 0, st>>>(x, ldx, rows, w, reinterpret_cast<__nv_bfloat16*>(h), ldh, d, dp, eps, \
                                                           n_rows, status)
  ARTB_BY_VECS(row_vecs(dp, th), ARTB_GN)
#undef ARTB_GN
  return static_cast<int>(cudaGetLastError());
}
