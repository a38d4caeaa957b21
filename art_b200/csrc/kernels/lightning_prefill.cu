// Lightning attention of prompt portions on tensor cores, in chunks of 64 tokens.
//
// With q, k, v (activated: the projection's epilogue applies the silu), a head's constant decay w and the state S before a
// chunk of n tokens
//
//   o_i = w^(i+1) q_i S + sum_{j <= i} w^(i-j) (q_i . k_j) v_j          S' = w^n S + sum_j k_j (w^(n-1-j) v_j)^T
//
// A CTA owns (sequence, head, 64 value columns) and walks over the portion.  The fp32 state lives in the accumulators of the
// warps; where it is an operand (q S), and where something enters it (w^(n-1-j) v_j), the operand is a bf16 pair (high part,
// remainder) and takes two products, so that the recurrence keeps fp32 accuracy.  The weights w^(i-j) (q_i . k_j) are a pair,
// too; q, k and v themselves are bf16, as projections are.  The next chunk's rows are loaded while the current one is worked
// on; two CTAs share an SM.
//
// Warp-level tiles: operands are made by the CUDA cores (decay, splitting) chunk by chunk in a serial chain, which leaves no
// long product to feed to the asynchronous tensor path.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "mma_tile.cuh"
#include "row_io.cuh"

namespace artb {

constexpr int LF_C = 64, LF_V = 64, LF_THREADS = 256;

struct Lightning {
  const __nv_bfloat16 *q, *k, *v;      // [M, ld]: heads of dim (q, k) and vdim (v) columns
  int ld;
  const float* decay;                  // [H]
  float* state;                        // [slots][H][vdim][ld_dim]
  long slot_stride;
  int ld_dim;
  long num_slots;
  const int *cu_q, *ctx, *state_slot;
  int H, dim, vdim;
  float* o;                            // [rows, ldo]
  int ldo, rows;
  int* status;
};

template <int D>
struct LfSmem {
  static constexpr int LD = D + 8, LV = LF_V + 8;
  static constexpr int Q = 0, K = Q + LF_C * LD, SH = K + LF_C * LD, SL = SH + LF_V * LD, V = SL + LF_V * LD, VH = V + LF_C * LV,
                       VL = VH + LF_C * LV, ELEMS = VL + LF_C * LV;
  static constexpr int BYTES = ELEMS * 2 + (LF_C + 1) * 4;
};

__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = pair_bf16(a, b);
  const float2 h = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&hi));
  lo = pair_bf16(a - h.x, b - h.y);
}

template <int D>
__global__ void __launch_bounds__(LF_THREADS, 2) lightning_prefill_kernel(const Lightning a) {
  using L = LfSmem<D>;
  constexpr int LD = L::LD, LV = L::LV, NQ = LF_C * (D / 8) / LF_THREADS, NV = LF_C * (LF_V / 8) / LF_THREADS;
  constexpr int NT = D / 16;                    // state tiles of a warp: 16 value columns x D / 2 channels
  extern __shared__ __align__(16) __nv_bfloat16 lf_s[];
  __nv_bfloat16 *sQ = lf_s + L::Q, *sK = lf_s + L::K, *sSh = lf_s + L::SH, *sSl = lf_s + L::SL, *sV = lf_s + L::V, *sVh = lf_s + L::VH,
                *sVl = lf_s + L::VL;
  float* pw = reinterpret_cast<float*>(lf_s + L::ELEMS);      // powers 0 .. 64 of the decay
  const int seq = blockIdx.y, h = blockIdx.x % a.H, v0 = blockIdx.x / a.H * LF_V;
  const int row0 = a.cu_q[seq], len = a.cu_q[seq + 1] - row0;
  if (len <= 0) return;
  if (row0 < 0 || len > a.rows - row0) {        // not a portion of this batch
    if (threadIdx.x == 0) atomicMax(a.status, ST_BAD_ARGS);
    return;
  }
  int slot = a.state_slot[seq];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3, jm = lane >> 3, rr = lane & 7;
  if (tid <= LF_C) {
    double p = 1.0, x = a.decay[h];
    for (int e = tid; e; e >>= 1, x *= x)
      if (e & 1) p *= x;
    pw[tid] = static_cast<float>(p);
  }
  const int mt = (warp & 3) * 16, nh = warp >> 2;      // rows of the warp's tiles (tokens, value columns) and its column half

  // state tiles: value columns mt + g (+ 8), channels nh * D / 2 + i * 8 + 2 t
  float S[NT][4];
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.slot_stride + static_cast<size_t>(h) * a.vdim * a.ld_dim;
  const bool resume = slot >= 0 && a.ctx[seq] != len;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int v = v0 + mt + g + 8 * e, d = nh * (D / 2) + i * 8 + 2 * t;
      float2 x = make_float2(0.f, 0.f);
      if (resume && v < a.vdim && d < a.ld_dim) x = *reinterpret_cast<const float2*>(sp + static_cast<size_t>(v) * a.ld_dim + d);
      S[i][2 * e] = x.x;
      S[i][2 * e + 1] = x.y;
    }

  uint4 rq[NQ], rk[NQ], rv[NV];
  const __nv_bfloat16 *gq = a.q + h * a.dim, *gk = a.k + h * a.dim, *gv = a.v + h * a.vdim + v0;
  auto fetch = [&](int t0) {
    const int n = len - t0;
    const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int x = tid + i * LF_THREADS, r = x / (D / 8), c = x % (D / 8) * 8;
      const bool ok = r < n && c < a.dim;
      const size_t off = static_cast<size_t>(row0 + t0 + r) * a.ld + c;
      rq[i] = ok ? *reinterpret_cast<const uint4*>(gq + off) : zero;
      rk[i] = ok ? *reinterpret_cast<const uint4*>(gk + off) : zero;
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int x = tid + i * LF_THREADS, r = x / (LF_V / 8), c = x % (LF_V / 8) * 8;
      rv[i] = r < n && v0 + c < a.vdim ? *reinterpret_cast<const uint4*>(gv + static_cast<size_t>(row0 + t0 + r) * a.ld + c) : zero;
    }
  };
  fetch(0);
  __syncthreads();
  for (int t0 = 0; t0 < len; t0 += LF_C) {
    const int n = min(LF_C, len - t0);
    // ---- operands of the chunk
#pragma unroll
    for (int i = 0; i < NQ; ++i) {
      const int x = tid + i * LF_THREADS, r = x / (D / 8), c = x % (D / 8) * 8;
      *reinterpret_cast<uint4*>(sQ + r * LD + c) = rq[i];
      *reinterpret_cast<uint4*>(sK + r * LD + c) = rk[i];
    }
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int x = tid + i * LF_THREADS, r = x / (LF_V / 8), c = x % (LF_V / 8) * 8;
      const float w = r < n ? pw[n - 1 - r] : 0.f;
      const uint4 y = rv[i];
      uint4 hi, lo;
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const float2 f = __bfloat1622float2(reinterpret_cast<const __nv_bfloat162*>(&y)[e]);
        split_pair(w * f.x, w * f.y, reinterpret_cast<uint32_t*>(&hi)[e], reinterpret_cast<uint32_t*>(&lo)[e]);
      }
      *reinterpret_cast<uint4*>(sV + r * LV + c) = y;
      *reinterpret_cast<uint4*>(sVh + r * LV + c) = hi;
      *reinterpret_cast<uint4*>(sVl + r * LV + c) = lo;
    }
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int at = (mt + g + 8 * e) * LD + nh * (D / 2) + i * 8 + 2 * t;
        uint32_t hi, lo;
        split_pair(S[i][2 * e], S[i][2 * e + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(sSh + at) = hi;
        *reinterpret_cast<uint32_t*>(sSl + at) = lo;
      }
    __syncthreads();
    if (t0 + LF_C < len) fetch(t0 + LF_C);

    // ---- outputs: tokens mt .. mt + 15, value columns nh * 32 .. + 31
    if (mt < n) {
      float O[4][4];
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) O[i][e] = 0.f;
#pragma unroll
      for (int ks = 0; ks < D / 16; ++ks) {
        uint32_t qf[4];
        ldmat_x4(qf, sQ + (mt + (jm & 1) * 8 + rr) * LD + ks * 16 + (jm >> 1) * 8);
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          const int at = (nh * 32 + np * 16 + (jm >> 1) * 8 + rr) * LD + ks * 16 + (jm & 1) * 8;
          uint32_t b[4];
          ldmat_x4(b, sSh + at);
          mma_bf16(O[2 * np], qf, b[0], b[1]);
          mma_bf16(O[2 * np + 1], qf, b[2], b[3]);
          ldmat_x4(b, sSl + at);
          mma_bf16(O[2 * np], qf, b[0], b[1]);
          mma_bf16(O[2 * np + 1], qf, b[2], b[3]);
        }
      }
      const float w0 = pw[mt + g + 1], w1 = pw[mt + g + 9];      // at most 64
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        O[i][0] *= w0;
        O[i][1] *= w0;
        O[i][2] *= w1;
        O[i][3] *= w1;
      }
      for (int kb = 0; kb <= mt; kb += 16) {           // keys up to the tile's own
        float P[2][4] = {};
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
          uint32_t qf[4], b[4];
          ldmat_x4(qf, sQ + (mt + (jm & 1) * 8 + rr) * LD + ks * 16 + (jm >> 1) * 8);
          ldmat_x4(b, sK + (kb + (jm >> 1) * 8 + rr) * LD + ks * 16 + (jm & 1) * 8);
          mma_bf16(P[0], qf, b[0], b[1]);
          mma_bf16(P[1], qf, b[2], b[3]);
        }
        uint32_t ph[4], pl[4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int dist = mt + g + 8 * e - (kb + j * 8 + 2 * t);
            const float p0 = dist >= 0 ? P[j][2 * e] * pw[dist] : 0.f, p1 = dist >= 1 ? P[j][2 * e + 1] * pw[dist - 1] : 0.f;
            split_pair(p0, p1, ph[2 * j + e], pl[2 * j + e]);
          }
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t b[4];
          ldmat_x4_t(b, sV + (kb + (jm & 1) * 8 + rr) * LV + nh * 32 + np * 16 + (jm >> 1) * 8);
          mma_bf16(O[2 * np], ph, b[0], b[1]);
          mma_bf16(O[2 * np + 1], ph, b[2], b[3]);
          mma_bf16(O[2 * np], pl, b[0], b[1]);
          mma_bf16(O[2 * np + 1], pl, b[2], b[3]);
        }
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int r = mt + g + 8 * e, v = v0 + nh * 32 + i * 8 + 2 * t;       // vdim is even
          if (r < n && v < a.vdim)
            *reinterpret_cast<float2*>(a.o + static_cast<size_t>(row0 + t0 + r) * a.ldo + h * a.vdim + v) = make_float2(O[i][2 * e], O[i][2 * e + 1]);
        }
    }

    // ---- state
    const float wn = pw[n];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) S[i][e] *= wn;
#pragma unroll
    for (int ks = 0; ks < LF_C / 16; ++ks) {
      if (ks * 16 >= n) break;                         // uniform
      uint32_t ah[4], al[4];
      const int at = (ks * 16 + (jm >> 1) * 8 + rr) * LV + mt + (jm & 1) * 8;
      ldmat_x4_t(ah, sVh + at);
      ldmat_x4_t(al, sVl + at);
#pragma unroll
      for (int np = 0; np < NT / 2; ++np) {
        uint32_t b[4];
        ldmat_x4_t(b, sK + (ks * 16 + (jm & 1) * 8 + rr) * LD + nh * (D / 2) + np * 16 + (jm >> 1) * 8);
        mma_bf16(S[2 * np], ah, b[0], b[1]);
        mma_bf16(S[2 * np + 1], ah, b[2], b[3]);
        mma_bf16(S[2 * np], al, b[0], b[1]);
        mma_bf16(S[2 * np + 1], al, b[2], b[3]);
      }
    }
    __syncthreads();
  }
  if (slot < 0) return;
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int v = v0 + mt + g + 8 * e, d = nh * (D / 2) + i * 8 + 2 * t;
      if (v < a.vdim && d < a.ld_dim) *reinterpret_cast<float2*>(sp + static_cast<size_t>(v) * a.ld_dim + d) = make_float2(S[i][2 * e], S[i][2 * e + 1]);
    }
}

template <int D>
static int launch_lightning(const Lightning& a, int n_seqs, cudaStream_t st) {
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(lightning_prefill_kernel<D>, cudaFuncAttributeMaxDynamicSharedMemorySize, LfSmem<D>::BYTES);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = true;
  }
  lightning_prefill_kernel<D><<<dim3(a.H * ((a.vdim + LF_V - 1) / LF_V), n_seqs), LF_THREADS, LfSmem<D>::BYTES, st>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace artb

using namespace artb;

// q, k, v bf16 [M, ld] (after the silu, 16-byte aligned; dim, vdim and ld multiples of 8, dim <= 128); o fp32 [rows, ldo]
// gets H * vdim columns.  State and sequence arguments as artb_linear_scan.
ARTB_EXPORT int artb_lightning_prefill(const void* q, const void* k, const void* v, int ld, const float* decay, float* state,
                                       long slot_stride, int ld_dim, long num_slots, const int* cu_q, const int* ctx,
                                       const int* state_slot, int n_seqs, int H, int dim, int vdim, float* o, int ldo, int rows,
                                       int* status, cudaStream_t st) {
  if (n_seqs <= 0) return 0;
  if (H <= 0 || dim <= 0 || vdim <= 0 || dim > 128 || ((dim | vdim | ld) & 7) || (ldo & 1) || ldo < H * vdim || (ld_dim & 3) || ld_dim < dim ||
      (slot_stride & 3) || n_seqs > 65535)
    return ERR_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(v) | reinterpret_cast<uintptr_t>(o) |
       reinterpret_cast<uintptr_t>(state)) & 15)
    return ERR_BAD_ALIGN;
  const Lightning a{reinterpret_cast<const __nv_bfloat16*>(q), reinterpret_cast<const __nv_bfloat16*>(k), reinterpret_cast<const __nv_bfloat16*>(v),
                    ld, decay, state, slot_stride, ld_dim, num_slots, cu_q, ctx, state_slot, H, dim, vdim, o, ldo, rows, status};
  return dim <= 64 ? launch_lightning<64>(a, n_seqs, st) : launch_lightning<128>(a, n_seqs, st);
}
