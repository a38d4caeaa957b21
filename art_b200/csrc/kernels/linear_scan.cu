// Linear attention with a decay per channel or per head, carried in an fp32 state S [dim, vdim] per sequence and head.
//
//   SCAN_HGRN2   f = l + (1 - l) sigmoid(g + b), q = silu(q);   S = f S + (1 - f) v^T ;  o = S^T q        (reads after)
//   SCAN_WKV     w = exp(-exp(g + b));   o = (S + (u k) v^T)^T r ;  S = w S + k v^T                       (reads before)
//   SCAN_FIXED   q, k, v = silu(q), silu(k), silu(v);               S = w S + k v^T ;  o = S^T q          (reads after)
//                w a constant of the head
//
// All of it is fp32 arithmetic on CUDA cores: a recurrence multiplies rounding errors, so its operands do not go through
// 16-bit tensor-core products.  The decay, the gates and the bonus are computed where they are used; q, k, v and g are
// the raw outputs of the projections.
//
// Two kernels share the state layout [slot][head][vdim][ld_dim] (a column of S is contiguous):
//
//   linear_scan_kernel     portions of prompts.  A CTA owns (sequence, head, a slice of 16 to 128 value columns) and
//                          walks over the portion.  The state lives in registers: eight threads share one to four
//                          columns, each with NR of their rows (interleaved in groups of four, so that operands are
//                          16-byte shared-memory reads without bank conflicts).  Four extra warps load the
//                          next 16 tokens and apply decay / gate functions while the others work on the current
//                          16; the partial sums of four tokens over eight threads are reduced by four exchanges
//                          instead of twelve.
//   linear_decode_kernel   one new token per sequence.  A CTA owns (sequence, head), streams the state through registers
//                          once (read, update, write) and finishes the head: RMSNorm over its vdim outputs, norm weight,
//                          optional silu gate, bf16 store.  Without a norm weight the fp32 outputs are stored as they are.
//
// A portion that starts a sequence (ctx == its length) begins with a zero state whatever the slot holds.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "row_io.cuh"

namespace artb {

enum ScanMode : int { SCAN_HGRN2 = 0, SCAN_WKV = 1, SCAN_FIXED = 2 };

struct ScanArgs {
  void* q;      // q (hgrn2) or r (wkv): [M, ldq], kind qkv_kind
  void* k;      // wkv and fixed
  void* v;
  void* g;      // decay projection, kind g_kind
  int ldq, ldk, ldv, ldg, qkv_kind, g_kind;
  const float* bias;    // [H * dim] added to g
  const float* aux;     // [H * dim] lower bound (hgrn2) or bonus u (wkv); [H] decay (fixed)
  float* state;
  long slot_stride;     // floats per slot
  int ld_dim;           // row pitch of a state column (multiple of 4, >= dim)
  long num_slots;
  const int* cu_q;
  const int* ctx;
  const int* state_slot;
  int H, dim, vdim;
  int* status;
};

struct ScanOut {
  float* o;             // fp32 [rows, ldo] (linear_scan_kernel)
  int ldo, rows;
};

struct DecodeOut {
  const float* w;       // norm weight [vdim] or [H * vdim]; null: out is fp32 [M, ldo], vdim columns per head, not normalised
  int w_per_head;
  void* gate;           // silu gate, kind gate_kind, or null
  int ldgate, gate_kind;
  void* out;            // T [M, ldo], vp columns per head
  int ldo, vp;
  float eps;
};

// packed fp32 pairs (one instruction per two multiply-adds)
__device__ __forceinline__ uint64_t pack2(float a, float b) {
  uint64_t r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(uint64_t v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
struct alignas(16) Pair2 {
  uint64_t lo, hi;
};

constexpr int SCAN_TC = 16;             // tokens per stage
constexpr int SCAN_RG = 8;              // threads that share a state column
constexpr int SCAN_LOADERS = 128;

template <int MODE>
constexpr int scan_arrays() { return MODE == SCAN_WKV ? 3 : 2; }      // q, k and decay, as far as they are operands
template <int MODE>
constexpr int scan_smem(int DP, int cw) {
  return 2 * SCAN_TC * (scan_arrays<MODE>() * DP + 2 * cw + 1) * 4;
}

// decay, gate and bonus of one channel from the raw projections; k of hgrn2 is 1 - f
template <int MODE>
__device__ __forceinline__ void scan_gates(float qr, float kr, float g, float aux, float& q, float& f, float& k, float& bonus) {
  if (MODE == SCAN_HGRN2) {
    q = __fdividef(qr, 1.f + expf(-qr));
    f = aux + (1.f - aux) * __fdividef(1.f, 1.f + expf(-g));
    k = 1.f - f;
    bonus = 0.f;
  } else if (MODE == SCAN_WKV) {
    q = qr;
    f = expf(-expf(g));
    k = kr;
    bonus = qr * aux * kr;
  } else {
    q = silu_f(qr);
    f = aux;
    k = silu_f(kr);
    bonus = 0.f;
  }
}

// All compute and loader warps; a named barrier because the two roles wait at different places of the code.  The
// instruction wants whole warps: lanes that took different ways through the code before it (a store that only some of them
// do) come together first.
template <int THREADS>
__device__ __forceinline__ void stage_barrier() {
  __syncwarp();
  asm volatile("bar.sync 1, %0;" ::"n"(THREADS) : "memory");
}

// A CTA's column slice is CW = NC * CPT wide: thread (rg, cg) holds rows {4 rg + 32 i} of columns {cg + NC j}.
template <int NR, int MODE, int CPT, int NC, typename T>
__global__ void __launch_bounds__(SCAN_RG * NC + SCAN_LOADERS, CPT * NR <= 64 && NC == 16 ? 2 : 1)
linear_scan_kernel(const ScanArgs a, const ScanOut so) {
  constexpr int DP = SCAN_RG * NR, CW = NC * CPT, COMP = SCAN_RG * NC, CH = DP / 32;
  constexpr bool HAS_K = MODE != SCAN_HGRN2, HAS_F = MODE != SCAN_FIXED;      // k as an operand, a decay per channel
  extern __shared__ __align__(16) float scan_s[];
  float* sq = scan_s;                                   // [2][TC][DP]
  float* sf = sq + 2 * SCAN_TC * DP;
  float* sk = sf + (HAS_F ? 2 * SCAN_TC * DP : 0);
  float* sv = sk + (HAS_K ? 2 * SCAN_TC * DP : 0);      // [2][TC][CW]
  float* sout = sv + 2 * SCAN_TC * CW;                  // [2][TC][CW]
  float* sb = sout + 2 * SCAN_TC * CW;                  // [2][TC] bonus
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, h = blockIdx.x % a.H, c0 = (blockIdx.x / a.H) * CW;
  const int row0 = a.cu_q[seq], len = a.cu_q[seq + 1] - row0;
  if (len <= 0) return;
  if (row0 < 0 || len > so.rows - row0) {      // not a portion of this batch
    if (threadIdx.x == 0) atomicMax(a.status, ST_BAD_ARGS);
    return;
  }
  int slot = a.state_slot[seq];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const bool comp = static_cast<int>(threadIdx.x) < COMP;
  const int chunks = (len + SCAN_TC - 1) / SCAN_TC;

  if (!comp) {
    // ---------------------------------------------------------------- loader warps: one token per warp at a time
    const int lt = static_cast<int>(threadIdx.x) - COMP, lane = lt & 31, lw = lt >> 5;
    constexpr int TB = 2;                               // tokens of a warp whose raw values are in flight together
    constexpr int PER = SCAN_TC / (SCAN_LOADERS / 32);  // tokens per warp and stage
    constexpr int CV = (CW + 31) / 32;
    float bias[CH], aux[CH];
#pragma unroll
    for (int i = 0; i < CH; ++i) {
      const int c = i * 32 + lane;
      bias[i] = HAS_F && c < a.dim ? a.bias[h * a.dim + c] : 0.f;
      aux[i] = HAS_F && c < a.dim ? a.aux[h * a.dim + c] : 0.f;
    }
    const T* __restrict__ gq = reinterpret_cast<const T*>(a.q) + h * a.dim;
    const T* __restrict__ gk = reinterpret_cast<const T*>(a.k) + h * a.dim;
    const T* __restrict__ gv = reinterpret_cast<const T*>(a.v) + h * a.vdim + c0;
    const float* __restrict__ gg = reinterpret_cast<const float*>(a.g) + h * a.dim;
    struct Raw {       // as loaded: converting them here would make the warp wait for them here
      T q[TB][CH], k[TB][HAS_K ? CH : 1], v[TB][CV];
      float g[TB][HAS_F ? CH : 1];
    };
    const T zero = T(0.f);
    auto fetch = [&](Raw& r, int chunk, int p) {        // raw values of tokens p, p + 1 of the warp's share of a stage
      const int t0 = chunk * SCAN_TC, nt = min(SCAN_TC, len - t0);
#pragma unroll
      for (int b = 0; b < TB; ++b) {
        const int t = lw + (p + b) * (SCAN_LOADERS / 32);
        const size_t m = static_cast<size_t>(row0 + t0 + t);
#pragma unroll
        for (int i = 0; i < CH; ++i) {
          const int c = i * 32 + lane;
          const bool ok = t < nt && c < a.dim;
          r.q[b][i] = ok ? gq[m * a.ldq + c] : zero;
          if (HAS_F) r.g[b][HAS_F ? i : 0] = ok ? gg[m * a.ldg + c] : 0.f;
          if (HAS_K) r.k[b][HAS_K ? i : 0] = ok ? gk[m * a.ldk + c] : zero;
        }
#pragma unroll
        for (int i = 0; i < CV; ++i) {
          const int c = i * 32 + lane;
          r.v[b][i] = t < nt && c < CW && c0 + c < a.vdim ? gv[m * a.ldv + c] : zero;
        }
      }
    };
    auto stage = [&](const Raw& r, int buf, int p) {    // gates of those tokens -> shared memory
#pragma unroll
      for (int b = 0; b < TB; ++b) {
        const int at = buf * SCAN_TC + lw + (p + b) * (SCAN_LOADERS / 32);
        float bsum = 0.f;
#pragma unroll
        for (int i = 0; i < CH; ++i) {
          const int c = i * 32 + lane;
          float q, f, k, bo;
          scan_gates<MODE>(ld1(&r.q[b][i]), ld1(&r.k[b][HAS_K ? i : 0]), r.g[b][HAS_F ? i : 0] + bias[i], aux[i], q, f, k, bo);
          const bool ok = c < a.dim;                    // channels past dim leave the state at zero
          sq[at * DP + c] = ok ? q : 0.f;
          if (HAS_F) sf[at * DP + c] = ok ? f : (MODE == SCAN_HGRN2 ? 1.f : 0.f);
          if (HAS_K) sk[at * DP + c] = ok ? k : 0.f;
          if (MODE == SCAN_WKV) bsum += ok ? bo : 0.f;
        }
        if (MODE == SCAN_WKV) {
          bsum = lane_sum(bsum);
          if (lane == 0) sb[at] = bsum;
        }
#pragma unroll
        for (int i = 0; i < CV; ++i)
          if (i * 32 + lane < CW) sv[at * CW + i * 32 + lane] = MODE == SCAN_FIXED ? silu_f(ld1(&r.v[b][i])) : ld1(&r.v[b][i]);
      }
    };
    // two register sets: the next tokens are on their way while the current ones go through their gates
    Raw ra, rb;
    auto load = [&](int chunk, int buf) {
      static_assert(PER == 2 * TB, "two batches per stage");
      fetch(rb, chunk, TB);
      stage(ra, buf, 0);
      if (chunk + 1 < chunks) fetch(ra, chunk + 1, 0);
      stage(rb, buf, TB);
    };
    auto flush = [&](int chunk, int buf) {      // outputs of a finished stage -> global memory
      const int t0 = chunk * SCAN_TC, nt = min(SCAN_TC, len - t0);
      for (int i = lt; i < nt * CW; i += SCAN_LOADERS) {
        const int t = i / CW, c = i % CW;
        if (c0 + c < a.vdim)
          so.o[static_cast<size_t>(row0 + t0 + t) * so.ldo + h * a.vdim + c0 + c] = sout[(buf * SCAN_TC + t) * CW + c];
      }
    };
    fetch(ra, 0, 0);
    load(0, 0);
    stage_barrier<COMP + SCAN_LOADERS>();
    for (int ch = 0; ch < chunks; ++ch) {
      if (ch + 1 < chunks) load(ch + 1, (ch + 1) & 1);
      if (ch > 0) flush(ch - 1, (ch - 1) & 1);
      stage_barrier<COMP + SCAN_LOADERS>();
    }
    flush(chunks - 1, (chunks - 1) & 1);
    return;
  }

  // ------------------------------------------------------------------ compute warps
  const int rg = threadIdx.x & (SCAN_RG - 1), cg = threadIdx.x >> 3;
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.slot_stride + static_cast<size_t>(h) * a.vdim * a.ld_dim;
  const bool resume = slot >= 0 && a.ctx[seq] != len;
  const uint64_t minus1 = pack2(-1.f, -1.f);
  const float head_decay = MODE == SCAN_FIXED ? a.aux[h] : 0.f;
  const uint64_t fd = pack2(head_decay, head_decay);
  uint64_t S[CPT][NR / 2];
#pragma unroll
  for (int j = 0; j < CPT; ++j)
#pragma unroll
    for (int i = 0; i < NR / 4; ++i) {
      const int r = i * 32 + rg * 4, c = c0 + cg + NC * j;
      Pair2 p{0ull, 0ull};
      if (resume && r < a.ld_dim && c < a.vdim) p = *reinterpret_cast<const Pair2*>(sp + static_cast<size_t>(c) * a.ld_dim + r);
      S[j][2 * i] = p.lo;
      S[j][2 * i + 1] = p.hi;
    }
  stage_barrier<COMP + SCAN_LOADERS>();
  for (int ch = 0; ch < chunks; ++ch) {
    const int buf = ch & 1, nt = min(SCAN_TC, len - ch * SCAN_TC);
#pragma unroll 1
    for (int t4 = 0; t4 < nt; t4 += 4) {
      float part[CPT][4];
#pragma unroll
      for (int t = 0; t < 4; ++t) {
#pragma unroll
        for (int j = 0; j < CPT; ++j) part[j][t] = 0.f;
        if (t4 + t < nt) {                       // uniform for the CTA
          const int at = buf * SCAN_TC + t4 + t;
          const float* qp = sq + at * DP + rg * 4;
          const float* fp = sf + at * DP + rg * 4;
          const float* kp = sk + at * DP + rg * 4;
          uint64_t v2[CPT], o0[CPT], o1[CPT];
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            const float v = sv[at * CW + cg + NC * j];
            v2[j] = pack2(v, v);
            o0[j] = o1[j] = 0ull;
          }
#pragma unroll
          for (int i = 0; i < NR / 4; ++i) {
            const Pair2 q = *reinterpret_cast<const Pair2*>(qp + i * 32);
            Pair2 f{fd, fd}, k{0ull, 0ull};
            if (HAS_F) f = *reinterpret_cast<const Pair2*>(fp + i * 32);
            if (HAS_K) k = *reinterpret_cast<const Pair2*>(kp + i * 32);
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
              if (MODE == SCAN_HGRN2) {            // f S + (1 - f) v  =  f (S - v) + v
                S[j][2 * i] = fma2(f.lo, fma2(v2[j], minus1, S[j][2 * i]), v2[j]);
                S[j][2 * i + 1] = fma2(f.hi, fma2(v2[j], minus1, S[j][2 * i + 1]), v2[j]);
                o0[j] = fma2(q.lo, S[j][2 * i], o0[j]);
                o1[j] = fma2(q.hi, S[j][2 * i + 1], o1[j]);
              } else if (MODE == SCAN_FIXED) {
                S[j][2 * i] = fma2(f.lo, S[j][2 * i], mul2(k.lo, v2[j]));
                S[j][2 * i + 1] = fma2(f.hi, S[j][2 * i + 1], mul2(k.hi, v2[j]));
                o0[j] = fma2(q.lo, S[j][2 * i], o0[j]);
                o1[j] = fma2(q.hi, S[j][2 * i + 1], o1[j]);
              } else {
                o0[j] = fma2(q.lo, S[j][2 * i], o0[j]);
                o1[j] = fma2(q.hi, S[j][2 * i + 1], o1[j]);
                S[j][2 * i] = fma2(f.lo, S[j][2 * i], mul2(k.lo, v2[j]));
                S[j][2 * i + 1] = fma2(f.hi, S[j][2 * i + 1], mul2(k.hi, v2[j]));
              }
            }
          }
#pragma unroll
          for (int j = 0; j < CPT; ++j) {
            const float2 s = unpack2(add2(o0[j], o1[j]));
            part[j][t] = s.x + s.y;
            if (MODE == SCAN_WKV && rg == 0) part[j][t] = fmaf(unpack2(v2[j]).x, sb[at], part[j][t]);
          }
        }
      }
      // four partial sums of four tokens over the eight threads of a column: thread rg ends with token t4 + (rg & 3)
#pragma unroll
      for (int j = 0; j < CPT; ++j) {
#pragma unroll
        for (int half = 2; half >= 1; half >>= 1) {
          const bool up = rg & half;
#pragma unroll
          for (int x = 0; x < 2; ++x)
            if (x < half) {
              const float send = up ? part[j][x] : part[j][x + half];
              const float keep = up ? part[j][x + half] : part[j][x];
              part[j][x] = keep + __shfl_xor_sync(0xffffffffu, send, half);
            }
        }
        part[j][0] += __shfl_xor_sync(0xffffffffu, part[j][0], 4);
        if (rg < 4 && t4 + rg < nt) sout[(buf * SCAN_TC + t4 + rg) * CW + cg + NC * j] = part[j][0];
      }
    }
    stage_barrier<COMP + SCAN_LOADERS>();
  }
  if (slot >= 0) {
#pragma unroll
    for (int j = 0; j < CPT; ++j)
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const int r = i * 32 + rg * 4, c = c0 + cg + NC * j;
        if (r < a.ld_dim && c < a.vdim)
          *reinterpret_cast<Pair2*>(sp + static_cast<size_t>(c) * a.ld_dim + r) = Pair2{S[j][2 * i], S[j][2 * i + 1]};
      }
  }
}

template <int NR, int MODE, typename T>
__global__ void __launch_bounds__(256)
linear_decode_kernel(const ScanArgs a, const DecodeOut d) {
  constexpr int DP = SCAN_RG * NR;
  constexpr int CW = 32;                       // columns per pass
  __shared__ __align__(16) float sq[DP], sf[DP], sk[DP];
  __shared__ float sv[256], so[256];
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.x, m = blockIdx.y;    // row m holds sequence m's one token
  int slot = a.state_slot[m];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const bool fresh = a.ctx[m] == 1 || slot < 0;
  const int rg = threadIdx.x & (SCAN_RG - 1), col0 = threadIdx.x >> 3;
  float* base = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.slot_stride + static_cast<size_t>(h) * a.vdim * a.ld_dim;
  float bpart = 0.f;
  for (int i = threadIdx.x; i < DP; i += 256) {
    float q = 0.f, f = 1.f, k = 0.f, b = 0.f;           // channels past dim leave the state at zero
    if (i < a.dim) {
      const int c = h * a.dim + i;
      const float qr = take1(a.q, static_cast<size_t>(m) * a.ldq + c, a.qkv_kind);
      const float g = MODE != SCAN_FIXED ? take1(a.g, static_cast<size_t>(m) * a.ldg + c, a.g_kind) + a.bias[c] : 0.f;
      const float kr = MODE != SCAN_HGRN2 ? take1(a.k, static_cast<size_t>(m) * a.ldk + c, a.qkv_kind) : 0.f;
      scan_gates<MODE>(qr, kr, g, a.aux[MODE == SCAN_FIXED ? h : c], q, f, k, b);
    }
    sq[i] = q;
    sf[i] = f;
    sk[i] = k;
    bpart += b;
  }
  for (int j = threadIdx.x; j < a.vdim; j += 256) {
    const float v = take1(a.v, static_cast<size_t>(m) * a.ldv + h * a.vdim + j, a.qkv_kind);
    sv[j] = MODE == SCAN_FIXED ? silu_f(v) : v;
  }
  float bonus = 0.f;
  if (MODE == SCAN_WKV) bonus = cta_sum(bpart, red);
  __syncthreads();
  for (int c = col0; c - col0 < a.vdim; c += CW) {       // the same trip count for every thread
    float o = 0.f;
    if (c < a.vdim) {
      const float v = sv[c];
      float* sp = base + static_cast<size_t>(c) * a.ld_dim;
      float4 S[NR / 4];
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const int r = i * 32 + rg * 4;
        S[i] = (!fresh && r < a.ld_dim) ? *reinterpret_cast<const float4*>(sp + r) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int i = 0; i < NR / 4; ++i) {
        const int r = i * 32 + rg * 4;
        const float4 q = ld4(sq + r), f = ld4(sf + r), k = ld4(sk + r);
        if (MODE == SCAN_WKV) o += q.x * S[i].x + q.y * S[i].y + q.z * S[i].z + q.w * S[i].w;
        S[i].x = fmaf(f.x, S[i].x, k.x * v);
        S[i].y = fmaf(f.y, S[i].y, k.y * v);
        S[i].z = fmaf(f.z, S[i].z, k.z * v);
        S[i].w = fmaf(f.w, S[i].w, k.w * v);
        if (MODE != SCAN_WKV) o += q.x * S[i].x + q.y * S[i].y + q.z * S[i].z + q.w * S[i].w;
        if (slot >= 0 && r < a.ld_dim) *reinterpret_cast<float4*>(sp + r) = S[i];
      }
    }
#pragma unroll
    for (int x = 1; x < SCAN_RG; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
    if (rg == 0 && c < a.vdim) so[c] = MODE == SCAN_WKV ? fmaf(sv[c], bonus, o) : o;
  }
  __syncthreads();
  if (!d.w) {
    for (int j = threadIdx.x; j < a.vdim; j += 256) reinterpret_cast<float*>(d.out)[static_cast<size_t>(m) * d.ldo + h * a.vdim + j] = so[j];
    return;
  }
  float ss = 0.f;
  for (int j = threadIdx.x; j < a.vdim; j += 256) ss += so[j] * so[j];
  const float r = 1.f / sqrtf(cta_sum(ss, red) / a.vdim + d.eps);
  T* out = reinterpret_cast<T*>(d.out) + static_cast<size_t>(m) * d.ldo + h * d.vp;
  for (int j = threadIdx.x; j < d.vp; j += 256) {
    float y = 0.f;
    if (j < a.vdim) {
      y = so[j] * r * d.w[d.w_per_head ? h * a.vdim + j : j];
      if (d.gate) y *= silu_f(take1(d.gate, static_cast<size_t>(m) * d.ldgate + h * a.vdim + j, d.gate_kind));
    }
    st1(out + j, y);
  }
}

// rows per thread for a head of `dim` channels: instantiated multiples of four; 0: too large
static int scan_rows(int dim) { return dim <= 32 ? 4 : dim <= 64 ? 8 : dim <= 96 ? 12 : dim <= 128 ? 16 : dim <= 192 ? 24 : dim <= 256 ? 32 : 0; }

template <int NR, int MODE, int CPT, int NC, typename T>
static int launch_scan_slices(const ScanArgs& a, const ScanOut& o, int n_seqs, cudaStream_t st) {
  constexpr int CW = NC * CPT;
  const int smem = scan_smem<MODE>(SCAN_RG * NR, CW);
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(linear_scan_kernel<NR, MODE, CPT, NC, T>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = true;
  }
  const dim3 grid(a.H * ((a.vdim + CW - 1) / CW), n_seqs);
  return static_cast<int>(launch_kernel(linear_scan_kernel<NR, MODE, CPT, NC, T>, grid, dim3(SCAN_RG * NC + SCAN_LOADERS), smem, st, a, o));
}

// Width of the column slices: wide ones share operand reads and the loaders' work, narrow ones give a small batch more CTAs.
template <int NR, int MODE>
static int launch_scan(const ScanArgs& a, const ScanOut& o, int n_seqs, cudaStream_t st) {
  if (a.qkv_kind == ROW_F32) return launch_scan_slices<NR, MODE, 1, 16, float>(a, o, n_seqs, st);      // the 32-bit mode
  const long units = static_cast<long>(n_seqs) * a.H, sms = sm_count();
  if (NR <= 16 && a.vdim > 64 && units * ((a.vdim + 127) / 128) >= sms * 3 / 4)
    return launch_scan_slices<(NR <= 16 ? NR : 16), MODE, 4, 32, __nv_bfloat16>(a, o, n_seqs, st);
  if (a.vdim > 32 && units * ((a.vdim + 63) / 64) >= sms) return launch_scan_slices<NR, MODE, 4, 16, __nv_bfloat16>(a, o, n_seqs, st);
  if (a.vdim > 16 && units * ((a.vdim + 31) / 32) >= sms / 2) return launch_scan_slices<NR, MODE, 2, 16, __nv_bfloat16>(a, o, n_seqs, st);
  return launch_scan_slices<NR, MODE, 1, 16, __nv_bfloat16>(a, o, n_seqs, st);
}

}  // namespace artb

using namespace artb;

#define ARTB_BY_ROWS(NR_, CALL)  \
  switch (NR_) {                 \
    case 4: CALL(4); break;      \
    case 8: CALL(8); break;      \
    case 12: CALL(12); break;    \
    case 16: CALL(16); break;    \
    case 24: CALL(24); break;    \
    case 32: CALL(32); break;    \
    default: return ERR_TOO_LARGE; \
  }

static bool scan_args_ok(const ScanArgs& a, int mode) {
  return a.H > 0 && a.dim > 0 && a.vdim > 0 && a.vdim <= 256 && (a.ld_dim & 3) == 0 && a.ld_dim >= a.dim && (a.slot_stride & 3) == 0 &&
         !(reinterpret_cast<uintptr_t>(a.state) & 15) && a.q && a.v && a.aux && (mode == SCAN_FIXED || (a.g && a.bias)) &&
         (mode == SCAN_HGRN2 || a.k) && mode >= SCAN_HGRN2 && mode <= SCAN_FIXED &&
         a.cu_q && a.ctx && a.state_slot;
}

// Portions of n_seqs sequences (rows cu_q[i] .. cu_q[i + 1] - 1); o fp32 [rows, ldo] gets H * vdim columns.
// q, k, v bf16 or fp32, g fp32; not ROW_F32_TAKE (several CTAs read them).
ARTB_EXPORT int artb_linear_scan(int mode, void* q, int ldq, void* k, int ldk, void* v, int ldv, int qkv_kind, void* g, int ldg,
                                 int g_kind, const float* bias, const float* aux, float* state, long slot_stride, int ld_dim,
                                 long num_slots, const int* cu_q, const int* ctx, const int* state_slot, int n_seqs, int H,
                                 int dim, int vdim, float* o, int ldo, int rows, int* status, cudaStream_t st) {
  if (n_seqs <= 0) return 0;
  const ScanArgs a{q, k, v, g, ldq, ldk, ldv, ldg, qkv_kind, g_kind, bias, aux, state, slot_stride, ld_dim, num_slots, cu_q, ctx,
                   state_slot, H, dim, vdim, status};
  if (!scan_args_ok(a, mode) || qkv_kind == ROW_F32_TAKE || (mode != SCAN_FIXED && g_kind != ROW_F32) || n_seqs > 65535 || ldo < H * vdim)
    return ERR_BAD_SHAPE;
  const ScanOut so{o, ldo, rows};
  const int nr = scan_rows(dim);
#define ARTB_SC(NR_)                                                              \
  return mode == SCAN_WKV     ? launch_scan<NR_, SCAN_WKV>(a, so, n_seqs, st)     \
         : mode == SCAN_FIXED ? launch_scan<NR_, SCAN_FIXED>(a, so, n_seqs, st)   \
                              : launch_scan<NR_, SCAN_HGRN2>(a, so, n_seqs, st)
  ARTB_BY_ROWS(nr, ARTB_SC)
#undef ARTB_SC
  return 0;
}

// One token of each of M sequences; out T [M, ldo] with vp >= vdim columns per head (padding zero), or fp32 without w.
ARTB_EXPORT int artb_linear_decode(int f32, int mode, void* q, int ldq, void* k, int ldk, void* v, int ldv, int qkv_kind, void* g,
                                   int ldg, int g_kind, const float* bias, const float* aux, float* state, long slot_stride,
                                   int ld_dim, long num_slots, const int* cu_q, const int* ctx, const int* state_slot, int M, int H,
                                   int dim, int vdim, const float* w, int w_per_head, void* gate, int ldgate, int gate_kind,
                                   void* out, int ldo, int vp, float eps, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  const ScanArgs a{q, k, v, g, ldq, ldk, ldv, ldg, qkv_kind, g_kind, bias, aux, state, slot_stride, ld_dim, num_slots, cu_q, ctx,
                   state_slot, H, dim, vdim, status};
  if (!scan_args_ok(a, mode) || M > 65535 || vp < vdim || ldo < H * (w ? vp : vdim) || !out) return ERR_BAD_SHAPE;
  const DecodeOut d{w, w_per_head, gate, ldgate, gate_kind, out, ldo, vp, eps};
  const dim3 grid(H, M);
  cudaError_t e = cudaSuccess;
#define ARTB_LD2(NR_, MODE_)                                                                                      \
  e = f32 ? launch_kernel(linear_decode_kernel<NR_, MODE_, float>, grid, dim3(256), 0, st, a, d)                   \
          : launch_kernel(linear_decode_kernel<NR_, MODE_, __nv_bfloat16>, grid, dim3(256), 0, st, a, d)
#define ARTB_LD(NR_)                                                                                              \
  if (mode == SCAN_WKV) ARTB_LD2(NR_, SCAN_WKV);                                                                   \
  else if (mode == SCAN_FIXED) ARTB_LD2(NR_, SCAN_FIXED);                                                          \
  else ARTB_LD2(NR_, SCAN_HGRN2)
  ARTB_BY_ROWS(scan_rows(dim), ARTB_LD)
#undef ARTB_LD
#undef ARTB_LD2
  return static_cast<int>(e);
}
