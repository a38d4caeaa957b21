// Linear attention with a per-channel decay, carried in an fp32 state S [dim, vdim] per sequence and head.
//
//   SCAN_HGRN2   f = l + (1 - l) sigmoid(g + b), q = silu(q);   S = f S + (1 - f) v^T ;  o = S^T q        (reads after)
//   SCAN_WKV     w = exp(-exp(g + b));   o = (S + (u k) v^T)^T r ;  S = w S + k v^T                       (reads before)
//
// All of it is fp32 arithmetic on CUDA cores: a recurrence multiplies rounding errors, so its operands do not go through
// 16-bit tensor-core products.  The decay, the gates and the bonus are computed where they are used; q, k, v and g are
// the raw outputs of the projections.
//
// Two kernels share the state layout [slot][head][vdim][ld_dim] (a column of S is contiguous):
//
//   linear_scan_kernel     portions of prompts.  A CTA owns (sequence, head, a slice of CW value columns) and walks over
//                          the portion.  The state lives in registers: eight threads share a column, each with NR of its
//                          rows (interleaved in groups of four, so that operands are 16-byte shared-memory reads without
//                          bank conflicts).  Four extra warps load the next 16 tokens and apply decay / gate functions
//                          while the others work on the current 16; the eight partial sums of eight tokens are reduced
//                          by a seven-step exchange instead of 24 shuffles.
//   linear_decode_kernel   one new token per sequence.  A CTA owns (sequence, head), streams the state through registers
//                          once (read, update, write) and finishes the head: RMSNorm over its vdim outputs, norm weight,
//                          optional silu gate, bf16 store.
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

enum ScanMode : int { SCAN_HGRN2 = 0, SCAN_WKV = 1 };

struct ScanArgs {
  void* q;      // q (hgrn2) or r (wkv): [M, ldq], kind qkv_kind
  void* k;      // wkv only
  void* v;
  void* g;      // decay projection, kind g_kind
  int ldq, ldk, ldv, ldg, qkv_kind, g_kind;
  const float* bias;    // [H * dim] added to g
  const float* aux;     // [H * dim] lower bound (hgrn2) or bonus u (wkv)
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
  float* o;             // fp32 [M, ldo] (linear_scan_kernel)
  int ldo;
};

struct DecodeOut {
  const float* w;       // norm weight [vdim] or [H * vdim]
  int w_per_head;
  void* gate;           // silu gate, kind gate_kind, or null
  int ldgate, gate_kind;
  void* out;            // T [M, ldo], vp columns per head
  int ldo, vp;
  float eps;
};

__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

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
constexpr int scan_arrays() { return MODE == SCAN_WKV ? 3 : 2; }
template <int MODE>
constexpr int scan_smem(int DP, int cw) {
  return 2 * SCAN_TC * (scan_arrays<MODE>() * DP + 2 * cw + 1) * 4;
}

// decay, gate and raw values of channel i of one token; channels past dim leave the state at zero
template <int MODE>
__device__ __forceinline__ void scan_channel(const ScanArgs& a, int m, int h, int i, float& q, float& f, float& k, float& bonus) {
  q = 0.f;
  k = 0.f;
  bonus = 0.f;
  f = MODE == SCAN_HGRN2 ? 1.f : 0.f;
  if (i >= a.dim) return;
  const int c = h * a.dim + i;
  const float qr = take1(a.q, static_cast<size_t>(m) * a.ldq + c, a.qkv_kind);
  const float g = take1(a.g, static_cast<size_t>(m) * a.ldg + c, a.g_kind) + a.bias[c];
  if (MODE == SCAN_HGRN2) {
    const float l = a.aux[c];
    q = silu_f(qr);
    f = l + (1.f - l) * sigmoid_f(g);
  } else {
    q = qr;
    f = expf(-expf(g));
    k = take1(a.k, static_cast<size_t>(m) * a.ldk + c, a.qkv_kind);
    bonus = q * a.aux[c] * k;
  }
}

template <int NR, int MODE>
__global__ void __launch_bounds__(SCAN_RG * 32 + SCAN_LOADERS)
linear_scan_kernel(const ScanArgs a, const ScanOut so, int cw) {
  constexpr int DP = SCAN_RG * NR;
  extern __shared__ __align__(16) float scan_s[];
  float* sq = scan_s;                                   // [2][TC][DP]
  float* sf = sq + 2 * SCAN_TC * DP;
  float* sk = sf + 2 * SCAN_TC * DP;                    // wkv only
  float* sv = sk + (MODE == SCAN_WKV ? 2 * SCAN_TC * DP : 0);   // [2][TC][cw]
  float* sout = sv + 2 * SCAN_TC * cw;                  // [2][TC][cw]
  float* sb = sout + 2 * SCAN_TC * cw;                  // [2][TC] bonus
  pdl_wait();
  pdl_launch_dependents();
  const int seq = blockIdx.y, h = blockIdx.x % a.H, c0 = (blockIdx.x / a.H) * cw;
  const int row0 = a.cu_q[seq], T = a.cu_q[seq + 1] - row0;
  if (T <= 0) return;
  int slot = a.state_slot[seq];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  const int n_comp = SCAN_RG * cw;
  const bool comp = static_cast<int>(threadIdx.x) < n_comp;
  const int lt = static_cast<int>(threadIdx.x) - n_comp, lane = threadIdx.x & 31;

  auto load = [&](int chunk, int buf) {       // loader warps: one token per warp at a time
    const int t0 = chunk * SCAN_TC, nt = min(SCAN_TC, T - t0);
    for (int t = lt >> 5; t < nt; t += SCAN_LOADERS / 32) {
      const int m = row0 + t0 + t, at = buf * SCAN_TC + t;
      float bsum = 0.f;
#pragma unroll
      for (int i0 = 0; i0 < DP; i0 += 32) {
        float q, f, k, b;
        const int i = i0 + lane;
        if (DP % 32 == 0 || i < DP) {
          scan_channel<MODE>(a, m, h, i, q, f, k, b);
          sq[at * DP + i] = q;
          sf[at * DP + i] = f;
          if (MODE == SCAN_WKV) {
            sk[at * DP + i] = k;
            bsum += b;
          }
        }
      }
      if (MODE == SCAN_WKV) {
        bsum = lane_sum(bsum);
        if (lane == 0) sb[at] = bsum;
      }
      for (int c = lane; c < cw; c += 32)
        sv[at * cw + c] = c0 + c < a.vdim ? take1(a.v, static_cast<size_t>(m) * a.ldv + h * a.vdim + c0 + c, a.qkv_kind) : 0.f;
    }
  };
  auto flush = [&](int chunk, int buf) {      // outputs of a finished stage -> global memory
    const int t0 = chunk * SCAN_TC, nt = min(SCAN_TC, T - t0);
    for (int i = lt; i < nt * cw; i += SCAN_LOADERS) {
      const int t = i / cw, c = i - t * cw;
      if (c0 + c < a.vdim)
        so.o[static_cast<size_t>(row0 + t0 + t) * so.ldo + h * a.vdim + c0 + c] = sout[(buf * SCAN_TC + t) * cw + c];
    }
  };

  const int rg = threadIdx.x & (SCAN_RG - 1), col = threadIdx.x >> 3;
  const bool live = comp && c0 + col < a.vdim;
  float* sp = a.state + static_cast<size_t>(slot < 0 ? 0 : slot) * a.slot_stride +
              (static_cast<size_t>(h) * a.vdim + c0 + col) * a.ld_dim;
  uint64_t S[NR / 2];
#pragma unroll
  for (int i = 0; i < NR / 2; ++i) S[i] = 0ull;
  if (live && slot >= 0 && a.ctx[seq] != T) {
#pragma unroll
    for (int i = 0; i < NR / 4; ++i) {
      const int r = i * 32 + rg * 4;
      if (r < a.ld_dim) {
        const Pair2 p = *reinterpret_cast<const Pair2*>(sp + r);
        S[2 * i] = p.lo;
        S[2 * i + 1] = p.hi;
      }
    }
  }

  const int chunks = (T + SCAN_TC - 1) / SCAN_TC;
  if (!comp) load(0, 0);
  __syncthreads();
  for (int ch = 0; ch < chunks; ++ch) {
    const int buf = ch & 1;
    if (comp) {
      const int nt = min(SCAN_TC, T - ch * SCAN_TC);
#pragma unroll 1
      for (int t8 = 0; t8 < nt; t8 += 8) {
        float part[8];
#pragma unroll
        for (int t = 0; t < 8; ++t) {
          part[t] = 0.f;
          if (t8 + t < nt) {                       // uniform for the CTA
            const int at = buf * SCAN_TC + t8 + t;
            const float v = sv[at * cw + col];
            const float* qp = sq + at * DP + rg * 4;
            const float* fp = sf + at * DP + rg * 4;
            const float* kp = sk + at * DP + rg * 4;
            const uint64_t v2 = pack2(v, v);
            uint64_t o0 = 0ull, o1 = 0ull;
#pragma unroll
            for (int i = 0; i < NR / 4; ++i) {
              const Pair2 q = *reinterpret_cast<const Pair2*>(qp + i * 32);
              const Pair2 f = *reinterpret_cast<const Pair2*>(fp + i * 32);
              if (MODE == SCAN_HGRN2) {            // f S + (1 - f) v  =  f (S - v) + v
                const uint64_t n2 = pack2(-v, -v);
                S[2 * i] = fma2(f.lo, add2(S[2 * i], n2), v2);
                S[2 * i + 1] = fma2(f.hi, add2(S[2 * i + 1], n2), v2);
                o0 = fma2(q.lo, S[2 * i], o0);
                o1 = fma2(q.hi, S[2 * i + 1], o1);
              } else {
                const Pair2 k = *reinterpret_cast<const Pair2*>(kp + i * 32);
                o0 = fma2(q.lo, S[2 * i], o0);
                o1 = fma2(q.hi, S[2 * i + 1], o1);
                S[2 * i] = fma2(f.lo, S[2 * i], mul2(k.lo, v2));
                S[2 * i + 1] = fma2(f.hi, S[2 * i + 1], mul2(k.hi, v2));
              }
            }
            const float2 s = unpack2(add2(o0, o1));
            part[t] = s.x + s.y;
            if (MODE == SCAN_WKV && rg == 0) part[t] = fmaf(v, sb[at], part[t]);
          }
        }
        // eight partial sums of eight tokens over the eight threads of a column: thread rg ends with token t8 + rg
#pragma unroll
        for (int half = 4; half >= 1; half >>= 1) {
          const bool up = rg & half;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if (j < half) {
              const float send = up ? part[j] : part[j + half];
              const float keep = up ? part[j + half] : part[j];
              part[j] = keep + __shfl_xor_sync(0xffffffffu, send, half);
            }
        }
        if (t8 + rg < nt) sout[(buf * SCAN_TC + t8 + rg) * cw + col] = part[0];
      }
    } else {
      if (ch + 1 < chunks) load(ch + 1, buf ^ 1);
      if (ch > 0) flush(ch - 1, buf ^ 1);
    }
    __syncthreads();
  }
  if (!comp) flush(chunks - 1, (chunks - 1) & 1);
  if (live && slot >= 0) {
#pragma unroll
    for (int i = 0; i < NR / 4; ++i) {
      const int r = i * 32 + rg * 4;
      if (r < a.ld_dim) *reinterpret_cast<Pair2*>(sp + r) = Pair2{S[2 * i], S[2 * i + 1]};
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
    float q, f, k, b;
    scan_channel<MODE>(a, m, h, i, q, f, k, b);
    sq[i] = q;
    sf[i] = f;
    sk[i] = MODE == SCAN_WKV ? k : (i < a.dim ? 1.f - f : 0.f);
    bpart += b;
  }
  for (int j = threadIdx.x; j < a.vdim; j += 256) sv[j] = take1(a.v, static_cast<size_t>(m) * a.ldv + h * a.vdim + j, a.qkv_kind);
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
        if (MODE == SCAN_HGRN2) o += q.x * S[i].x + q.y * S[i].y + q.z * S[i].z + q.w * S[i].w;
        if (slot >= 0 && r < a.ld_dim) *reinterpret_cast<float4*>(sp + r) = S[i];
      }
    }
#pragma unroll
    for (int x = 1; x < SCAN_RG; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
    if (rg == 0 && c < a.vdim) so[c] = MODE == SCAN_WKV ? fmaf(sv[c], bonus, o) : o;
  }
  __syncthreads();
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

template <int NR, int MODE>
static int launch_scan(const ScanArgs& a, const ScanOut& o, int n_seqs, int cw, cudaStream_t st) {
  const int smem = scan_smem<MODE>(SCAN_RG * NR, cw);
  static int configured[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured[dev & 63] < smem) {
    cudaError_t e = cudaFuncSetAttribute(linear_scan_kernel<NR, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = smem;
  }
  const dim3 grid(a.H * ((a.vdim + cw - 1) / cw), n_seqs);
  return static_cast<int>(launch_kernel(linear_scan_kernel<NR, MODE>, grid, dim3(SCAN_RG * cw + SCAN_LOADERS), smem, st, a, o, cw));
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
         !(reinterpret_cast<uintptr_t>(a.state) & 15) && a.q && a.v && a.g && a.bias && a.aux && (mode != SCAN_WKV || a.k) &&
         a.cu_q && a.ctx && a.state_slot;
}

// Portions of n_seqs sequences (rows cu_q[i] .. cu_q[i + 1] - 1); o fp32 [M, ldo] gets H * vdim columns.
// Inputs must not be of kind ROW_F32_TAKE (several CTAs read them).
ARTB_EXPORT int artb_linear_scan(int mode, void* q, int ldq, void* k, int ldk, void* v, int ldv, int qkv_kind, void* g, int ldg,
                                 int g_kind, const float* bias, const float* aux, float* state, long slot_stride, int ld_dim,
                                 long num_slots, const int* cu_q, const int* ctx, const int* state_slot, int n_seqs, int H,
                                 int dim, int vdim, float* o, int ldo, int* status, cudaStream_t st) {
  if (n_seqs <= 0) return 0;
  const ScanArgs a{q, k, v, g, ldq, ldk, ldv, ldg, qkv_kind, g_kind, bias, aux, state, slot_stride, ld_dim, num_slots, cu_q, ctx,
                   state_slot, H, dim, vdim, status};
  if (!scan_args_ok(a, mode) || qkv_kind == ROW_F32_TAKE || g_kind == ROW_F32_TAKE || n_seqs > 65535 || ldo < H * vdim)
    return ERR_BAD_SHAPE;
  const ScanOut so{o, ldo};
  // column slices: as wide as 32 (the loaders' work is shared by more columns), narrower while CTAs are scarce
  int cw = vdim <= 8 ? 8 : vdim <= 16 ? 16 : 32;
  while (cw > 8 && static_cast<long>(n_seqs) * H * ((vdim + cw - 1) / cw) < sm_count() / 2) cw >>= 1;
  const int nr = scan_rows(dim);
#define ARTB_SC(NR_) return mode == SCAN_WKV ? launch_scan<NR_, SCAN_WKV>(a, so, n_seqs, cw, st) : launch_scan<NR_, SCAN_HGRN2>(a, so, n_seqs, cw, st)
  ARTB_BY_ROWS(nr, ARTB_SC)
#undef ARTB_SC
  return 0;
}

// One token of each of M sequences; out T [M, ldo] with vp >= vdim columns per head (padding zero).
ARTB_EXPORT int artb_linear_decode(int f32, int mode, void* q, int ldq, void* k, int ldk, void* v, int ldv, int qkv_kind, void* g,
                                   int ldg, int g_kind, const float* bias, const float* aux, float* state, long slot_stride,
                                   int ld_dim, long num_slots, const int* cu_q, const int* ctx, const int* state_slot, int M, int H,
                                   int dim, int vdim, const float* w, int w_per_head, void* gate, int ldgate, int gate_kind,
                                   void* out, int ldo, int vp, float eps, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  const ScanArgs a{q, k, v, g, ldq, ldk, ldv, ldg, qkv_kind, g_kind, bias, aux, state, slot_stride, ld_dim, num_slots, cu_q, ctx,
                   state_slot, H, dim, vdim, status};
  if (!scan_args_ok(a, mode) || M > 65535 || vp < vdim || ldo < H * vp || !w || !out) return ERR_BAD_SHAPE;
  const DecodeOut d{w, w_per_head, gate, ldgate, gate_kind, out, ldo, vp, eps};
  const dim3 grid(H, M);
  cudaError_t e = cudaSuccess;
#define ARTB_LD2(NR_, MODE_)                                                                                      \
  e = f32 ? launch_kernel(linear_decode_kernel<NR_, MODE_, float>, grid, dim3(256), 0, st, a, d)                   \
          : launch_kernel(linear_decode_kernel<NR_, MODE_, __nv_bfloat16>, grid, dim3(256), 0, st, a, d)
#define ARTB_LD(NR_)                                                                                              \
  if (mode == SCAN_WKV) ARTB_LD2(NR_, SCAN_WKV);                                                                   \
  else ARTB_LD2(NR_, SCAN_HGRN2)
  ARTB_BY_ROWS(scan_rows(dim), ARTB_LD)
#undef ARTB_LD
#undef ARTB_LD2
  return static_cast<int>(e);
}
