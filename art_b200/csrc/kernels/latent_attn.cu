// Latent attention over a paged cache of latents.
//
// A token's cache row is [ c: rank_p | rotated key part: rot_p ] (both padded to a multiple of 16 with zeros): the latent
// that every head expands into its keys and values, and one rotated key part that all heads share.  Position i sees the
// keys j with 0 <= i - j < window.
//
//   latent_finish_kernel   what follows the q | latent projection, one CTA per token: RMSNorm of the latent, rotation of the
//                          shared key part and of every head's rotated query part (angles reduced in fp64), cache write, and
//                          the queries in the layout the attention form of the row reads
//   latent_attend_kernel   attention in latent space ("absorbed" form): q~ = W_uk^T q per head is taken against the cached
//                          latents themselves, the weighted latents are expanded by W_uv afterwards.  Scalar fp32
//                          arithmetic: the 32-bit mode runs on it (bf16: latent_decode.cu, latent_prefill.cu).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "key_weights.cuh"
#include "row_io.cuh"

namespace artb {

struct LatentFinish {
  void* p;                  // [M, ldp] of kind `kind`: q (H heads of dim | rot) | latent (rank) | rotated part (rot)
  int ldp, kind;
  const float* w;           // latent norm weight [rank]
  const double* freq;       // angle of pair i of position p: p * freq[i], rot / 2 pairs
  float rot_scale;          // factor of sine and cosine
  int next;                 // a dimension's partner: its neighbour, or (0) rot / 2 dimensions further
  const int* pos;
  const int* slot;          // cache row of every token, < 0: not written
  void* cache;              // T [num_slots, ldc]
  int ldc;
  long num_slots;
  int n_abs;                // rows below n_abs go to the absorbed layout
  void* qn;                 // T [H][pitch][dim_p]
  void* qr;                 // T [H][pitch][rot_p]
  int pitch;
  void* qe;                 // T [M - n_abs][ldqe], heads of (dim_p + rot_p), padding zero
  int ldqe;
  int H, dim, dim_p, rot, rot_p, rank, rank_p;
  float eps;
  int* status;
};

// V neighbouring elements at a time (V = 4 when every size and offset allows it)
template <int V>
__device__ __forceinline__ void take_v(void* p, size_t off, int kind, float (&f)[V]) {
  if (V == 4) {
    const float4 v = take4(p, off, kind);
    f[0] = v.x, f[1 % V] = v.y, f[2 % V] = v.z, f[3 % V] = v.w;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = take1(p, off + i, kind);
  }
}
template <typename T, int V>
__device__ __forceinline__ void put_v(T* p, const float (&f)[V]) {
  if (V == 4) {
    st4(p, make_float4(f[0], f[1 % V], f[2 % V], f[3 % V]));
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) st1(p + i, f[i]);
  }
}

// W: elements per access of the unrotated parts; RW: of the rotated parts (whole pairs)
template <typename T, int W, int RW>
__global__ void __launch_bounds__(256) latent_finish_kernel(const LatentFinish a) {
  __shared__ float red[32];
  extern __shared__ float cs[];            // cos, sin of rot / 2 angles
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, tid = threadIdx.x, hp = a.rot >> 1, hq = a.dim + a.rot;
  float *cc = cs, *sn = cs + hp;
  const size_t row = static_cast<size_t>(m) * a.ldp;
  const int pk = peek_kind(a.kind);        // a workspace is cleared at the end
  for (int i = tid; i < hp; i += blockDim.x) {
    const float2 t = position_pair(a.pos[m], a.freq[i]);
    sn[i] = a.rot_scale * t.x;
    cc[i] = a.rot_scale * t.y;
  }
  int slot = a.slot[m];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  T* crow = reinterpret_cast<T*>(a.cache) + static_cast<size_t>(slot < 0 ? 0 : slot) * a.ldc;
  const bool absorbed = m < a.n_abs;
  const int he = a.dim_p + a.rot_p;
  T* erow = reinterpret_cast<T*>(a.qe) + static_cast<size_t>(absorbed ? 0 : m - a.n_abs) * a.ldqe;
  T* qn = reinterpret_cast<T*>(a.qn) + static_cast<size_t>(m) * a.dim_p;
  T* qr = reinterpret_cast<T*>(a.qr) + static_cast<size_t>(m) * a.rot_p;
  // unrotated query parts first: they wait for nothing
  const int du = a.dim / W;
  for (int j = tid; j < a.H * du; j += blockDim.x) {
    const int h = j / du, i = (j - h * du) * W;
    float x[W];
    take_v<W>(a.p, row + h * hq + i, pk, x);
    put_v(absorbed ? qn + static_cast<size_t>(h) * a.pitch * a.dim_p + i : erow + h * he + i, x);
  }
  // latent: two passes over the row (the second finds it in L1 / L2)
  const int c0 = a.H * hq;
  float ss = 0.f;
  for (int i = tid * W; i < a.rank; i += blockDim.x * W) {
    float x[W];
    take_v<W>(a.p, row + c0 + i, pk, x);
#pragma unroll
    for (int e = 0; e < W; ++e) ss += x[e] * x[e];
  }
  const float r = 1.f / sqrtf(cta_sum(ss, red) / a.rank + a.eps);      // also the barrier behind cos / sin
  for (int i = tid * W; i < a.rank; i += blockDim.x * W) {
    float x[W];
    take_v<W>(a.p, row + c0 + i, pk, x);
#pragma unroll
    for (int e = 0; e < W; ++e) x[e] = x[e] * r * a.w[i + e];
    if (slot >= 0) put_v(crow + i, x);
  }
  // rotated parts: heads 0 .. H - 1 of the query, then the shared key part as "head" H
  auto rotated = [&](int h) {              // where its part goes, null: nowhere
    if (h < a.H) return absorbed ? qr + static_cast<size_t>(h) * a.pitch * a.rot_p : erow + h * he + a.dim_p;
    return slot >= 0 ? crow + a.rank_p : static_cast<T*>(nullptr);
  };
  if (!a.next) {                           // a unit: W neighbours and their partners half the dimensions further
    const int ru = hp / W;
    for (int j = tid; j < (a.H + 1) * ru; j += blockDim.x) {
      const int h = j / ru, i = (j - h * ru) * W;
      const size_t src = row + (h < a.H ? h * hq + a.dim : c0 + a.rank) + i;
      float x[W], z[W], y0[W], y1[W];
      take_v<W>(a.p, src, pk, x);
      take_v<W>(a.p, src + hp, pk, z);
#pragma unroll
      for (int e = 0; e < W; ++e) {
        y0[e] = x[e] * cc[i + e] - z[e] * sn[i + e];
        y1[e] = z[e] * cc[i + e] + x[e] * sn[i + e];
      }
      T* dst = rotated(h);
      if (dst) {
        put_v(dst + i, y0);
        put_v(dst + hp + i, y1);
      }
    }
  }
  const int ru = a.next ? a.rot / RW : 0;
  for (int j = tid; j < (a.H + 1) * ru; j += blockDim.x) {
    const int h = j / ru, i = (j - h * ru) * RW;
    float x[RW], y[RW];
    take_v<RW>(a.p, row + (h < a.H ? h * hq + a.dim : c0 + a.rank) + i, pk, x);
#pragma unroll
    for (int e = 0; e < RW; e += 2) {
      const float c = cc[(i + e) >> 1], s = sn[(i + e) >> 1];
      y[e] = x[e] * c - x[e + 1] * s;
      y[e + 1] = x[e + 1] * c + x[e] * s;
    }
    T* dst = rotated(h);
    if (dst) put_v(dst + i, y);
  }
  if (!absorbed) {
    const int np = he - a.dim - a.rot;       // padding columns of a head: behind the first part, behind the rotated part
    for (int j = tid; j < a.H * np; j += blockDim.x) {
      const int h = j / np, i = j - h * np;
      st1(erow + h * he + (i < a.dim_p - a.dim ? a.dim + i : a.dim + i + a.rot), 0.f);
    }
  }
  if (a.kind == ROW_F32_TAKE) {
    __syncthreads();
    for (int i = tid * W; i < c0 + a.rank + a.rot; i += blockDim.x * W) {
      if (W == 4) clear4(a.p, row + i, a.kind);
      else clear1(a.p, row + i, a.kind);
    }
  }
}

struct LatentAttend {
  const void* ql;           // T [H][pitch][rank_p]   queries in latent space
  const void* qr;           // T [H][pitch][rot_p]
  int pitch;
  const void* cache;        // T [num_blocks * block_size, ldc]
  int ldc;
  const int* block_table;
  int max_blocks, block_size;
  long num_blocks;
  const int* row_seq;
  const int* pos;           // position of the row's token
  const int* ctx;           // tokens of the sequence; 0: padding sequence
  int window;               // <= 0: every earlier key
  float scale;
  const float* sink;        // fp32 [H] sinks of the softmax, or null
  void* o;                  // T [H][pitch][rank_p]   weighted latents
  int rank_p, rot_p;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(128) latent_attend_kernel(const LatentAttend a) {
  constexpr int KT = 128;
  extern __shared__ float la_s[];
  float* sq = la_s;                          // [rank_p + rot_p]
  __shared__ float sp[KT];
  __shared__ long srow[KT];
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int D = a.rank_p + a.rot_p;
  const int seq = a.row_seq[m], p = a.pos[m];
  const int len = a.ctx[seq] > 0 ? p + 1 : 0;
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const size_t qo = static_cast<size_t>(h) * a.pitch + m;
  for (int i = tid; i < a.rank_p; i += 128) sq[i] = take1(const_cast<void*>(a.ql), qo * a.rank_p + i, sizeof(T) == 2 ? ROW_BF16 : ROW_F32);
  for (int i = tid; i < a.rot_p; i += 128) sq[a.rank_p + i] = take1(const_cast<void*>(a.qr), qo * a.rot_p + i, sizeof(T) == 2 ? ROW_BF16 : ROW_F32);
  constexpr int OV = 8;                      // up to 1024 latent dimensions
  float acc[OV];
#pragma unroll
  for (int i = 0; i < OV; ++i) acc[i] = 0.f;
  float mx = a.sink ? a.sink[h] : -INFINITY, sum = a.sink ? 1.f : 0.f;
  const T* cache = reinterpret_cast<const T*>(a.cache);
  for (int k0 = lo; k0 < len; k0 += KT) {
    __syncthreads();
    const int j = k0 + tid;
    float s = -INFINITY;
    long cr = -1;
    if (j < len) {
      const int blk = a.block_table[static_cast<size_t>(seq) * a.max_blocks + j / a.block_size];
      if (index_ok(blk, a.num_blocks, a.status)) {
        cr = static_cast<long>(blk) * a.block_size + j % a.block_size;
        const T* c = cache + cr * a.ldc;
        float t = 0.f;
        for (int i = 0; i < D; i += 4) {
          const float4 x = ld4(c + i);
          t = fmaf(x.x, sq[i], t);
          t = fmaf(x.y, sq[i + 1], t);
          t = fmaf(x.z, sq[i + 2], t);
          t = fmaf(x.w, sq[i + 3], t);
        }
        s = t * a.scale;
      }
    }
    float tm = s;
#pragma unroll
    for (int x = 16; x > 0; x >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, x));
    if ((tid & 31) == 0) red[tid >> 5] = tm;
    __syncthreads();
    tm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
    const float mn = fmaxf(mx, tm);
    if (mn == -INFINITY) continue;           // uniform: no usable key so far
    const float corr = mx == -INFINITY ? 0.f : expf(mx - mn);
    const float e = s == -INFINITY ? 0.f : expf(s - mn);
    mx = mn;
    sp[tid] = e;
    srow[tid] = cr;
    sum = sum * corr + cta_sum(e, red);      // barriers publish sp / srow
    const int nk = min(KT, len - k0);
#pragma unroll
    for (int i = 0; i < OV; ++i) {
      const int dcol = tid + i * 128;
      if (dcol < a.rank_p) {
        float t = acc[i] * corr;
        for (int k = 0; k < nk; ++k)
          if (srow[k] >= 0) t = fmaf(sp[k], take1(const_cast<void*>(a.cache), srow[k] * a.ldc + dcol, sizeof(T) == 2 ? ROW_BF16 : ROW_F32), t);
        acc[i] = t;
      }
    }
  }
  const float inv = sum > 0.f ? 1.f / sum : 0.f;
#pragma unroll
  for (int i = 0; i < OV; ++i) {
    const int dcol = tid + i * 128;
    if (dcol < a.rank_p) st1(reinterpret_cast<T*>(const_cast<void*>(static_cast<const void*>(a.o))) + qo * a.rank_p + dcol, acc[i] * inv);
  }
}

}  // namespace artb

using namespace artb;

ARTB_EXPORT int artb_latent_finish(int f32, void* p, int ldp, int kind, const float* w, const double* freq, float rot_scale, int next,
                                   const int* pos, const int* slot, void* cache, int ldc, long num_slots, int n_abs, void* qn, void* qr, int pitch,
                                   void* qe, int ldqe, int M, int H, int dim, int dim_p, int rot, int rot_p, int rank, int rank_p,
                                   float eps, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || (rot & 1) || (rot && !freq) || dim_p < dim || rot_p < rot || rank_p < rank || ldc < rank_p + rot_p) return ERR_BAD_SHAPE;
  if ((n_abs > 0 && (!qn || !qr || pitch < n_abs)) || (n_abs < M && (!qe || ldqe < H * (dim_p + rot_p)))) return ERR_BAD_SHAPE;
  const LatentFinish a{p, ldp, kind, w, freq, rot_scale, next, pos, slot, cache, ldc, num_slots, n_abs, qn, qr, pitch, qe, ldqe, H, dim, dim_p,
                       rot, rot_p, rank, rank_p, eps, status};
  const size_t smem = static_cast<size_t>(rot) * 4;
  const bool v4 = !((dim | rot | rank | ldp) & 3) && (next || !(rot & 7)) && !(reinterpret_cast<uintptr_t>(p) & 15);
#define ARTB_LF(T_, W_, R_) return static_cast<int>(launch_kernel(latent_finish_kernel<T_, W_, R_>, dim3(M), dim3(256), smem, st, a))
  if (f32) {
    if (v4) ARTB_LF(float, 4, 4);
    ARTB_LF(float, 1, 2);
  }
  if (v4) ARTB_LF(__nv_bfloat16, 4, 4);
  ARTB_LF(__nv_bfloat16, 1, 2);
#undef ARTB_LF
}

ARTB_EXPORT int artb_latent_attend(int f32, const void* ql, const void* qr, int pitch, const void* cache, int ldc,
                                   const int* block_table, int max_blocks, int block_size, long num_blocks, const int* row_seq,
                                   const int* pos, const int* ctx, int window, float scale, const float* sink, void* o, int M, int H,
                                   int rank_p, int rot_p, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || H > 65535 || rank_p > 1024 || (rank_p & 3) || (rot_p & 3) || (ldc & 3) || ldc < rank_p + rot_p || pitch < M ||
      block_size <= 0)
    return ERR_BAD_SHAPE;
  const LatentAttend a{ql, qr, pitch, cache, ldc, block_table, max_blocks, block_size, num_blocks, row_seq, pos, ctx, window, scale, sink,
                       o, rank_p, rot_p, status};
  const size_t smem = static_cast<size_t>(rank_p + rot_p) * 4;
  return static_cast<int>(f32 ? launch_kernel(latent_attend_kernel<float>, dim3(M, H), dim3(128), smem, st, a)
                              : launch_kernel(latent_attend_kernel<__nv_bfloat16>, dim3(M, H), dim3(128), smem, st, a));
}
