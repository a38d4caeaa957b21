// Grouped-query attention over a paged cache with a key mask (window or chunk), value heads of their own size, optionally
// squashed scores, a bias by distance with sigmoid weights instead of a softmax (key_weights.cuh), a factor per row and head
// or per row and column.
//
// A token's cache row is [ keys of the Hkv heads: dk_p each | values of the Hkv heads: dv_p each ], padded with zeros.
//
//   gqa_finish_kernel    what follows the q | k | v projection, one CTA per token: biases, cache write, padded queries
//   gqa_finish_norm_kernel   the same with a norm over all heads of q, and of k, or over each head, a rotation of the first
//                        columns of every head (angles reduced in fp64, as for position vectors) and the heads' or columns'
//                        gates
//   gqa_finish_heads_kernel  a norm over each head and no rotation, heads of a power of two up to 128: in registers alone
//   gqa_gather_kernel    the cache rows a batch's portions see, contiguous: keys row by row, values transposed, as the
//                        tcgen05 kernel of latent_prefill_tc.cu wants them (sizes that do not suit it: latent_gather and
//                        latent_prefill)
//   gqa_decode_kernel    rows with few new tokens: a CTA owns (row, key head, split); the query heads of the key head are the
//                        rows of one m16 tile, four warps walk 32-key tiles through their own staging areas
//   gqa_attend_kernel    the same in scalar fp32 arithmetic, any sizes: the 32-bit mode runs on it
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "key_mask.cuh"
#include "key_weights.cuh"
#include "mma_tile.cuh"
#include "row_io.cuh"
#include "softcap.cuh"

namespace artb {

struct GqaFinish {
  void* p;                  // [M, ldp] of kind `kind`: q (H heads of dim) | k (Hkv heads of dim) | v (Hkv heads of vdim)
  int ldp, kind;
  const float* bias;        // fp32 over the same columns, or null
  const int* slot;          // cache row of every token, < 0: not written
  void* cache;              // T [num_slots, ldc]
  int ldc;
  long num_slots;
  void* q;                  // T [M, ldq], heads of dk_p
  int ldq;
  int H, Hkv, dim, dk_p, vdim, dv_p;      // Hkv = 0: q alone (keys and values are another layer's)
  int* status;
  // gqa_finish_norm_kernel alone
  const float *wq, *wk;     // fp32 norm weights over all heads of q and of k, or null; per_head: one head's, shared by all
  int per_head;             // a norm over each head instead
  const float* q_scale;     // fp32 [H] factor of every query head (per_head alone), or null
  float eps;
  const double* freq;       // angle of pair i of position p: p * freq[i], rot / 2 pairs
  float rot_scale;          // factor of sine and cosine
  int rot, next;            // rotated columns of a head; partner: the neighbour (next) or rot / 2 columns further
  const int* pos;
  float* gate;              // fp32 [M, H]: the sigmoid of the columns behind v, or null
  void* cols;               // T [M, ldcols], heads of colp: the H * vdim columns behind v, or null
  int ldcols, colp;
};

template <typename T, int V>
__global__ void __launch_bounds__(256) gqa_finish_kernel(const GqaFinish a) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x;
  int slot = a.slot[m];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  T* crow = reinterpret_cast<T*>(a.cache) + static_cast<size_t>(slot < 0 ? 0 : slot) * a.ldc;
  T* qrow = reinterpret_cast<T*>(a.q) + static_cast<size_t>(m) * a.ldq;
  const int nq = a.H * a.dim, nk = a.Hkv * a.dim, n = nq + nk + a.Hkv * a.vdim;
  for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
    float x[V];
    if (V == 4) {
      const float4 v = take4(a.p, static_cast<size_t>(m) * a.ldp + c, peek_kind(a.kind));
      x[0] = v.x, x[1 % V] = v.y, x[2 % V] = v.z, x[3 % V] = v.w;
    } else {
      x[0] = take1(a.p, static_cast<size_t>(m) * a.ldp + c, peek_kind(a.kind));
    }
#pragma unroll
    for (int e = 0; e < V; ++e)
      if (a.bias) x[e] += a.bias[c + e];
    T* dst;
    if (c < nq) {
      dst = qrow + c / a.dim * a.dk_p + c % a.dim;
    } else if (slot < 0) {
      continue;
    } else if (c < nq + nk) {
      dst = crow + (c - nq) / a.dim * a.dk_p + (c - nq) % a.dim;
    } else {
      dst = crow + a.Hkv * a.dk_p + (c - nq - nk) / a.vdim * a.dv_p + (c - nq - nk) % a.vdim;
    }
    if (V == 4) st4(dst, make_float4(x[0], x[1 % V], x[2 % V], x[3 % V]));
    else st1(dst, x[0]);
  }
  if (a.kind == ROW_F32_TAKE)
    for (int c = threadIdx.x * V; c < n; c += blockDim.x * V) {
      if (V == 4) clear4(a.p, static_cast<size_t>(m) * a.ldp + c, a.kind);
      else clear1(a.p, static_cast<size_t>(m) * a.ldp + c, a.kind);
    }
  const int np = a.dk_p - a.dim;
  for (int j = threadIdx.x; j < a.H * np; j += blockDim.x) st1(qrow + j / np * a.dk_p + a.dim + j % np, 0.f);
}

// n / d without a division, for n * d < 2^32
struct QuickDiv {
  unsigned d, m;
  static QuickDiv by(int d) { return {static_cast<unsigned>(d), d > 1 ? 0xffffffffu / d + 1 : 0u}; }
  __device__ __forceinline__ int operator()(int n) const { return d > 1 ? static_cast<int>(__umulhi(static_cast<unsigned>(n), m)) : n; }
};

template <typename T, int V>
__device__ __forceinline__ void put_vec(T* dst, const float (&y)[V]) {
  if (V == 4) st4(dst, make_float4(y[0], y[1 % V], y[2 % V], y[3 % V]));
  else st1(dst, y[0]);
}
template <int V>
__device__ __forceinline__ void get_vec(const float* src, float (&y)[V]) {
  if (V == 4) {
    const float4 v = ld4(src);
    y[0] = v.x, y[1 % V] = v.y, y[2 % V] = v.z, y[3 % V] = v.w;
  } else {
    y[0] = *src;
  }
}

// V = 4: dim, vdim and the projection's pitch are multiples of 4, rot of 8; everything 16-byte aligned
template <typename T, int V>
__global__ void __launch_bounds__(256, 5) gqa_finish_norm_kernel(const GqaFinish a, const QuickDiv by_dim, const QuickDiv by_vdim, const QuickDiv by_units) {
  extern __shared__ __align__(16) float gn_smem[];      // [nq + nk] columns times their norm weights, then cos [rot / 2], sin [rot / 2]
  __shared__ float red[2][8];
  constexpr int B = 4;                                  // loads of a thread in flight
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, tid = threadIdx.x;
  int slot = a.slot[m];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  T* crow = reinterpret_cast<T*>(a.cache) + static_cast<size_t>(slot < 0 ? 0 : slot) * a.ldc;
  T* qrow = reinterpret_cast<T*>(a.q) + static_cast<size_t>(m) * a.ldq;
  const int nq = a.H * a.dim, nqk = nq + a.Hkv * a.dim, n = nqk + a.Hkv * a.vdim, half = a.rot >> 1;
  const size_t row = static_cast<size_t>(m) * a.ldp;
  float *cosine = gn_smem + ((nqk + 3) & ~3), *sine = cosine + ((half + 3) & ~3);
  float ssq = 0.f, ssk = 0.f;
  const int n_cols = a.cols ? a.H * a.vdim : 0, pk = peek_kind(a.kind);
  for (int c0 = tid * V; c0 < n + n_cols; c0 += blockDim.x * V * B) {
    float x[B][V];
#pragma unroll
    for (int u = 0; u < B; ++u) {
      const int c = c0 + u * blockDim.x * V;
      if (c >= n + n_cols) continue;
      if (V == 4) {
        const float4 v = take4(a.p, row + c, pk);
        x[u][0] = v.x, x[u][1 % V] = v.y, x[u][2 % V] = v.z, x[u][3 % V] = v.w;
      } else {
        x[u][0] = take1(a.p, row + c, pk);
      }
    }
#pragma unroll
    for (int u = 0; u < B; ++u) {
      const int c = c0 + u * blockDim.x * V;
      if (c >= n + n_cols) continue;
      if (c >= n) {
        put_vec(reinterpret_cast<T*>(a.cols) + static_cast<size_t>(m) * a.ldcols + by_vdim(c - n) * (a.colp - a.vdim) + c - n, x[u]);
        continue;
      }
      float t[V];
      if (a.bias) {
        get_vec(a.bias + c, t);
#pragma unroll
        for (int e = 0; e < V; ++e) x[u][e] += t[e];
      }
      if (c >= nqk) {
        if (slot < 0) continue;
        const int hd = by_vdim(c - nqk);
        put_vec(crow + a.Hkv * a.dk_p + hd * (a.dv_p - a.vdim) + c - nqk, x[u]);
        continue;
      }
      const bool isq = c < nq;
      float s = 0.f;
#pragma unroll
      for (int e = 0; e < V; ++e) s = fmaf(x[u][e], x[u][e], s);
      ssq += isq ? s : 0.f;
      ssk += isq ? 0.f : s;
      const float* w = isq ? a.wq : a.wk;
      if (w && !a.per_head) {
        get_vec(w + (isq ? c : c - nq), t);
#pragma unroll
        for (int e = 0; e < V; ++e) x[u][e] *= t[e];
      }
      put_vec(gn_smem + c, x[u]);
    }
    if (a.kind == ROW_F32_TAKE) {
#pragma unroll
      for (int u = 0; u < B; ++u) {
        const int c = c0 + u * blockDim.x * V;
        if (c >= n + n_cols) continue;
        if (V == 4) clear4(a.p, row + c, a.kind);
        else clear1(a.p, row + c, a.kind);
      }
    }
  }
  if (a.gate)
    for (int h = tid; h < a.H; h += blockDim.x) a.gate[static_cast<size_t>(m) * a.H + h] = logistic_f(take1(a.p, row + n + h, a.kind));
  for (int i = tid; i < half; i += blockDim.x) {
    const float2 t = position_pair(a.pos[m], a.freq[i]);
    cosine[i] = a.rot_scale * t.y;
    sine[i] = a.rot_scale * t.x;
  }
  const int warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5;
  const int heads = slot < 0 ? a.H : a.H + a.Hkv;       // the heads of q, then those of k
  float rq = 1.f, rk = 1.f;
  if (a.per_head) {                                     // a warp norms a head where it lies
    __syncthreads();
    for (int hd = warp; hd < heads; hd += nw) {
      float* x = gn_smem + hd * a.dim;
      const float* w = hd < a.H ? a.wq : a.wk;
      float ss = 0.f;
      for (int c = lane * V; c < a.dim; c += 32 * V) {
        float y[V];
        get_vec(x + c, y);
#pragma unroll
        for (int e = 0; e < V; ++e) ss = fmaf(y[e], y[e], ss);
      }
      float r = 1.f / sqrtf(lane_sum(ss) / a.dim + a.eps);
      if (hd < a.H && a.q_scale) r *= a.q_scale[hd];
      for (int c = lane * V; c < a.dim; c += 32 * V) {
        float y[V], g[V];
        get_vec(x + c, y);
        get_vec(w + c, g);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] *= r * g[e];
        put_vec(x + c, y);
      }
    }
    __syncthreads();
  } else {
    ssq = lane_sum(ssq);
    ssk = lane_sum(ssk);
    if (lane == 0) red[0][warp] = ssq, red[1][warp] = ssk;
    __syncthreads();
    ssq = lane_sum(lane < nw ? red[0][lane] : 0.f);
    ssk = lane_sum(lane < nw ? red[1][lane] : 0.f);
    if (a.wq) rq = 1.f / sqrtf(ssq / nq + a.eps);
    if (a.wk) rk = 1.f / sqrtf(ssk / max(1, nqk - nq) + a.eps);
  }
  auto out = [&](int hd) { return hd < a.H ? qrow + hd * a.dk_p : crow + (hd - a.H) * a.dk_p; };
  // rotated columns, a unit being V pairs (halves) or the pairs of V columns (neighbours), then the others
  const int units = a.next ? a.rot / (V == 4 ? 4 : 2) : half / V;
  for (int j = tid; j < heads * units; j += blockDim.x) {
    const int hd = by_units(j), i = j - hd * units;
    const float r = hd < a.H ? rq : rk;
    const float* src = gn_smem + hd * a.dim;
    T* dst = out(hd);
    if (!a.next) {
      float x[V], z[V], c[V], s[V], y0[V], y1[V];
      get_vec(src + i * V, x);
      get_vec(src + half + i * V, z);
      get_vec(cosine + i * V, c);
      get_vec(sine + i * V, s);
#pragma unroll
      for (int e = 0; e < V; ++e) {
        y0[e] = (x[e] * c[e] - z[e] * s[e]) * r;
        y1[e] = (z[e] * c[e] + x[e] * s[e]) * r;
      }
      put_vec(dst + i * V, y0);
      put_vec(dst + half + i * V, y1);
    } else if (V == 4) {
      const float4 x = ld4(src + i * 4);
      const float2 c = *reinterpret_cast<const float2*>(cosine + i * 2), s = *reinterpret_cast<const float2*>(sine + i * 2);
      st4(dst + i * 4, make_float4((x.x * c.x - x.y * s.x) * r, (x.y * c.x + x.x * s.x) * r, (x.z * c.y - x.w * s.y) * r, (x.w * c.y + x.z * s.y) * r));
    } else {
      const float x = src[2 * i], z = src[2 * i + 1], c = cosine[i], s = sine[i];
      st1(dst + 2 * i, (x * c - z * s) * r);
      st1(dst + 2 * i + 1, (z * c + x * s) * r);
    }
  }
  if (a.rot < a.dim)
    for (int c = tid * V; c < heads * a.dim; c += blockDim.x * V) {
      const int hd = by_dim(c), d = c - hd * a.dim;
      if (d < a.rot) continue;
      float x[V];
      get_vec(gn_smem + c, x);
#pragma unroll
      for (int e = 0; e < V; ++e) x[e] *= hd < a.H ? rq : rk;
      put_vec(out(hd) + d, x);
    }
  const int np = a.dk_p - a.dim;
  for (int j = tid; j < a.H * np; j += blockDim.x) st1(qrow + j / np * a.dk_p + a.dim + j % np, 0.f);
}

// A warp takes 128 columns at a time, a lane four: a head is dim / 4 neighbouring lanes.
template <typename T>
__global__ void __launch_bounds__(256) gqa_finish_heads_kernel(const GqaFinish a, const QuickDiv by_vdim) {
  constexpr int B = 4;                                  // loads of a thread in flight
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, lane = threadIdx.x & 31, step = blockDim.x * 4;
  int slot = a.slot[m];
  if (slot >= 0 && !index_ok(slot, a.num_slots, a.status)) slot = -1;
  T* crow = reinterpret_cast<T*>(a.cache) + static_cast<size_t>(slot < 0 ? 0 : slot) * a.ldc;
  T* qrow = reinterpret_cast<T*>(a.q) + static_cast<size_t>(m) * a.ldq;
  T* grow = reinterpret_cast<T*>(a.cols) + static_cast<size_t>(a.cols ? m : 0) * a.ldcols;
  const int nq = a.H * a.dim, nqk = nq + a.Hkv * a.dim, n = nqk + a.Hkv * a.vdim, total = n + (a.cols ? a.H * a.vdim : 0);
  const size_t row = static_cast<size_t>(m) * a.ldp;
  const int pk = peek_kind(a.kind), shift = 31 - __clz(a.dim), d0 = (lane * 4) & (a.dim - 1);
  const float4 wq = ld4(a.wq + d0), wk = a.Hkv ? ld4(a.wk + d0) : wq;
  const float inv_dim = 1.f / a.dim;
  for (int c0 = (threadIdx.x - lane) * 4; c0 < total; c0 += step * B) {      // the same for a warp
    float4 x[B];
#pragma unroll
    for (int u = 0; u < B; ++u) {
      const int c = c0 + u * step + lane * 4;
      x[u] = c < total ? take4(a.p, row + c, pk) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
#pragma unroll
    for (int u = 0; u < B; ++u) {
      const int c = c0 + u * step + lane * 4;
      if (a.bias && c < n) {
        const float4 b = ld4(a.bias + c);
        x[u] = make_float4(x[u].x + b.x, x[u].y + b.y, x[u].z + b.z, x[u].w + b.w);
      }
      float ss = sq4(x[u]);
      for (int o = a.dim >> 3; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (c < nqk) {
        const int hd = c >> shift;
        const bool isq = hd < a.H;
        float r = rsqrtf(fmaf(ss, inv_dim, a.eps));
        if (isq && a.q_scale) r *= __ldg(a.q_scale + hd);
        const float4 w = isq ? wq : wk;
        x[u] = make_float4(x[u].x * r * w.x, x[u].y * r * w.y, x[u].z * r * w.z, x[u].w * r * w.w);
        if (isq) st4(qrow + hd * a.dk_p + d0, x[u]);
        else if (slot >= 0) st4(crow + (hd - a.H) * a.dk_p + d0, x[u]);
      } else if (c < n) {
        if (slot >= 0) st4(crow + a.Hkv * a.dk_p + by_vdim(c - nqk) * (a.dv_p - a.vdim) + c - nqk, x[u]);
      } else if (c < total) {
        st4(grow + by_vdim(c - n) * (a.colp - a.vdim) + c - n, x[u]);
      }
    }
    if (a.kind == ROW_F32_TAKE) {
#pragma unroll
      for (int u = 0; u < B; ++u) {
        const int c = c0 + u * step + lane * 4;
        if (c < total) clear4(a.p, row + c, a.kind);
      }
    }
  }
  const int np = a.dk_p - a.dim;
  for (int j = threadIdx.x; j < a.H * np; j += blockDim.x) st1(qrow + j / np * a.dk_p + a.dim + j % np, 0.f);
}

struct GqaGather {
  const __nv_bfloat16* cache;
  int ldc;
  const int* block_table;
  int max_blocks, block_size;
  long num_blocks;
  const int *seq_of, *key_off, *key_pos0, *key_cnt;
  int n_seqs, n_keys;
  __nv_bfloat16* k;         // [n_keys, kcols]
  __nv_bfloat16* vt;        // [vcols, n_keys]
  int kcols, vcols;         // multiples of 64
  int* status;
};

// blockIdx.x: 64 keys; blockIdx.y: 64 columns, the key columns first
__global__ void __launch_bounds__(256) gqa_gather_kernel(const GqaGather a) {
  __shared__ long src[64];
  __shared__ __align__(16) __nv_bfloat16 tile[64][72];
  const int k0 = blockIdx.x * 64, c0 = blockIdx.y * 64, tid = threadIdx.x;
  if (tid < 64) {
    const int r = k0 + tid;
    long s = -1;
    if (r < a.n_keys) {
      int lo = 0, hi = a.n_seqs - 1;
      while (lo < hi) {
        const int mid = (lo + hi + 1) >> 1;
        if (a.key_off[mid] <= r) lo = mid;
        else hi = mid - 1;
      }
      const int i = r - a.key_off[lo];
      if (i < a.key_cnt[lo]) {
        const int j = a.key_pos0[lo] + i;
        const int blk = a.block_table[static_cast<size_t>(a.seq_of[lo]) * a.max_blocks + j / a.block_size];
        if (index_ok(blk, a.num_blocks, a.status)) s = static_cast<long>(blk) * a.block_size + j % a.block_size;
      }
    }
    src[tid] = s;
  }
  __syncthreads();
  for (int v = tid; v < 512; v += 256) {
    const int r = v >> 3, c = (v & 7) * 8;
    const uint4 x = src[r] >= 0 ? *reinterpret_cast<const uint4*>(a.cache + src[r] * a.ldc + c0 + c) : make_uint4(0, 0, 0, 0);
    if (c0 < a.kcols) {
      if (k0 + r < a.n_keys) *reinterpret_cast<uint4*>(a.k + static_cast<size_t>(k0 + r) * a.kcols + c0 + c) = x;
    } else {
      *reinterpret_cast<uint4*>(&tile[r][c]) = x;
    }
  }
  if (c0 < a.kcols) return;
  __syncthreads();
  for (int v = tid; v < 512; v += 256) {
    const int c = v & 63, r = (v >> 6) * 8;          // eight keys of one column
    if (k0 + r >= a.n_keys) continue;                // n_keys is a multiple of 8
    __align__(16) __nv_bfloat16 y[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] = tile[r + i][c];
    *reinterpret_cast<uint4*>(a.vt + static_cast<size_t>(c0 - a.kcols + c) * a.n_keys + k0 + r) = *reinterpret_cast<const uint4*>(y);
  }
}

struct GqaAttend {
  const void* q;            // T [M, ldq], heads of dk_p
  int ldq;
  const void* cache;        // T [num_blocks * block_size, ldc]
  int ldc;
  const int* block_table;
  int max_blocks, block_size;
  long num_blocks;
  const int* row_seq;
  const int* pos;
  const int* ctx;           // tokens of the sequence; 0: padding sequence
  KeyMask mask;
  float scale, softcap;
  ScoreScale score;         // the same for base-2 exponents
  float out_scale;
  const float* gate;        // fp32 [M][ldg] factor per row and head, or null
  int ldg;
  int sigmoid;              // weights are sigmoids of score + bias, not a softmax
  DistanceBias bias;        // of every query head (sigmoid weights)
  const void* cols;         // T [M][ldcols] gate logits of the result's columns, heads of colp, or null
  int ldcols, colp;
  void* o;                  // T [M, ldo], heads of vp; padding columns zero
  int ldo, vp;
  float* ws;                // [M][H][splits][dv_p + 2]
  int splits;
  int H, Hkv, dk_p, vdim, dv_p;
  int* status;

  __device__ __forceinline__ float factor(int m, int h) const { return gate ? out_scale * gate[static_cast<size_t>(m) * ldg + h] : out_scale; }
};

constexpr int GD_KT = 32;   // keys per warp tile

template <int DK, int DV>
constexpr int gqa_decode_smem() { return (16 * (DK + 8) + 4 * GD_KT * (DK + 8 + DV + 8)) * 2 + 2 * 4 * 16 * 4; }

// SIG: sigmoid weights
template <int DK, int DV, bool SIG>
__global__ void __launch_bounds__(128) gqa_decode_kernel(const GqaAttend a) {
  constexpr int LK = DK + 8, LV = DV + 8, WARP_ELEMS = GD_KT * (LK + LV);
  static_assert(16 * DV * 4 <= WARP_ELEMS * 2, "a warp's accumulators must fit its staging area");
  extern __shared__ __align__(16) uint8_t gd_smem[];
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(gd_smem);      // [16][LK]
  __nv_bfloat16* sKV = sQ + 16 * LK;                                   // [4 warps][keys | values]
  float* sM = reinterpret_cast<float*>(sKV + 4 * WARP_ELEMS);          // [4][16] maxima, [4][16] sums
  pdl_wait();
  pdl_launch_dependents();
  const int G = a.H / a.Hkv, groups = (G + 15) / 16;
  const int m = blockIdx.x, hk = blockIdx.y / groups, g0 = (blockIdx.y % groups) * 16, split = blockIdx.z;
  const int ng = min(16, G - g0), h0 = hk * G + g0;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3, jm = lane >> 3, rr = lane & 7;
  const int seq = a.row_seq[m], p = a.pos[m];
  const int len = a.ctx[seq] > 0 ? p + 1 : 0, first = a.mask.first(p);
  const int* bt = a.block_table + static_cast<size_t>(seq) * a.max_blocks;
  const int bs_shift = (a.block_size & (a.block_size - 1)) == 0 ? 31 - __clz(a.block_size) : -1;
  const __nv_bfloat16* q = reinterpret_cast<const __nv_bfloat16*>(a.q) + static_cast<size_t>(m) * a.ldq;

  for (int v = tid; v < 16 * (DK / 8); v += 128) {
    const int r = v / (DK / 8), c = (v % (DK / 8)) * 8;
    uint4 val = make_uint4(0, 0, 0, 0);
    if (r < ng && c < a.dk_p) val = *reinterpret_cast<const uint4*>(q + (h0 + r) * a.dk_p + c);
    *reinterpret_cast<uint4*>(sQ + r * LK + c) = val;
  }
  __syncthreads();
  uint32_t qf[DK / 16][4];
#pragma unroll
  for (int ks = 0; ks < DK / 16; ++ks) ldmat_x4(qf[ks], sQ + ((jm & 1) * 8 + rr) * LK + ks * 16 + (jm >> 1) * 8);

  // the splits share [first, len) in whole tiles, the warps of a split take its tiles in turn
  const int tiles = (len - first + GD_KT - 1) / GD_KT, per = (tiles + a.splits - 1) / a.splits;
  const int tile_hi = min(tiles, (split + 1) * per);
  float acc[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float* tab[2];                                 // bias of the thread's two heads, and what it is far away
  float far[2];
  if (SIG) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      tab[e] = a.bias.head(h0 + min(g + 8 * e, ng - 1));
      far[e] = a.bias.last(tab[e]);
    }
  }
  __nv_bfloat16 *wK = sKV + warp * WARP_ELEMS, *wV = wK + GD_KT * LK;
  const __nv_bfloat16* kc = reinterpret_cast<const __nv_bfloat16*>(a.cache) + hk * a.dk_p;
  const __nv_bfloat16* vc = reinterpret_cast<const __nv_bfloat16*>(a.cache) + a.Hkv * a.dk_p + hk * a.dv_p;

  for (int tile = split * per + warp; tile < tile_hi; tile += 4) {
    const int k0 = first + tile * GD_KT;
    // lane i looks up key i of the tile, the copies take the row from it
    long my_row = -1;
    {
      const int kt = k0 + lane;
      if (kt < len) {
        const int blk = bt[bs_shift >= 0 ? kt >> bs_shift : kt / a.block_size];
        if (index_ok(blk, a.num_blocks, a.status))
          my_row = static_cast<long>(blk) * a.block_size + (bs_shift >= 0 ? kt & (a.block_size - 1) : kt % a.block_size);
      }
    }
    auto load = [&](__nv_bfloat16* dst, int ld, const __nv_bfloat16* src, int width, auto tag) {
      constexpr int W = decltype(tag)::value, CPR = W / 8, RPI = CPR >= 32 ? 1 : 32 / CPR;
      const int c = (lane % CPR) * 8;
#pragma unroll 4
      for (int r0 = 0; r0 < GD_KT; r0 += RPI) {
        const int r = r0 + lane / CPR;
        const long row = __shfl_sync(0xffffffffu, my_row, r);
        const bool ok = row >= 0 && c < width;
        copy16_async(dst + r * ld + c, src + (ok ? row * a.ldc + c : 0), ok);
      }
    };
    load(wK, LK, kc, a.dk_p, std::integral_constant<int, DK>());
    load(wV, LV, vc, a.dv_p, std::integral_constant<int, DV>());
    copy_commit();
    copy_wait<0>();
    __syncwarp();
    float s[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) s[i][j] = 0.f;
#pragma unroll
    for (int ks = 0; ks < DK / 16; ++ks)
#pragma unroll
      for (int np = 0; np < 2; ++np) {
        uint32_t b[4];
        ldmat_x4(b, wK + (np * 16 + (jm >> 1) * 8 + rr) * LK + ks * 16 + (jm & 1) * 8);
        mma_bf16(s[np * 2], qf[ks], b[0], b[1]);
        mma_bf16(s[np * 2 + 1], qf[ks], b[2], b[3]);
      }
    uint32_t pf[2][4];
    if (SIG) {
      const bool near = !a.bias.beyond(p, min(k0 + GD_KT, len) - 1);
#pragma unroll
      for (int e = 0; e < 2; ++e)
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (e == 1 && ng <= 8) {                       // rows without a head
            pf[i >> 1][(i & 1) * 2 + e] = 0;
            continue;
          }
          float w[2] = {s[i][2 * e], s[i][2 * e + 1]};
          const int kt = k0 + i * 8 + 2 * t;
          a.score(w[0], w[1]);
          w[0] += near ? a.bias.at(tab[e], p - kt) : far[e];
          w[1] += near ? a.bias.at(tab[e], p - kt - 1) : far[e];
          sigmoid_pair(w[0], w[1]);
          pf[i >> 1][(i & 1) * 2 + e] = pair_bf16(kt < len ? w[0] : 0.f, kt + 1 < len ? w[1] : 0.f);
        }
    } else {
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (e == 1 && ng <= 8) {                         // rows without a head
#pragma unroll
          for (int i = 0; i < 4; ++i) pf[i >> 1][(i & 1) * 2 + e] = 0;
          continue;
        }
        float mn = mx[e];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 2; ++j) {
            float& x = s[i][2 * e + j];
            x = k0 + i * 8 + 2 * t + j < len ? a.score(x) : -INFINITY;
            mn = fmaxf(mn, x);
          }
        mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 1));
        mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 2));
        const float ms = mn == -INFINITY ? 0.f : mn, corr = exp2f(mx[e] - ms);
        mx[e] = mn;
        float sum = 0.f;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float p0 = exp2f(s[i][2 * e] - ms), p1 = exp2f(s[i][2 * e + 1] - ms);
          sum += p0 + p1;
          pf[i >> 1][(i & 1) * 2 + e] = pair_bf16(p0, p1);
        }
        l[e] = l[e] * corr + sum;
#pragma unroll
        for (int i = 0; i < DV / 8; ++i) {
          acc[i][2 * e] *= corr;
          acc[i][2 * e + 1] *= corr;
        }
      }
    }
#pragma unroll
    for (int ks = 0; ks < 2; ++ks)
#pragma unroll
      for (int dp = 0; dp < DV / 16; ++dp) {
        uint32_t b[4];
        ldmat_x4_t(b, wV + (ks * 16 + (jm & 1) * 8 + rr) * LV + dp * 16 + (jm >> 1) * 8);
        mma_bf16(acc[dp * 2], pf[ks], b[0], b[1]);
        mma_bf16(acc[dp * 2 + 1], pf[ks], b[2], b[3]);
      }
    __syncwarp();
  }
  if (SIG) {                                           // nothing to rescale; the first part alone counts as the sum
#pragma unroll
    for (int e = 0; e < 2; ++e) mx[e] = 0.f, l[e] = split == 0 && warp == 0 && t == 0 ? 1.f : 0.f;
  }
  const auto cols = ColumnGate<__nv_bfloat16>::of(a.cols, a.ldcols, a.colp, a.vdim);
  auto warp_acc = [&](int w) { return reinterpret_cast<float*>(sKV + w * WARP_ELEMS); };
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
    l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
    if (t == 0) {
      sM[warp * 16 + g + 8 * e] = mx[e];
      sM[64 + warp * 16 + g + 8 * e] = l[e];
    }
#pragma unroll
    for (int i = 0; i < DV / 8; ++i)
      *reinterpret_cast<float2*>(warp_acc(warp) + (g + 8 * e) * DV + i * 8 + 2 * t) = make_float2(acc[i][2 * e], acc[i][2 * e + 1]);
  }
  __syncthreads();
  for (int idx = tid; idx < ng * a.vp; idx += 128) {
    const int r = idx / a.vp, d = idx % a.vp;
    float mm = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) mm = fmaxf(mm, sM[w * 16 + r]);
    float ls = 0.f, o = 0.f;
    if (mm != -INFINITY) {
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float sc = exp2f(sM[w * 16 + r] - mm);
        ls += sM[64 + w * 16 + r] * sc;
        o += warp_acc(w)[r * DV + d] * sc;
      }
    }
    if (a.splits == 1) {
      __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.o) + static_cast<size_t>(m) * a.ldo + (h0 + r) * a.vp;
      out[d] = __float2bfloat16(ls > 0.f ? o / ls * a.factor(m, h0 + r) * cols(m, h0 + r, d) : 0.f);
    } else {
      float* w = a.ws + ((static_cast<size_t>(m) * a.H + h0 + r) * a.splits + split) * (a.vp + 2);
      w[d] = o;
      if (d == 0) {
        w[a.vp] = mm;
        w[a.vp + 1] = ls;
      }
    }
  }
}

__global__ void __launch_bounds__(128) gqa_merge_kernel(const GqaAttend a) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, h = blockIdx.y;
  const auto cols = ColumnGate<__nv_bfloat16>::of(a.cols, a.ldcols, a.colp, a.vdim);
  const float* base = a.ws + (static_cast<size_t>(m) * a.H + h) * a.splits * (a.vp + 2);
  float mm = -INFINITY;
  for (int s = 0; s < a.splits; ++s) mm = fmaxf(mm, base[s * (a.vp + 2) + a.vp]);
  for (int d = threadIdx.x; d < a.vp; d += 128) {
    float ls = 0.f, o = 0.f;
    if (mm != -INFINITY)
      for (int s = 0; s < a.splits; ++s) {
        const float* w = base + s * (a.vp + 2);
        const float sc = exp2f(w[a.vp] - mm);
        ls += w[a.vp + 1] * sc;
        o += w[d] * sc;
      }
    reinterpret_cast<__nv_bfloat16*>(a.o)[static_cast<size_t>(m) * a.ldo + h * a.vp + d] = __float2bfloat16(ls > 0.f ? o / ls * a.factor(m, h) * cols(m, h, d) : 0.f);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) gqa_attend_kernel(const GqaAttend a) {
  constexpr int KT = 128, OV = 8;            // up to 1024 value columns
  extern __shared__ float ga_q[];            // [dk_p]
  __shared__ float sp[KT];
  __shared__ long srow[KT];
  __shared__ float red[32];
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, h = blockIdx.y, hk = h / (a.H / a.Hkv), tid = threadIdx.x;
  const int seq = a.row_seq[m], p = a.pos[m], len = a.ctx[seq] > 0 ? p + 1 : 0;
  const T* q = reinterpret_cast<const T*>(a.q) + static_cast<size_t>(m) * a.ldq + h * a.dk_p;
  for (int i = tid; i < a.dk_p; i += 128) ga_q[i] = ld1(q + i);
  float acc[OV];
#pragma unroll
  for (int i = 0; i < OV; ++i) acc[i] = 0.f;
  float mx = -INFINITY, sum = 0.f;
  const T* keys = reinterpret_cast<const T*>(a.cache) + hk * a.dk_p;
  const T* vals = reinterpret_cast<const T*>(a.cache) + a.Hkv * a.dk_p + hk * a.dv_p;
  for (int k0 = a.mask.first(p); k0 < len; k0 += KT) {
    __syncthreads();
    const int j = k0 + tid;
    float s = -INFINITY;
    long cr = -1;
    if (j < len) {
      const int blk = a.block_table[static_cast<size_t>(seq) * a.max_blocks + j / a.block_size];
      if (index_ok(blk, a.num_blocks, a.status)) {
        cr = static_cast<long>(blk) * a.block_size + j % a.block_size;
        const T* k = keys + cr * a.ldc;
        float d = 0.f;
        for (int i = 0; i < a.dk_p; i += 4) {
          const float4 x = ld4(k + i);
          d = fmaf(x.x, ga_q[i], d);
          d = fmaf(x.y, ga_q[i + 1], d);
          d = fmaf(x.z, ga_q[i + 2], d);
          d = fmaf(x.w, ga_q[i + 3], d);
        }
        s = d * a.scale;
        if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      }
    }
    float corr = 1.f, e;
    if (a.sigmoid) {
      e = s == -INFINITY ? 0.f : 1.f / (1.f + exp2f(-fmaf(s, KW_LOG2E, a.bias.at(a.bias.head(h), p - j))));
      sp[tid] = e;
      srow[tid] = cr;
      __syncthreads();
    } else {
      float tm = s;
#pragma unroll
      for (int x = 16; x > 0; x >>= 1) tm = fmaxf(tm, __shfl_xor_sync(0xffffffffu, tm, x));
      if ((tid & 31) == 0) red[tid >> 5] = tm;
      __syncthreads();
      tm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
      const float mn = fmaxf(mx, tm);
      if (mn == -INFINITY) continue;           // uniform: no usable key so far
      corr = mx == -INFINITY ? 0.f : expf(mx - mn);
      e = s == -INFINITY ? 0.f : expf(s - mn);
      mx = mn;
      sp[tid] = e;
      srow[tid] = cr;
      sum = sum * corr + cta_sum(e, red);      // its barriers publish sp / srow
    }
    const int nk = min(KT, len - k0);
#pragma unroll
    for (int i = 0; i < OV; ++i) {
      const int d = tid + i * 128;
      if (d < a.vdim) {
        float x = acc[i] * corr;
        for (int k = 0; k < nk; ++k)
          if (srow[k] >= 0) x = fmaf(sp[k], ld1(vals + srow[k] * a.ldc + d), x);
        acc[i] = x;
      }
    }
  }
  const float inv = a.sigmoid ? a.factor(m, h) : sum > 0.f ? a.factor(m, h) / sum : 0.f;
  const auto cols = ColumnGate<T>::of(a.cols, a.ldcols, a.colp, a.vdim);
  T* o = reinterpret_cast<T*>(a.o) + static_cast<size_t>(m) * a.ldo + h * a.vp;
#pragma unroll
  for (int i = 0; i < OV; ++i) {
    const int d = tid + i * 128;
    if (d < a.vp) st1(o + d, acc[i] * inv * cols(m, h, d));
  }
}

template <int DK, int DV, bool SIG>
static int launch_gqa_decode(const GqaAttend& a, int M, cudaStream_t st) {
  constexpr int smem = gqa_decode_smem<DK, DV>();
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(gqa_decode_kernel<DK, DV, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = true;
  }
  const int groups = (a.H / a.Hkv + 15) / 16;
  cudaError_t e = launch_kernel(gqa_decode_kernel<DK, DV, SIG>, dim3(M, a.Hkv * groups, a.splits), dim3(128), smem, st, a);
  if (e == cudaSuccess && a.splits > 1) e = launch_kernel(gqa_merge_kernel, dim3(M, a.H), dim3(128), 0, st, a);
  return static_cast<int>(e);
}

static bool gqa_ok(const GqaAttend& a, int M) {
  return a.H > 0 && a.H <= 65535 && a.Hkv > 0 && a.H % a.Hkv == 0 && a.block_size > 0 && a.ldc >= a.Hkv * (a.dk_p + a.dv_p) && a.vp >= a.vdim &&
         a.dv_p >= a.vp && a.ldo >= a.H * a.vp && a.ldq >= a.H * a.dk_p && (!a.sigmoid || (a.bias.tab && a.bias.n > 0)) &&
         (!a.cols || (a.colp >= a.vdim && a.ldcols >= a.H * a.colp - (a.colp - a.vdim)));
}

}  // namespace artb

using namespace artb;

ARTB_EXPORT int artb_gqa_finish(int f32, void* p, int ldp, int kind, const float* bias, const int* slot, void* cache, int ldc,
                                long num_slots, void* q, int ldq, int M, int H, int Hkv, int dim, int dk_p, int vdim, int dv_p,
                                int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || Hkv <= 0 || H % Hkv || dk_p < dim || dv_p < vdim || ldc < Hkv * (dk_p + dv_p) || ldq < H * dk_p || ((dk_p | dv_p | ldc | ldq) & 3))
    return ERR_BAD_SHAPE;
  const GqaFinish a{p, ldp, kind, bias, slot, cache, ldc, num_slots, q, ldq, H, Hkv, dim, dk_p, vdim, dv_p, status,
                    nullptr, nullptr, 0, nullptr, 0.f, nullptr, 1.f, 0, 0, nullptr, nullptr, nullptr, 0, 0};
  const bool v4 = !((dim | vdim | ldp) & 3) && !(reinterpret_cast<uintptr_t>(p) & 15);
#define ARTB_GF(T_, V_) return static_cast<int>(launch_kernel(gqa_finish_kernel<T_, V_>, dim3(M), dim3(256), 0, st, a))
  if (f32) {
    if (v4) ARTB_GF(float, 4);
    ARTB_GF(float, 1);
  }
  if (v4) ARTB_GF(__nv_bfloat16, 4);
  ARTB_GF(__nv_bfloat16, 1);
#undef ARTB_GF
}

// As artb_gqa_finish, with norms (wq, wk; per_head: over each head, q_scale its factor), the rotation of the first `rot` columns
// of every head of q and k, and gates: of the heads, or the column gates' logits (cols), one or the other; Hkv = 0: the
// projection holds q (and gate) columns alone and the cache is not touched.
ARTB_EXPORT int artb_gqa_finish_norm(int f32, void* p, int ldp, int kind, const float* bias, const int* slot, void* cache, int ldc,
                                     long num_slots, void* q, int ldq, int M, int H, int Hkv, int dim, int dk_p, int vdim, int dv_p,
                                     const float* wq, const float* wk, int per_head, const float* q_scale, float eps, const double* freq,
                                     float rot_scale, int rot, int next, const int* pos, float* gate, void* cols, int ldcols, int colp,
                                     int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || Hkv < 0 || (Hkv && H % Hkv) || dim <= 0 || vdim <= 0 || dk_p < dim || dv_p < vdim || (Hkv && ldc < Hkv * (dk_p + dv_p)) ||
      ldq < H * dk_p || ((dk_p | dv_p | ldc | ldq) & 3) || (rot & 1) || rot < 0 || rot > dim || (rot && (!freq || !pos)) ||
      ldp < H * dim + Hkv * (dim + vdim) + (gate ? H : cols ? H * vdim : 0) || (gate && cols) || (cols && (colp < vdim || ldcols < H * colp)) ||
      (per_head && (!wq || (Hkv && !wk))) || (q_scale && !per_head))
    return ERR_BAD_SHAPE;
  const GqaFinish a{p, ldp, kind, bias, slot, cache, ldc, num_slots, q, ldq, H, Hkv, dim, dk_p, vdim, dv_p, status,
                    wq, wk, per_head, q_scale, eps, freq, rot_scale, rot, next, pos, gate, cols, ldcols, colp};
  const size_t smem = (static_cast<size_t>((H + Hkv) * dim + 3) / 4 * 4 + (rot / 2 + 3) / 4 * 8) * 4;
  if (smem > 224 * 1024) return ERR_TOO_LARGE;
  const auto aligned = [](const void* x) { return !(reinterpret_cast<uintptr_t>(x) & 15); };
  const bool v4 = !((dim | vdim | ldp) & 3) && !(rot & 7) && aligned(p) && aligned(bias) && aligned(wq) && aligned(wk) &&
                  !((ldcols | colp) & 3) && aligned(cols);
  const QuickDiv by_dim = QuickDiv::by(dim), by_vdim = QuickDiv::by(vdim),
                 by_units = QuickDiv::by(rot ? (next ? rot / (v4 ? 4 : 2) : rot / 2 / (v4 ? 4 : 1)) : 1);
  if (per_head && !rot && v4 && !gate && dim <= 128 && !(dim & (dim - 1)))
    return static_cast<int>(f32 ? launch_kernel(gqa_finish_heads_kernel<float>, dim3(M), dim3(256), 0, st, a, by_vdim)
                                : launch_kernel(gqa_finish_heads_kernel<__nv_bfloat16>, dim3(M), dim3(256), 0, st, a, by_vdim));
#define ARTB_GN(T_, V_)                                                                                                        \
  do {                                                                                                                         \
    if (smem > 48 * 1024) {                                                                                                    \
      const cudaError_t e = cudaFuncSetAttribute(gqa_finish_norm_kernel<T_, V_>, cudaFuncAttributeMaxDynamicSharedMemorySize,  \
                                                 static_cast<int>(smem));                                                      \
      if (e != cudaSuccess) return static_cast<int>(e);                                                                        \
    }                                                                                                                          \
    return static_cast<int>(launch_kernel(gqa_finish_norm_kernel<T_, V_>, dim3(M), dim3(256), smem, st, a, by_dim, by_vdim,    \
                                          by_units));                                                                     \
  } while (0)
  if (f32) {
    if (v4) ARTB_GN(float, 4);
    ARTB_GN(float, 1);
  }
  if (v4) ARTB_GN(__nv_bfloat16, 4);
  ARTB_GN(__nv_bfloat16, 1);
#undef ARTB_GN
}

// k [n_keys, kcols] and vt [vcols, n_keys] of the gathered rows (see artb_latent_gather); kcols and vcols multiples of 64,
// n_keys a multiple of 8
ARTB_EXPORT int artb_gqa_gather(const void* cache, int ldc, const int* block_table, int max_blocks, int block_size, long num_blocks,
                                const int* seq_of, const int* key_off, const int* key_pos0, const int* key_cnt, int n_seqs, int n_keys,
                                void* k, void* vt, int kcols, int vcols, int* status, cudaStream_t st) {
  if (n_keys <= 0 || n_seqs <= 0) return 0;
  if ((ldc & 7) || (kcols & 63) || (vcols & 63) || (n_keys & 7) || kcols <= 0 || vcols <= 0 || ldc < kcols + vcols || block_size <= 0 ||
      (kcols + vcols) / 64 > 65535)
    return ERR_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(k) | reinterpret_cast<uintptr_t>(vt) | reinterpret_cast<uintptr_t>(cache)) & 15) return ERR_BAD_ALIGN;
  const GqaGather a{reinterpret_cast<const __nv_bfloat16*>(cache), ldc, block_table, max_blocks, block_size, num_blocks, seq_of, key_off,
                    key_pos0, key_cnt, n_seqs, n_keys, reinterpret_cast<__nv_bfloat16*>(k), reinterpret_cast<__nv_bfloat16*>(vt), kcols,
                    vcols, status};
  gqa_gather_kernel<<<dim3((n_keys + 63) / 64, (kcols + vcols) / 64), 256, 0, st>>>(a);
  return static_cast<int>(cudaGetLastError());
}

// sigmoid: weights sigmoid(score + bias) with bias fp32 [H][n_bias + 2 * DistanceBias::PAD]; cols: column gates (key_weights.cuh).
// Rows 0 .. M - 1, each its own query; bf16, dk_p and dv_p multiples of 8 up to 256.  splits > 1: ws fp32 [M * H * splits * (vp + 2)].
ARTB_EXPORT int artb_gqa_decode(const void* q, int ldq, const void* cache, int ldc, const int* block_table, int max_blocks,
                                int block_size, long num_blocks, const int* row_seq, const int* pos, const int* ctx, int window,
                                int chunk, float scale, float softcap, float out_scale, const float* gate, int ldg, int sigmoid,
                                const float* bias, int n_bias, const void* cols, int ldcols, int colp, void* o, int ldo, int vp, float* ws, int splits, int M, int H,
                                int Hkv, int dk_p, int vdim, int dv_p, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  const GqaAttend a{q, ldq, cache, ldc, block_table, max_blocks, block_size, num_blocks, row_seq, pos, ctx, {window, chunk}, scale, softcap,
                    ScoreScale::of(scale, softcap), out_scale, gate, ldg, sigmoid, {bias, n_bias}, cols, ldcols, colp, o, ldo, vp, ws, splits, H, Hkv, dk_p, vdim, dv_p, status};
  if (!gqa_ok(a, M) || ((dk_p | dv_p | ldc | ldq) & 7) || splits < 1 || splits > 65535 || (splits > 1 && !ws)) return ERR_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache)) & 15) return ERR_BAD_ALIGN;
#define ARTB_GD(K_, S_)                                               \
  do {                                                                \
    if (dv_p <= 64) return launch_gqa_decode<K_, 64, S_>(a, M, st);   \
    if (dv_p <= 128) return launch_gqa_decode<K_, 128, S_>(a, M, st); \
    if (dv_p <= 256) return launch_gqa_decode<K_, 256, S_>(a, M, st); \
    return ERR_TOO_LARGE;                                             \
  } while (0)
  if (sigmoid) {
    if (dk_p <= 64) ARTB_GD(64, true);
    if (dk_p <= 128) ARTB_GD(128, true);
    if (dk_p <= 256) ARTB_GD(256, true);
    return ERR_TOO_LARGE;
  }
  if (dk_p <= 64) ARTB_GD(64, false);
  if (dk_p <= 128) ARTB_GD(128, false);
  if (dk_p <= 256) ARTB_GD(256, false);
#undef ARTB_GD
  return ERR_TOO_LARGE;
}

ARTB_EXPORT int artb_gqa_attend(int f32, const void* q, int ldq, const void* cache, int ldc, const int* block_table, int max_blocks,
                                int block_size, long num_blocks, const int* row_seq, const int* pos, const int* ctx, int window,
                                int chunk, float scale, float softcap, float out_scale, const float* gate, int ldg, int sigmoid,
                                const float* bias, int n_bias, const void* cols, int ldcols, int colp, void* o, int ldo, int vp, int M, int H, int Hkv, int dk_p, int vdim, int dv_p, int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  const GqaAttend a{q, ldq, cache, ldc, block_table, max_blocks, block_size, num_blocks, row_seq, pos, ctx, {window, chunk}, scale, softcap,
                    ScoreScale::of(scale, softcap), out_scale, gate, ldg, sigmoid, {bias, n_bias}, cols, ldcols, colp, o, ldo, vp, nullptr, 1, H, Hkv, dk_p, vdim, dv_p, status};
  if (!gqa_ok(a, M) || ((dk_p | dv_p | ldc) & 3) || vp > 1024 || dk_p > 8192) return ERR_BAD_SHAPE;
  const size_t smem = static_cast<size_t>(dk_p) * 4;
  return static_cast<int>(f32 ? launch_kernel(gqa_attend_kernel<float>, dim3(M, H), dim3(128), smem, st, a)
                              : launch_kernel(gqa_attend_kernel<__nv_bfloat16>, dim3(M, H), dim3(128), smem, st, a));
}
