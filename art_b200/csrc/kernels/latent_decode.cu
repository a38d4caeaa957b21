// Latent attention of single tokens on tensor cores: the absorbed form over the paged latent cache.
//
// All heads of a token read the same cache rows [ c: rank_p | rotated part: rot_p ], so the heads are the rows of the
// matrix products:  S = [q~ | q_rot] [c | k_rot]^T  and  O = P c  per tile of 64 keys, one load of the tile serving both.
// A CTA owns (token, up to 16 * MT heads, a part of the window) and has eight warps: in the score product a warp takes
// eight of the tile's keys, in the value product a share of the latent columns (pairs of 8-column tiles, strided by
// eight warps).  Tiles are double-buffered with asynchronous copies; scores, softmax and accumulators are fp32.
//
// With several splits the partial (output, max, sum) triples go to a workspace and latent_merge_kernel combines them: a
// small batch then still covers the machine, although a window has few tiles.
#include <math.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "mma_tile.cuh"

namespace artb {

constexpr int LD_KT = 64;          // keys per tile
constexpr int LD_WARPS = 8;

struct LatentDecode {
  const __nv_bfloat16* ql;         // [H][pitch][rank_p]
  const __nv_bfloat16* qr;         // [H][pitch][rot_p]
  int pitch;
  const __nv_bfloat16* cache;      // [slots][ldc]
  int ldc;
  const int* block_table;
  int max_blocks, block_size;
  long num_blocks;
  const int* row_seq;
  const int* pos;
  const int* ctx;
  int window;
  float scale_log2;
  __nv_bfloat16* o;                // [H][pitch][rank_p]
  float* ws;                       // [M][H][splits][rank_p + 2]
  int splits, H, rank_p, rot_p;
  int* status;
};

// NP: pairs of 8-column tiles per warp (16 * 8 * NP >= rank_p)
template <int MT, int NP>
__global__ void __launch_bounds__(32 * LD_WARPS, 1) latent_decode_kernel(const LatentDecode a) {
  extern __shared__ __align__(16) uint8_t ld_smem[];
  const int D = a.rank_p + a.rot_p, LD = D + 8;
  constexpr int R = 16 * MT, LP = LD_KT + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(ld_smem);       // [R][LD]
  __nv_bfloat16* sK = sQ + R * LD;                                       // [2][KT][LD]
  __nv_bfloat16* sP = sK + 2 * LD_KT * LD;                               // [R][LP]
  float* sMax = reinterpret_cast<float*>(sP + R * LP);                   // [warps][R]
  float* sSum = sMax + LD_WARPS * R;                                     // [warps][R]

  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, h0 = blockIdx.y * R, split = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3, jm = lane >> 3, rr = lane & 7;
  const int seq = a.row_seq[m], p = a.pos[m];
  const int len = a.ctx[seq] > 0 ? p + 1 : 0;
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const int tiles = len > lo ? (len - lo + LD_KT - 1) / LD_KT : 0;
  const int per = (tiles + a.splits - 1) / a.splits;
  const int t_lo = split * per, t_hi = min(tiles, t_lo + per);
  const int vec = D >> 3;
  const int* bt = a.block_table + static_cast<size_t>(seq) * a.max_blocks;

  auto load_tile = [&](int tile, int buf) {
    const int k0 = lo + tile * LD_KT;
    for (int i = warp; i < LD_KT; i += LD_WARPS) {       // a warp copies a key's row
      const int j = k0 + i;
      bool ok = j < len;
      size_t s = 0;
      if (ok) {
        const int blk = bt[j / a.block_size];
        ok = index_ok(blk, a.num_blocks, a.status);
        s = static_cast<size_t>(blk) * a.block_size + j % a.block_size;
      }
      const __nv_bfloat16* src = a.cache + (ok ? s * a.ldc : 0);
      __nv_bfloat16* dst = sK + (buf * LD_KT + i) * LD;
      for (int c = lane; c < vec; c += 32) copy16_async(dst + c * 8, src + c * 8, ok);
    }
    copy_commit();
  };

  if (t_lo < t_hi) load_tile(t_lo, 0);
  for (int v = tid; v < R * vec; v += 32 * LD_WARPS) {
    const int r = v / vec, c = (v - r * vec) * 8;
    uint4 val = make_uint4(0, 0, 0, 0);
    if (h0 + r < a.H) {
      const size_t row = static_cast<size_t>(h0 + r) * a.pitch + m;
      val = c < a.rank_p ? *reinterpret_cast<const uint4*>(a.ql + row * a.rank_p + c)
                         : *reinterpret_cast<const uint4*>(a.qr + row * a.rot_p + (c - a.rank_p));
    }
    *reinterpret_cast<uint4*>(sQ + r * LD + c) = val;
  }

  float acc[MT][2 * NP][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < 2 * NP; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  float mrow[MT][2], lrow[MT][2];
#pragma unroll
  for (int i = 0; i < MT; ++i) mrow[i][0] = mrow[i][1] = -INFINITY, lrow[i][0] = lrow[i][1] = 0.f;

  for (int tile = t_lo; tile < t_hi; ++tile) {
    const int buf = (tile - t_lo) & 1;
    if (tile + 1 < t_hi) {
      load_tile(tile + 1, buf ^ 1);
      copy_wait<1>();
    } else {
      copy_wait<0>();
    }
    __syncthreads();
    const __nv_bfloat16* K = sK + buf * LD_KT * LD;
    // scores of this warp's eight keys; two k16 steps per K fragment load
    float s[MT][4];
#pragma unroll
    for (int i = 0; i < MT; ++i) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
    const __nv_bfloat16* kp = K + (warp * 8 + rr) * LD + jm * 8;
    const __nv_bfloat16* qp = sQ + ((jm & 1) * 8 + rr) * LD + (jm >> 1) * 8;
    int c = 0;
    for (; c + 32 <= D; c += 32) {
      uint32_t b[4];
      ldmat_x4(b, kp + c);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        uint32_t q0[4], q1[4];
        ldmat_x4(q0, qp + i * 16 * LD + c);
        ldmat_x4(q1, qp + i * 16 * LD + c + 16);
        mma_bf16(s[i], q0, b[0], b[1]);
        mma_bf16(s[i], q1, b[2], b[3]);
      }
    }
    if (c < D) {       // one step of 16 left: lanes 16..31 would address the row's padding, so they repeat the others'
      uint32_t b[4];
      ldmat_x4(b, K + (warp * 8 + rr) * LD + c + (jm & 1) * 8);
#pragma unroll
      for (int i = 0; i < MT; ++i) {
        uint32_t q0[4];
        ldmat_x4(q0, qp + i * 16 * LD + c);
        mma_bf16(s[i], q0, b[0], b[1]);
      }
    }
    const int k0 = lo + tile * LD_KT + warp * 8 + 2 * t;
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      float x0 = -INFINITY, x1 = -INFINITY;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const bool ok = k0 + j < len;
        s[i][j] = ok ? s[i][j] * a.scale_log2 : -INFINITY;
        s[i][2 + j] = ok ? s[i][2 + j] * a.scale_log2 : -INFINITY;
        x0 = fmaxf(x0, s[i][j]);
        x1 = fmaxf(x1, s[i][2 + j]);
      }
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 1));
      x0 = fmaxf(x0, __shfl_xor_sync(0xffffffffu, x0, 2));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 1));
      x1 = fmaxf(x1, __shfl_xor_sync(0xffffffffu, x1, 2));
      if (t == 0) {
        sMax[warp * R + i * 16 + g] = x0;
        sMax[warp * R + i * 16 + g + 8] = x1;
      }
    }
    __syncthreads();
    float corr[MT][2];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        float mx = mrow[i][e];
#pragma unroll
        for (int w = 0; w < LD_WARPS; ++w) mx = fmaxf(mx, sMax[w * R + i * 16 + g + 8 * e]);
        const float base = mx == -INFINITY ? 0.f : mx;
        corr[i][e] = exp2f(mrow[i][e] - base);
        mrow[i][e] = mx;
        const float p0 = exp2f(s[i][2 * e] - base), p1 = exp2f(s[i][2 * e + 1] - base);
        lrow[i][e] = lrow[i][e] * corr[i][e] + p0 + p1;
        *reinterpret_cast<uint32_t*>(sP + (i * 16 + g + 8 * e) * LP + warp * 8 + 2 * t) = pair_bf16(p0, p1);
      }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < 2 * NP; ++j) {
        acc[i][j][0] *= corr[i][0];
        acc[i][j][1] *= corr[i][0];
        acc[i][j][2] *= corr[i][1];
        acc[i][j][3] *= corr[i][1];
      }
#pragma unroll
    for (int ks = 0; ks < LD_KT / 16; ++ks) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmat_x4(pf[i], sP + (i * 16 + (jm & 1) * 8 + rr) * LP + ks * 16 + (jm >> 1) * 8);
#pragma unroll
      for (int n = 0; n < NP; ++n) {
        const int col = (warp + n * LD_WARPS) * 16;
        if (col < a.rank_p) {           // uniform for the warp
          uint32_t b[4];
          ldmat_x4_t(b, K + (ks * 16 + (jm & 1) * 8 + rr) * LD + col + (jm >> 1) * 8);
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            mma_bf16(acc[i][2 * n], pf[i], b[0], b[1]);
            mma_bf16(acc[i][2 * n + 1], pf[i], b[2], b[3]);
          }
        }
      }
    }
    __syncthreads();                    // before the next copies land in the buffer just read
  }
  // every warp has the row maxima; the sums are spread over the warps' keys
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float l = lrow[i][e];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if (t == 0) sSum[warp * R + i * 16 + g + 8 * e] = l;
    }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = i * 16 + g + 8 * e, h = h0 + r;
      float l = 0.f;
#pragma unroll
      for (int w = 0; w < LD_WARPS; ++w) l += sSum[w * R + r];
      if (h >= a.H) continue;
      const float inv = l > 0.f ? 1.f / l : 0.f;
      float* w = a.ws + ((static_cast<size_t>(m) * a.H + h) * a.splits + split) * (a.rank_p + 2);
      __nv_bfloat16* o = a.o + (static_cast<size_t>(h) * a.pitch + m) * a.rank_p;
#pragma unroll
      for (int n = 0; n < NP; ++n) {
        const int col = (warp + n * LD_WARPS) * 16;
        if (col < a.rank_p) {
#pragma unroll
          for (int k = 0; k < 2; ++k) {
            const int d = col + k * 8 + 2 * t;
            const float v0 = acc[i][2 * n + k][2 * e], v1 = acc[i][2 * n + k][2 * e + 1];
            if (a.splits == 1) {
              *reinterpret_cast<uint32_t*>(o + d) = pair_bf16(v0 * inv, v1 * inv);
            } else {
              *reinterpret_cast<float2*>(w + d) = make_float2(v0, v1);
            }
          }
        }
      }
      if (a.splits > 1 && warp == 0 && t == 0) {
        w[a.rank_p] = mrow[i][e];
        w[a.rank_p + 1] = l;
      }
    }
}

__global__ void __launch_bounds__(128) latent_merge_kernel(const LatentDecode a) {
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, h = blockIdx.y, W = a.rank_p + 2;
  const float* base = a.ws + (static_cast<size_t>(m) * a.H + h) * a.splits * W;
  float mx = -INFINITY;
  for (int s = 0; s < a.splits; ++s) mx = fmaxf(mx, base[s * W + a.rank_p]);
  float l = 0.f;
  if (mx != -INFINITY)
    for (int s = 0; s < a.splits; ++s) l += base[s * W + a.rank_p + 1] * exp2f(base[s * W + a.rank_p] - mx);
  const float inv = l > 0.f ? 1.f / l : 0.f;
  __nv_bfloat16* o = a.o + (static_cast<size_t>(h) * a.pitch + m) * a.rank_p;
  for (int d = threadIdx.x * 2; d < a.rank_p; d += 256) {
    float x = 0.f, y = 0.f;
    if (mx != -INFINITY)
      for (int s = 0; s < a.splits; ++s) {
        const float sc = exp2f(base[s * W + a.rank_p] - mx);
        const float2 v = *reinterpret_cast<const float2*>(base + s * W + d);
        x = fmaf(v.x, sc, x);
        y = fmaf(v.y, sc, y);
      }
    *reinterpret_cast<uint32_t*>(o + d) = pair_bf16(x * inv, y * inv);
  }
}

static size_t latent_decode_smem(int R, int D) {
  return static_cast<size_t>(R) * (D + 8) * 2 + 2ull * LD_KT * (D + 8) * 2 + static_cast<size_t>(R) * (LD_KT + 8) * 2 +
         2ull * LD_WARPS * R * 4;
}

template <int MT, int NP>
static int launch_latent_decode(const LatentDecode& a, int M, cudaStream_t st) {
  const size_t smem = latent_decode_smem(16 * MT, a.rank_p + a.rot_p);
  static size_t configured[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured[dev & 63] < smem) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = smem;
  }
  return static_cast<int>(launch_kernel(latent_decode_kernel<MT, NP>, dim3(M, (a.H + 16 * MT - 1) / (16 * MT), a.splits),
                                        dim3(32 * LD_WARPS), smem, st, a));
}

}  // namespace artb

using namespace artb;

// Rows 0 .. M - 1 (single tokens; row m of every head-major operand).  ws: M * H * splits * (rank_p + 2) floats when
// splits > 1.  rank_p, rot_p multiples of 16; rank_p <= 1024.
ARTB_EXPORT int artb_latent_decode(const void* ql, const void* qr, int pitch, const void* cache, int ldc, const int* block_table,
                                   int max_blocks, int block_size, long num_blocks, const int* row_seq, const int* pos, const int* ctx,
                                   int window, float scale, void* o, float* ws, int splits, int M, int H, int rank_p, int rot_p,
                                   int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || (rank_p & 15) || (rot_p & 15) || rank_p <= 0 || (ldc & 7) || ldc < rank_p + rot_p || pitch < M || splits < 1 ||
      splits > 64 || (splits > 1 && !ws) || block_size <= 0)
    return ERR_BAD_SHAPE;
  if (rank_p > 1024) return ERR_TOO_LARGE;
  if ((reinterpret_cast<uintptr_t>(ql) | reinterpret_cast<uintptr_t>(qr) | reinterpret_cast<uintptr_t>(cache)) & 15) return ERR_BAD_ALIGN;
  const LatentDecode a{reinterpret_cast<const __nv_bfloat16*>(ql), reinterpret_cast<const __nv_bfloat16*>(qr), pitch,
                       reinterpret_cast<const __nv_bfloat16*>(cache), ldc, block_table, max_blocks, block_size, num_blocks, row_seq, pos,
                       ctx, window, scale * 1.4426950408889634f, reinterpret_cast<__nv_bfloat16*>(o), ws, splits, H, rank_p, rot_p,
                       status};
  const bool wide = H > 16 && latent_decode_smem(32, rank_p + rot_p) <= 225 * 1024;
  if (!wide && latent_decode_smem(16, rank_p + rot_p) > 225 * 1024) return ERR_TOO_LARGE;
  const int np = (rank_p + 127) / 128;
  int e;
  if (wide) e = np <= 1 ? launch_latent_decode<2, 1>(a, M, st) : np <= 2 ? launch_latent_decode<2, 2>(a, M, st)
              : np <= 4 ? launch_latent_decode<2, 4>(a, M, st) : launch_latent_decode<2, 8>(a, M, st);
  else e = np <= 1 ? launch_latent_decode<1, 1>(a, M, st) : np <= 2 ? launch_latent_decode<1, 2>(a, M, st)
         : np <= 4 ? launch_latent_decode<1, 4>(a, M, st) : launch_latent_decode<1, 8>(a, M, st);
  if (e || splits == 1) return e;
  return static_cast<int>(launch_kernel(latent_merge_kernel, dim3(M, H), dim3(128), 0, st, a));
}
