// Latent attention of single tokens on tensor cores: the absorbed form over the paged latent cache.
//
// All heads of a token read the same cache rows [ c: rank_p | rotated part: rot_p ], so the heads are the rows of the
// matrix products:  S = [q~ | q_rot] [c | k_rot]^T  and  O = P c  per tile of 32 or 64 keys, one load serving both.
// A CTA owns (token, up to 16 * MT heads, a part of the window) and has eight warps.  In the score product a warp takes
// half of the tile's keys and a quarter of the D channels, so that its query fragments stay in registers and every key
// element is read from shared memory once; the four partial scores are added in the softmax step, where a warp owns
// 2 * MT rows.  In the value product a warp takes a share of the latent columns (16 at a time, strided by eight warps).
// Tiles are double-buffered with bulk copies (one per key row); scores, softmax and accumulators are fp32.
//
// With several splits the partial (output, max, sum) triples go to a workspace and latent_merge_kernel combines them: a
// small batch then still covers the machine, although a window has few tiles.
#include <math.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "key_weights.cuh"
#include "mma_tile.cuh"

namespace artb {

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
  const float* sink;               // fp32 [H] sinks of the softmax, or null
  __nv_bfloat16* o;                // [H][pitch][rank_p]
  float* ws;                       // [M][H][splits][rank_p + 2]
  int splits, H, rank_p, rot_p;
  int* status;
};

// NP: pairs of 8-column tiles per warp (128 * NP >= rank_p); KS: 16-channel steps per quarter (64 * KS >= D); LD_KT: keys
// per tile (32 or 64); RANK, ROT: the sizes when they are known at compile time (addresses then fold into immediates: with
// runtime sizes the address arithmetic outnumbers the other instructions), 0: runtime
template <int MT, int NP, int KS, int LD_KT, int RANK, int ROT>
__global__ void __launch_bounds__(32 * LD_WARPS, LD_KT == 32 && KS < 17 ? 2 : 1) latent_decode_kernel(const LatentDecode a) {
  extern __shared__ __align__(16) uint8_t ld_smem[];
  const int rank_p = RANK ? RANK : a.rank_p, rot_p = RANK ? ROT : a.rot_p;
  const int D = rank_p + rot_p, LD = D + 8;
  constexpr int R = 16 * MT, LP = LD_KT + 8, RPW = R / LD_WARPS, NK = LD_KT / 32;
  __nv_bfloat16* sK = reinterpret_cast<__nv_bfloat16*>(ld_smem);        // [2][KT][LD]
  __nv_bfloat16* sP = sK + 2 * LD_KT * LD;                                // [R][LP]
  float* sS = reinterpret_cast<float*>(sP + R * LP);                      // [4][R][LP]  partial scores
  float* sCorr = sS + 4 * R * LP;                                         // [R] rescaling of the accumulators
  float* sM = sCorr + R;                                                  // [R] final maximum
  float* sL = sM + R;                                                     // [R] final sum
  __shared__ uint64_t full[2];

  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.y, h0 = blockIdx.x * R, split = blockIdx.z;      // head groups of a token run side by side
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3, jm = lane >> 3, rr = lane & 7;
  const int dq = warp & 3, kh = warp >> 2;
  const int seq = a.row_seq[m], p = a.pos[m];
  const int len = a.ctx[seq] > 0 ? p + 1 : 0;
  const int lo = a.window > 0 ? max(0, p - a.window + 1) : 0;
  const int tiles = len > lo ? (len - lo + LD_KT - 1) / LD_KT : 0;
  const int per = (tiles + a.splits - 1) / a.splits;
  const int t_lo = split * per, t_hi = min(tiles, t_lo + per);
  const int* bt = a.block_table + static_cast<size_t>(seq) * a.max_blocks;

  // A tile arrives as one bulk copy per key row, completion on the buffer's mbarrier; every warp issues an eighth of the
  // copies (a warp issues them one by one).  The rows are looked up in the block table one tile ahead, so that the copies
  // wait for nothing.  Keys past the end repeat the last one (finite values; their scores are masked).
  constexpr int PW = LD_KT / LD_WARPS;
  int blk = 0;
  auto key_of = [&](int tile) { return min(lo + tile * LD_KT + warp * PW + lane, len - 1); };
  auto look_up = [&](int tile) {
    if (lane < PW) blk = bt[key_of(tile) / a.block_size];
  };
  auto load_tile = [&](int tile, int buf) {
    if (lane < PW) {
      size_t row = 0;
      if (index_ok(blk, a.num_blocks, a.status)) row = static_cast<size_t>(blk) * a.block_size + key_of(tile) % a.block_size;
      bulk_load(sK + (buf * LD_KT + warp * PW + lane) * LD, a.cache + row * a.ldc, D * 2, &full[buf]);
    }
  };

  if (tid == 0) {
    mbar_init(&full[0], 1);
    mbar_init(&full[1], 1);
    fence_mbar_init();
    if (t_lo < t_hi) mbar_expect_tx(&full[0], LD_KT * D * 2);
  }
  __syncthreads();
  if (t_lo < t_hi) {
    look_up(t_lo);
    load_tile(t_lo, 0);
    look_up(t_lo + 1);
  }
  // query fragments of this warp's channels: steps dq * KS .. of the concatenated [q~ | q_rot]
  const int ks0 = dq * KS, ks_n = min(KS, (D >> 4) - ks0);              // may be <= 0 for the last quarters
  uint32_t qf[MT][KS][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int k = 0; k < KS; ++k)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int h = h0 + i * 16 + g + (e & 1) * 8, c = (ks0 + k) * 16 + 2 * t + (e >> 1) * 8;
        uint32_t v = 0;
        if (k < ks_n && h < a.H) {
          const size_t row = static_cast<size_t>(h) * a.pitch + m;
          v = c < rank_p ? *reinterpret_cast<const uint32_t*>(a.ql + row * rank_p + c)
                           : *reinterpret_cast<const uint32_t*>(a.qr + row * rot_p + (c - rank_p));
        }
        qf[i][k][e] = v;
      }

  float acc[MT][2 * NP][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < 2 * NP; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  float mrow[RPW], lrow[RPW];          // of rows warp * RPW + j, the same in every lane
#pragma unroll
  for (int j = 0; j < RPW; ++j) {
    const int h = h0 + warp * RPW + j;
    const bool sink = a.sink && split == 0 && h < a.H;      // counted by one split
    mrow[j] = sink ? a.sink[h] * KW_LOG2E : -INFINITY;
    lrow[j] = sink ? 1.f : 0.f;
  }

  for (int tile = t_lo; tile < t_hi; ++tile) {
    const int buf = (tile - t_lo) & 1, k0 = lo + tile * LD_KT;
    const bool landed = mbar_wait_timed(&full[buf], ((tile - t_lo) >> 1) & 1);
    if (!__syncthreads_and(landed)) {  // also: everyone is done with the other buffer
      if (tid == 0) atomicMax(a.status, ST_TIMEOUT_FULL);
      for (int i = 0; i < 2000; ++i) __nanosleep(1000);      // let a copy in flight land before shared memory is released
      return;                          // the same for every thread
    }
    if (tile + 1 < t_hi) {
      if (tid == 0) mbar_expect_tx(&full[buf ^ 1], LD_KT * D * 2);
      load_tile(tile + 1, buf ^ 1);
      look_up(tile + 2);
    }
    __syncwarp();                      // the matrix loads below are executed by whole warps
    const __nv_bfloat16* K = sK + buf * LD_KT * LD;
    float s[MT][2 * NK][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int j = 0; j < 2 * NK; ++j) s[i][j][0] = s[i][j][1] = s[i][j][2] = s[i][j][3] = 0.f;
    const __nv_bfloat16* kp = K + (kh * 16 * NK + (jm >> 1) * 8 + rr) * LD + ks0 * 16 + (jm & 1) * 8;
#pragma unroll
    for (int k = 0; k < KS; ++k)
      if (k < ks_n) {
#pragma unroll
        for (int n = 0; n < NK; ++n) {
          uint32_t b[4];
          ldmat_x4(b, kp + n * 16 * LD + k * 16);
#pragma unroll
          for (int i = 0; i < MT; ++i) {
            mma_bf16(s[i][2 * n], qf[i][k], b[0], b[1]);
            mma_bf16(s[i][2 * n + 1], qf[i][k], b[2], b[3]);
          }
        }
      }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int n = 0; n < 2 * NK; ++n)
#pragma unroll
        for (int e = 0; e < 2; ++e)
          *reinterpret_cast<float2*>(sS + (dq * R + i * 16 + g + 8 * e) * LP + kh * 16 * NK + n * 8 + 2 * t) =
              make_float2(s[i][n][2 * e], s[i][n][2 * e + 1]);
    __syncthreads();
#pragma unroll
    for (int j = 0; j < RPW; ++j) {
      const int row = warp * RPW + j;
      float x[NK], mx = mrow[j];
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        const int c = k * 32 + lane;
        const float* y = sS + row * LP + c;
        x[k] = ((y[0] + y[R * LP]) + (y[2 * R * LP] + y[3 * R * LP])) * a.scale_log2;
        if (k0 + c >= len) x[k] = -INFINITY;
        mx = fmaxf(mx, x[k]);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      // finite from here on: a visited tile has at least one key
      const float corr = exp2f(mrow[j] - mx);
      float sum = 0.f;
#pragma unroll
      for (int k = 0; k < NK; ++k) {
        const float p = exp2f(x[k] - mx);
        sum += p;
        sP[row * LP + k * 32 + lane] = __float2bfloat16(p);
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
      mrow[j] = mx;
      lrow[j] = lrow[j] * corr + sum;
      if (lane == 0) sCorr[row] = corr;
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const float c0 = sCorr[i * 16 + g], c1 = sCorr[i * 16 + g + 8];
      if (!__all_sync(0xffffffffu, c0 == 1.f && c1 == 1.f))      // most tiles raise no row's maximum
#pragma unroll
      for (int j = 0; j < 2 * NP; ++j) {
        acc[i][j][0] *= c0;
        acc[i][j][1] *= c0;
        acc[i][j][2] *= c1;
        acc[i][j][3] *= c1;
      }
    }
#pragma unroll
    for (int ks = 0; ks < LD_KT / 16; ++ks) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmat_x4(pf[i], sP + (i * 16 + (jm & 1) * 8 + rr) * LP + ks * 16 + (jm >> 1) * 8);
#pragma unroll
      for (int n = 0; n < NP; ++n) {
        const int col = (warp + n * LD_WARPS) * 16;
        if (col < rank_p) {           // uniform for the warp
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
  }
  if (lane == 0) {
#pragma unroll
    for (int j = 0; j < RPW; ++j) {
      sM[warp * RPW + j] = mrow[j];
      sL[warp * RPW + j] = lrow[j];
    }
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int r = i * 16 + g + 8 * e, h = h0 + r;
      if (h >= a.H) continue;
      const float l = sL[r], inv = l > 0.f ? 1.f / l : 0.f;
      float* w = a.ws + ((static_cast<size_t>(m) * a.H + h) * a.splits + split) * (rank_p + 2);
      __nv_bfloat16* o = a.o + (static_cast<size_t>(h) * a.pitch + m) * rank_p;
#pragma unroll
      for (int n = 0; n < NP; ++n) {
        const int col = (warp + n * LD_WARPS) * 16;
        if (col < rank_p) {
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
        w[rank_p] = sM[r];
        w[rank_p + 1] = l;
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

static size_t latent_decode_smem(int R, int D, int kt) {
  return 2ull * kt * (D + 8) * 2 + static_cast<size_t>(R) * (kt + 8) * 2 + 4ull * R * (kt + 8) * 4 + 3ull * R * 4;
}

template <int MT, int NP, int KS, int KT, int RANK = 0, int ROT = 0>
static int launch_latent_decode(const LatentDecode& a, int M, cudaStream_t st) {
  const size_t smem = latent_decode_smem(16 * MT, a.rank_p + a.rot_p, KT);
  if (smem > 226 * 1024) return ERR_TOO_LARGE;
  static size_t configured[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured[dev & 63] < smem) {
    cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<MT, NP, KS, KT, RANK, ROT>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = smem;
  }
  return static_cast<int>(launch_kernel(latent_decode_kernel<MT, NP, KS, KT, RANK, ROT>, dim3((a.H + 16 * MT - 1) / (16 * MT), M, a.splits),
                                        dim3(32 * LD_WARPS), smem, st, a));
}

}  // namespace artb

using namespace artb;

// Rows 0 .. M - 1 (single tokens; row m of every head-major operand).  ws: M * H * splits * (rank_p + 2) floats when
// splits > 1.  rank_p, rot_p multiples of 16; rank_p <= 1024.
ARTB_EXPORT int artb_latent_decode(const void* ql, const void* qr, int pitch, const void* cache, int ldc, const int* block_table,
                                   int max_blocks, int block_size, long num_blocks, const int* row_seq, const int* pos, const int* ctx,
                                   int window, float scale, const float* sink, void* o, float* ws, int splits, int M, int H, int rank_p, int rot_p,
                                   int* status, cudaStream_t st) {
  if (M <= 0) return 0;
  if (H <= 0 || (rank_p & 15) || (rot_p & 15) || rank_p <= 0 || (ldc & 7) || ldc < rank_p + rot_p || pitch < M || splits < 1 ||
      splits > 64 || (splits > 1 && !ws) || block_size <= 0)
    return ERR_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(ql) | reinterpret_cast<uintptr_t>(qr) | reinterpret_cast<uintptr_t>(cache)) & 15) return ERR_BAD_ALIGN;
  const LatentDecode a{reinterpret_cast<const __nv_bfloat16*>(ql), reinterpret_cast<const __nv_bfloat16*>(qr), pitch,
                       reinterpret_cast<const __nv_bfloat16*>(cache), ldc, block_table, max_blocks, block_size, num_blocks, row_seq, pos,
                       ctx, window, scale * KW_LOG2E, sink, reinterpret_cast<__nv_bfloat16*>(o), ws, splits, H, rank_p, rot_p,
                       status};
  const int D = rank_p + rot_p;
  if (M > 65535) return ERR_BAD_SHAPE;
  int e;
  if (rank_p == 512 && rot_p == 64)
    e = H > 16 ? launch_latent_decode<2, 4, 9, 64, 512, 64>(a, M, st) : launch_latent_decode<1, 4, 9, 32, 512, 64>(a, M, st);
  else if (rank_p <= 128 && D <= 192) e = launch_latent_decode<1, 1, 3, 32>(a, M, st);
  else if (rank_p <= 256 && D <= 320) e = launch_latent_decode<1, 2, 5, 32>(a, M, st);
  else if (rank_p <= 512 && D <= 576) 
    e = H > 16 ? launch_latent_decode<2, 4, 9, 64>(a, M, st) : launch_latent_decode<1, 4, 9, 32>(a, M, st);
  else if (D <= 1088) e = launch_latent_decode<1, 8, 17, 32>(a, M, st);
  else return ERR_TOO_LARGE;
  if (e || splits == 1) return e;
  return static_cast<int>(launch_kernel(latent_merge_kernel, dim3(M, H), dim3(128), 0, st, a));
}
