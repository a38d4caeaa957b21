// Latent attention of prompt portions: the expanded form.
//
//   latent_gather_kernel    the cache rows a portion's window reaches, page by page, into one contiguous row range per
//                           sequence (a GEMM then expands their latents into every head's keys and values)
//   latent_prefill_kernel   windowed flash attention for any sizes (whole 64-column blocks: latent_prefill_tc.cu); a head's key is [ expanded part: dk | rotated part: rot_p ], the
//                           rotated part coming from the gathered rows all heads share
// Without a rotated part, and with G query heads per key head, the same kernel is grouped-query attention.  Sigmoid weights
// with a bias by distance, sinks and column gates: key_weights.cuh.
//
// A CTA owns 128 query rows of one sequence and one head: four warps with 32 rows each, key tiles of 32, keys and values
// double-buffered with asynchronous copies.  Scores, softmax and accumulators are fp32; only the probabilities enter the
// value product as bf16.  Tiles outside every row's window are not visited, tiles inside every row's window are not masked.
#include <math.h>

#include "bounds_check.cuh"
#include "host_utils.h"
#include "key_mask.cuh"
#include "key_weights.cuh"
#include "mma_tile.cuh"
#include "softcap.cuh"

namespace artb {

constexpr int LP_BM = 128, LP_BN = 32, LP_WARPS = 4;

__global__ void latent_gather_kernel(const __nv_bfloat16* __restrict__ cache, int ldc, const int* __restrict__ block_table, int max_blocks,
                                     int block_size, long num_blocks, const int* __restrict__ seq_of, const int* __restrict__ key_off,
                                     const int* __restrict__ key_pos0, const int* __restrict__ key_cnt, int n_seqs, __nv_bfloat16* __restrict__ out,
                                     int n_keys, int* status) {
  const int vec = ldc >> 3;
  const long total = static_cast<long>(n_keys) * vec;
  for (long i = blockIdx.x * static_cast<long>(blockDim.x) + threadIdx.x; i < total; i += static_cast<long>(gridDim.x) * blockDim.x) {
    const int r = i / vec, c = static_cast<int>(i % vec) * 8;
    int lo = 0, hi = n_seqs - 1;              // the last sequence whose range starts at or before row r
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (key_off[mid] <= r) lo = mid;
      else hi = mid - 1;
    }
    if (r - key_off[lo] >= key_cnt[lo]) {      // rows between two sequences
      *reinterpret_cast<uint4*>(out + static_cast<size_t>(r) * ldc + c) = make_uint4(0, 0, 0, 0);
      continue;
    }
    const int j = key_pos0[lo] + r - key_off[lo];
    const int blk = block_table[static_cast<size_t>(seq_of[lo]) * max_blocks + j / block_size];
    if (!index_ok(blk, num_blocks, status)) continue;
    const size_t s = static_cast<size_t>(blk) * block_size + j % block_size;
    *reinterpret_cast<uint4*>(out + static_cast<size_t>(r) * ldc + c) = *reinterpret_cast<const uint4*>(cache + s * ldc + c);
  }
}

struct LatentPrefill {
  const __nv_bfloat16* q;        // [rows][ldq]: heads of (dk | rot_p)
  int ldq;
  const __nv_bfloat16* kv;       // [n_keys][ldkv]: keys of all heads (dk each), then values of all heads (dv each)
  int ldkv;
  const __nv_bfloat16* c;        // [n_keys][ldc]: gathered cache rows, the rotated part from column rank_p on
  int ldc, rank_p;
  const int* tile_seq;           // per query tile: index into key_off / key_pos0 / row arrays
  const int* tile_row;           // first query row of the tile (row of q)
  const int* row_end;            // per sequence: row after its last one
  const int* row_pos0;           // per sequence: position of row 0 of q if it belonged to the sequence (position - row)
  const int* key_off;            // per sequence: first gathered row
  const int* key_pos0;           // per sequence: position of that row
  KeyMask mask;
  ScoreScale score;
  float out_scale;               // multiplies the result
  const float* gate;             // [rows][ldg] factor per row and head, or null
  int ldg;
  const float* sink;             // fp32 [H] sinks of the softmax, or null
  DistanceBias bias;             // of every query head (sigmoid weights)
  ColumnGate<__nv_bfloat16> cols;
  __nv_bfloat16* o;              // [rows][ldo]: heads of vp columns
  int ldo, vp, vdim;
  int H, G, dk, dv, rot_p;       // G heads share a key head; dk, dv, rot_p multiples of 16
};

// DV: value columns held in registers (dv <= DV); SIG: sigmoid weights
template <int DV, bool SIG>
__global__ void __launch_bounds__(32 * LP_WARPS, DV <= 128 ? 2 : 1) latent_prefill_kernel(const LatentPrefill a) {
  extern __shared__ __align__(16) uint8_t lp_smem[];
  const int DQ = a.dk + a.rot_p, LQ = DQ + 8, LV = a.dv + 8;
  __nv_bfloat16* sQ = reinterpret_cast<__nv_bfloat16*>(lp_smem);        // [BM][LQ]
  __nv_bfloat16* sK = sQ + LP_BM * LQ;                                    // [2][BN][LQ]
  __nv_bfloat16* sV = sK + 2 * LP_BN * LQ;                                // [2][BN][LV]
  const int h = blockIdx.x, sq = a.tile_seq[blockIdx.y];
  const int r0 = a.tile_row[blockIdx.y], nrow = min(LP_BM, a.row_end[sq] - r0);
  const int p0 = r0 + a.row_pos0[sq], p1 = p0 + nrow - 1;                 // positions of the tile's first and last row
  const int kp0 = a.key_pos0[sq];
  const int lo = max(kp0, a.mask.first(p0));
  const int tiles = (p1 - lo) / LP_BN + 1;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int g = lane >> 2, t = lane & 3, jm = lane >> 3, rr = lane & 7;
  const __nv_bfloat16* kbase = a.kv + static_cast<size_t>(h / a.G) * a.dk;
  const __nv_bfloat16* vbase = a.kv + static_cast<size_t>(a.H / a.G) * a.dk + static_cast<size_t>(h / a.G) * a.dv;
  const __nv_bfloat16* rbase = a.c + a.rank_p;
  const int kv8 = a.dk >> 3, rv8 = a.rot_p >> 3, vv8 = a.dv >> 3, row8 = kv8 + rv8 + vv8;

  auto load_tile = [&](int tile, int buf) {
    const int k0 = lo + tile * LP_BN;
    for (int v = tid; v < LP_BN * row8; v += 32 * LP_WARPS) {
      const int i = v / row8, c = v - i * row8;
      const bool ok = k0 + i <= p1;
      const size_t kr = ok ? static_cast<size_t>(a.key_off[sq] + k0 + i - kp0) : 0;
      if (c < kv8) copy16_async(sK + (buf * LP_BN + i) * LQ + c * 8, kbase + kr * a.ldkv + c * 8, ok);
      else if (c < kv8 + rv8) copy16_async(sK + (buf * LP_BN + i) * LQ + c * 8, rbase + kr * a.ldc + (c - kv8) * 8, ok);
      else copy16_async(sV + (buf * LP_BN + i) * LV + (c - kv8 - rv8) * 8, vbase + kr * a.ldkv + (c - kv8 - rv8) * 8, ok);
    }
    copy_commit();
  };

  for (int v = tid; v < LP_BM * (kv8 + rv8); v += 32 * LP_WARPS) {
    const int i = v / (kv8 + rv8), c = v - i * (kv8 + rv8);
    copy16_async(sQ + i * LQ + c * 8, a.q + static_cast<size_t>(r0 + min(i, nrow - 1)) * a.ldq + static_cast<size_t>(h) * DQ + c * 8, i < nrow);
  }
  load_tile(0, 0);

  float acc[2][DV / 8][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < DV / 8; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[i][j][e] = 0.f;
  float mrow[2][2], lrow[2][2];
#pragma unroll
  for (int i = 0; i < 2; ++i) mrow[i][0] = mrow[i][1] = -INFINITY, lrow[i][0] = lrow[i][1] = 0.f;
  if (!SIG && a.sink) {                           // counted by one of the four lanes of a row
    const float sk = a.sink[h] * KW_LOG2E;
#pragma unroll
    for (int i = 0; i < 2; ++i) mrow[i][0] = mrow[i][1] = sk, lrow[i][0] = lrow[i][1] = t == 0 ? 1.f : 0.f;
  }
  const float* tab = SIG ? a.bias.head(h) : nullptr;
  const float far = SIG ? a.bias.last(tab) : 0.f;
  const int w0 = warp * 32;                       // first row of the warp inside the tile

  for (int tile = 0; tile < tiles; ++tile) {
    const int buf = tile & 1, k0 = lo + tile * LP_BN;
    if (tile + 1 < tiles) {
      load_tile(tile + 1, buf ^ 1);
      copy_wait<1>();
    } else {
      copy_wait<0>();
    }
    __syncthreads();
    // a row at p sees positions first(p) .. p, first() never falls: skip a tile no row of the warp sees
    const int wp0 = p0 + w0, wp1 = min(p0 + w0 + 31, p1);
    const bool any = w0 < nrow && k0 <= wp1 && k0 + LP_BN - 1 >= a.mask.first(wp0);
    if (any) {
      const __nv_bfloat16* K = sK + buf * LP_BN * LQ;
      float s[2][4][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) s[i][j][e] = 0.f;
      for (int c = 0; c < DQ; c += 16) {
        uint32_t qf[2][4], b[2][4];
#pragma unroll
        for (int i = 0; i < 2; ++i) ldmat_x4(qf[i], sQ + (w0 + i * 16 + (jm & 1) * 8 + rr) * LQ + c + (jm >> 1) * 8);
#pragma unroll
        for (int n = 0; n < 2; ++n) ldmat_x4(b[n], K + (n * 16 + (jm >> 1) * 8 + rr) * LQ + c + (jm & 1) * 8);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            mma_bf16(s[i][2 * n], qf[i], b[n][0], b[n][1]);
            mma_bf16(s[i][2 * n + 1], qf[i], b[n][2], b[n][3]);
          }
      }
      // no masking needed when every row of the warp sees the whole tile
      const bool inside = k0 + LP_BN - 1 <= wp0 && k0 >= a.mask.first(wp1);
      const bool near = SIG && !a.bias.beyond(wp0, k0 + LP_BN - 1);
      uint32_t pf[2][2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int p = p0 + w0 + i * 16 + g + 8 * e, first = a.mask.first(p);
          if (SIG) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              float w[2] = {s[i][j][2 * e], s[i][j][2 * e + 1]};
              const int kp = k0 + j * 8 + 2 * t;
              a.score(w[0], w[1]);
              w[0] += near ? a.bias.at(tab, p - kp) : far;
              w[1] += near ? a.bias.at(tab, p - kp - 1) : far;
              sigmoid_pair(w[0], w[1]);
              if (!inside) {
                if (kp > p || kp < first) w[0] = 0.f;
                if (kp + 1 > p || kp + 1 < first) w[1] = 0.f;
              }
              pf[i][j >> 1][(j & 1) * 2 + e] = pair_bf16(w[0], w[1]);
            }
            continue;
          }
          float mx = mrow[i][e];
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int k = 0; k < 2; ++k) {
              float& x = s[i][j][2 * e + k];
              const int kp = k0 + j * 8 + 2 * t + k;
              x = a.score(x);
              if (!inside && (kp > p || kp < first)) x = -INFINITY;
              mx = fmaxf(mx, x);
            }
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
          mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          const float base = mx == -INFINITY ? 0.f : mx;
          const float corr = exp2f(mrow[i][e] - base);
          mrow[i][e] = mx;
          float sum = 0.f;
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float q0 = exp2f(s[i][j][2 * e] - base), q1 = exp2f(s[i][j][2 * e + 1] - base);
            sum += q0 + q1;
            pf[i][j >> 1][(j & 1) * 2 + e] = pair_bf16(q0, q1);
          }
          lrow[i][e] = lrow[i][e] * corr + sum;
#pragma unroll
          for (int j = 0; j < DV / 8; ++j) {
            acc[i][j][2 * e] *= corr;
            acc[i][j][2 * e + 1] *= corr;
          }
        }
      const __nv_bfloat16* V = sV + buf * LP_BN * LV;
#pragma unroll
      for (int ks = 0; ks < 2; ++ks)
#pragma unroll
        for (int n = 0; n < DV / 16; ++n)
          if (n * 16 < a.dv) {                       // uniform
            uint32_t b[4];
            ldmat_x4_t(b, V + (ks * 16 + (jm & 1) * 8 + rr) * LV + n * 16 + (jm >> 1) * 8);
#pragma unroll
            for (int i = 0; i < 2; ++i) {
              mma_bf16(acc[i][2 * n], pf[i][ks], b[0], b[1]);
              mma_bf16(acc[i][2 * n + 1], pf[i][ks], b[2], b[3]);
            }
          }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float l = lrow[i][e];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      const int r = w0 + i * 16 + g + 8 * e;
      if (r >= nrow) continue;
      float inv = SIG ? a.out_scale : l > 0.f ? a.out_scale / l : 0.f;
      if (a.gate) inv *= a.gate[static_cast<size_t>(r0 + r) * a.ldg + h];
      __nv_bfloat16* o = a.o + static_cast<size_t>(r0 + r) * a.ldo + static_cast<size_t>(h) * a.vp;
#pragma unroll
      for (int n = 0; n < DV / 8; ++n) {
        const int d = n * 8 + 2 * t;
        if (d < a.vp)
          *reinterpret_cast<uint32_t*>(o + d) = pair_bf16(acc[i][n][2 * e] * inv * a.cols(r0 + r, h, d), acc[i][n][2 * e + 1] * inv * a.cols(r0 + r, h, d + 1));
      }
    }
}

static size_t latent_prefill_smem(int DQ, int dv) { return (static_cast<size_t>(LP_BM + 2 * LP_BN) * (DQ + 8) + 2ull * LP_BN * (dv + 8)) * 2; }

template <int DV, bool SIG>
static int launch_latent_prefill(const LatentPrefill& a, int n_tiles, cudaStream_t st) {
  const size_t smem = latent_prefill_smem(a.dk + a.rot_p, a.dv);
  if (smem > 225 * 1024) return ERR_TOO_LARGE;
  static size_t configured[64] = {0};
  int dev = 0;
  cudaGetDevice(&dev);
  if (configured[dev & 63] < smem) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_kernel<DV, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = smem;
  }
  latent_prefill_kernel<DV, SIG><<<dim3(a.H, n_tiles), 32 * LP_WARPS, smem, st>>>(a);
  return static_cast<int>(cudaGetLastError());
}

}  // namespace artb

using namespace artb;
typedef __nv_bfloat16 bf16;

// Gathered row r of sequence i (key_off[i] <= r < key_off[i] + key_cnt[i]) is position key_pos0[i] + r - key_off[i] of the
// sequence seq_of[i] of the block table; rows up to the next sequence (or n_keys) are zero.
ARTB_EXPORT int artb_latent_gather(const void* cache, int ldc, const int* block_table, int max_blocks, int block_size, long num_blocks,
                                   const int* seq_of, const int* key_off, const int* key_pos0, const int* key_cnt, int n_seqs, void* out, int n_keys,
                                   int* status, cudaStream_t st) {
  if (n_keys <= 0 || n_seqs <= 0) return 0;
  if ((ldc & 7) || block_size <= 0) return ERR_BAD_SHAPE;
  long blocks = (static_cast<long>(n_keys) * (ldc / 8) + 255) / 256;
  if (blocks > 148L * 16) blocks = 148L * 16;
  latent_gather_kernel<<<static_cast<unsigned>(blocks), 256, 0, st>>>((const bf16*)cache, ldc, block_table, max_blocks, block_size, num_blocks,
                                                                  seq_of, key_off, key_pos0, key_cnt, n_seqs, (bf16*)out, n_keys, status);
  return static_cast<int>(cudaGetLastError());
}

ARTB_EXPORT int artb_latent_prefill(const void* q, int ldq, const void* kv, int ldkv, const void* c, int ldc, int rank_p, const int* tile_seq,
                                    const int* tile_row, int n_tiles, const int* row_end, const int* row_pos0, const int* key_off,
                                    const int* key_pos0, int window, int chunk, float scale, float softcap, float out_scale, const float* gate, int ldg, const float* sink, int sigmoid, const float* bias, int n_bias, const void* cols, int ldcols, int colp,
                                    void* o, int ldo, int vp, int vdim, int H, int G, int dk, int dv, int rot_p, cudaStream_t st) {
  if (n_tiles <= 0) return 0;
  if (H <= 0 || G <= 0 || H % G || (dk & 15) || (dv & 15) || (rot_p & 15) || (ldq & 7) || (ldkv & 7) || (ldc & 7) || (rank_p & 7) || (ldo & 1) || (vp & 1) ||
      vp > dv || vdim > vp || n_tiles > 65535 || (sigmoid && (!bias || n_bias <= 0 || sink)) || (cols && colp < vdim))
    return ERR_BAD_SHAPE;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(c)) & 15) return ERR_BAD_ALIGN;
  const LatentPrefill a{(const bf16*)q, ldq, (const bf16*)kv, ldkv, (const bf16*)c, ldc, rank_p, tile_seq, tile_row, row_end, row_pos0,
                        key_off, key_pos0, {window, chunk}, ScoreScale::of(scale, softcap), out_scale, gate, ldg, sink, {bias, n_bias},
                        ColumnGate<bf16>::of(cols, ldcols, colp, vdim), (bf16*)o, ldo, vp, vdim, H, G, dk, dv, rot_p};
#define ARTB_LP(V_)                                                                                                          \
  if (dv <= V_) return sigmoid ? launch_latent_prefill<V_, true>(a, n_tiles, st) : launch_latent_prefill<V_, false>(a, n_tiles, st)
  ARTB_LP(32);
  ARTB_LP(64);
  ARTB_LP(96);
  ARTB_LP(128);
#undef ARTB_LP
  return ERR_TOO_LARGE;
}
