// Windowed attention of prompt portions on tcgen05, for heads whose key parts are whole 64-column blocks.
//
// The same operation as latent_prefill_kernel (expanded keys of dk columns, a rotated part of rot_p columns shared by all
// heads, values of dv columns), with S = Q K^T and O = P V as tcgen05.mma with accumulators in TMEM:
//
// With G query heads per key head and no rotated part it is grouped-query attention.  With sigmoid weights (key_weights.cuh)
// nothing is rescaled: P V of all tiles adds up in one TMEM accumulator, and the warps of a row need not agree on a maximum.
//
//   warp 0      TMA producer: Q once; per tile of 128 keys the key blocks (expanded part from k, rotated part from the
//               gathered cache rows) and the value block, which a GEMM has written transposed ([H * dv, keys])
//   warp 1      MMA issuer: S of tile i, then P V of tile i - 1; S and P V accumulators are double-buffered in TMEM
//   warps 2-9   softmax: two warps per TMEM lane quarter, each with half of the tile's columns; scores are read from TMEM
//               once, probabilities leave as bf16 in the swizzled operand layout, the output accumulates in registers
//
// Keys are double-buffered in shared memory, values have one stage: they are needed one softmax later than their keys, which
// is when the previous tile's product has released them.  All waits are bounded; an expiry records a status, raises the
// CTA's abort flag and every role unwinds.
#include <math.h>

#include "host_utils.h"
#include "key_mask.cuh"
#include "key_weights.cuh"
#include "ptx_sm100.cuh"
#include "softcap.cuh"

namespace artb {

constexpr int LT_B = 128;                    // queries per CTA, keys per tile
constexpr int LT_BLK = LT_B * 64 * 2;        // 16 KB: 128 rows of one 64-column block
constexpr int LT_THREADS = 320;

struct LatentTc {
  const int* tile_seq;
  const int* tile_row;
  const int* row_end;
  const int* row_pos0;
  const int* key_off;
  const int* key_pos0;
  KeyMask mask;
  ScoreScale score;
  float out_scale;
  const float* gate;      // [rows][ldg] factor per row and head, or null
  int ldg;
  const float* sink;      // fp32 [H] sinks of the softmax, or null
  DistanceBias bias;      // of every query head (sigmoid weights)
  ColumnGate<__nv_bfloat16> cols;
  __nv_bfloat16* o;
  int ldo, vp;
  int rank_p, dk, rot_p, G;
  int* status;
};

template <int NQ, int DV>        // 64-column blocks of a key (expanded + rotated); value columns (64 or 128)
struct LtSmem {
  static constexpr int Q = 0;
  static constexpr int K = Q + NQ * LT_BLK;               // [2]
  static constexpr int V = K + 2 * NQ * LT_BLK;           // two 64-key blocks of [DV rows][64]
  static constexpr int VBLK = DV * 128;
  static constexpr int P = V + 2 * VBLK;                  // two 64-key blocks
  static constexpr int XCH = P + 2 * LT_BLK;              // float [2][2][128]
  static constexpr int BAR = XCH + 2 * 256 * 4;
  static constexpr int TOTAL = BAR + 28 * 8 + 1024;
};

__device__ __forceinline__ float lt_ex2(float x) { return exp2_approx(x); }

// SIG: sigmoid weights
template <int NQ, int DV, bool SIG>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                         const __grid_constant__ CUtensorMap tmC, const __grid_constant__ CUtensorMap tmVt, const LatentTc a) {
  using L = LtSmem<NQ, DV>;
  constexpr int OC = DV / 2;                 // output columns per softmax warp
  extern __shared__ uint8_t lt_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(lt_raw) + 1023) & ~static_cast<uintptr_t>(1023));
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L::BAR);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;      // [2]
  uint64_t* k_empty = bars + 3;     // [2]
  uint64_t* v_full = bars + 5;
  uint64_t* v_empty = bars + 6;
  uint64_t* s_full = bars + 7;      // [2]
  uint64_t* s_empty = bars + 9;     // [2]
  uint64_t* p_full = bars + 11;
  uint64_t* p_empty = bars + 12;
  uint64_t* pv_full = bars + 13;    // [2]
  uint64_t* pv_empty = bars + 15;   // [2]
  uint64_t* x_bar = bars + 17;      // [4] one per lane quarter, two arrivals (the warp pair)
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 21);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* xch = reinterpret_cast<float*>(smem + L::XCH);

  const int h = blockIdx.y, hk = h / a.G, sq = a.tile_seq[blockIdx.x];
  const int r0 = a.tile_row[blockIdx.x], nrow = min(LT_B, a.row_end[sq] - r0);
  const int p0 = r0 + a.row_pos0[sq], p1 = p0 + nrow - 1;
  const int kp0 = a.key_pos0[sq], koff = a.key_off[sq];
  // first tile: down to a multiple of 8 keys, where the value load may start
  const int lo_rel = max(0, a.mask.first(p0) - kp0) & ~7;
  const int tiles = (p1 - kp0 - lo_rel) / LT_B + 1;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (koff & 7) {                            // the value loads would not start on a 16-byte boundary
    if (threadIdx.x == 0) atomicMax(a.status, ST_BAD_ARGS);
    return;
  }

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    mbar_init(v_full, 1);
    mbar_init(v_empty, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(&k_full[i], 1);
      mbar_init(&k_empty[i], 1);
      mbar_init(&s_full[i], 1);
      mbar_init(&s_empty[i], 8);
      mbar_init(&pv_full[i], 1);
      mbar_init(&pv_empty[i], 8);
    }
    for (int i = 0; i < 4; ++i) mbar_init(&x_bar[i], 2);
    mbar_init(p_full, 8);
    mbar_init(p_empty, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;

  if (warp == 0) {
    // ------------------------------------------------------------------ TMA producer
    if (lane == 0) {
      tma_prefetch_desc(&tmQ);
      tma_prefetch_desc(&tmK);
      tma_prefetch_desc(&tmC);
      tma_prefetch_desc(&tmVt);
      mbar_expect_tx(q_full, NQ * LT_BLK);
#pragma unroll
      for (int b = 0; b < NQ; ++b) tma_load_2d(smem + L::Q + b * LT_BLK, &tmQ, h * (a.dk + a.rot_p) + b * 64, r0, q_full);
      const int nk = a.dk >> 6;
      for (int it = 0; it < tiles && !*abort_flag; ++it) {
        const int s = it & 1, krow = koff + lo_rel + it * LT_B;
        if (!mbar_wait_timed(&k_empty[s], ((it >> 1) & 1) ^ 1)) {
          atomicMax(a.status, ST_TIMEOUT_EMPTY);
          *abort_flag = 1;
          break;
        }
        uint8_t* sk = smem + L::K + s * NQ * LT_BLK;
        mbar_expect_tx(&k_full[s], NQ * LT_BLK);
#pragma unroll
        for (int b = 0; b < NQ; ++b) {
          if (b < nk) tma_load_2d(sk + b * LT_BLK, &tmK, hk * a.dk + b * 64, krow, &k_full[s]);
          else tma_load_2d(sk + b * LT_BLK, &tmC, a.rank_p + (b - nk) * 64, krow, &k_full[s]);
        }
        if (!mbar_wait_timed(v_empty, (it & 1) ^ 1)) {
          atomicMax(a.status, ST_TIMEOUT_EMPTY);
          *abort_flag = 1;
          break;
        }
        mbar_expect_tx(v_full, 2 * L::VBLK);
        tma_load_2d(smem + L::V, &tmVt, krow, hk * DV, v_full);
        tma_load_2d(smem + L::V + L::VBLK, &tmVt, krow + 64, hk * DV, v_full);
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------------ MMA issuer
    if (lane == 0) {
      constexpr uint32_t idesc_s = umma_idesc_bf16(LT_B, LT_B), idesc_o = umma_idesc_bf16(LT_B, DV);
      const uint32_t sq_ = smem_u32(smem + L::Q), sp = smem_u32(smem + L::P), sv = smem_u32(smem + L::V);
      bool ok = mbar_wait_timed(q_full, 0);
      auto issue_pv = [&](int i) -> bool {
        const int s = i & 1;
        if (!mbar_wait_timed(v_full, i & 1) || !mbar_wait_timed(p_full, i & 1)) return false;
        if (!SIG && !mbar_wait_timed(&pv_empty[s], ((i >> 1) & 1) ^ 1)) return false;
        tc_fence_after_sync();
        const uint32_t d = tmem + 256 + (SIG ? 0 : s * 128);
#pragma unroll
        for (int kk = 0; kk < 8; ++kk)
          tc_mma_f16(d, umma_smem_desc_k128(sp + (kk >> 2) * LT_BLK) + 2 * (kk & 3),
                     umma_smem_desc_k128(sv + (kk >> 2) * L::VBLK) + 2 * (kk & 3), idesc_o, kk != 0 || (SIG && i > 0));
        if (!SIG) tc_commit(&pv_full[s]);
        else if (i == tiles - 1) tc_commit(&pv_full[0]);
        tc_commit(v_empty);
        tc_commit(p_empty);
        return true;
      };
      int it = 0;
      for (; it < tiles && ok && !*abort_flag; ++it) {
        const int s = it & 1;
        const uint32_t ph = (it >> 1) & 1;
        if (!mbar_wait_timed(&k_full[s], ph) || !mbar_wait_timed(&s_empty[s], ph ^ 1)) {
          ok = false;
          break;
        }
        tc_fence_after_sync();
        const uint32_t sk = smem_u32(smem + L::K + s * NQ * LT_BLK);
#pragma unroll
        for (int kk = 0; kk < 4 * NQ; ++kk)
          tc_mma_f16(tmem + s * LT_B, umma_smem_desc_k128(sq_ + (kk >> 2) * LT_BLK) + 2 * (kk & 3),
                     umma_smem_desc_k128(sk + (kk >> 2) * LT_BLK) + 2 * (kk & 3), idesc_s, kk != 0);
        tc_commit(&s_full[s]);
        tc_commit(&k_empty[s]);
        if (it > 0 && !issue_pv(it - 1)) {
          ok = false;
          break;
        }
      }
      if (ok && !*abort_flag && tiles > 0 && !issue_pv(tiles - 1)) ok = false;
      if (!ok) {
        atomicMax(a.status, ST_TIMEOUT_TMEM_EMPTY);
        *abort_flag = 1;
      }
    }
  } else {
    // ------------------------------------------------------------------ softmax / output warps
    const int q = warp & 3;                 // TMEM lane quarter of this warp
    const int hf = (warp - 2) >> 2;         // which half of the columns
    const int r = q * 32 + lane;            // query row inside the tile
    const int qpos = p0 + r, first = a.mask.first(qpos);
    const uint32_t lane_off = static_cast<uint32_t>(q * 32) << 16;
    uint8_t* prow = smem + L::P + hf * LT_BLK + r * 128;
    const int sw = r & 7;
    if (a.cols.g && r < nrow && hf * OC < a.cols.vdim) a.cols.prefetch(r0 + r, h, hf * OC);      // the epilogue's loads then hit the L2
    float O[OC];
#pragma unroll
    for (int i = 0; i < OC; ++i) O[i] = 0.f;
    float m = -INFINITY, l = 0.f, m_o = 0.f, ms_prev = 0.f;
    if (!SIG && a.sink) {                   // counted by one warp of the pair
      m = a.sink[h] * KW_LOG2E;
      l = hf == 0 ? 1.f : 0.f;
    }
    const float* tab = SIG ? a.bias.head(h) : nullptr;
    const float far = SIG ? a.bias.last(tab) : 0.f;
    bool dead = false;
    uint32_t xph = 0;

    auto fail = [&](int code) {
      if (lane == 0) {
        atomicMax(a.status, code);
        *abort_flag = 1;
      }
      dead = true;
    };
    // exchange one float with the partner thread (same row, other half); false on timeout
    auto swap_with_partner = [&](float mine, float& other) -> bool {
      float* slot = xch + (xph & 1) * 256;
      slot[hf * 128 + r] = mine;
      __syncwarp();
      if (lane == 0) mbar_arrive(&x_bar[q]);
      const int okw = mbar_wait_timed(&x_bar[q], xph & 1) ? 1 : 0;
      if (!__all_sync(0xffffffffu, okw)) return false;
      other = slot[(hf ^ 1) * 128 + r];
      ++xph;
      return true;
    };
    auto add_pv = [&](int i, float ms_i) -> bool {
      const int s = i & 1;
      const int okw = mbar_wait_timed(&pv_full[s], (i >> 1) & 1) ? 1 : 0;
      if (!__all_sync(0xffffffffu, okw)) return false;
      tc_fence_after_sync();
      // maxima only grow, but a row that has seen no key yet stands at 0: nothing to rescale then
      const float f = lt_ex2(fminf(m_o - ms_i, 0.f));
      m_o = ms_i;
#pragma unroll
      for (int c = 0; c < OC; c += 32) {
        uint32_t v[32];
        tmem_ld_32x32(tmem + lane_off + 256 + s * 128 + hf * OC + c, v);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) O[c + j] = fmaf(O[c + j], f, __uint_as_float(v[j]));
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&pv_empty[s]);
      return true;
    };

    for (int it = 0; it < tiles; ++it) {
      if (__shfl_sync(0xffffffffu, *abort_flag, 0)) {
        dead = true;
        break;
      }
      const int s = it & 1;
      const int k0 = kp0 + lo_rel + it * LT_B;                         // position of the tile's first key
      const bool inside = k0 + LT_B - 1 <= p0 && k0 >= a.mask.first(p0 + LT_B - 1);
      const int okw = mbar_wait_timed(&s_full[s], (it >> 1) & 1) ? 1 : 0;
      if (!__all_sync(0xffffffffu, okw)) {
        fail(ST_TIMEOUT_TMEM_FULL);
        break;
      }
      tc_fence_after_sync();
      float x[64];
      {
        uint32_t v0[32], v1[32];
        tmem_ld_32x32(tmem + lane_off + s * LT_B + hf * 64, v0);
        tmem_ld_32x32(tmem + lane_off + s * LT_B + hf * 64 + 32, v1);
        tmem_ld_wait();
#pragma unroll
        for (int j = 0; j < 32; ++j) {
          x[j] = __uint_as_float(v0[j]);
          x[32 + j] = __uint_as_float(v1[j]);
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&s_empty[s]);
      if (a.score.capped()) {
#pragma unroll
        for (int j = 0; j < 64; j += 2) a.score.squash(x[j], x[j + 1]);
      }
      if (SIG) {
        if (a.bias.beyond(p0, k0 + LT_B - 1)) {
#pragma unroll
          for (int j = 0; j < 64; ++j) x[j] = fmaf(x[j], a.score.scale_log2, far);
        } else {                              // distances of the tile stay within the table's padding
          const float* td = tab + qpos - (k0 + hf * 64);
#pragma unroll
          for (int j = 0; j < 64; ++j) x[j] = fmaf(x[j], a.score.scale_log2, __ldg(td - j));
        }
#pragma unroll
        for (int j = 0; j < 64; j += 2) sigmoid_pair(x[j], x[j + 1]);
        if (!inside) {
          const int hi = qpos - (k0 + hf * 64), lo = first - (k0 + hf * 64);
#pragma unroll
          for (int j = 0; j < 64; ++j)
            if (j > hi || j < lo) x[j] = 0.f;
        }
        const int okp = mbar_wait_timed(p_empty, (it & 1) ^ 1) ? 1 : 0;
        if (!__all_sync(0xffffffffu, okp)) {
          fail(ST_TIMEOUT_EMPTY);
          break;
        }
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          uint4 w;
          w.x = pack_bf16x2(x[8 * i], x[8 * i + 1]);
          w.y = pack_bf16x2(x[8 * i + 2], x[8 * i + 3]);
          w.z = pack_bf16x2(x[8 * i + 4], x[8 * i + 5]);
          w.w = pack_bf16x2(x[8 * i + 6], x[8 * i + 7]);
          *reinterpret_cast<uint4*>(prow + ((i ^ sw) << 4)) = w;
        }
        fence_proxy_async_smem();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_full);
        continue;
      }
      if (!inside) {
        const int hi = qpos - (k0 + hf * 64), lo = first - (k0 + hf * 64);      // visible: lo <= j <= hi
#pragma unroll
        for (int j = 0; j < 64; ++j)
          if (j > hi || j < lo) x[j] = -INFINITY;
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int j = 0; j < 64; ++j) mx4[j & 3] = fmaxf(mx4[j & 3], x[j]);
      const float mx_mine = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3])) * a.score.scale_log2;   // scale > 0
      float mx_other;
      if (!swap_with_partner(mx_mine, mx_other)) {
        fail(ST_TIMEOUT_PEER);
        break;
      }
      const float mn = fmaxf(m, fmaxf(mx_mine, mx_other));
      const float ms = mn == -INFINITY ? 0.f : mn;
      l *= lt_ex2(m - ms);
      m = mn;
      // the previous tile's product has left shared memory P free once it was consumed
      const int okp = mbar_wait_timed(p_empty, (it & 1) ^ 1) ? 1 : 0;
      if (!__all_sync(0xffffffffu, okp)) {
        fail(ST_TIMEOUT_EMPTY);
        break;
      }
      float rs4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        float pe[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          pe[e] = lt_ex2(fmaf(x[8 * i + e], a.score.scale_log2, -ms));
          rs4[e & 3] += pe[e];
        }
        uint4 w;
        w.x = pack_bf16x2(pe[0], pe[1]);
        w.y = pack_bf16x2(pe[2], pe[3]);
        w.z = pack_bf16x2(pe[4], pe[5]);
        w.w = pack_bf16x2(pe[6], pe[7]);
        *reinterpret_cast<uint4*>(prow + ((i ^ sw) << 4)) = w;
      }
      l += (rs4[0] + rs4[1]) + (rs4[2] + rs4[3]);
      fence_proxy_async_smem();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
      if (it > 0 && !add_pv(it - 1, ms_prev)) {
        fail(ST_TIMEOUT_TMEM_FULL);
        break;
      }
      ms_prev = ms;
    }
    uint4 gates[OC / 8];                      // they arrive while the last product ends
    const bool gated = a.cols.g && r < nrow;
    if (gated) {
#pragma unroll
      for (int c = 0; c < OC; c += 8) gates[c / 8] = a.cols.load8(r0 + r, h, hf * OC + c);
    }
    float l_other = 0.f;
    if (SIG) {
      const int okw = !dead && mbar_wait_timed(&pv_full[0], 0) ? 1 : 0;
      if (!__all_sync(0xffffffffu, okw)) {
        if (!dead) fail(ST_TIMEOUT_TMEM_FULL);
      } else {
        tc_fence_after_sync();
#pragma unroll
        for (int c = 0; c < OC; c += 32) {
          uint32_t v[32];
          tmem_ld_32x32(tmem + lane_off + 256 + hf * OC + c, v);
          tmem_ld_wait();
#pragma unroll
          for (int j = 0; j < 32; ++j) O[c + j] = __uint_as_float(v[j]);
        }
      }
    } else {
      if (!dead && tiles > 0 && !add_pv(tiles - 1, ms_prev)) fail(ST_TIMEOUT_TMEM_FULL);
      if (!dead && !swap_with_partner(l, l_other)) fail(ST_TIMEOUT_PEER);
    }
    if (!dead && r < nrow) {
      const float lt = l + l_other;
      float inv = SIG ? a.out_scale : lt > 0.f ? a.out_scale / lt : 0.f;
      if (a.gate) inv *= a.gate[static_cast<size_t>(r0 + r) * a.ldg + h];
      __nv_bfloat16* o = a.o + static_cast<size_t>(r0 + r) * a.ldo + static_cast<size_t>(h) * a.vp + hf * OC;
#pragma unroll
      for (int c = 0; c < OC; c += 8) {
        if (hf * OC + c < a.vp) {
          float y[8];
#pragma unroll
          for (int j = 0; j < 8; ++j) y[j] = O[c + j] * inv;
          if (gated) a.cols.apply8(gates[c / 8], y);
          uint4 w;
          w.x = pack_bf16x2(y[0], y[1]);
          w.y = pack_bf16x2(y[2], y[3]);
          w.z = pack_bf16x2(y[4], y[5]);
          w.w = pack_bf16x2(y[6], y[7]);
          *reinterpret_cast<uint4*>(o + c) = w;
        }
      }
    }
  }

  tc_fence_before_sync();
  __syncthreads();
  if (*abort_flag) {
    for (int i = 0; i < 2000; ++i) __nanosleep(1000);
    __syncthreads();
  }
  if (warp == 1) {
    __syncwarp();
    tc_fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

template <int NQ, int DV, bool SIG>
static int launch_latent_tc_form(const CUtensorMap& tQ, const CUtensorMap& tK, const CUtensorMap& tC, const CUtensorMap& tV, const LatentTc& a,
                            int n_tiles, int H, cudaStream_t st) {
  using L = LtSmem<NQ, DV>;
  static_assert(L::TOTAL <= 227 * 1024, "shared memory");
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(latent_prefill_tc_kernel<NQ, DV, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = true;
  }
  latent_prefill_tc_kernel<NQ, DV, SIG><<<dim3(n_tiles, H), LT_THREADS, L::TOTAL, st>>>(tQ, tK, tC, tV, a);
  return static_cast<int>(cudaGetLastError());
}

template <int NQ, int DV>
static int launch_latent_tc(const CUtensorMap& tQ, const CUtensorMap& tK, const CUtensorMap& tC, const CUtensorMap& tV, const LatentTc& a,
                            int n_tiles, int H, cudaStream_t st) {
  return a.bias.tab ? launch_latent_tc_form<NQ, DV, true>(tQ, tK, tC, tV, a, n_tiles, H, st)
                    : launch_latent_tc_form<NQ, DV, false>(tQ, tK, tC, tV, a, n_tiles, H, st);
}

}  // namespace artb

using namespace artb;

// As artb_latent_prefill, with keys k [n_keys, H / G * dk] and values transposed: vt [H / G * dv, n_keys].  dk and rot_p multiples
// of 64 (dk + rot_p <= 192), dv 64 or 128, n_keys and every key_off a multiple of 8, scale > 0.  Gathered rows between two
// sequences must be finite.
ARTB_EXPORT int artb_latent_prefill_tc(const void* q, int ldq, int rows, const void* k, int ldk, const void* c, int ldc, int rank_p,
                                       const void* vt, int ldvt, int n_keys, const int* tile_seq, const int* tile_row, int n_tiles,
                                       const int* row_end, const int* row_pos0, const int* key_off, const int* key_pos0, int window,
                                       int chunk, float scale, float softcap, float out_scale, const float* gate, int ldg, const float* sink, int sigmoid, const float* bias, int n_bias, const void* cols, int ldcols, int colp,
                                       void* o, int ldo, int vp, int vdim, int H, int G, int dk, int dv, int rot_p,
                                       int* status, cudaStream_t st) {
  if (n_tiles <= 0) return 0;
  if (H <= 0 || H > 65535 || G <= 0 || H % G || dk <= 0 || (dk & 63) || (rot_p & 63) || dk + rot_p > 192 || (dv != 64 && dv != 128) || (n_keys & 7) || (ldo & 7) ||
      (vp & 7) || vp > dv || vdim > vp || !(scale > 0.f) || (rank_p & 7) || (sigmoid ? !bias || n_bias <= 0 || sink : bias != nullptr) ||
      (cols && colp < vdim))
    return ERR_BAD_SHAPE;
  if (reinterpret_cast<uintptr_t>(o) & 15) return ERR_BAD_ALIGN;
  CUtensorMap tQ, tK, tC, tV;
  int e;
  if ((e = make_tmap_bf16_2d(&tQ, q, rows, static_cast<uint64_t>(H) * (dk + rot_p), ldq, LT_B, 64))) return e;
  if ((e = make_tmap_bf16_2d(&tK, k, n_keys, static_cast<uint64_t>(H / G) * dk, ldk, LT_B, 64))) return e;
  if ((e = make_tmap_bf16_2d(&tC, c, n_keys, ldc, ldc, LT_B, 64))) return e;
  if ((e = make_tmap_bf16_2d(&tV, vt, static_cast<uint64_t>(H / G) * dv, n_keys, ldvt, dv, 64))) return e;
  const LatentTc a{tile_seq, tile_row, row_end, row_pos0, key_off, key_pos0, {window, chunk}, ScoreScale::of(scale, softcap), out_scale, gate, ldg,
                   sink, {bias, n_bias}, ColumnGate<__nv_bfloat16>::of(cols, ldcols, colp, vdim), reinterpret_cast<__nv_bfloat16*>(o), ldo, vp, rank_p, dk, rot_p, G, status};
  const int nq = (dk + rot_p) / 64;
  if (dv == 128) {
    if (nq == 1) return launch_latent_tc<1, 128>(tQ, tK, tC, tV, a, n_tiles, H, st);
    if (nq == 2) return launch_latent_tc<2, 128>(tQ, tK, tC, tV, a, n_tiles, H, st);
    return launch_latent_tc<3, 128>(tQ, tK, tC, tV, a, n_tiles, H, st);
  }
  if (nq == 1) return launch_latent_tc<1, 64>(tQ, tK, tC, tV, a, n_tiles, H, st);
  if (nq == 2) return launch_latent_tc<2, 64>(tQ, tK, tC, tV, a, n_tiles, H, st);
  return launch_latent_tc<3, 64>(tQ, tK, tC, tV, a, n_tiles, H, st);
}
