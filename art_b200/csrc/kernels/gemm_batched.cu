// Batched bf16 GEMM on the tcgen05 pipeline:  C_b[m, n] = A_b[m, :] . B_b[n, :]   for b < batch.
//
// A is [batch][pitch][K] with the row pitch a multiple of 128 (an M tile then belongs to one batch member; rows past M
// are computed and not stored), B the members' matrices stacked along rows [batch * N, K].  C_b starts c_batch elements
// after C_{b-1}, with leading dimension ldc: c_batch = N, ldc = batch * N interleaves the members' columns in one row
// (per-head projections next to each other), c_batch = pitch * N, ldc = N keeps them apart.
//
// One launch serves the per-head projections of latent attention (batch = heads) and the projections of a token-shift
// mixer, each of which reads its own mix of the tokens (batch = r, k, v, g).
#include "gemm_epilogue.cuh"
#include "host_utils.h"

namespace artb {

struct SchedBatched {
  int batch, m_tiles, tiles_pitch, n_tiles, b_rows;
  __device__ int tiles_for_cta(int cta, int ncta) const {
    const int total = batch * m_tiles * n_tiles;
    return cta < total ? (total - cta + ncta - 1) / ncta : 0;
  }
  __device__ TileInfo get(int cta, int ncta, int i) const {
    const int t = cta + i * ncta;
    const int m = t % m_tiles, r = t / m_tiles, n = r % n_tiles, b = r / n_tiles;
    TileInfo ti = make_tile(b * tiles_pitch + m, n);
    ti.group = b;
    ti.b_row = b * b_rows;
    return ti;
  }
};

template <int BN>
struct EpiBatched {
  EpiStore<BN, 1> st;
  int tiles_pitch;
  long c_batch_bytes;
  uint8_t* base;
  __device__ TileInfo local(const TileInfo& ti) {
    TileInfo t = ti;
    t.m_blk = ti.m_blk - ti.group * tiles_pitch;
    st.C = base + ti.group * c_batch_bytes;
    return t;
  }
  __device__ void tile_begin(const TileInfo&, int) {}
  __device__ void tile_end(const TileInfo&, int) {}
  __device__ void chunk(const TileInfo& ti, int row, int c, uint32_t (&acc)[32]) { st.chunk(local(ti), row, c, acc); }
};

template <int BN, int STAGES>
static int launch_batched(const CUtensorMap& tA, const CUtensorMap& tB, int kb, const SchedBatched& sched, const EpiBatched<BN>& epi,
                          int* status, cudaStream_t stream) {
  using L = GemmSmemLayout<BN, STAGES>;
  auto kern = gemm_tcgen05_kernel<BN, STAGES, SchedBatched, EpiBatched<BN>>;
  static bool configured[64] = {false};
  int dev = 0;
  cudaGetDevice(&dev);
  if (!configured[dev & 63]) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL);
    if (e != cudaSuccess) return static_cast<int>(e);
    configured[dev & 63] = true;
  }
  int grid = sched.batch * sched.m_tiles * sched.n_tiles;
  if (grid > sm_count()) grid = sm_count();
  return static_cast<int>(launch_kernel(kern, dim3(grid), dim3(GEMM_THREADS), L::TOTAL, stream, tA, tB, tA, tB, kb, 0, sched, epi,
                                        status, NoComm{}));
}

}  // namespace artb

using namespace artb;

ARTB_EXPORT int artb_gemm_batched_bf16_tn(const void* A, int lda, int pitch, const void* B, int ldb, void* C, int ldc, long c_batch,
                                          int out_f32, int batch, int M, int N, int K, int* status, cudaStream_t stream) {
  if (batch <= 0 || M <= 0 || N <= 0 || K <= 0 || pitch < M || pitch % GEMM_BM) return ERR_BAD_SHAPE;
  if ((K & 7) || (N & 7) || (out_f32 ? (ldc & 3) || (c_batch & 3) : (ldc & 7) || (c_batch & 7))) return ERR_BAD_SHAPE;
  if (reinterpret_cast<uintptr_t>(C) & 15) return ERR_BAD_ALIGN;
  const int m_tiles = (M + GEMM_BM - 1) / GEMM_BM;
  int bn = N > 128 ? 256 : N > 64 ? 128 : 64;
  while (bn > 64 && static_cast<long>(batch) * m_tiles * ((N + bn - 1) / bn) < sm_count() / 2) bn >>= 1;
  CUtensorMap tA, tB;
  int e;
  if ((e = make_tmap_bf16_2d(&tA, A, static_cast<uint64_t>(batch) * pitch, K, lda, GEMM_BM, GEMM_BK))) return e;
  if ((e = make_tmap_bf16_2d(&tB, B, static_cast<uint64_t>(batch) * N, K, ldb, bn, GEMM_BK))) return e;
  const int kb = (K + GEMM_BK - 1) / GEMM_BK;
#define ARTB_LAUNCH(BN_, ST_)                                                                                             \
  {                                                                                                                       \
    const SchedBatched sched{batch, m_tiles, pitch / GEMM_BM, (N + BN_ - 1) / BN_, N};                                    \
    EpiBatched<BN_> epi{EpiStore<BN_, 1>{C, nullptr, nullptr, nullptr, ldc, 0, 0, M, N, out_f32 ? 1 : 0, N},               \
                        pitch / GEMM_BM, c_batch * (out_f32 ? 4 : 2), reinterpret_cast<uint8_t*>(C)};                      \
    return launch_batched<BN_, ST_>(tA, tB, kb, sched, epi, status, stream);                                               \
  }
  if (bn == 256) ARTB_LAUNCH(256, 4)
  if (bn == 128) ARTB_LAUNCH(128, 6)
  ARTB_LAUNCH(64, 8)
#undef ARTB_LAUNCH
}
