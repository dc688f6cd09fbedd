// tcgen05 products of token groups with several weight matrices of one shape (experts): gemm_kernel.cuh with the table of
// token tiles that moe_route.cu writes.
#include "gemm_kernel.cuh"

namespace ti {

// Token tiles that walk the weight tiles together: about 2048 rows, so that their activations and the matrices they meet
// (a few experts) stay in L2 while every weight tile is used by all of them.
static int group_tiles(int BN, int max_tiles) { return std::max(1, std::min(2048 / BN, max_tiles)); }

template <bool BF16>
static int run_grouped(GemmParams& p, int BN, int BMH, cudaStream_t st) {
  p.group_m = group_tiles(BN, p.max_tiles);
  const int rows = kBM * BMH;
  p.tiles_n = (p.w_tiles * 8 + rows - 1) / rows;
  const dim3 grid((p.max_tiles + p.group_m - 1) / p.group_m * p.group_m * p.tiles_n, 1, 1);
  if (BN == 32) return launch_gemm<32, BF16, 1, kGemmShortRingKb, true>(p, grid, st);
  if (BN == 64) return launch_gemm<64, BF16, 1, kGemmShortRingKb, true>(p, grid, st);
  // two CTAs per SM (bf16: 2 x 256 TMEM columns): the epilogue of one overlaps the main loop of the other
  constexpr int RK = BF16 ? kGemmShortRingKb : TI_GEMM_RING_KB;
  if (BMH == 2) return launch_gemm<128, BF16, 2, RK, true>(p, grid, st);
  return launch_gemm<128, BF16, 1, RK, true>(p, grid, st);
}

static int prepare_grouped(GemmParams& p, const void* w, int E, int KB, int BN, int BMH) {
  if (BN != 32 && BN != 64 && BN != 128) return -2;
  p.kb_per_split = (KB + kKS - 1) / kKS;
  return cached_map(&p.map_w, w, KB, E * p.w_tiles, BMH == 2 ? -32 : 0);
}

// 256-row weight tiles when the matrices have them and there are many token rows
static int grouped_bmh(int BN, int w_tiles, int rows) { return BN == 128 && w_tiles >= 32 && rows >= 4096 ? 2 : 1; }

}  // namespace ti

extern "C" {

// y[r] = x[r] W_e^T for the rows r of every token tile and its matrix e.  w: bf16, E matrices of n_tiles 8-row tiles each
// ([E * n_tiles][K/32][8][32]); x: [rows][K] bf16; tiles: int32 [3][max_tiles]; num_tiles: device counter.  N: columns
// of a matrix; epi as in ti_gemm_bf16 without the residual and split-k forms.
int ti_gemm_grouped_bf16(const void* w, int E, int n_tiles, int N, int K, const void* x, int rows, const void* tiles,
                         const void* num_tiles, int max_tiles, int BN, void* out, int ldo, int epi, void* status,
                         const ti::GemmEpilogue* ex, void* stream) {
  if (rows <= 0 || max_tiles <= 0) return 0;
  if (K % 32 || N < 1 || N > n_tiles * 8 || (epi != ti::GEPI_STORE && epi != ti::GEPI_F32 && epi != ti::GEPI_SPLIT_GLU)) return -2;
  ti::GemmParams p = {};
  const int BMH = ti::grouped_bmh(BN, n_tiles, rows);
  p.w_tiles = n_tiles;
  p.M = rows; p.N = N; p.K = 2 * K; p.ldo = ldo; p.epi = epi;
  p.out = out;
  p.status = (unsigned*)status;
  p.tiles = (const int*)tiles;
  p.num_tiles = (const int*)num_tiles;
  p.max_tiles = max_tiles;
  int rc = ti::prepare_grouped(p, w, E, K / 32, BN, BMH);
  if (rc) return rc;
  rc = ti::cached_map(&p.map_xh, x, 2 * K, rows, BN);
  if (rc) return rc;
  rc = ti::set_epilogue(p, ex);
  if (rc) return rc;
  return ti::run_grouped<true>(p, BN, BMH, (cudaStream_t)stream);
}

// The same for int8 matrices ([E * n_tiles][K/64][8][64], one bf16 scale per row) and the limb planes of x.  The row
// scales of a matrix follow each other, matrix after matrix.
int ti_gemm_grouped_w8a16(const void* w, const void* wscale, int E, int n_tiles, int N, int K, const void* xh, const void* xl,
                          const void* xscale, int rows, const void* tiles, const void* num_tiles, int max_tiles, int BN,
                          void* out, int ldo, int epi, void* status, const ti::GemmEpilogue* ex, void* stream) {
  if (rows <= 0 || max_tiles <= 0) return 0;
  if (K % 64 || N < 1 || N > n_tiles * 8 || (epi != ti::GEPI_STORE && epi != ti::GEPI_F32 && epi != ti::GEPI_SPLIT_GLU)) return -2;
  ti::GemmParams p = {};
  const int BMH = ti::grouped_bmh(BN, n_tiles, rows);
  p.w_tiles = n_tiles;
  p.M = rows; p.N = N; p.K = K; p.ldo = ldo; p.epi = epi;
  p.out = out;
  p.status = (unsigned*)status;
  p.xscale = (const float*)xscale;
  p.wscale = (const __nv_bfloat16*)wscale;
  p.tiles = (const int*)tiles;
  p.num_tiles = (const int*)num_tiles;
  p.max_tiles = max_tiles;
  int rc = ti::prepare_grouped(p, w, E, K / 64, BN, BMH);
  if (rc) return rc;
  rc = ti::cached_map(&p.map_xh, xh, K, rows, BN);
  if (rc) return rc;
  rc = ti::cached_map(&p.map_xl, xl, K, rows, BN);
  if (rc) return rc;
  rc = ti::set_epilogue(p, ex);
  if (rc) return rc;
  return ti::run_grouped<false>(p, BN, BMH, (cudaStream_t)stream);
}

}  // extern "C"
