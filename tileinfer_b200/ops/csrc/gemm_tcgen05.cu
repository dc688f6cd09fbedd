// Entry points of the tcgen05 products (gemm_kernel.cuh) and the activation quantisation of the int8 form.
#include "gemm_kernel.cuh"

namespace ti {

// ---------------------------------------------------------------- activation limbs
// One block per row: optional RMSNorm(1+w), rounding to bf16, row maximum, quantisation to two int8 planes.
__global__ void __launch_bounds__(256) quant_rows_kernel(const __nv_bfloat16* __restrict__ x, int ldx,
                                                         const __nv_bfloat16* __restrict__ norm_w, float eps, int K,
                                                         int8_t* __restrict__ xh, uint8_t* __restrict__ xl,
                                                         float* __restrict__ xscale) {
  __shared__ float red[8], bcast[2];
  const int m = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const __nv_bfloat16* row = x + (size_t)m * ldx;
  float rr = 1.f;
  if (norm_w != nullptr) {
    float ss = 0.f;
    for (int k = tid; k < K; k += 256) {
      const float v = __bfloat162float(row[k]);
      ss += v * v;
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    if (tid == 0) {
      float t = 0.f;
      for (int w = 0; w < 8; ++w) t += red[w];
      bcast[0] = rsqrtf(t / (float)K + eps);
    }
    __syncthreads();
    rr = bcast[0];
  }
  float mx = 0.f;
  for (int k = tid; k < K; k += 256) {
    float v = __bfloat162float(row[k]);
    if (norm_w != nullptr) v = round_bf16(v * rr * (1.f + __bfloat162float(norm_w[k])));
    mx = fmaxf(mx, fabsf(v));
  }
  mx = warp_max(mx);
  __syncthreads();
  if (lane == 0) red[warp] = mx;
  __syncthreads();
  if (tid == 0) {
    float a = 0.f;
    for (int w = 0; w < 8; ++w) a = fmaxf(a, red[w]);
    int e = (int)((__float_as_uint(a) >> 23) & 0xffu) - 127;
    e = max(e, -100);
    if (!(a < 3.0e38f)) e = 127;
    bcast[1] = exp2f((float)(14 - e));
    xscale[m] = exp2f((float)(e - 14));
  }
  __syncthreads();
  const float qs = bcast[1];
  for (int k = tid; k < K; k += 256) {
    float v = __bfloat162float(row[k]);
    if (norm_w != nullptr) v = round_bf16(v * rr * (1.f + __bfloat162float(norm_w[k])));
    const int q = max(-32768, min(32767, __float2int_rn(v * qs)));
    xh[(size_t)m * K + k] = (int8_t)(q >> 8);
    xl[(size_t)m * K + k] = (uint8_t)(q & 0xff);
  }
}

// The same for rows of up to 512 * 5 * 8 = 20480 elements in ONE pass: every thread keeps its (up to five) 16-byte
// chunks of the row in registers between the statistics and the quantisation, so the row is read once.  The block is
// as small as the row allows (K / 40 threads, rounded up to warps: 128 threads at K = 5120), so that many rows are in
// flight per SM: a row is a load -> reduce -> reduce -> store chain of a few microseconds, and 8192 rows of 512 threads
// each pass through an SM only four at a time.
__global__ void __launch_bounds__(512) quant_rows_fast_kernel(const __nv_bfloat16* __restrict__ x, int ldx,
                                                              const __nv_bfloat16* __restrict__ norm_w, float eps, int K,
                                                              int8_t* __restrict__ xh, uint8_t* __restrict__ xl,
                                                              float* __restrict__ xscale) {
  __shared__ float red[16], red2[16];
  const int m = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const __nv_bfloat16* row = x + (size_t)m * ldx;
  const int nchunk = K >> 3;
  const int nthr = blockDim.x, nwarp = nthr >> 5;
  pdl_trigger();
  pdl_wait();
  float v[5][8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < 5; ++j) {
    const int c = tid + j * nthr;
    uint4 q = make_uint4(0, 0, 0, 0);
    if (c < nchunk) q = *reinterpret_cast<const uint4*>(row + (size_t)c * 8);
    const uint32_t w4[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      v[j][2 * i] = bf16lo(w4[i]);
      v[j][2 * i + 1] = bf16hi(w4[i]);
      ss += v[j][2 * i] * v[j][2 * i] + v[j][2 * i + 1] * v[j][2 * i + 1];
    }
  }
  if (norm_w != nullptr) {
    uint4 nwv[5];
#pragma unroll
    for (int j = 0; j < 5; ++j) {
      const int c = tid + j * nthr;
      nwv[j] = c < nchunk ? *reinterpret_cast<const uint4*>(norm_w + (size_t)c * 8) : make_uint4(0, 0, 0, 0);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    float tot = 0.f;
#pragma unroll
    for (int w = 0; w < 16; ++w) tot += w < nwarp ? red[w] : 0.f;
    const float rr = rsqrtf(tot / (float)K + eps);
#pragma unroll
    for (int j = 0; j < 5; ++j) {
      const uint32_t n4[4] = {nwv[j].x, nwv[j].y, nwv[j].z, nwv[j].w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        v[j][2 * i] = round_bf16(v[j][2 * i] * rr * (1.f + bf16lo(n4[i])));
        v[j][2 * i + 1] = round_bf16(v[j][2 * i + 1] * rr * (1.f + bf16hi(n4[i])));
      }
    }
  }
  float mx = 0.f;
#pragma unroll
  for (int j = 0; j < 5; ++j)
#pragma unroll
    for (int i = 0; i < 8; ++i) mx = fmaxf(mx, fabsf(v[j][i]));
  mx = warp_max(mx);
  if (lane == 0) red2[warp] = mx;
  __syncthreads();
  float a = 0.f;
#pragma unroll
  for (int w = 0; w < 16; ++w) a = fmaxf(a, w < nwarp ? red2[w] : 0.f);
  int e = (int)((__float_as_uint(a) >> 23) & 0xffu) - 127;
  e = max(e, -100);
  if (!(a < 3.0e38f)) e = 127;
  const float qs = exp2f((float)(14 - e));
  if (tid == 0) xscale[m] = exp2f((float)(e - 14));
#pragma unroll
  for (int j = 0; j < 5; ++j) {
    const int c = tid + j * nthr;
    if (c >= nchunk) continue;
    uint32_t hw[2] = {0, 0}, lw[2] = {0, 0};
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int q = max(-32768, min(32767, __float2int_rn(v[j][i] * qs)));
      hw[i >> 2] |= (uint32_t)((q >> 8) & 0xff) << (8 * (i & 3));
      lw[i >> 2] |= (uint32_t)(q & 0xff) << (8 * (i & 3));
    }
    *reinterpret_cast<uint2*>(xh + (size_t)m * K + (size_t)c * 8) = make_uint2(hw[0], hw[1]);
    *reinterpret_cast<uint2*>(xl + (size_t)m * K + (size_t)c * 8) = make_uint2(lw[0], lw[1]);
  }
}

}  // namespace ti

extern "C" {

int ti_gemm_epilogue_size() { return (int)sizeof(ti::GemmEpilogue); }

// xh/xl/xscale <- limbs of x (optionally RMS-normalised with (1+norm_w)); one launch, M blocks.
int ti_quant_rows(const void* x, int ldx, const void* norm_w, float eps, int M, int K, void* xh, void* xl, void* xscale,
                  void* stream) {
  if (M <= 0) return 0;
  const bool aligned = (K % 8 == 0) && (ldx % 8 == 0) && (((uintptr_t)x | (uintptr_t)xh | (uintptr_t)xl) % 16 == 0) &&
                       (norm_w == nullptr || (uintptr_t)norm_w % 16 == 0);
  if (aligned && K <= 512 * 5 * 8)
    ti::launch_kernel(ti::quant_rows_fast_kernel, dim3(M), dim3(std::min(512, ((K / 8 + 4) / 5 + 31) / 32 * 32)), 0, (cudaStream_t)stream, true, (const __nv_bfloat16*)x, ldx,
                      (const __nv_bfloat16*)norm_w, eps, K, (int8_t*)xh, (uint8_t*)xl, (float*)xscale);
  else
    ti::quant_rows_kernel<<<M, 256, 0, (cudaStream_t)stream>>>((const __nv_bfloat16*)x, ldx, (const __nv_bfloat16*)norm_w,
                                                               eps, K, (int8_t*)xh, (uint8_t*)xl, (float*)xscale);
  return (int)cudaGetLastError();
}

// y = x W^T for tiled int8 weights `w` ([n_tiles][K/64][8][64]) and the limb planes of x.
// `part` / `tile_count`: split-k workspace (fp32 [S][M][N]) and zeroed per-tile counters, may be null (no split);
// `part_bytes` / `n_count` are their capacities.  The token tile (32 / 64 / 128) and the k split follow from M, N.
int ti_gemm_w8a16(const void* w, const void* wscale, int n_tiles, int N, int K, const void* xh, const void* xl,
                  const void* xscale, int M, const void* resid, void* out, int ldo, int epi, void* status, void* part,
                  size_t part_bytes, void* tile_count, int n_count, const ti::GemmEpilogue* ex, void* stream) {
  if (M <= 0) return 0;
  if (K % 64 || N < 1 || epi < 0 || epi > 6) return -2;
  ti::GemmParams p = {};
  const int KB = K / 64, KS = (KB + ti::kKS - 1) / ti::kKS;      // 64-byte slabs of the weight layout; 128-byte stages
  const int BN = M <= 32 ? 32 : (M <= 64 ? 64 : 128);
  const int BMH = ti::pick_bmh(M, n_tiles);
  int rc = ti::cached_map(&p.map_w, w, KB, n_tiles, BMH == 2 ? -32 : 0);
  if (rc) return rc;
  rc = ti::cached_map(&p.map_xh, xh, K, M, BN);
  if (rc) return rc;
  rc = ti::cached_map(&p.map_xl, xl, K, M, BN);
  if (rc) return rc;
  p.xscale = (const float*)xscale;
  p.wscale = (const __nv_bfloat16*)wscale;
  p.resid = (const __nv_bfloat16*)resid;
  p.out = out;
  p.status = (unsigned*)status;
  p.M = M;
  p.N = N;
  p.K = K;
  p.ldo = ldo;
  p.epi = epi;
  rc = ti::set_epilogue(p, ex);
  if (rc) return rc;
  const int rows = ti::kBM * BMH;
  const int tiles_n = (n_tiles * 8 + rows - 1) / rows, tiles_m = (M + BN - 1) / BN;
  const int S = ti::plan_split(p, KS, tiles_n * tiles_m, M, N, ldo, part, part_bytes, tile_count, n_count);
  dim3 grid(tiles_m, tiles_n, S);
  cudaStream_t st = (cudaStream_t)stream;
  if (BMH == 2 && BN == 32) return ti::launch_gemm<32, false, 2>(p, grid, st);
  if (BMH == 2 && BN == 64) return ti::launch_gemm<64, false, 2>(p, grid, st);
  if (BMH == 2) return ti::launch_gemm<128, false, 2>(p, grid, st);
  if (BN == 32) return ti::launch_gemm<32, false>(p, grid, st);
  if (BN == 64) return ti::launch_gemm<64, false>(p, grid, st);
  return ti::launch_gemm<128, false>(p, grid, st);
}

// The same for bf16 weights tiled [n_tiles][K/32][8][32] (lm_head, unquantised mode) and bf16 activations x [M][K]
// (contiguous rows): tcgen05.mma kind::f16, fp32 accumulation.  epi 3 stores fp32 (logits).
int ti_gemm_bf16(const void* w, int n_tiles, int N, int K, const void* x, int M, const void* resid, void* out, int ldo,
                 int epi, void* status, void* part, size_t part_bytes, void* tile_count, int n_count, const ti::GemmEpilogue* ex,
                 void* stream) {
  if (M <= 0) return 0;
  if (K % 32 || N < 1 || epi < 0 || epi > 6) return -2;
  ti::GemmParams p = {};
  const int KB = K / 32, KS = (KB + ti::kKS - 1) / ti::kKS;    // 64-byte slabs; 128-byte stages
  // a single weight tile (a router): smaller token tiles, so that there are enough of them for all SMs
  const int BN = M <= 32 || (N <= 128 && M <= 64 * 148) ? 32 : (M <= 64 || N <= 128 ? 64 : 128);
  const int BMH = ti::pick_bmh(M, n_tiles);
  int rc = ti::cached_map(&p.map_w, w, KB, n_tiles, BMH == 2 ? -32 : 0);
  if (rc) return rc;
  rc = ti::cached_map(&p.map_xh, x, 2 * K, M, BN);
  if (rc) return rc;
  p.resid = (const __nv_bfloat16*)resid;
  p.out = out;
  p.status = (unsigned*)status;
  p.M = M;
  p.N = N;
  p.K = 2 * K;                                                 // bytes of k: the kernel counts 64-byte slabs
  p.ldo = ldo;
  p.epi = epi;
  rc = ti::set_epilogue(p, ex);
  if (rc) return rc;
  const int rows = ti::kBM * BMH;
  const int tiles_n = (n_tiles * 8 + rows - 1) / rows, tiles_m = (M + BN - 1) / BN;
  const int S = ti::plan_split(p, KS, tiles_n * tiles_m, M, N, ldo, part, part_bytes, tile_count, n_count);
  dim3 grid(tiles_m, tiles_n, S);
  cudaStream_t st = (cudaStream_t)stream;
  if (S == 1 && ti::short_k(KS, BN, (long long)tiles_n * tiles_m))
    return BMH == 2 ? ti::launch_gemm<128, true, 2, ti::kGemmShortRingKb>(p, grid, st) : ti::launch_gemm<128, true, 1, ti::kGemmShortRingKb>(p, grid, st);
  if (N <= 128 && M > 64 && BN == 32) return ti::launch_gemm<32, true, 1, ti::kGemmShortRingKb>(p, grid, st);   // two CTAs per SM
  if (BMH == 2 && BN == 32) return ti::launch_gemm<32, true, 2>(p, grid, st);
  if (BMH == 2 && BN == 64) return ti::launch_gemm<64, true, 2>(p, grid, st);
  if (BMH == 2) return ti::launch_gemm<128, true, 2>(p, grid, st);
  if (BN == 32) return ti::launch_gemm<32, true>(p, grid, st);
  if (BN == 64) return ti::launch_gemm<64, true>(p, grid, st);
  return ti::launch_gemm<128, true>(p, grid, st);
}

}  // extern "C"
