// Row operations and small products around latent attention: the latent's norm and its store into cache pages (beside a
// rotated key part, with the rotation of the queries), and the per-head products that absorb W_uk into the query and W_uv into the output.
//
// Every kernel is templated on the activation type (bf16, or float in 32-bit mode).  Row pitches are padded to
// multiples of 64 elements and the pad columns hold zeros (zero weight rows, zero norm weights), so that rows are read
// in whole vectors; means divide by the true length.
#include "row_vec.cuh"

namespace ti {

// ---------------------------------------------------------------- latent -> cache
// One warp per token: c = rmsnorm(proj[t, col0 : col0 + R]) * w into the token's cache slot (pages of 16 rows of Rp
// columns, so a slot is a row).  Slots outside the cache (-1: do not store) are skipped.
template <typename T>
__global__ void __launch_bounds__(128) latent_store_kernel(const T* __restrict__ proj, int ld, int col0, const float* __restrict__ w,
                                                           const long long* __restrict__ slots, T* __restrict__ cache,
                                                           long long num_slots, int M, int R, int Rp, float eps) {
  pdl_trigger();
  pdl_wait();
  const int m = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= M) return;
  const long long slot = slots[m];
  if (slot < 0 || slot >= num_slots) return;
  const T* src = proj + (size_t)m * ld + col0;
  float ss = 0.f;
  for (int c = lane * 8; c < Rp; c += 256) {
    float v[8];
    load8(src + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
  }
  const float rr = rsqrtf(warp_sum(ss) / (float)R + eps);
  T* dst = cache + (size_t)slot * Rp;
  for (int c = lane * 8; c < Rp; c += 256) {
    float v[8], g[8];
    load8(src + c, v);
    load8(w + c, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= rr * g[i];
    store8(dst + c, v);
  }
}

// The same with a rotated part: a block per token.  Warp 0 writes the cache row [rmsnorm(latent) * w | turned key part | 0],
// the others turn the trailing part of every query head in place.  Dimension i of a part turns with dimension i + half.
struct LatentRopeParams {
  void* proj;                    // [M, ld]: query heads at h * dp (dim plain, then 2 * half turned), latent and key part at col0
  const float* w;                // [R]
  const float* inv_freq;         // [half]
  const int* positions;          // [M]
  const long long* slots;        // [M]
  void* cache;                   // [num_slots][Rp]
  long long num_slots;
  int ld, H, dp, dim, col0, half, M, R, Rp;
  float eps;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_rope_kernel(const __grid_constant__ LatentRopeParams p) {
  extern __shared__ float cs[];                            // [half] cosines, [half] sines
  const int m = blockIdx.x, tid = threadIdx.x;
  pdl_trigger();
  pdl_wait();
  T* row = static_cast<T*>(p.proj) + (size_t)m * p.ld;
  const float pos = (float)p.positions[m];
  for (int i = tid; i < p.half; i += 256) sincosf(pos * p.inv_freq[i], &cs[p.half + i], &cs[i]);
  __syncthreads();
  auto turn = [&](const T* src, T* dst, int i) {
    const float u = to_f<T>(src[i]), v = to_f<T>(src[i + p.half]), co = cs[i], si = cs[p.half + i];
    dst[i] = from_f<T>(u * co - v * si);
    dst[i + p.half] = from_f<T>(v * co + u * si);
  };
  if (tid >= 32) {
    for (int k = tid - 32; k < p.H * p.half; k += 224) {
      const int h = k / p.half;
      T* part = row + (size_t)h * p.dp + p.dim;
      turn(part, part, k - h * p.half);
    }
    return;
  }
  const long long slot = p.slots[m];
  if (slot < 0 || slot >= p.num_slots) return;
  const T* src = row + p.col0;
  T* dst = static_cast<T*>(p.cache) + (size_t)slot * p.Rp;
  float ss = 0.f;
#pragma unroll 4
  for (int c = tid; c < p.R; c += 32) {
    const float v = to_f<T>(src[c]);
    ss += v * v;
  }
  const float rr = rsqrtf(warp_sum(ss) / (float)p.R + p.eps);
#pragma unroll 4
  for (int c = tid; c < p.R; c += 32) dst[c] = from_f<T>(to_f<T>(src[c]) * rr * p.w[c]);
  for (int c = p.R + 2 * p.half + tid; c < p.Rp; c += 32) dst[c] = from_f<T>(0.f);
  for (int i = tid; i < p.half; i += 32) turn(src + p.R, dst + p.R, i);
}

// Latent rows of listed cache slots -> dense rows (keys of a prefill step).  Negative or out-of-range slots give zeros.
template <typename T>
__global__ void __launch_bounds__(128) latent_gather_kernel(const T* __restrict__ cache, const long long* __restrict__ slots,
                                                            long long num_slots, T* __restrict__ out, int M, int Rp) {
  pdl_trigger();
  pdl_wait();
  const int m = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (m >= M) return;
  const long long slot = slots[m];
  const bool ok = slot >= 0 && slot < num_slots;
  for (int c = lane * 8; c < Rp; c += 256) {
    float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (ok) load8(cache + (size_t)slot * Rp + c, v);
    store8(out + (size_t)m * Rp + c, v);
  }
}

// ---------------------------------------------------------------- per-head products
// out[t, h, n] = sum_k x[t, h, k] W[h, n, k] (* sigmoid(gate[t, h])).  K a multiple of 32, N a multiple of 64.
struct HeadProductParams {
  const void* x;      // [M, ldx], head h at column h * K
  const void* w;      // [H][N][K]
  const void* gate;   // null, or [M, ldg]: gate of head h at column gcol + h
  void* out;          // [M, ldo], head h at column h * N
  int M, H, N, K, ldx, ldo, ldg, gcol;
};

// 16 tokens x 64 outputs of one head per block.  The four warps take k steps of 32 in turn (a long contraction is then a
// short chain of loads per warp) and their partial sums meet in shared memory.  The contraction index is permuted alike
// in both operands (a lane's 16-byte load feeds two k steps), so fragments come straight from global memory.
__global__ void __launch_bounds__(128) head_product_bf16_kernel(const __grid_constant__ HeadProductParams p) {
  __shared__ float part[4][16][68];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int h = blockIdx.y, n0 = blockIdx.x * 64, m0 = blockIdx.z * 16;
  const bf16* w = static_cast<const bf16*>(p.w) + ((size_t)h * p.N + n0) * p.K;
  const bf16* x = static_cast<const bf16*>(p.x) + (size_t)h * p.K;
  const bf16* xa = x + (size_t)min(m0 + g, p.M - 1) * p.ldx;
  const bf16* xb = x + (size_t)min(m0 + g + 8, p.M - 1) * p.ldx;
  pdl_trigger();
  pdl_wait();
  float d[8][4] = {};
#pragma unroll 2
  for (int k = 32 * warp + 8 * t; k < p.K; k += 128) {
    const uint4 a = *reinterpret_cast<const uint4*>(xa + k), b = *reinterpret_cast<const uint4*>(xb + k);
    uint4 u[8];
#pragma unroll
    for (int n = 0; n < 8; ++n) u[n] = ldg_cached16(w + (size_t)(n * 8 + g) * p.K + k);
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      mma_bf16_16816(d[n], a.x, b.x, a.y, b.y, u[n].x, u[n].y);
      mma_bf16_16816(d[n], a.z, b.z, a.w, b.w, u[n].z, u[n].w);
    }
  }
#pragma unroll
  for (int n = 0; n < 8; ++n) {
    *reinterpret_cast<float2*>(&part[warp][g][n * 8 + 2 * t]) = make_float2(d[n][0], d[n][1]);
    *reinterpret_cast<float2*>(&part[warp][g + 8][n * 8 + 2 * t]) = make_float2(d[n][2], d[n][3]);
  }
  __syncthreads();
  const int r = tid >> 3, c = (tid & 7) * 8;
  if (m0 + r >= p.M) return;
  float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int e = 0; e < 8; ++e) v[e] += part[i][r][c + e];
  const bf16* gate = static_cast<const bf16*>(p.gate);
  const float s = gate == nullptr ? 1.f : sigmoid_f(__bfloat162float(gate[(size_t)(m0 + r) * p.ldg + p.gcol + h]));
#pragma unroll
  for (int e = 0; e < 8; ++e) v[e] *= s;
  store8(static_cast<bf16*>(p.out) + (size_t)(m0 + r) * p.ldo + (size_t)h * p.N + n0 + c, v);
}

__global__ void __launch_bounds__(128) head_product_f32_kernel(const __grid_constant__ HeadProductParams p) {
  const int h = blockIdx.y, n = blockIdx.x * 64 + (threadIdx.x & 63), m0 = blockIdx.z * 16 + (threadIdx.x >> 6) * 8;
  const float* w = static_cast<const float*>(p.w) + ((size_t)h * p.N + n) * p.K;
  const float* x = static_cast<const float*>(p.x) + (size_t)h * p.K;
  pdl_trigger();
  pdl_wait();
  float acc[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  for (int k = 0; k < p.K; k += 4) {
    const float4 b = *reinterpret_cast<const float4*>(w + k);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float4 a = *reinterpret_cast<const float4*>(x + (size_t)min(m0 + i, p.M - 1) * p.ldx + k);
      acc[i] += a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w;
    }
  }
  const float* gate = static_cast<const float*>(p.gate);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (m0 + i >= p.M) continue;
    const float s = gate == nullptr ? 1.f : sigmoid_exact(gate[(size_t)(m0 + i) * p.ldg + p.gcol + h]);
    static_cast<float*>(p.out)[(size_t)(m0 + i) * p.ldo + (size_t)h * p.N + n] = acc[i] * s;
  }
}

}  // namespace ti

extern "C" {

int ti_latent_store(const void* proj, int ld, int col0, const void* w, const void* slots, void* cache, long long num_slots,
                    int M, int R, int Rp, float eps, int f32, void* stream) {
  if (M <= 0) return 0;
  if (Rp % 8 || R > Rp || ld % 8 || col0 % 8) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  const dim3 grid((M + 3) / 4);
  if (f32)
    ti::launch_kernel(ti::latent_store_kernel<float>, grid, dim3(128), 0, st, true, (const float*)proj, ld, col0, (const float*)w,
                      (const long long*)slots, (float*)cache, num_slots, M, R, Rp, eps);
  else
    ti::launch_kernel(ti::latent_store_kernel<ti::bf16>, grid, dim3(128), 0, st, true, (const ti::bf16*)proj, ld, col0, (const float*)w,
                      (const long long*)slots, (ti::bf16*)cache, num_slots, M, R, Rp, eps);
  return (int)cudaGetLastError();
}

int ti_latent_rope(void* proj, int ld, int H, int dp, int dim, int col0, const void* w, const void* inv_freq, int half, const void* positions,
                   const void* slots, void* cache, long long num_slots, int M, int R, int Rp, float eps, int f32, void* stream) {
  if (M <= 0) return 0;
  if (dim + 2 * half > dp || R + 2 * half > Rp || half < 0 || half > 4096 || H < 0) return -2;
  const ti::LatentRopeParams p = {proj, (const float*)w, (const float*)inv_freq, (const int*)positions, (const long long*)slots, cache,
                                  num_slots, ld, H, dp, dim, col0, half, M, R, Rp, eps};
  ti::launch_kernel(f32 ? ti::latent_rope_kernel<float> : ti::latent_rope_kernel<ti::bf16>, dim3(M), dim3(256), (size_t)half * 8,
                    (cudaStream_t)stream, true, p);
  return (int)cudaGetLastError();
}

int ti_latent_gather(const void* cache, const void* slots, long long num_slots, void* out, int M, int Rp, int f32, void* stream) {
  if (M <= 0) return 0;
  if (Rp % 8) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  const dim3 grid((M + 3) / 4);
  if (f32)
    ti::launch_kernel(ti::latent_gather_kernel<float>, grid, dim3(128), 0, st, true, (const float*)cache, (const long long*)slots,
                      num_slots, (float*)out, M, Rp);
  else
    ti::launch_kernel(ti::latent_gather_kernel<ti::bf16>, grid, dim3(128), 0, st, true, (const ti::bf16*)cache, (const long long*)slots,
                      num_slots, (ti::bf16*)out, M, Rp);
  return (int)cudaGetLastError();
}

int ti_head_product(const void* x, const void* w, const void* gate, void* out, int M, int H, int N, int K, int ldx, int ldo,
                    int ldg, int gcol, int f32, void* stream) {
  if (M <= 0) return 0;
  if (K % 32 || N % 64 || ldx % 8 || ldo % 8 || (((uintptr_t)x | (uintptr_t)w | (uintptr_t)out) & 15)) return -2;
  ti::HeadProductParams p = {x, w, gate, out, M, H, N, K, ldx, ldo, ldg, gcol};
  const dim3 grid(N / 64, H, (M + 15) / 16);
  ti::launch_kernel(f32 ? ti::head_product_f32_kernel : ti::head_product_bf16_kernel, grid, dim3(128), 0, (cudaStream_t)stream, true, p);
  return (int)cudaGetLastError();
}

}  // extern "C"
