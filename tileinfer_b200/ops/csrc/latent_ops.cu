// Row operations and small products around latent attention and an fp32 residual stream: token + position embedding
// with a norm, plain RMSNorm of fp32 rows, the latent's norm and its store into cache pages, the per-head products that
// absorb W_uk into the query and W_uv into the output, and the fp32 matrix product of the 32-bit mode.
//
// Every kernel is templated on the activation type (bf16, or float in 32-bit mode).  Row pitches are padded to
// multiples of 64 elements and the pad columns hold zeros (zero weight rows, zero norm weights), so that rows are read
// in whole vectors; means divide by the true length.
#include "common.cuh"

namespace ti {

typedef __nv_bfloat16 bf16;

template <typename T> TI_DEVICE void load8(const T* p, float (&v)[8]);
template <> TI_DEVICE void load8<bf16>(const bf16* p, float (&v)[8]) {
  const uint4 q = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) { v[2 * i] = bf16lo(w[i]); v[2 * i + 1] = bf16hi(w[i]); }
}
template <> TI_DEVICE void load8<float>(const float* p, float (&v)[8]) {
  const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
  v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}
template <typename T> TI_DEVICE void store8(T* p, const float (&v)[8]);
template <> TI_DEVICE void store8<bf16>(bf16* p, const float (&v)[8]) {
  *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
}
template <> TI_DEVICE void store8<float>(float* p, const float (&v)[8]) {
  *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4*>(p + 4) = make_float4(v[4], v[5], v[6], v[7]);
}
template <typename T> TI_DEVICE float to_f(T v);
template <> TI_DEVICE float to_f<bf16>(bf16 v) { return __bfloat162float(v); }
template <> TI_DEVICE float to_f<float>(float v) { return v; }
TI_DEVICE float sigmoid_exact(float x) { return 1.f / (1.f + expf(-x)); }

TI_DEVICE float block_sum32(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < nw; ++w) t += red[w];
  return t;
}

// ---------------------------------------------------------------- embedding
// x[m, :] = rmsnorm(embed[ids[m]] + pos[positions[m]]) * w in fp32.  Either of `pos` and `w` may be null.  Block 0 also
// advances the device step counter.
template <typename T>
__global__ void __launch_bounds__(256) embed_pos_kernel(const long long* __restrict__ ids, const int* __restrict__ positions,
                                                        const T* __restrict__ embed, const T* __restrict__ pos,
                                                        const float* __restrict__ w, float* __restrict__ x, int W, int P,
                                                        int vocab, int max_pos, float eps, unsigned* step) {
  __shared__ float red[8];
  pdl_trigger();
  pdl_wait();
  const int m = blockIdx.x;
  long long id = ids[m];
  if (id < 0 || id >= vocab) id = 0;
  const int ps = min(max(positions[m], 0), max_pos - 1);
  const T* e = embed + (size_t)id * P;
  const T* q = pos == nullptr ? nullptr : pos + (size_t)ps * P;
  float ss = 0.f;
  for (int c = threadIdx.x * 8; c < P; c += blockDim.x * 8) {
    float a[8], b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    load8(e + c, a);
    if (q != nullptr) load8(q + c, b);
#pragma unroll
    for (int i = 0; i < 8; ++i) { const float v = a[i] + b[i]; ss += v * v; }
  }
  const float rr = w == nullptr ? 1.f : rsqrtf(block_sum32(ss, red) / (float)W + eps);
  for (int c = threadIdx.x * 8; c < P; c += blockDim.x * 8) {
    float a[8], b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, g[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
    load8(e + c, a);
    if (q != nullptr) load8(q + c, b);
    if (w != nullptr) load8(w + c, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] = (a[i] + b[i]) * rr * g[i];
    store8(x + (size_t)m * P + c, a);
  }
  if (step != nullptr && m == 0 && threadIdx.x == 0) *step = *step + 1u;
}

// ---------------------------------------------------------------- RMSNorm of fp32 rows
// y[m, :] = x[m, :] / sqrt(mean(x^2) + eps) * w.  The row is kept in registers between the two passes when it fits.
template <typename T>
__global__ void __launch_bounds__(256) rmsnorm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w,
                                                          T* __restrict__ y, int W, int P, float eps) {
  __shared__ float red[8];
  constexpr int kKeep = 4;                                // 256 threads x 4 x 8 = 8192 columns
  pdl_trigger();
  pdl_wait();
  const float* row = x + (size_t)blockIdx.x * P;
  T* out = y + (size_t)blockIdx.x * P;
  const int step = blockDim.x * 8;
  float keep[kKeep][8];
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int c = threadIdx.x * 8 + j * step;
    if (c < P) {
      load8(row + c, keep[j]);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += keep[j][i] * keep[j][i];
    }
  }
  for (int c = threadIdx.x * 8 + kKeep * step; c < P; c += step) {
    float v[8];
    load8(row + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
  }
  const float rr = rsqrtf(block_sum32(ss, red) / (float)W + eps);
#pragma unroll
  for (int j = 0; j < kKeep; ++j) {
    const int c = threadIdx.x * 8 + j * step;
    if (c < P) {
      float g[8];
      load8(w + c, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) g[i] *= keep[j][i] * rr;
      store8(out + c, g);
    }
  }
  for (int c = threadIdx.x * 8 + kKeep * step; c < P; c += step) {
    float v[8], g[8];
    load8(row + c, v);
    load8(w + c, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= rr * g[i];
    store8(out + c, v);
  }
}

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

// ---------------------------------------------------------------- fp32 matrix product (32-bit mode)
// y[M, N] = x[M, K] W[N, K]^T in plain fp32 FMAs, 64 x 64 tiles, with the epilogues of the tcgen05 product that an fp32
// residual stream uses.  K a multiple of 16.
struct GemmF32Params {
  const float* w;       // [N][K]
  const float* x;       // [M][ldx]
  const float* resid;   // epi 4: [M][ldo]
  float* out;           // [M][ldo]
  float* out2;          // epi 5: [M][ldo2], column (n - n_split) / 2 for the pairs of rows from n_split on
  int M, N, K, ldx, ldo, ldo2, n_split, epi;
  float scale, glu_limit, glu_alpha, glu_bias;
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ GemmF32Params p) {
  __shared__ float xs[16][68], ws[16][68];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  const float* xrow = p.x + (size_t)min(m0 + lr, p.M - 1) * p.ldx;
  const float* wrow = p.w + (size_t)min(n0 + lr, p.N - 1) * p.K;
  pdl_trigger();
  pdl_wait();
  float acc[4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += 16) {
    const float4 a = *reinterpret_cast<const float4*>(xrow + k0 + lk), b = *reinterpret_cast<const float4*>(wrow + k0 + lk);
    xs[lk][lr] = a.x; xs[lk + 1][lr] = a.y; xs[lk + 2][lr] = a.z; xs[lk + 3][lr] = a.w;
    ws[lk][lr] = b.x; ws[lk + 1][lr] = b.y; ws[lk + 2][lr] = b.z; ws[lk + 3][lr] = b.w;
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 u = *reinterpret_cast<const float4*>(&xs[k][ty * 4]), v = *reinterpret_cast<const float4*>(&ws[k][tx * 4]);
      const float xm[4] = {u.x, u.y, u.z, u.w}, wn[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xm[i], wn[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.M) continue;
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      if (p.epi == 5 && n >= p.n_split) {               // (gate, up) pair
        const float g = fminf(acc[i][j], p.glu_limit), u = fminf(fmaxf(acc[i][j + 1], -p.glu_limit), p.glu_limit);
        p.out2[(size_t)m * p.ldo2 + ((n - p.n_split) >> 1)] = g * sigmoid_exact(p.glu_alpha * g) * (u + p.glu_bias);
        continue;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (n + e >= p.N) continue;
        const size_t at = (size_t)m * p.ldo + n + e;
        p.out[at] = p.epi == 4 ? p.resid[at] + acc[i][j + e] : acc[i][j + e] * p.scale;
      }
    }
  }
}

}  // namespace ti

extern "C" {

// f32 selects the activation / table type: 0 bf16, 1 float.  P: row pitch (a multiple of 8), W: true width.
int ti_embed_pos(const void* ids, const void* positions, const void* embed, const void* pos, const void* w, void* x, int M,
                 int W, int P, int vocab, int max_pos, float eps, void* step, int f32, void* stream) {
  if (M <= 0) return 0;
  if (P % 8 || W > P || vocab < 1 || (pos != nullptr && max_pos < 1)) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    ti::launch_kernel(ti::embed_pos_kernel<float>, dim3(M), dim3(256), 0, st, true, (const long long*)ids, (const int*)positions,
                      (const float*)embed, (const float*)pos, (const float*)w, (float*)x, W, P, vocab, max_pos, eps, (unsigned*)step);
  else
    ti::launch_kernel(ti::embed_pos_kernel<ti::bf16>, dim3(M), dim3(256), 0, st, true, (const long long*)ids, (const int*)positions,
                      (const ti::bf16*)embed, (const ti::bf16*)pos, (const float*)w, (float*)x, W, P, vocab, max_pos, eps, (unsigned*)step);
  return (int)cudaGetLastError();
}

int ti_rmsnorm_f32(const void* x, const void* w, void* y, int M, int W, int P, float eps, int f32, void* stream) {
  if (M <= 0) return 0;
  if (P % 8 || W > P) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  const dim3 block(P >= 2048 ? 256 : 128);
  if (f32)
    ti::launch_kernel(ti::rmsnorm_f32_kernel<float>, dim3(M), block, 0, st, true, (const float*)x, (const float*)w, (float*)y, W, P, eps);
  else
    ti::launch_kernel(ti::rmsnorm_f32_kernel<ti::bf16>, dim3(M), block, 0, st, true, (const float*)x, (const float*)w, (ti::bf16*)y, W, P, eps);
  return (int)cudaGetLastError();
}

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

int ti_gemm_f32(const void* w, const void* x, const void* resid, void* out, void* out2, int M, int N, int K, int ldx, int ldo,
                int ldo2, int n_split, int epi, float scale, float glu_limit, float glu_alpha, float glu_bias, void* stream) {
  if (M <= 0) return 0;
  if (K % 16 || ldx % 4 || n_split % 2 || (epi != 3 && epi != 4 && epi != 5)) return -2;
  ti::GemmF32Params p = {(const float*)w, (const float*)x, (const float*)resid, (float*)out, (float*)out2, M, N, K, ldx, ldo,
                         ldo2, n_split, epi, scale, glu_limit, glu_alpha, glu_bias};
  ti::launch_kernel(ti::gemm_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, (cudaStream_t)stream, true, p);
  return (int)cudaGetLastError();
}

}  // extern "C"
