// Row operations around an fp32 residual stream and the products of the 32-bit mode: token (+ position) embedding with
// an optional norm, plain RMSNorm of fp32 rows, and matrix products in fp32 FMAs.
//
// Every kernel is templated on the activation type (bf16, or float in 32-bit mode).  Row pitches are padded to
// multiples of 64 elements and the pad columns hold zeros (zero weight rows, zero norm weights), so that rows are read
// in whole vectors; means divide by the true length.
#include "resid_norm.cuh"

namespace ti {

// ---------------------------------------------------------------- embedding
// x[m, :] = rmsnorm(embed[ids[m]] + pos[positions[m]]) * w * scale in fp32.  Either of `pos` and `w` may be null (no w: no norm).  With `h`
// the row is stored as T as well.  Block 0 also advances the device step counter.
template <typename T>
__global__ void __launch_bounds__(256) embed_pos_kernel(const long long* __restrict__ ids, const int* __restrict__ positions,
                                                        const T* __restrict__ embed, const T* __restrict__ pos,
                                                        const float* __restrict__ w, float* __restrict__ x, int W, int P,
                                                        int vocab, int max_pos, float eps, float scale, unsigned* step, T* __restrict__ h) {
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
  const float rr = scale * (w == nullptr ? 1.f : rsqrtf(block_sum32(ss, red) / (float)W + eps));
  for (int c = threadIdx.x * 8; c < P; c += blockDim.x * 8) {
    float a[8], b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, g[8] = {1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f, 1.f};
    load8(e + c, a);
    if (q != nullptr) load8(q + c, b);
    if (w != nullptr) load8(w + c, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) a[i] = (a[i] + b[i]) * rr * g[i];
    store8(x + (size_t)m * P + c, a);
    if (h != nullptr) store8(h + (size_t)m * P + c, a);
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

// ---------------------------------------------------------------- sublayer output -> residual -> next sublayer's input
template <typename T, int KEEP, bool ROUTED, bool FEW>
__global__ void __launch_bounds__(256) resid_norm_kernel(const __grid_constant__ ResidNormParams p) {
  __shared__ float red[64];
  float y[KEEP][8];
  pdl_trigger();
  pdl_wait();
  resid_norm_row<T, KEEP, ROUTED, FEW>(p, blockIdx.x, y, red);
}

template <typename T, int KEEP>
__global__ void __launch_bounds__(256) gated_norm_kernel(const __grid_constant__ GatedNormParams p) {
  __shared__ float red[96];
  pdl_trigger();
  pdl_wait();
  gated_norm_row<T, KEEP>(p, blockIdx.x, red);
}

// ---------------------------------------------------------------- fp32 matrix product (32-bit mode)
// y[M, N] = x[M, K] W[N, K]^T in plain fp32 FMAs, 64 x 64 tiles, with the epilogues of the tcgen05 product that an fp32
// residual stream uses.  K a multiple of 16.
struct GemmF32Params {
  const float* w;       // [N][K]
  const float* x;       // [M][ldx]
  const float* resid;   // epi 4: [M][ldo]
  float* out;           // [M][ldo]
  float* out2;          // epi 5: [M][ldo2], column (n - n_split) / 2 for the pairs of rows from n_split on; epi 6: column n - n_split, squared positive part
  int M, N, K, ldx, ldo, ldo2, n_split, epi;
  float scale, glu_limit, glu_alpha, glu_bias;
  // several weight matrices side by side: [3][max_tiles] weight matrix, first row of x, rows (at most 64) of a row tile
  const int* tiles;
  const int* num_tiles;
  int max_tiles;
  float softcap;        // epi 3: > 0 stores softcap * tanh(value / softcap)
  const float* bias;    // null, or [N]
};

__global__ void __launch_bounds__(256) gemm_f32_kernel(const __grid_constant__ GemmF32Params p) {
  __shared__ float xs[16][68], ws[16][68];
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int lr = tid >> 2, lk = (tid & 3) * 4;
  pdl_trigger();
  pdl_wait();
  int m0 = blockIdx.y * 64, m_end = p.M;
  const int n0 = blockIdx.x * 64;
  const float* w = p.w;
  if (p.tiles != nullptr) {
    if ((int)blockIdx.y >= *p.num_tiles) return;
    w += (size_t)p.tiles[blockIdx.y] * p.N * p.K;
    m0 = p.tiles[p.max_tiles + blockIdx.y];
    m_end = m0 + p.tiles[2 * p.max_tiles + blockIdx.y];
  }
  const float* xrow = p.x + (size_t)min(m0 + lr, m_end - 1) * p.ldx;
  const float* wrow = w + (size_t)min(n0 + lr, p.N - 1) * p.K;
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
    if (m >= m_end) continue;
#pragma unroll
    for (int j = 0; j < 4; j += 2) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      if (p.bias != nullptr) {
        acc[i][j] += p.bias[n];
        if (n + 1 < p.N) acc[i][j + 1] += p.bias[n + 1];
      }
      if (p.epi == 5 && n >= p.n_split) {               // (gate, up) pair
        const float g = fminf(acc[i][j], p.glu_limit), u = fminf(fmaxf(acc[i][j + 1], -p.glu_limit), p.glu_limit);
        p.out2[(size_t)m * p.ldo2 + ((n - p.n_split) >> 1)] = g * sigmoid_exact(p.glu_alpha * g) * (u + p.glu_bias);
        continue;
      }
      if (p.epi == 6 && n >= p.n_split) {
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const float v = fmaxf(acc[i][j + e], 0.f);
          if (n + e < p.N) p.out2[(size_t)m * p.ldo2 + n + e - p.n_split] = v * v;
        }
        continue;
      }
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (n + e >= p.N) continue;
        const size_t at = (size_t)m * p.ldo + n + e;
        if (p.epi == 4) {
          p.out[at] = p.resid[at] + acc[i][j + e];
        } else {
          const float v = acc[i][j + e] * p.scale;
          p.out[at] = p.softcap > 0.f ? p.softcap * tanhf(v / p.softcap) : v;
        }
      }
    }
  }
}

}  // namespace ti

extern "C" {

// f32 selects the activation / table type: 0 bf16, 1 float.  P: row pitch (a multiple of 8), W: true width.
int ti_embed_pos(const void* ids, const void* positions, const void* embed, const void* pos, const void* w, void* x, int M,
                 int W, int P, int vocab, int max_pos, float eps, float scale, void* step, void* h, int f32, void* stream) {
  if (M <= 0) return 0;
  if (P % 8 || W > P || vocab < 1 || (pos != nullptr && max_pos < 1)) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    ti::launch_kernel(ti::embed_pos_kernel<float>, dim3(M), dim3(256), 0, st, true, (const long long*)ids, (const int*)positions,
                      (const float*)embed, (const float*)pos, (const float*)w, (float*)x, W, P, vocab, max_pos, eps, scale, (unsigned*)step, (float*)h);
  else
    ti::launch_kernel(ti::embed_pos_kernel<ti::bf16>, dim3(M), dim3(256), 0, st, true, (const long long*)ids, (const int*)positions,
                      (const ti::bf16*)embed, (const ti::bf16*)pos, (const float*)w, (float*)x, W, P, vocab, max_pos, eps, scale, (unsigned*)step, (ti::bf16*)h);
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

int ti_resid_norm_params_size() { return (int)sizeof(ti::ResidNormParams); }

int ti_resid_norm(const ti::ResidNormParams* p, int M, int f32, void* stream) {
  if (M <= 0) return 0;
  if (p->P % 8 || p->ldy % 8 || p->W > p->P || p->P > 256 * 8 * 8) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  // one, two, four or eight vectors per thread
  const int threads = p->P >= 2048 ? 256 : (p->P / 8 + 31) / 32 * 32, keep = (p->P / 8 + threads - 1) / threads;
  const dim3 grid(M), block(threads);
#define TI_RN(T, K)                                                                                                             \
  (p->slot == nullptr ? ti::launch_kernel(ti::resid_norm_kernel<T, K, false, false>, grid, block, 0, st, true, *p)             \
   : M <= 512         ? ti::launch_kernel(ti::resid_norm_kernel<T, K, true, true>, grid, block, 0, st, true, *p)               \
                      : ti::launch_kernel(ti::resid_norm_kernel<T, K, true, false>, grid, block, 0, st, true, *p))
  if (f32) {
    if (keep <= 1) TI_RN(float, 1); else if (keep <= 2) TI_RN(float, 2); else if (keep <= 4) TI_RN(float, 4); else TI_RN(float, 8);
  } else {
    if (keep <= 1) TI_RN(ti::bf16, 1); else if (keep <= 2) TI_RN(ti::bf16, 2); else if (keep <= 4) TI_RN(ti::bf16, 4); else TI_RN(ti::bf16, 8);
  }
#undef TI_RN
  return (int)cudaGetLastError();
}

int ti_gated_norm_params_size() { return (int)sizeof(ti::GatedNormParams); }

int ti_gated_norm(const ti::GatedNormParams* p, int M, int f32, void* stream) {
  if (M <= 0) return 0;
  if (p->P % 8 || p->ldy % 8 || p->ldg % 8 || p->W > p->P || p->P > 256 * 8 * 8 || (p->y2 != nullptr && (p->w_y == nullptr || p->w_y2 == nullptr)) ||
      (((uintptr_t)p->y | (uintptr_t)p->y2 | (uintptr_t)p->gate | (uintptr_t)p->x | (uintptr_t)p->h) & 15))
    return -2;
  cudaStream_t st = (cudaStream_t)stream;
  const int threads = p->P >= 2048 ? 256 : (p->P / 8 + 31) / 32 * 32, keep = (p->P / 8 + threads - 1) / threads;
#define TI_GN(T, K) ti::launch_kernel(ti::gated_norm_kernel<T, K>, dim3(M), dim3(threads), 0, st, true, *p)
  if (f32) {
    if (keep <= 1) TI_GN(float, 1); else if (keep <= 2) TI_GN(float, 2); else if (keep <= 4) TI_GN(float, 4); else TI_GN(float, 8);
  } else {
    if (keep <= 1) TI_GN(ti::bf16, 1); else if (keep <= 2) TI_GN(ti::bf16, 2); else if (keep <= 4) TI_GN(ti::bf16, 4); else TI_GN(ti::bf16, 8);
  }
#undef TI_GN
  return (int)cudaGetLastError();
}

int ti_gemm_f32(const void* w, const void* x, const void* resid, void* out, void* out2, int M, int N, int K, int ldx, int ldo,
                int ldo2, int n_split, int epi, float scale, float glu_limit, float glu_alpha, float glu_bias, const void* tiles,
                const void* num_tiles, int max_tiles, float softcap, const void* bias, void* stream) {
  if (M <= 0) return 0;
  if (K % 16 || ldx % 4 || n_split % 2 || epi < 3 || epi > 6) return -2;
  ti::GemmF32Params p = {(const float*)w, (const float*)x, (const float*)resid, (float*)out, (float*)out2, M, N, K, ldx, ldo,
                         ldo2, n_split, epi, scale, glu_limit, glu_alpha, glu_bias, (const int*)tiles, (const int*)num_tiles, max_tiles, softcap, (const float*)bias};
  ti::launch_kernel(ti::gemm_f32_kernel, dim3((N + 63) / 64, tiles != nullptr ? max_tiles : (M + 63) / 64), dim3(256), 0, (cudaStream_t)stream, true, p);
  return (int)cudaGetLastError();
}

}  // extern "C"
