// State-space mixer (Mamba-2, Dao and Gu), token by token: a state S [Np, V] per head,
//     S <- exp(-exp(A_log) dt) S + dt B x^T      y = S^T C + D x
// with B and C shared by the heads of a group.  Decode steps and short portions run here; long portions run in chunks
// (ssd_chunk.cu).  A block owns 64 columns of one head's state of one sequence in registers while it walks the sequence's
// tokens; step sizes, decays and states are fp32.  `ssd_finish_kernel` applies silu(z) and then the norm of equal parts.
#include "ssd.cuh"

namespace ti {

// thread = (row group of 16, four columns): rows rg + 16 i, i < NR
template <typename T, int NR>
__global__ void __launch_bounds__(256) ssd_step_kernel(const __grid_constant__ SsdParams p) {
  constexpr int NP = NR * 16;
  __shared__ float b_s[2][NP], c_s[2][NP];
  __shared__ __align__(16) float red[2][8][64];
  const int tid = threadIdx.x, rg = tid >> 4, cq = (tid & 15) * 4, warp = tid >> 5, lane = tid & 31;
  const int col0 = blockIdx.x * 64, h = blockIdx.y, s = p.seqs == nullptr ? (int)blockIdx.z : p.seqs[blockIdx.z];
  const int vp = p.vp, grp = h / (p.H / p.G);
  float* state = p.state + (((size_t)p.slots[s] * p.H + h) * NP) * vp + col0 + cq;
  float4 S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = *reinterpret_cast<const float4*>(state + (size_t)(rg + 16 * i) * vp);
  pdl_trigger();
  pdl_wait();                                              // the inputs come from the kernels before
  const int t0 = p.cu == nullptr ? s : p.cu[s], t1 = p.cu == nullptr ? s + 1 : p.cu[s + 1];
  for (int t = t0; t < t1; ++t) {
    const int b = t & 1;
    const T* row = static_cast<const T*>(p.xbc) + (size_t)t * p.ldx;
    for (int n = tid; n < NP; n += 256) {
      b_s[b][n] = to_f<T>(row[p.b_col + grp * NP + n]);
      c_s[b][n] = to_f<T>(row[p.c_col + grp * NP + n]);
    }
    const float dt = ssd_step_size(p, static_cast<const T*>(p.proj) + (size_t)t * p.ld, h), a = expf(p.neg_a[h] * dt);
    const T* xp = row + p.x_col + h * vp + col0;
    const float4 x = make_float4(dt * to_f<T>(xp[cq]), dt * to_f<T>(xp[cq + 1]), dt * to_f<T>(xp[cq + 2]), dt * to_f<T>(xp[cq + 3]));
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const float k = b_s[b][rg + 16 * i], q = c_s[b][rg + 16 * i];
      S[i].x = fmaf(a, S[i].x, k * x.x); S[i].y = fmaf(a, S[i].y, k * x.y);
      S[i].z = fmaf(a, S[i].z, k * x.z); S[i].w = fmaf(a, S[i].w, k * x.w);
      o.x = fmaf(q, S[i].x, o.x); o.y = fmaf(q, S[i].y, o.y);
      o.z = fmaf(q, S[i].z, o.z); o.w = fmaf(q, S[i].w, o.w);
    }
    o.x += __shfl_xor_sync(0xffffffffu, o.x, 16);
    o.y += __shfl_xor_sync(0xffffffffu, o.y, 16);
    o.z += __shfl_xor_sync(0xffffffffu, o.z, 16);
    o.w += __shfl_xor_sync(0xffffffffu, o.w, 16);
    if (lane < 16) *reinterpret_cast<float4*>(&red[b][warp][cq]) = o;
    __syncthreads();
    if (tid < 64) {
      float sum = p.D[h] * to_f<T>(xp[tid]);
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[b][w][tid];
      p.y[(size_t)t * p.H * vp + h * vp + col0 + tid] = sum;
    }
    for (int j = 0; j < p.num_snap; ++j) {                 // snapshot points of this sequence
      if (p.snap_rel[s * p.num_snap + j] != t - t0 + 1) continue;
      float* dst = p.snap + (((size_t)p.snap_idx[s * p.num_snap + j] * p.H + h) * NP) * vp + col0 + cq;
#pragma unroll
      for (int i = 0; i < NR; ++i) *reinterpret_cast<float4*>(dst + (size_t)(rg + 16 * i) * vp) = S[i];
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) *reinterpret_cast<float4*>(state + (size_t)(rg + 16 * i) * vp) = S[i];
}

// out = norm(y * silu(z)) in equal parts of the true channels; a block per (token, part).  Channel i is column i % V of head
// i / V.  VEC 8 when a part and a head are whole vectors.
template <typename T, int VEC>
__global__ void __launch_bounds__(128) ssd_finish_kernel(const __grid_constant__ SsdParams p) {
  constexpr int KEEP = 2;
  __shared__ float red[4];
  const int t = blockIdx.x, len = p.H * p.V / p.norm_groups, first = blockIdx.y * len, step = 128 * VEC;
  pdl_trigger();
  pdl_wait();
  const float* y = p.y + (size_t)t * p.H * p.vp;
  const T* z = static_cast<const T*>(p.proj) + (size_t)t * p.ld + p.z_col;
  T* out = static_cast<T*>(p.out) + (size_t)t * p.ldo;
  auto gated = [&](int at, float (&v)[VEC]) {
    if constexpr (VEC == 8) {
      float g[8];
      load8(y + at, v);
      load8(z + at, g);
#pragma unroll
      for (int k = 0; k < 8; ++k) v[k] *= g[k] * sigmoid_exact(g[k]);
    } else {
      const float g = to_f<T>(z[at]);
      v[0] = y[at] * g * sigmoid_exact(g);
    }
  };
  auto place = [&](int i) {
    const int h = i / p.V;
    return h * p.vp + i - h * p.V;
  };
  float v[KEEP][VEC], ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int i = threadIdx.x * VEC + j * step;
    if (i >= len) continue;
    gated(place(first + i), v[j]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += v[j][k] * v[j][k];
  }
  for (int i = threadIdx.x * VEC + KEEP * step; i < len; i += step) {
    float u[VEC];
    gated(place(first + i), u);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += u[k] * u[k];
  }
  const float rr = rsqrtf(block_sum32(ss, red) / (float)len + p.eps);
  auto put = [&](int i, float (&u)[VEC]) {
    const int at = place(first + i), off = (first + i) % p.V;
    if constexpr (VEC == 8) {
      float w[8];
      load8(p.norm + at, w);
#pragma unroll
      for (int k = 0; k < 8; ++k) u[k] *= rr * w[k];
      store8(out + at, u);
    } else {
      out[at] = from_f<T>(u[0] * rr * p.norm[at]);
    }
    if (off + VEC == p.V)                                  // the end of a head: its padding holds zeros
      for (int k = VEC; k < p.vp - p.V + VEC; ++k) out[at + k] = from_f<T>(0.f);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if ((int)threadIdx.x * VEC + j * step < len) put(threadIdx.x * VEC + j * step, v[j]);
  for (int i = threadIdx.x * VEC + KEEP * step; i < len; i += step) {
    float u[VEC];
    gated(place(first + i), u);
    put(i, u);
  }
}

template <typename T>
static int launch_step(const SsdParams& p, int S, int Np, cudaStream_t st) {
  const dim3 grid(p.vp / 64, p.H, S);
  switch (Np) {
    case 64: launch_kernel(ssd_step_kernel<T, 4>, grid, dim3(256), 0, st, true, p); break;
    case 128: launch_kernel(ssd_step_kernel<T, 8>, grid, dim3(256), 0, st, true, p); break;
    case 256: launch_kernel(ssd_step_kernel<T, 16>, grid, dim3(256), 0, st, true, p); break;
    case 512: launch_kernel(ssd_step_kernel<T, 32>, grid, dim3(256), 0, st, true, p); break;
    default: return -3;
  }
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_finish(const SsdParams& p, int M, cudaStream_t st) {
  const bool vec = p.V % 8 == 0 && (p.H * p.V / p.norm_groups) % 8 == 0;
  launch_kernel(vec ? ssd_finish_kernel<T, 8> : ssd_finish_kernel<T, 1>, dim3(M, p.norm_groups), dim3(128), 0, st, true, p);
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_ssd_params_size() { return (int)sizeof(ti::SsdParams); }

static bool ssd_fits(const ti::SsdParams* p) {
  return p->ld % 8 == 0 && p->ldx % 8 == 0 && p->ldo % 8 == 0 && p->vp % 64 == 0 && p->V >= 1 && p->V <= p->vp && p->G >= 1 &&
         p->H % p->G == 0 && p->norm_groups >= 1 && (p->H * p->V) % p->norm_groups == 0 && p->z_col % 8 == 0 && p->x_col % 8 == 0 &&
         p->b_col % 8 == 0 && p->c_col % 8 == 0 &&
         (((uintptr_t)p->proj | (uintptr_t)p->xbc | (uintptr_t)p->out | (uintptr_t)p->y | (uintptr_t)p->state | (uintptr_t)p->norm) & 15) == 0;
}

// y[t, h] and the states for the tokens cu[s] .. cu[s+1] of the S sequences (all, or those of `seqs`; cu null: one token each).
// Np: padded state size (64, 128, 256 or 512).
int ti_ssd_step(const ti::SsdParams* p, int S, int Np, int f32, void* stream) {
  if (S <= 0) return 0;
  if (!ssd_fits(p)) return -2;
  return f32 ? ti::launch_step<float>(*p, S, Np, (cudaStream_t)stream) : ti::launch_step<ti::bf16>(*p, S, Np, (cudaStream_t)stream);
}

// out[t] = norm(y[t] * silu(z[t])) for M tokens
int ti_ssd_finish(const ti::SsdParams* p, int M, int f32, void* stream) {
  if (M <= 0) return 0;
  if (!ssd_fits(p)) return -2;
  return f32 ? ti::launch_finish<float>(*p, M, (cudaStream_t)stream) : ti::launch_finish<ti::bf16>(*p, M, (cudaStream_t)stream);
}

}  // extern "C"
