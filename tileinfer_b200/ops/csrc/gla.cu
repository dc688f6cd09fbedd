// Gated linear attention, token by token: a state S [dim, vdim] per head decays per key channel and takes one outer product
// per token,
//     a_t = sigmoid(W_a2 x_t + b)^(1/tau)      S <- diag(a_t) S + k_t v_t^T      o_t = S^T q_t / sqrt(dim)
// with x_t the narrow inner product of the decay.  Decode steps and short portions run here; long portions run in chunks
// (gla_chunk.cu).  A block owns 64 columns of one head's state of one sequence in registers while it walks the sequence's
// tokens; everything but the projections is fp32.  `head_norm_kernel` applies the head's RMSNorm and the silu gate.
#include "gla.cuh"
#include "head_norm.cuh"

namespace ti {

// thread = (row group of 16, four columns): rows rg + 16 i, i < NR
template <typename T, int NR>
__global__ void __launch_bounds__(256) gla_step_kernel(const __grid_constant__ GlaParams p) {
  constexpr int DK = NR * 16;
  __shared__ float a_s[2][DK], k_s[2][DK], q_s[2][DK];
  __shared__ __align__(16) float red[2][8][64];
  const int tid = threadIdx.x, rg = tid >> 4, cq = (tid & 15) * 4, warp = tid >> 5, lane = tid & 31;
  const int col0 = blockIdx.x * 64, h = blockIdx.y, s = p.seqs == nullptr ? (int)blockIdx.z : p.seqs[blockIdx.z];
  const int dv = gridDim.x * 64;
  float* state = p.state + (((size_t)p.slots[s] * p.H + h) * DK) * dv + col0 + cq;
  float4 S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = *reinterpret_cast<const float4*>(state + (size_t)(rg + 16 * i) * dv);
  pdl_trigger();
  pdl_wait();                                              // the projections come from the kernel before
  const int t0 = p.cu == nullptr ? s : p.cu[s], t1 = p.cu == nullptr ? s + 1 : p.cu[s + 1];
  const T* proj = static_cast<const T*>(p.proj);
  for (int t = t0; t < t1; ++t) {
    const int b = t & 1;
    const T* row = proj + (size_t)t * p.ld;
    for (int d = tid; d < DK; d += 256) {
      a_s[b][d] = expf(gla_log_decay(p, row, h * DK + d, p.H * DK));
      k_s[b][d] = to_f<T>(row[p.k_col + h * DK + d]);
      q_s[b][d] = to_f<T>(row[p.q_col + h * DK + d]) * p.q_scale;
    }
    const T* vp = row + p.v_col + h * dv + col0 + cq;
    const float4 v = make_float4(to_f<T>(vp[0]), to_f<T>(vp[1]), to_f<T>(vp[2]), to_f<T>(vp[3]));
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 16 * i;
      const float a = a_s[b][d], k = k_s[b][d], q = q_s[b][d];
      S[i].x = fmaf(a, S[i].x, k * v.x); S[i].y = fmaf(a, S[i].y, k * v.y);
      S[i].z = fmaf(a, S[i].z, k * v.z); S[i].w = fmaf(a, S[i].w, k * v.w);
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
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) sum += red[b][w][tid];
      p.o[(size_t)t * p.H * dv + h * dv + col0 + tid] = sum;
    }
    for (int j = 0; j < p.num_snap; ++j) {                 // snapshot points of this sequence
      if (p.snap_rel[s * p.num_snap + j] != t - t0 + 1) continue;
      float* dst = p.snap + (((size_t)p.snap_idx[s * p.num_snap + j] * p.H + h) * DK) * dv + col0 + cq;
#pragma unroll
      for (int i = 0; i < NR; ++i) *reinterpret_cast<float4*>(dst + (size_t)(rg + 16 * i) * dv) = S[i];
    }
  }
#pragma unroll
  for (int i = 0; i < NR; ++i) *reinterpret_cast<float4*>(state + (size_t)(rg + 16 * i) * dv) = S[i];
}

template <typename T>
static int launch_step(const GlaParams& p, int S, int DK, int dv, cudaStream_t st) {
  const dim3 grid(dv / 64, p.H, S);
  switch (DK) {
    case 64: launch_kernel(gla_step_kernel<T, 4>, grid, dim3(256), 0, st, true, p); break;
    case 128: launch_kernel(gla_step_kernel<T, 8>, grid, dim3(256), 0, st, true, p); break;
    case 256: launch_kernel(gla_step_kernel<T, 16>, grid, dim3(256), 0, st, true, p); break;
    case 512: launch_kernel(gla_step_kernel<T, 32>, grid, dim3(256), 0, st, true, p); break;
    default: return -3;
  }
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_gla_params_size() { return (int)sizeof(ti::GlaParams); }

static bool gla_aligned(const ti::GlaParams* p) {
  return p->ld % 8 == 0 && p->ldo % 8 == 0 && p->q_col % 8 == 0 && p->k_col % 8 == 0 && p->v_col % 8 == 0 && p->g_col % 8 == 0 &&
         (((uintptr_t)p->proj | (uintptr_t)p->out | (uintptr_t)p->o | (uintptr_t)p->state) & 15) == 0;
}

// o[t, h] and the states for the tokens cu[s] .. cu[s+1] of the S sequences (all, or those of `seqs`; cu null: one token each)
int ti_gla_step(const ti::GlaParams* p, int S, int dk, int dv, int f32, void* stream) {
  if (S <= 0) return 0;
  if (dv % 64 || !gla_aligned(p)) return -2;
  return f32 ? ti::launch_step<float>(*p, S, dk, dv, (cudaStream_t)stream) : ti::launch_step<ti::bf16>(*p, S, dk, dv, (cudaStream_t)stream);
}

// out[t, h] = rmsnorm(o[t, h]) * norm * silu(gate)
int ti_gla_finish(const ti::GlaParams* p, int T, int dv, int f32, void* stream) {
  const ti::HeadNormParams n = {p->o, p->proj, p->norm, p->out, p->ld, p->ldo, p->g_col, p->H, dv, p->vdim, 0, 1, p->eps};
  return ti::launch_head_norm(n, T, f32, (cudaStream_t)stream);
}

}  // extern "C"
