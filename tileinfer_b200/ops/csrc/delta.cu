// The gated and the general delta rule (delta.cuh), token by token.  Decode steps and short portions run here, and all of the
// 32-bit mode; long portions run in chunks (delta_chunk.cu).  A block owns 64 columns of one head's state of one sequence in
// registers while it walks the sequence's tokens; everything but the projections is fp32.
//
// A token takes one pass over the old state: u^T S and (w q)^T S are summed together, and
//     o = (w q)^T S - (p.q) (u^T S) + (c.q) v
// is the read-out of the new state, so that both sums meet behind one barrier.
#include "delta.cuh"
#include "head_norm.cuh"

namespace ti {

constexpr int kW2Smem = 64 * 1024;       // the head's rows of a decay's second matrix go to shared memory if they fit

TI_DEVICE void copy16_async(float* dst, const float* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(smem_u32(dst)), "l"(src));
}

// Threads own the state as (row group of 16, four columns): rows rg + 16 i, i < NR.  For the second product of a general decay
// they are (key channel, part of the ranks).
template <typename T, int NR, bool GENERAL>
__global__ void __launch_bounds__(256, NR <= 4 ? 4 : NR <= 8 ? 3 : 1) delta_step_kernel(const __grid_constant__ DeltaParams p) {
  constexpr int DK = NR * 16, PARTS = DK >= 256 ? 1 : 256 / DK, CH = DK > 256 ? DK / 256 : 1;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float w_s[2][GENERAL ? DK : 1], p_s[2][GENERAL ? DK : 1], u_s[2][DK], c_s[2][GENERAL ? DK : 1], q_s[2][DK];
  __shared__ float z_s[GENERAL ? PARTS : 1][GENERAL ? DK : 1], x_s[GENERAL ? 256 : 1];
  __shared__ __align__(16) float red[2][8][128];
  __shared__ float dots[2][8][2];
  const int tid = threadIdx.x, rg = tid >> 4, cq = (tid & 15) * 4, warp = tid >> 5, lane = tid & 31;
  const int col0 = blockIdx.x * 64, h = blockIdx.y, s = p.seqs == nullptr ? (int)blockIdx.z : p.seqs[blockIdx.z];
  const int dv = gridDim.x * 64, kh = h / p.rep;
  float* state = p.state + (((size_t)p.slots[s] * p.H + h) * DK) * dv + col0 + cq;
  float4 S[NR];
#pragma unroll
  for (int i = 0; i < NR; ++i) S[i] = *reinterpret_cast<const float4*>(state + (size_t)(rg + 16 * i) * dv);
  // ranks of this thread: r0 + PARTS i
  const int ch = PARTS > 1 ? tid % DK : tid, r0 = PARTS > 1 ? tid / DK : 0, cols = p.H * DK;
  const float* w2 = GENERAL ? p.w2 + h * DK : nullptr;
  int w2_ld = cols;
  if (GENERAL && (size_t)p.R * DK * 4 <= kW2Smem) {
    float* dst = reinterpret_cast<float*>(smem);           // [R][DK]
    for (int i = tid * 4; i < p.R * DK; i += 1024) copy16_async(dst + i, w2 + (size_t)(i / DK) * cols + i % DK);
    w2 = dst;
    w2_ld = DK;
  }
  pdl_trigger();
  pdl_wait();                                              // the inputs come from the kernels before
  const int t0 = p.cu == nullptr ? s : p.cu[s], t1 = p.cu == nullptr ? s + 1 : p.cu[s + 1];
  if (GENERAL) asm volatile("cp.async.wait_all;\n" ::: "memory");            // visible behind the first barrier
  for (int t = t0; t < t1; ++t) {
    const int b = t & 1;
    const T* src = static_cast<const T*>(p.src) + (size_t)t * p.lds;
    const T* row = static_cast<const T*>(p.proj) + (size_t)t * p.ld;
    const T *kp = src + p.k_col + kh * DK, *qp = src + p.q_col + kh * DK;
    float z[CH];
    if (GENERAL) {
      // z = W_2 tanh(x) + w_0, 256 ranks at a time
#pragma unroll
      for (int j = 0; j < CH; ++j) z[j] = 0.f;
      for (int rb = 0; rb < p.R; rb += 256) {
        if (rb) __syncthreads();
        if (rb + tid < p.R) x_s[tid] = tanhf(to_f<T>(row[p.a_col + rb + tid]));
        __syncthreads();
        const int rn = min(256, p.R - rb);
#pragma unroll 4
        for (int r = r0; r < rn; r += PARTS)
#pragma unroll
          for (int j = 0; j < CH; ++j) z[j] = fmaf(w2[(size_t)(rb + r) * w2_ld + ch + 256 * j], x_s[r], z[j]);
      }
      if (PARTS > 1) {
        z_s[r0][ch] = z[0];
        __syncthreads();
        z[0] = 0.f;
        if (tid < DK) {
#pragma unroll
          for (int i = 0; i < PARTS; ++i) z[0] += z_s[i][ch];
        }
      }
    }
    // every warp takes the lengths by itself
    float kk = 0.f, qq = 0.f;
#pragma unroll
    for (int d = lane; d < DK; d += 32) {
      const float k = to_f<T>(kp[d]), q = to_f<T>(qp[d]);
      kk = fmaf(k, k, kk);
      qq = fmaf(q, q, qq);
    }
    const float rk = rsqrtf(warp_sum(kk) + kUnitEps);
    const float qf = GENERAL ? 1.f : rsqrtf(warp_sum(qq) + kUnitEps) * p.q_scale;
    float g = 1.f, beta = 1.f;
    if (!GENERAL) {
      g = expf(p.neg_a[h] * softplus_exact(to_f<T>(row[p.a_col + h]) + p.bias[h]));
      beta = sigmoid_exact(to_f<T>(row[p.b_col + h]));
    }
#pragma unroll
    for (int j = 0; j < CH; ++j) {
      const int d = tid + 256 * j;
      if (d >= DK) continue;
      const float k = to_f<T>(kp[d]), u = k * rk;
      u_s[b][d] = u;
      q_s[b][d] = to_f<T>(qp[d]) * qf;
      if (GENERAL) {
        const int col = h * DK + d;
        w_s[b][d] = expf(-p.decay_scale * sigmoid_exact(z[j] + p.w0[col]));
        p_s[b][d] = sigmoid_exact(to_f<T>(row[p.b_col + col]) + p.bias[col]) * u;
        c_s[b][d] = k;
      }
    }
    const T* vp = src + p.v_col + h * dv + col0;
    const float4 v = make_float4(to_f<T>(vp[cq]), to_f<T>(vp[cq + 1]), to_f<T>(vp[cq + 2]), to_f<T>(vp[cq + 3]));
    __syncthreads();
    float4 y = make_float4(0.f, 0.f, 0.f, 0.f), o = y;
    float pq = 0.f, cd = 0.f;                              // p.q and c.q
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 16 * i;
      const float u = u_s[b][d], q = q_s[b][d], wq = (GENERAL ? w_s[b][d] : g) * q;
      pq = fmaf(GENERAL ? p_s[b][d] : u, q, pq);
      if (GENERAL) cd = fmaf(c_s[b][d], q, cd);
      y.x = fmaf(u, S[i].x, y.x); y.y = fmaf(u, S[i].y, y.y);
      y.z = fmaf(u, S[i].z, y.z); y.w = fmaf(u, S[i].w, y.w);
      o.x = fmaf(wq, S[i].x, o.x); o.y = fmaf(wq, S[i].y, o.y);
      o.z = fmaf(wq, S[i].z, o.z); o.w = fmaf(wq, S[i].w, o.w);
    }
    y.x += __shfl_xor_sync(0xffffffffu, y.x, 16); y.y += __shfl_xor_sync(0xffffffffu, y.y, 16);
    y.z += __shfl_xor_sync(0xffffffffu, y.z, 16); y.w += __shfl_xor_sync(0xffffffffu, y.w, 16);
    o.x += __shfl_xor_sync(0xffffffffu, o.x, 16); o.y += __shfl_xor_sync(0xffffffffu, o.y, 16);
    o.z += __shfl_xor_sync(0xffffffffu, o.z, 16); o.w += __shfl_xor_sync(0xffffffffu, o.w, 16);
    pq += __shfl_xor_sync(0xffffffffu, pq, 16);
    cd += __shfl_xor_sync(0xffffffffu, cd, 16);
    *reinterpret_cast<float4*>(&red[b][warp][(lane < 16 ? 0 : 64) + cq]) = lane < 16 ? y : o;
    if (lane == 0) { dots[b][warp][0] = pq; dots[b][warp][1] = cd; }
    __syncthreads();
    y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 8; ++w) {
      const float4 a = *reinterpret_cast<const float4*>(&red[b][w][cq]);
      y.x += a.x; y.y += a.y; y.z += a.z; y.w += a.w;
    }
    if (tid < 64) {
      float yt = 0.f, ot = 0.f, pt = 0.f, ct = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        yt += red[b][w][tid];
        ot += red[b][w][64 + tid];
        pt += dots[b][w][0];
        ct += dots[b][w][1];
      }
      const float vt = to_f<T>(vp[tid]);
      p.o[(size_t)t * p.H * dv + h * dv + col0 + tid] = GENERAL ? fmaf(ct, vt, fmaf(-pt, yt, ot)) : fmaf(pt * beta, fmaf(-g, yt, vt), ot);
    }
    // gated: S <- g S + u (beta (v - g y))
    const float4 n = make_float4(beta * fmaf(-g, y.x, v.x), beta * fmaf(-g, y.y, v.y), beta * fmaf(-g, y.z, v.z), beta * fmaf(-g, y.w, v.w));
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int d = rg + 16 * i;
      if (GENERAL) {
        const float w = w_s[b][d], c = c_s[b][d], r = -p_s[b][d];
        S[i].x = fmaf(w, S[i].x, fmaf(r, y.x, c * v.x)); S[i].y = fmaf(w, S[i].y, fmaf(r, y.y, c * v.y));
        S[i].z = fmaf(w, S[i].z, fmaf(r, y.z, c * v.z)); S[i].w = fmaf(w, S[i].w, fmaf(r, y.w, c * v.w));
      } else {
        const float u = u_s[b][d];
        S[i].x = fmaf(g, S[i].x, u * n.x); S[i].y = fmaf(g, S[i].y, u * n.y);
        S[i].z = fmaf(g, S[i].z, u * n.z); S[i].w = fmaf(g, S[i].w, u * n.w);
      }
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

template <typename T, int NR, bool GENERAL>
static void launch_delta_rows(const DeltaParams& p, dim3 grid, cudaStream_t st) {
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(delta_step_kernel<T, NR, GENERAL>, cudaFuncAttributeMaxDynamicSharedMemorySize, kW2Smem);
    configured = true;
  }
  const size_t need = GENERAL ? (size_t)p.R * NR * 64 : 0;
  launch_kernel(delta_step_kernel<T, NR, GENERAL>, grid, dim3(256), need <= kW2Smem ? need : 0, st, true, p);
}

template <typename T, bool GENERAL>
static int launch_delta(const DeltaParams& p, int S, int DK, int dv, cudaStream_t st) {
  const dim3 grid(dv / 64, p.H, S);
  switch (DK) {
    case 64: launch_delta_rows<T, 4, GENERAL>(p, grid, st); break;
    case 128: launch_delta_rows<T, 8, GENERAL>(p, grid, st); break;
    case 256: launch_delta_rows<T, 16, GENERAL>(p, grid, st); break;
    case 512: launch_delta_rows<T, 32, GENERAL>(p, grid, st); break;
    default: return -3;
  }
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_delta_params_size() { return (int)sizeof(ti::DeltaParams); }
int ti_head_norm_params_size() { return (int)sizeof(ti::HeadNormParams); }

// o[t, h] and the states for the tokens cu[s] .. cu[s+1] of the S sequences (all, or those of `seqs`; cu null: one token each)
int ti_delta_step(const ti::DeltaParams* p, int S, int dk, int dv, int general, int f32, void* stream) {
  if (S <= 0) return 0;
  if (dv % 64 || p->rep < 1 || p->H % p->rep || (general && (p->R < 1 || p->rep != 1 || ((uintptr_t)p->w2 & 15))) || ((uintptr_t)p->state & 15)) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (general) return f32 ? ti::launch_delta<float, true>(*p, S, dk, dv, st) : ti::launch_delta<ti::bf16, true>(*p, S, dk, dv, st);
  return f32 ? ti::launch_delta<float, false>(*p, S, dk, dv, st) : ti::launch_delta<ti::bf16, false>(*p, S, dk, dv, st);
}

// out[t, h] = rmsnorm(o[t, h]) * norm * gate
int ti_head_norm(const ti::HeadNormParams* p, int T, int f32, void* stream) { return ti::launch_head_norm(*p, T, f32, (cudaStream_t)stream); }

}  // extern "C"
