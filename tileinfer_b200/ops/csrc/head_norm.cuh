// The end of a recurrent mixer: every head's output divided by its root mean square, times a weight, times a gate.
#pragma once
#include "row_vec.cuh"

namespace ti {

struct HeadNormParams {
  const float* o;          // [T][H * dv]
  const void* gate;        // [T, ld]: column g_col + h * dv + d
  const float* norm;       // weight of head h's column d at h * norm_stride + d
  void* out;               // [T, ldo], head h at column h * dv
  int ld, ldo, g_col, H, dv, vdim, norm_stride;
  int silu;                // 1: silu(gate), 0: sigmoid(gate)
  float eps;
};

// LPI lanes per (token, head), eight columns each at a time
template <typename T, int LPI>
__global__ void __launch_bounds__(256) head_norm_kernel(const __grid_constant__ HeadNormParams p, int items) {
  const int item = (blockIdx.x * 256 + threadIdx.x) / LPI, lane = threadIdx.x & (LPI - 1), dv = p.dv;
  pdl_trigger();
  pdl_wait();
  const bool live = item < items;                          // the lanes of a warp meet in the shuffles
  const int t = live ? item / p.H : 0, h = live ? item - t * p.H : 0;
  const float* o = p.o + (size_t)t * p.H * dv + h * dv;
  const float* norm = p.norm + (size_t)h * p.norm_stride;
  const T* g = static_cast<const T*>(p.gate) + (size_t)t * p.ld + p.g_col + h * dv;
  T* out = static_cast<T*>(p.out) + (size_t)t * p.ldo + h * dv;
  float v[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, z[8], ss = 0.f;
  if (LPI < 32 || lane * 8 < dv) {
    load8(o + lane * 8, v);
    load8(g + lane * 8, z);
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
  if (LPI == 32)
    for (int c = lane * 8 + 256; c < dv; c += 256) {
      float u[8];
      load8(o + c, u);
#pragma unroll
      for (int i = 0; i < 8; ++i) ss += u[i] * u[i];
    }
#pragma unroll
  for (int s = LPI / 2; s > 0; s >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, s);
  if (!live) return;
  const float rr = rsqrtf(ss / (float)p.vdim + p.eps);
  for (int c = lane * 8; c < dv; c += LPI * 8) {
    float w[8];
    load8(norm + c, w);
    if (LPI == 32 && c >= 256) {
      load8(o + c, v);
      load8(g + c, z);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= rr * w[i] * sigmoid_exact(z[i]) * (p.silu ? z[i] : 1.f);
    store8(out + c, v);
  }
}

inline int launch_head_norm(const HeadNormParams& p, int T, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (p.dv % 64 || p.ld % 8 || p.ldo % 8 || p.g_col % 8 || p.norm_stride % 4 || (((uintptr_t)p.gate | (uintptr_t)p.out | (uintptr_t)p.o | (uintptr_t)p.norm) & 15)) return -2;
  const int items = T * p.H;
#define TI_HN(L)                                                                                                           \
  launch_kernel(f32 ? head_norm_kernel<float, L> : head_norm_kernel<bf16, L>, dim3((items + 256 / L - 1) / (256 / L)), dim3(256), 0, st, true, p, items)
  if (p.dv == 64) TI_HN(8);
  else if (p.dv == 128) TI_HN(16);
  else TI_HN(32);
#undef TI_HN
  return (int)cudaGetLastError();
}

}  // namespace ti
