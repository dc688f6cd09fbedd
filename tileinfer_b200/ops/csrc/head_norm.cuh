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

// a warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) head_norm_kernel(const __grid_constant__ HeadNormParams p, int items) {
  const int item = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, dv = p.dv;
  pdl_trigger();
  pdl_wait();
  if (item >= items) return;
  const int t = item / p.H, h = item - t * p.H;
  const float* o = p.o + (size_t)t * p.H * dv + h * dv;
  const float* norm = p.norm + (size_t)h * p.norm_stride;
  const T* g = static_cast<const T*>(p.gate) + (size_t)t * p.ld + p.g_col + h * dv;
  T* out = static_cast<T*>(p.out) + (size_t)t * p.ldo + h * dv;
  float ss = 0.f;
  for (int c = lane * 8; c < dv; c += 256) {
    float v[8];
    load8(o + c, v);
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += v[i] * v[i];
  }
  const float rr = rsqrtf(warp_sum(ss) / (float)p.vdim + p.eps);
  for (int c = lane * 8; c < dv; c += 256) {
    float v[8], w[8], z[8];
    load8(o + c, v);
    load8(norm + c, w);
    load8(g + c, z);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= rr * w[i] * sigmoid_exact(z[i]) * (p.silu ? z[i] : 1.f);
    store8(out + c, v);
  }
}

inline int launch_head_norm(const HeadNormParams& p, int T, int f32, cudaStream_t st) {
  if (T <= 0) return 0;
  if (p.dv % 64 || p.ld % 8 || p.ldo % 8 || p.g_col % 8 || p.norm_stride % 4 || (((uintptr_t)p.gate | (uintptr_t)p.out | (uintptr_t)p.o | (uintptr_t)p.norm) & 15)) return -2;
  const int items = T * p.H;
  launch_kernel(f32 ? head_norm_kernel<float> : head_norm_kernel<bf16>, dim3((items + 7) / 8), dim3(256), 0, st, true, p, items);
  return (int)cudaGetLastError();
}

}  // namespace ti
