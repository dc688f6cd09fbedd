// Vector access to rows of bf16 or float (eight elements per thread) and a block-wide sum, shared by the row operations.
#pragma once
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
template <typename T> TI_DEVICE T from_f(float v);
template <> TI_DEVICE bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }
template <> TI_DEVICE float from_f<float>(float v) { return v; }
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

}  // namespace ti
