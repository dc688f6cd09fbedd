// A sublayer's output into the fp32 residual, with the norms on both sides: one row by one block, kept in registers.
#pragma once
#include "row_vec.cuh"

namespace ti {

// x[m] += rmsnorm(y[m]) * w_out (w_out null: x[m] += y[m]; y null as well: x stays), then h[m] = rmsnorm(x[m]) * w_next
// (w_next null: no h).  y[m] is a row, or, with `slot`,
// the weighted sum over k < top of the rows slot[m, k] of y plus the input row h_in[m] times the weights whose slot is
// negative (-1; -2 adds nothing).
struct ResidNormParams {
  const void* y;           // [rows][ldy] or null
  float* x;                // [M][P]
  const float* w_out;      // [P] or null
  const float* w_next;     // [P] or null
  void* h;                 // [M][P]
  const int* slot;         // [M][top] or null
  const float* weight;     // [M][top]
  const void* h_in;        // [M][P]
  int W, P, ldy, top;
  float eps;
};

// KEEP x 8 columns per thread; on return `y` holds the thread's part of h (fp32, before it was stored as T).  `red`: 64
// floats of shared memory.
template <typename T, int KEEP, bool ROUTED, bool FEW = false>
TI_DEVICE void resid_norm_row(const ResidNormParams& p, int m, float (&y)[KEEP][8], float* red) {
  const int step = blockDim.x * 8;
  float* xr = p.x + (size_t)m * p.P;
  float ss = 0.f, x[KEEP][8];
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * 8 + j * step;
#pragma unroll
    for (int i = 0; i < 8; ++i) y[j][i] = 0.f;
    if (c >= p.P) continue;
    if (!ROUTED) {
      load8(xr + c, x[j]);
      if (p.y != nullptr) load8(static_cast<const T*>(p.y) + (size_t)m * p.ldy + c, y[j]);
    } else {
      float own = 0.f;
      int k0 = 0;
      if (FEW) {                                           // four rows in flight: a chain of loads is all such a step is
        for (; k0 + 4 <= p.top; k0 += 4) {
          int sl[4];
          float a[4], v[4][8];
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            sl[k] = p.slot[(size_t)m * p.top + k0 + k];
            a[k] = p.weight[(size_t)m * p.top + k0 + k];
          }
#pragma unroll
          for (int k = 0; k < 4; ++k) load8(static_cast<const T*>(p.y) + (size_t)max(sl[k], 0) * p.ldy + c, v[k]);
#pragma unroll
          for (int k = 0; k < 4; ++k) {
            own += sl[k] == -1 ? a[k] : 0.f;
            // a row that is not the token's may hold anything
#pragma unroll
            for (int i = 0; i < 8; ++i) y[j][i] = sl[k] < 0 ? y[j][i] : fmaf(a[k], v[k][i], y[j][i]);
          }
        }
      }
      for (int k = k0; k < p.top; ++k) {
        const int sl = p.slot[(size_t)m * p.top + k];
        const float a = p.weight[(size_t)m * p.top + k];
        if (sl == -1) own += a;
        if (sl < 0) continue;
        float v[8];
        load8(static_cast<const T*>(p.y) + (size_t)sl * p.ldy + c, v);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[j][i] = fmaf(a, v[i], y[j][i]);
      }
      if (own != 0.f) {
        float v[8];
        load8(static_cast<const T*>(p.h_in) + (size_t)m * p.P + c, v);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[j][i] = fmaf(own, v[i], y[j][i]);
      }
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += y[j][i] * y[j][i];
  }
  const bool normed = p.w_out != nullptr;                  // uniform over the grid
  const float ry = normed ? rsqrtf(block_sum32(ss, red) / (float)p.W + p.eps) : 1.f;
  ss = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * 8 + j * step;
    if (c >= p.P) continue;
    float g[8];
    if (ROUTED) load8(xr + c, x[j]);                       // later: the sum above needs the registers
    if (normed) {
      load8(p.w_out + c, g);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[j][i] *= ry * g[i];
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      y[j][i] = x[j][i] + y[j][i];
      ss += y[j][i] * y[j][i];
    }
    if (p.y != nullptr) store8(xr + c, y[j]);
  }
  if (p.w_next == nullptr) return;
  const float rx = rsqrtf(block_sum32(ss, red + 32) / (float)p.W + p.eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * 8 + j * step;
    if (c >= p.P) continue;
    float g[8];
    load8(p.w_next + c, g);
#pragma unroll
    for (int i = 0; i < 8; ++i) y[j][i] *= rx * g[i];
    store8(static_cast<T*>(p.h) + (size_t)m * p.P + c, y[j]);
  }
}

// x[m] += rmsnorm(sigmoid(gate[m]) * Y) * w_out and h[m] = x[m], with Y = y[m], or of two branches
// scale * (rmsnorm(y[m]) * w_y + rmsnorm(y2[m]) * w_y2).  `gate` holds logits.
struct GatedNormParams {
  const void* y;           // [M][ldy]
  const void* y2;          // [M][ldy] or null
  const void* gate;        // [M][ldg]
  const float* w_y;        // [P], with y2
  const float* w_y2;       // [P], with y2
  const float* w_out;      // [P]
  float* x;                // [M][P]
  void* h;                 // [M][P] or null
  int W, P, ldy, ldg;
  float eps, scale;
};

// KEEP x 8 columns per thread; `red`: 96 floats of shared memory
template <typename T, int KEEP>
TI_DEVICE void gated_norm_row(const GatedNormParams& p, int m, float* red) {
  const int step = blockDim.x * 8;
  const bool two = p.y2 != nullptr;                        // uniform over the grid
  float y[KEEP][8], z[KEEP][8], g[KEEP][8], s1 = 0.f, s2 = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * 8 + j * step;
    if (c >= p.P) continue;
    load8(static_cast<const T*>(p.y) + (size_t)m * p.ldy + c, y[j]);
    load8(static_cast<const T*>(p.gate) + (size_t)m * p.ldg + c, g[j]);
    if (two) load8(static_cast<const T*>(p.y2) + (size_t)m * p.ldy + c, z[j]);
  }
  if (two) {
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      if (threadIdx.x * 8 + j * step >= p.P) continue;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        s1 = fmaf(y[j][i], y[j][i], s1);
        s2 = fmaf(z[j][i], z[j][i], s2);
      }
    }
    const float r1 = p.scale * rsqrtf(block_sum32(s1, red) / (float)p.W + p.eps), r2 = p.scale * rsqrtf(block_sum32(s2, red + 32) / (float)p.W + p.eps);
#pragma unroll
    for (int j = 0; j < KEEP; ++j) {
      const int c = threadIdx.x * 8 + j * step;
      if (c >= p.P) continue;
      float a[8], b[8];
      load8(p.w_y + c, a);
      load8(p.w_y2 + c, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) y[j][i] = y[j][i] * r1 * a[i] + z[j][i] * r2 * b[i];
    }
  }
  s1 = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    if (threadIdx.x * 8 + j * step >= p.P) continue;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      y[j][i] *= sigmoid_exact(g[j][i]);
      s1 = fmaf(y[j][i], y[j][i], s1);
    }
  }
  const float rr = rsqrtf(block_sum32(s1, red + 64) / (float)p.W + p.eps);
#pragma unroll
  for (int j = 0; j < KEEP; ++j) {
    const int c = threadIdx.x * 8 + j * step;
    if (c >= p.P) continue;
    float x[8], w[8];
    load8(p.x + (size_t)m * p.P + c, x);
    load8(p.w_out + c, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) x[i] = fmaf(y[j][i] * rr, w[i], x[i]);
    store8(p.x + (size_t)m * p.P + c, x);
    if (p.h != nullptr) store8(static_cast<T*>(p.h) + (size_t)m * p.P + c, x);
  }
}

}  // namespace ti
