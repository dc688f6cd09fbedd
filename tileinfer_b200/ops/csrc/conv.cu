// Short causal convolutions over time on columns of a projection, one filter per channel:
//     y_t = sum_j w[j] u_(t - taps + 1 + j) (+ bias),   u before the sequence's first token is zero
// The last taps - 1 inputs of a sequence are carried in its state slot.  What becomes of y is a parameter: it is stored,
// optionally through silu, or its channels are the query, key and value heads of an attention layer, which go to the query
// rows (times a factor that grows with the logarithm of the position) and into the cache pages.
//
// A thread owns eight channels of four neighbouring tokens, with all their inputs in flight at once.  In a
// decode step (one token per sequence) it reads the state, which no kernel of the step writes before, ahead of the wait for
// the projection, and moves it on; in a step with longer portions several tiles read a sequence's state, so
// `conv_tail_kernel` does that afterwards, with the snapshots.
#include "row_vec.cuh"

namespace ti {

struct ConvParams {
  const void* proj;              // [T, ld], channels at column col
  const float* w;                // [taps][C]
  const float* bias;             // [C] or null
  void* state;                   // [slots][taps - 1][C]
  const int* slots;              // [S]
  const int* cu;                 // [S + 1] token offsets, or null: one token per sequence
  const int* tiles;              // [3][num_tiles] sequence, first flat token, tokens (at most 16); unused without cu
  void* out;                     // [T, ldo], or null: heads
  const int* positions;          // heads: [T]
  const long long* slot_mapping; // heads: [T] flat cache slot = block * 16 + offset; outside the cache: not stored
  void* q_out;                   // heads: [T, H * dp]
  void* kcache;                  // heads: [block][G][16][dp]
  void* vcache;                  // heads: [block][G][vp][16]
  const int* snap_rel;           // [S][num_snap] tokens of the step after which the inputs are kept (<= 0: unused)
  const int* snap_idx;           // [S][num_snap] entry of `snap`
  void* snap;                    // [entries][taps - 1][C]
  int T, S, ld, col, C, taps, num_tiles, ldo, silu, H, G, dp, vp, num_blocks, temp_every, num_snap;
  float temp_coef;               // heads: factor of a query at position p is 1 + coef ln(floor((p + 1) / every) + 1)
};

template <typename T>
TI_DEVICE void conv_emit(const ConvParams& p, int t, int c, float (&y)[8]) {
  if (p.out != nullptr) {
    if (p.silu) {
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] *= sigmoid_exact(y[i]);
    }
    store8(static_cast<T*>(p.out) + (size_t)t * p.ldo + c, y);
    return;
  }
  const int nq = p.H * p.dp, nk = p.G * p.dp;
  if (c < nq) {
    const float f = 1.f + p.temp_coef * logf((float)((p.positions[t] + 1) / p.temp_every + 1));
#pragma unroll
    for (int i = 0; i < 8; ++i) y[i] *= f;
    store8(static_cast<T*>(p.q_out) + (size_t)t * nq + c, y);
    return;
  }
  const long long slot = p.slot_mapping[t], blk = slot >> 4;
  if (slot < 0 || blk >= p.num_blocks) return;
  const int off = (int)(slot & 15);
  c -= nq;
  if (c < nk) {
    const int g = c / p.dp;
    store8(static_cast<T*>(p.kcache) + (((size_t)blk * p.G + g) * 16 + off) * p.dp + (c - g * p.dp), y);
    return;
  }
  c -= nk;
  T* v = static_cast<T*>(p.vcache) + ((size_t)blk * p.G * p.vp + c) * 16 + off;      // head g, dimension d: g * vp + d = c
#pragma unroll
  for (int i = 0; i < 8; ++i) v[(size_t)i * 16] = from_f<T>(y[i]);
}

constexpr int kConvTile = 16, kConvTokens = 4;             // tokens of a tile, and of a thread

// TAPS 0: any number of taps, the window read again for every token
template <typename T, int TAPS>
__global__ void __launch_bounds__(128) conv_kernel(const __grid_constant__ ConvParams p) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  pdl_trigger();
  if (c >= p.C) {
    pdl_wait();
    return;
  }
  constexpr int K = TAPS > 0 ? TAPS : 1;
  const int taps = TAPS > 0 ? TAPS : p.taps;
  float w[K][8], b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
  if (TAPS > 0) {
#pragma unroll
    for (int j = 0; j < K; ++j) load8(p.w + (size_t)j * p.C + c, w[j]);
  }
  if (p.bias != nullptr) load8(p.bias + c, b);
  const bool single = p.cu == nullptr;
  const int s = single ? (int)blockIdx.y : p.tiles[blockIdx.y];
  const int t0 = single ? s : p.tiles[p.num_tiles + blockIdx.y] + (int)blockIdx.z * kConvTokens;
  const int nt = single ? 1 : min(kConvTokens, p.tiles[2 * p.num_tiles + blockIdx.y] - (int)blockIdx.z * kConvTokens);
  const int begin = single ? s : p.cu[s];
  T* state = static_cast<T*>(p.state) + (size_t)p.slots[s] * (taps - 1) * p.C + c;
  const T* proj = static_cast<const T*>(p.proj) + p.col + c;
  // input of flat token t, which may lie before the portion
  auto input = [&](int t, float (&v)[8]) {
    if (t >= begin) load8(proj + (size_t)t * p.ld, v);
    else load8(state + (size_t)(taps - 1 + t - begin) * p.C, v);
  };
  float u[K - 1 + kConvTokens][8];
  if (TAPS > 0 && single) {
#pragma unroll
    for (int j = 0; j < K - 1; ++j) load8(state + (size_t)j * p.C, u[j]);
  }
  pdl_wait();
  if (TAPS > 0) {
    if (nt <= 0) return;
    if (!single) {
#pragma unroll
      for (int j = 0; j < K - 1; ++j) input(t0 - (K - 1) + j, u[j]);
    }
#pragma unroll
    for (int k = 0; k < kConvTokens; ++k)
      if (k < nt) load8(proj + (size_t)(t0 + k) * p.ld, u[K - 1 + k]);
#pragma unroll
    for (int k = 0; k < kConvTokens; ++k) {
      if (k >= nt) break;
      float y[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        y[i] = b[i];
#pragma unroll
        for (int j = 0; j < K; ++j) y[i] = fmaf(w[j][i], u[k + j][i], y[i]);
      }
      conv_emit<T>(p, t0 + k, c, y);
    }
    if (single) {
#pragma unroll
      for (int j = 0; j < K - 1; ++j) store8(state + (size_t)j * p.C, u[j + 1]);
    }
  } else {
    for (int t = t0; t < t0 + nt; ++t) {
      float y[8], v[8], f[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) y[i] = b[i];
      for (int j = 0; j < taps; ++j) {
        input(t - (taps - 1) + j, v);
        load8(p.w + (size_t)j * p.C + c, f);
#pragma unroll
        for (int i = 0; i < 8; ++i) y[i] = fmaf(f[i], v[i], y[i]);
      }
      conv_emit<T>(p, t, c, y);
    }
    if (single) {
      float v[8];
      for (int j = 0; j < taps - 1; ++j) {                 // the thread's own channels: what is read was not written yet
        input(t0 - (taps - 1) + j + 1, v);
        store8(state + (size_t)j * p.C, v);
      }
    }
  }
}

// The inputs a sequence carries on (and those wanted for snapshots) after a step with longer portions.
template <typename T>
__global__ void __launch_bounds__(128) conv_tail_kernel(const __grid_constant__ ConvParams p) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8, s = blockIdx.y;
  pdl_trigger();
  pdl_wait();
  if (c >= p.C) return;
  const int begin = p.cu[s], n = p.cu[s + 1] - begin, keep = p.taps - 1;
  T* state = static_cast<T*>(p.state) + (size_t)p.slots[s] * keep * p.C + c;
  const T* proj = static_cast<const T*>(p.proj) + p.col + c;
  // row i of what is carried after r tokens
  auto copy = [&](int r, int i, T* dst) {
    const int rel = r - keep + i;
    float v[8];
    if (rel >= 0) load8(proj + (size_t)(begin + rel) * p.ld, v);
    else load8(state + (size_t)(keep + rel) * p.C, v);
    store8(dst, v);
  };
  for (int k = 0; k < p.num_snap; ++k) {
    const int r = p.snap_rel[s * p.num_snap + k];
    if (r <= 0 || r > n) continue;
    T* dst = static_cast<T*>(p.snap) + (size_t)p.snap_idx[s * p.num_snap + k] * keep * p.C + c;
    for (int i = 0; i < keep; ++i) copy(r, i, dst + (size_t)i * p.C);
  }
  if (n <= 0) return;
  for (int i = 0; i < keep; ++i) copy(n, i, state + (size_t)i * p.C);      // reads row i + n, which is still the old one
}

template <typename T>
static int launch_conv(const ConvParams& p, cudaStream_t st) {
  const dim3 grid((p.C / 8 + 127) / 128, p.cu == nullptr ? p.S : p.num_tiles, p.cu == nullptr ? 1 : kConvTile / kConvTokens);
  switch (p.taps) {
    case 2: launch_kernel(conv_kernel<T, 2>, grid, dim3(128), 0, st, true, p); break;
    case 3: launch_kernel(conv_kernel<T, 3>, grid, dim3(128), 0, st, true, p); break;
    case 4: launch_kernel(conv_kernel<T, 4>, grid, dim3(128), 0, st, true, p); break;
    default: launch_kernel(conv_kernel<T, 0>, grid, dim3(128), 0, st, true, p);
  }
  if (p.cu != nullptr && p.taps > 1) launch_kernel(conv_tail_kernel<T>, dim3(grid.x, p.S), dim3(128), 0, st, true, p);
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_conv_params_size() { return (int)sizeof(ti::ConvParams); }

// The convolution of a step's tokens and the inputs its sequences carry on (one kernel without cu, else two).
int ti_conv(const ti::ConvParams* p, int f32, void* stream) {
  if (p->S <= 0 || (p->cu != nullptr && p->num_tiles <= 0)) return 0;
  if (p->taps < 1 || p->C < 8 || p->C % 8 || p->ld % 8 || p->col % 8 || ((uintptr_t)p->proj | (uintptr_t)p->state | (uintptr_t)p->w | (uintptr_t)p->bias) % 16)
    return -2;
  if (p->out != nullptr) {
    if (p->ldo % 8 || (uintptr_t)p->out % 16) return -2;
  } else if (p->dp % 8 || p->vp % 8 || p->C != (p->H + p->G) * p->dp + p->G * p->vp || p->temp_every < 1 || p->num_blocks < 1 ||
             ((uintptr_t)p->q_out | (uintptr_t)p->kcache | (uintptr_t)p->vcache) % 16) {
    return -2;
  }
  return f32 ? ti::launch_conv<float>(*p, (cudaStream_t)stream) : ti::launch_conv<ti::bf16>(*p, (cudaStream_t)stream);
}

}  // extern "C"
