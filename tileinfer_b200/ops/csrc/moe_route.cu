// Routing of tokens to experts: softmax scores over experts and identity experts (or over the chosen ones alone), an
// optionally corrected choice inside the best groups of neighbouring experts, and the layout the grouped products work on (gemm_grouped.cu).
//
// `moe_route_kernel` takes a warp per token, from logits that a product has computed.  `moe_norm_route_kernel`, for few
// tokens, is a block per token that first finishes the sublayer before (norm, residual add, next norm), computes the
// logits itself and copies the row to its experts.  The chosen experts draw their place inside the expert from a counter per expert (a block's tokens first
// among themselves); the last block to finish turns the counters into the first row of every expert and the table of token tiles, and
// clears them for the next layer.  The order of the rows of an expert depends on which token came first, but no result
// does: a product's row depends on nothing but its own input.  `moe_permute_kernel` copies the token rows to their places.
#include <algorithm>

#include "resid_norm.cuh"

namespace ti {

struct MoeRouteParams {
  const float* logits;     // [M][ldl], E + identity columns
  const float* correction; // [E + identity], or null: the weights are a softmax over the chosen logits alone
  const long long* valid;  // null, or [M]: tokens with a negative entry go nowhere (padding of captured steps)
  int* ids;                // [M][top] chosen expert (>= E: identity; -1: token goes nowhere)
  float* weight;           // [M][top] its score
  int* pos;                // [M][top] place inside the expert
  int* counts;             // [E], zero between launches
  unsigned* ticket;        // zero between launches
  int* first;              // [E] first row of every expert
  int* tiles;              // [3][max_tiles]: expert, first row, rows
  int* num_tiles;
  int M, E, identity, top, groups, keep, ldl, tile_rows, max_tiles;
  int row_stride;          // 0: the rows of the experts follow each other; else expert e's rows start at e * row_stride
};

constexpr int kRouteWarps = 8;

// Order-preserving map of floats to integers above 0 (0 marks what is out of the running), for the warp-wide integer
// maximum.
TI_DEVICE unsigned order_key(float v) {
  const unsigned u = __float_as_uint(v);
  return u & 0x80000000u ? ~u : u | 0x80000000u;
}
// The index of the largest of n keys, which is then set to 0; key e belongs to lane e % 32, equal keys go to the smaller
// index.  `best`, `at`: the lane's own largest key and its index, kept from call to call.
TI_DEVICE void lane_best(const unsigned* key, int n, unsigned& best, int& at) {
  best = 0;
  at = n;
  for (int e = threadIdx.x & 31; e < n; e += 32)
    if (key[e] > best) { best = key[e]; at = e; }
}
TI_DEVICE int take_best(unsigned* key, int n, unsigned& best, int& at) {
  const unsigned top = __reduce_max_sync(0xffffffffu, best);
  const int idx = min(__reduce_min_sync(0xffffffffu, best == top ? at : n), n - 1);
  if ((int)(threadIdx.x & 31) == (idx & 31)) {
    key[idx] = 0;
    lane_best(key, n, best, at);
  }
  return idx;
}

// Scores -> chosen experts of one token, by one warp.  `s`: the token's logits in shared memory (the scores on return);
// `key`, `grp`, `sel`: scratch of E + identity, `groups` and `top` words.  `counts`: places are drawn here.
TI_DEVICE void route_token(const MoeRouteParams& p, int m, float* s, unsigned* key, unsigned* grp, int* sel, int* counts) {
  const int lane = threadIdx.x & 31, n = p.E + p.identity, size = n / p.groups;
  float mx = __int_as_float(0xff800000), sum = 0.f;
  for (int e = lane; e < n; e += 32) mx = fmaxf(mx, s[e]);
  mx = warp_max(mx);
  const bool chosen_only = p.correction == nullptr;
  for (int e = lane; e < n; e += 32) {
    if (chosen_only) key[e] = order_key(s[e]);
    s[e] = expf(s[e] - mx);
    sum += s[e];
  }
  if (!chosen_only) {
    sum = warp_sum(sum);
    for (int e = lane; e < n; e += 32) {
      s[e] = s[e] / sum;
      key[e] = order_key(s[e] + p.correction[e]);          // corrected scores may be negative
    }
  }
  __syncwarp();
  unsigned best;
  int at;
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      unsigned b = 0;
      for (int e = g * size; e < (g + 1) * size; ++e) b = max(b, key[e]);
      grp[g] = b;
    }
    lane_best(grp, p.groups, best, at);
    for (int r = 0; r < p.keep; ++r) take_best(grp, p.groups, best, at);     // 0: kept
    __syncwarp();
    for (int e = lane; e < n; e += 32)
      if (grp[e / size] != 0) key[e] = 0;
  }
  lane_best(key, n, best, at);
  for (int k = 0; k < p.top; ++k) {
    const int e = take_best(key, n, best, at);
    if (lane == 0) sel[k] = e;
  }
  __syncwarp();
  float total = 1.f;
  if (chosen_only) {                                       // the largest logit is among the chosen ones: total >= 1
    total = 0.f;
    for (int k = lane; k < p.top; k += 32) total += s[sel[k]];
    total = warp_sum(total);
  }
  const bool goes = p.valid == nullptr || p.valid[m] >= 0;
  for (int k = lane; k < p.top; k += 32) {
    const int e = sel[k];
    const size_t o = (size_t)m * p.top + k;
    p.ids[o] = goes ? e : -1;
    p.weight[o] = s[e] / total;
    const int pos = goes && e < p.E ? atomicAdd(counts + e, 1) : 0;
    p.pos[o] = pos;
    if (p.row_stride > 0) sel[k] = !goes ? -2 : e >= p.E ? -1 : e * p.row_stride + pos;
  }
  __syncwarp();
}

// Counters -> first rows and token tiles; counters cleared.  By the last block of the grid to get here.
TI_DEVICE void route_finish(const MoeRouteParams& p) {
  __shared__ int s_last, s_rows[32], s_tiles[32];
  __syncthreads();
  if (gridDim.x > 1) {
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) s_last = atomicAdd(p.ticket, 1u) + 1u == gridDim.x;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
  }
  const int tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5, per = (p.E + nt - 1) / nt;
  const int e0 = min(tid * per, p.E), e1 = min(e0 + per, p.E);
  int rows = 0, tiles = 0;
  for (int e = e0; e < e1; ++e) {
    const int c = __ldcg(p.counts + e);
    rows += c;
    tiles += (c + p.tile_rows - 1) / p.tile_rows;
  }
  int r0 = rows, t0 = tiles;                               // inclusive sums over the warp, then over the warps
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int r = __shfl_up_sync(0xffffffffu, r0, o), t = __shfl_up_sync(0xffffffffu, t0, o);
    if (lane >= o) { r0 += r; t0 += t; }
  }
  if (lane == 31) { s_rows[warp] = r0; s_tiles[warp] = t0; }
  __syncthreads();
  r0 -= rows;
  t0 -= tiles;
  for (int w = 0; w < warp; ++w) { r0 += s_rows[w]; t0 += s_tiles[w]; }
  for (int e = e0; e < e1; ++e) {
    const int c = __ldcg(p.counts + e);
    if (p.row_stride > 0) r0 = e * p.row_stride;
    p.first[e] = r0;
    for (int a = 0; a < c; a += p.tile_rows, ++t0) {
      if (t0 >= p.max_tiles) continue;
      p.tiles[t0] = e;
      p.tiles[p.max_tiles + t0] = r0 + a;
      p.tiles[2 * p.max_tiles + t0] = min(p.tile_rows, c - a);
    }
    r0 += c;
    p.counts[e] = 0;
  }
  if (tid == nt - 1) *p.num_tiles = min(t0, p.max_tiles);
  if (tid == 0) *p.ticket = 0;
}

// Tokens blockIdx.x * 8 * tpw ..: a warp takes tpw of them one after the other.
__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const __grid_constant__ MoeRouteParams p, int tpw) {
  extern __shared__ float sh[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, n = p.E + p.identity;
  int* counts = reinterpret_cast<int*>(sh);                 // [E] of this block, then its first place in each expert
  float* s = sh + p.E + (size_t)warp * (2 * n + p.groups + p.top);
  for (int e = tid; e < p.E; e += kRouteWarps * 32) counts[e] = 0;
  pdl_trigger();
  pdl_wait();
  __syncthreads();
  const int m0 = (blockIdx.x * kRouteWarps + warp) * tpw, m1 = min(m0 + tpw, p.M);
  for (int m = m0; m < m1; ++m) {
    for (int e = lane; e < n; e += 32) s[e] = p.logits[(size_t)m * p.ldl + e];
    __syncwarp();
    route_token(p, m, s, reinterpret_cast<unsigned*>(s + n), reinterpret_cast<unsigned*>(s + 2 * n), reinterpret_cast<int*>(s + 2 * n + p.groups), counts);
    __syncwarp();
  }
  __syncthreads();
  for (int e = tid; e < p.E; e += kRouteWarps * 32)
    if (counts[e] > 0) counts[e] = atomicAdd(p.counts + e, counts[e]);
  __syncthreads();
  for (int i = m0 * p.top + lane; i < m1 * p.top; i += 32) {
    const int e = p.ids[i];
    if (e >= 0 && e < p.E) p.pos[i] += counts[e];
  }
  route_finish(p);
}

// Few tokens: a block per token finishes the sublayer before (resid_norm.cuh), computes the router's logits of the row it
// has just normalised (w: [E + identity][P] in the activation type), routes it and copies it to its experts: their rows
// have fixed places (row_stride), so no other token has to be waited for.
template <typename T>
__global__ void __launch_bounds__(1024) moe_norm_route_kernel(const __grid_constant__ ResidNormParams r, const __grid_constant__ MoeRouteParams p,
                                                              const T* __restrict__ w, int* __restrict__ slot, T* __restrict__ xs) {
  extern __shared__ __align__(16) float hs[];               // [P] the row, then logits, keys, groups, rows
  __shared__ float red[64];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = (int)blockDim.x >> 5, n = p.E + p.identity, m = blockIdx.x;
  float* s = hs + r.P;
  int* sel = reinterpret_cast<int*>(s + 2 * n + p.groups);
  float y[1][8];
  pdl_trigger();
  pdl_wait();
  resid_norm_row<T, 1, false>(r, m, y, red);
  if (tid * 8 < r.P) {
    float v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = to_f<T>(from_f<T>(y[0][i]));       // the row as it was stored
    store8(hs + tid * 8, v);
  }
  __syncthreads();
  for (int e = warp; e < n; e += 2 * nw) {                  // two router rows at a time
    const T *w0 = w + (size_t)e * r.P, *w1 = w + (size_t)min(e + nw, n - 1) * r.P;
    float a0 = 0.f, a1 = 0.f;
#pragma unroll 4
    for (int c = lane * 8; c < r.P; c += 256) {
      float u[8], v[8], b[8];
      load8(w0 + c, u);
      load8(w1 + c, v);
      load8(hs + c, b);
#pragma unroll
      for (int i = 0; i < 8; ++i) { a0 = fmaf(u[i], b[i], a0); a1 = fmaf(v[i], b[i], a1); }
    }
    a0 = warp_sum(a0);
    a1 = warp_sum(a1);
    if (lane == 0) {
      s[e] = a0;
      if (e + nw < n) s[e + nw] = a1;
    }
  }
  __syncthreads();
  if (warp == 0) {
    route_token(p, m, s, reinterpret_cast<unsigned*>(s + n), reinterpret_cast<unsigned*>(s + 2 * n), sel, p.counts);
    for (int k = lane; k < p.top; k += 32) slot[(size_t)m * p.top + k] = sel[k];
  }
  __syncthreads();
  if (tid * 8 < r.P)
    for (int k = 0; k < p.top; ++k)
      if (sel[k] >= 0) store8(xs + (size_t)sel[k] * r.P + tid * 8, y[0]);
  route_finish(p);
}

// Row m of h -> row slot of xs for every expert it goes to; slot[m, k] = that row, -1 for an identity expert, -2 for a
// token that goes nowhere.
template <typename T>
__global__ void __launch_bounds__(128) moe_permute_kernel(const T* __restrict__ h, int P, const int* __restrict__ ids,
                                                          const int* __restrict__ pos, const int* __restrict__ first,
                                                          int* __restrict__ slot, T* __restrict__ xs, int E, int top, int rows) {
  extern __shared__ int dst[];
  const int m = blockIdx.x;
  pdl_trigger();
  pdl_wait();
  for (int k = threadIdx.x; k < top; k += blockDim.x) {
    const size_t o = (size_t)m * top + k;
    const int e = ids[o];
    int d = e < 0 ? -2 : e >= E ? -1 : first[e] + pos[o];
    if (d >= rows) d = -2;
    slot[o] = d;
    dst[k] = d;
  }
  __syncthreads();
  for (int c = threadIdx.x * 8; c < P; c += blockDim.x * 8) {
    float v[8];
    load8(h + (size_t)m * P + c, v);
    for (int k = 0; k < top; ++k)
      if (dst[k] >= 0) store8(xs + (size_t)dst[k] * P + c, v);
  }
}

}  // namespace ti

extern "C" {

int ti_moe_route_params_size() { return (int)sizeof(ti::MoeRouteParams); }

static int check_route(const ti::MoeRouteParams* p) {
  const int n = p->E + p->identity;
  return p->E < 1 || p->identity < 0 || p->groups < 1 || n % p->groups || p->keep < 1 || p->keep > p->groups || p->top < 1 ||
         p->top > n / p->groups * p->keep || p->tile_rows < 1 || p->max_tiles < 1 || n > 1024 || p->row_stride < 0;
}

int ti_moe_route(const ti::MoeRouteParams* p, void* stream) {
  if (p->M <= 0) return 0;
  if (check_route(p)) return -2;
  const size_t smem = ((size_t)p->E + (size_t)ti::kRouteWarps * (2 * (p->E + p->identity) + p->groups + p->top)) * 4;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(ti::moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
    configured = true;
  }
  const int tpw = p->M >= 4096 ? 4 : p->M >= 1024 ? 2 : 1, per = ti::kRouteWarps * tpw;
  ti::launch_kernel(ti::moe_route_kernel, dim3((p->M + per - 1) / per), dim3(ti::kRouteWarps * 32), smem, (cudaStream_t)stream, true, *p, tpw);
  return (int)cudaGetLastError();
}

// The residual step of `r` (whose rows are the tokens), the routing of its h with router weights w [E + identity][P], and
// h's rows to their experts' rows of xs [E * row_stride][P].
int ti_moe_norm_route(const ti::ResidNormParams* r, const ti::MoeRouteParams* p, const void* w, void* slot, void* xs, int f32, void* stream) {
  if (p->M <= 0) return 0;
  if (check_route(p) || r->P % 8 || r->ldy % 8 || r->W > r->P || r->P > 8192 || r->w_next == nullptr || p->row_stride < p->M) return -2;
  const int threads = r->P <= 512 ? 256 : 1024;
  const size_t smem = ((size_t)2 * (p->E + p->identity) + p->groups + p->top + r->P) * 4;
  cudaStream_t st = (cudaStream_t)stream;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(ti::moe_norm_route_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
    cudaFuncSetAttribute(ti::moe_norm_route_kernel<ti::bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
    configured = true;
  }
  if (f32) ti::launch_kernel(ti::moe_norm_route_kernel<float>, dim3(p->M), dim3(threads), smem, st, true, *r, *p, (const float*)w, (int*)slot, (float*)xs);
  else ti::launch_kernel(ti::moe_norm_route_kernel<ti::bf16>, dim3(p->M), dim3(threads), smem, st, true, *r, *p, (const ti::bf16*)w, (int*)slot, (ti::bf16*)xs);
  return (int)cudaGetLastError();
}

int ti_moe_permute(const void* h, int M, int P, const void* ids, const void* pos, const void* first, void* slot, void* xs, int E,
                   int top, int rows, int f32, void* stream) {
  if (M <= 0) return 0;
  if (P % 8 || top < 1 || top > 1024) return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    ti::launch_kernel(ti::moe_permute_kernel<float>, dim3(M), dim3(128), top * sizeof(int), st, true, (const float*)h, P, (const int*)ids,
                      (const int*)pos, (const int*)first, (int*)slot, (float*)xs, E, top, rows);
  else
    ti::launch_kernel(ti::moe_permute_kernel<ti::bf16>, dim3(M), dim3(128), top * sizeof(int), st, true, (const ti::bf16*)h, P, (const int*)ids,
                      (const int*)pos, (const int*)first, (int*)slot, (ti::bf16*)xs, E, top, rows);
  return (int)cudaGetLastError();
}

}  // extern "C"
