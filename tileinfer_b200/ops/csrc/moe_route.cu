// Routing of tokens to experts: softmax scores over experts and identity experts, a corrected choice inside the best
// groups of neighbouring experts, and the layout the grouped products work on (gemm_grouped.cu).
//
// `moe_route_kernel` takes a warp per token.  The chosen experts draw their place inside the expert from a counter per
// expert; the last block to finish turns the counters into the first row of every expert and the table of token tiles, and
// clears them for the next layer.  The order of the rows of an expert depends on which token came first, but no result
// does: a product's row depends on nothing but its own input.  `moe_permute_kernel` copies the token rows to their places.
#include "row_vec.cuh"

namespace ti {

struct MoeRouteParams {
  const float* logits;     // [M][ldl], E + identity columns
  const float* correction; // [E + identity]
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
};

constexpr int kRouteWarps = 4;

// (value, index) of the largest value of a warp; equal values go to the smaller index
TI_DEVICE void warp_argmax(float& v, int& i) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v2 = __shfl_xor_sync(0xffffffffu, v, o);
    const int i2 = __shfl_xor_sync(0xffffffffu, i, o);
    if (v2 > v || (v2 == v && i2 < i)) { v = v2; i = i2; }
  }
}

// Scores -> chosen experts of one token, by one warp.  `s`: the token's logits in shared memory (the scores on return);
// `choice`, `grp`: scratch of E + identity and `groups` floats.
TI_DEVICE void route_token(const MoeRouteParams& p, int m, float* s, float* choice, float* grp) {
  const int lane = threadIdx.x & 31, n = p.E + p.identity, size = n / p.groups;
  const float kNone = __int_as_float(0xff800000);          // -infinity: corrected scores may be negative
  float mx = kNone, sum = 0.f;
  for (int e = lane; e < n; e += 32) mx = fmaxf(mx, s[e]);
  mx = warp_max(mx);
  for (int e = lane; e < n; e += 32) {
    s[e] = expf(s[e] - mx);
    sum += s[e];
  }
  sum = warp_sum(sum);
  for (int e = lane; e < n; e += 32) {
    s[e] = s[e] / sum;
    choice[e] = s[e] + p.correction[e];
  }
  __syncwarp();
  if (p.keep < p.groups) {
    for (int g = lane; g < p.groups; g += 32) {
      float best = kNone;
      for (int e = g * size; e < (g + 1) * size; ++e) best = fmaxf(best, choice[e]);
      grp[g] = best;
    }
    __syncwarp();
    for (int r = 0; r < p.keep; ++r) {                      // NaN marks a kept group
      float v = kNone;
      int at = p.groups;
      for (int g = lane; g < p.groups; g += 32)
        if (grp[g] > v || (grp[g] == v && g < at)) { v = grp[g]; at = g; }
      warp_argmax(v, at);
      if (lane == 0 && at < p.groups) grp[at] = __int_as_float(0x7fc00000);
      __syncwarp();
    }
    for (int e = lane; e < n; e += 32)
      if (grp[e / size] == grp[e / size]) choice[e] = kNone;
    __syncwarp();
  }
  const bool goes = p.valid == nullptr || p.valid[m] >= 0;
  for (int k = 0; k < p.top; ++k) {
    float v = kNone;
    int at = n;
    for (int e = lane; e < n; e += 32)
      if (choice[e] > v || (choice[e] == v && e < at)) { v = choice[e]; at = e; }
    warp_argmax(v, at);
    at = min(at, n - 1);
    if (lane == 0) {
      choice[at] = kNone;
      const size_t o = (size_t)m * p.top + k;
      p.ids[o] = goes ? at : -1;
      p.weight[o] = s[at];
      p.pos[o] = goes && at < p.E ? atomicAdd(p.counts + at, 1) : 0;
    }
    __syncwarp();
  }
}

// Counters -> first rows and token tiles; counters cleared.  By the last block of the grid to get here.
TI_DEVICE void route_finish(const MoeRouteParams& p) {
  __shared__ int s_last, s_rows[256], s_tiles[256];
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) s_last = atomicAdd(p.ticket, 1u) + 1u == gridDim.x;
  __syncthreads();
  if (!s_last) return;
  __threadfence();
  const int tid = threadIdx.x, nt = blockDim.x, per = (p.E + nt - 1) / nt;
  const int e0 = min(tid * per, p.E), e1 = min(e0 + per, p.E);
  int rows = 0, tiles = 0;
  for (int e = e0; e < e1; ++e) {
    const int c = __ldcg(p.counts + e);
    rows += c;
    tiles += (c + p.tile_rows - 1) / p.tile_rows;
  }
  s_rows[tid] = rows;
  s_tiles[tid] = tiles;
  __syncthreads();
  int r0 = 0, t0 = 0;
  for (int i = 0; i < tid; ++i) { r0 += s_rows[i]; t0 += s_tiles[i]; }
  for (int e = e0; e < e1; ++e) {
    const int c = __ldcg(p.counts + e);
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

__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const __grid_constant__ MoeRouteParams p) {
  extern __shared__ float sh[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = p.E + p.identity;
  const int m = blockIdx.x * kRouteWarps + warp;
  float* s = sh + (size_t)warp * (2 * n + p.groups);
  pdl_trigger();
  pdl_wait();
  if (m < p.M) {
    for (int e = lane; e < n; e += 32) s[e] = p.logits[(size_t)m * p.ldl + e];
    __syncwarp();
    route_token(p, m, s, s + n, s + 2 * n);
  }
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

int ti_moe_route(const ti::MoeRouteParams* p, void* stream) {
  if (p->M <= 0) return 0;
  const int n = p->E + p->identity;
  if (p->E < 1 || p->identity < 0 || p->groups < 1 || n % p->groups || p->keep < 1 || p->keep > p->groups || p->top < 1 ||
      p->top > n / p->groups * p->keep || p->tile_rows < 1 || p->max_tiles < 1 || n > 2048)
    return -2;
  const size_t smem = (size_t)ti::kRouteWarps * (2 * n + p->groups) * 4;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(ti::moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
    configured = true;
  }
  ti::launch_kernel(ti::moe_route_kernel, dim3((p->M + ti::kRouteWarps - 1) / ti::kRouteWarps), dim3(ti::kRouteWarps * 32), smem,
                    (cudaStream_t)stream, true, *p);
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
