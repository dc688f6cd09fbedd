// Around the paged attention kernels: the preparation of rotated heads that are root-mean-square normalised one by one, or
// all together before they are split, and a plain attention
// kernel for what the tensor-core kernels do not take (32-bit mode, heads wider than 256).
//
// Cache layout as in attn_paged.cu, in bf16 or float: K pages [block][kv_head][16 tokens][dp], V pages transposed
// [block][kv_head][vp][16 tokens].  Head sizes are padded to multiples of 64 with zeros; means divide by the true size.
#include "row_vec.cuh"

namespace ti {

struct RopeUnitParams {
  const void* proj;              // [T, ld]: H query heads at q_col, G key heads at k_col (dp each), G value heads at v_col (vp)
  const float* inv_freq;         // [half] angle per position of pair i, i + half (pairs: 2i, 2i + 1)
  const int* positions;          // [T]
  const long long* slot_mapping; // [T] flat slot = block * 16 + offset; outside the cache: not stored
  void* q_out;                   // [T, H, dp]
  void* kcache;
  void* vcache;
  unsigned* status;
  int T, ld, q_col, k_col, v_col, H, G, dim, dp, vp, half, num_blocks;
  float eps;
  int pairs;                     // neighbouring dimensions turn together
  const float* q_w;              // null, or [H * dp]: factors of the normed head, ahead of the rotation (0 in the padding)
  const float* k_w;              // [G * dp]
};

// A warp per (token, head): x / sqrt(mean(x^2) + eps), optionally times a weight, and the rotation of the first 2 * half
// dimensions; values (which may be the columns of the keys) are only stored.  Everything up to the store is fp32.
template <typename T, int E>
__global__ void __launch_bounds__(128) rope_unit_kernel(const __grid_constant__ RopeUnitParams p) {
  extern __shared__ float sh[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, heads = p.H + 2 * p.G;
  const long long item = (long long)blockIdx.x * 4 + warp;
  pdl_trigger();
  pdl_wait();
  if (item >= (long long)p.T * heads) return;
  const int t = (int)(item / heads), head = (int)(item - (long long)t * heads);
  const T* row = static_cast<const T*>(p.proj) + (size_t)t * p.ld;
  const long long slot = p.slot_mapping[t], blk = slot >> 4;
  const int off = (int)(slot & 15);
  const bool stored = slot >= 0 && blk < p.num_blocks;
  if (head >= p.H + p.G) {
    if (!stored) return;
    const int g = head - p.H - p.G;
    const T* src = row + p.v_col + (size_t)g * p.vp;
    T* dst = static_cast<T*>(p.vcache) + ((size_t)blk * p.G + g) * p.vp * 16 + off;
    for (int c = lane; c < p.vp; c += 32) dst[(size_t)c * 16] = src[c];
    return;
  }
  const bool is_q = head < p.H;
  if (!is_q && !stored) return;
  const T* src = row + (is_q ? p.q_col + (size_t)head * p.dp : p.k_col + (size_t)(head - p.H) * p.dp);
  const float* w = p.q_w == nullptr ? nullptr : is_q ? p.q_w + (size_t)head * p.dp : p.k_w + (size_t)(head - p.H) * p.dp;
  float* buf = sh + (size_t)warp * p.dp;
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int c = lane + 32 * i;
    if (c < p.dp) {
      const float v = to_f<T>(src[c]);
      buf[c] = w == nullptr ? v : v * w[c];
      ss += v * v;                                         // a rotation keeps the sum of squares
    }
  }
  __syncwarp();
  const float rr = rsqrtf(warp_sum(ss) / (float)p.dim + p.eps);
  const float pos = (float)p.positions[t];
  for (int i = lane; i < p.half; i += 32) {
    float sn, cs;
    sincosf(pos * p.inv_freq[i], &sn, &cs);
    const int a = p.pairs ? 2 * i : i, b = p.pairs ? 2 * i + 1 : i + p.half;
    const float u = buf[a], v = buf[b];
    buf[a] = u * cs - v * sn;
    buf[b] = v * cs + u * sn;
  }
  __syncwarp();
  T* dst = is_q ? static_cast<T*>(p.q_out) + ((size_t)t * p.H + head) * p.dp
                : static_cast<T*>(p.kcache) + (((size_t)blk * p.G + head - p.H) * 16 + off) * p.dp;
#pragma unroll
  for (int i = 0; i < E; ++i) {
    const int c = lane + 32 * i;
    if (c < p.dp) dst[c] = from_f<T>(buf[c] * rr);
  }
}

struct NormRopeParams {
  const void* proj;              // [T, ld]: H query heads at q_col, G key heads at k_col (dp each), G value heads at v_col (vp)
  const float* q_w;              // [H * dp] weights of the norm over all query heads together (0 in the padding)
  const float* k_w;              // [G * dp]
  const float* inv_freq;         // [half] angle per position of dimensions 2i, 2i + 1
  const int* positions;          // [T]
  const long long* slot_mapping; // [T] flat slot = block * 16 + offset; outside the cache: not stored
  void* q_out;                   // [T, H, dp]
  void* kcache;
  void* vcache;
  int T, ld, q_col, k_col, v_col, H, G, dim, dp, vp, half, num_blocks;
  float eps;
};

// A block per token: x / sqrt(mean over all heads of x^2 + eps) * w for the queries and for the keys, then the rotation of
// neighbouring dimensions; values are only stored.
template <typename T>
__global__ void __launch_bounds__(1024) norm_rope_kernel(const __grid_constant__ NormRopeParams p) {
  extern __shared__ float cs[];                            // [half] cosines, [half] sines
  __shared__ float red[2][32];
  const int tid = threadIdx.x, nt = blockDim.x, t = blockIdx.x, nq = p.H * p.dp, nk = p.G * p.dp, nv = p.G * p.vp, step = nt * 8;
  pdl_trigger();
  pdl_wait();
  const T* row = static_cast<const T*>(p.proj) + (size_t)t * p.ld;
  const long long slot = p.slot_mapping[t], blk = slot >> 4;
  const int off = (int)(slot & 15);
  const bool stored = slot >= 0 && blk < p.num_blocks;
  auto source = [&](int c) { return c < nq ? row + p.q_col + c : row + p.k_col + c - nq; };
  constexpr int KEEP = 1;                                  // vectors a thread keeps between the two passes
  float keep[KEEP][8], sq = 0.f, sk = 0.f;
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (tid * 8 + j * step < nq + nk) load8(source(tid * 8 + j * step), keep[j]);
  const float pos = (float)p.positions[t];
  for (int i = tid; i < p.half; i += nt) sincosf(pos * p.inv_freq[i], &cs[p.half + i], &cs[i]);
  auto square = [&](int c, const float (&v)[8]) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) s += v[i] * v[i];
    if (c < nq) sq += s;
    else sk += s;
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (tid * 8 + j * step < nq + nk) square(tid * 8 + j * step, keep[j]);
  for (int c = tid * 8 + KEEP * step; c < nq + nk; c += step) {
    float v[8];
    load8(source(c), v);
    square(c, v);
  }
  if (stored) {                                            // values while the sums meet
    T* dst = static_cast<T*>(p.vcache) + (size_t)blk * nv * 16 + off;
    for (int c = (nt - 1 - tid) * 8; c < nv; c += step) {
      float v[8];
      load8(row + p.v_col + c, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) dst[(size_t)(c + i) * 16] = from_f<T>(v[i]);
    }
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = sq;
    red[1][tid >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
  for (int w = 0; w < nt >> 5; ++w) {
    sq += red[0][w];
    sk += red[1][w];
  }
  const float rq = rsqrtf(sq / (float)(p.H * p.dim) + p.eps), rk = rsqrtf(sk / (float)(p.G * p.dim) + p.eps);
  auto put = [&](int c, float (&v)[8]) {
    const bool is_q = c < nq;
    if (!is_q && !stored) return;
    const int e = is_q ? c : c - nq, g = e / p.dp, d = e - g * p.dp;
    float w[8];
    load8((is_q ? p.q_w : p.k_w) + e, w);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] *= (is_q ? rq : rk) * w[i];
#pragma unroll
    for (int i = 0; i < 8; i += 2) {
      const int f = (d + i) >> 1;
      if (f < p.half) {
        const float a = v[i], b = v[i + 1], co = cs[f], si = cs[p.half + f];
        v[i] = a * co - b * si;
        v[i + 1] = b * co + a * si;
      }
    }
    store8(is_q ? static_cast<T*>(p.q_out) + (size_t)t * nq + e : static_cast<T*>(p.kcache) + (((size_t)blk * p.G + g) * 16 + off) * p.dp + d, v);
  };
#pragma unroll
  for (int j = 0; j < KEEP; ++j)
    if (tid * 8 + j * step < nq + nk) put(tid * 8 + j * step, keep[j]);
  for (int c = tid * 8 + KEEP * step; c < nq + nk; c += step) {
    float v[8];
    load8(source(c), v);
    put(c, v);
  }
}

struct AttnGeneralParams {
  const void* q;           // [T, H, dp]
  const void* kcache;
  const void* vcache;
  const int* block_tables; // [S, max_blocks]
  const int* positions;    // [T]
  const int* qg_seq;       // [num_qg] sequence of a query token
  const int* qg_tok0;      // [num_qg] its flat index
  const int* qg_ntok;      // [num_qg] 1, or 0: padding
  void* out;               // [T, ldo], head h at column h * vp
  unsigned* status;
  int H, G, dp, vp, max_blocks, num_qg, num_blocks, ldo;
  float scale, softcap;    // softcap 0: none
  int window;              // keys seen, the token itself included (0: all earlier ones)
  const float* slopes;     // null, or [H]: taken off a score per token of distance
  const void* head_gate;   // null, or [T, ldg]: the sigmoid of column gcol + h scales head h
  int ldg, gcol;
  float out_scale;         // factor of the output
  const void* gate;        // null, or [T, ldg]: the sigmoid of column gcol + h * vp + d scales dimension d of head h
};

// One query token and head per block; the four warps take the pages in turn and keep running maxima, sums and outputs.
template <typename T, int NV>
__global__ void __launch_bounds__(128) attn_general_kernel(const __grid_constant__ AttnGeneralParams p) {
  extern __shared__ float sh[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, qg = blockIdx.x, h = blockIdx.y;
  float *qs = sh, *acc_s = sh + p.dp, *ml = acc_s + 4 * p.vp, *ps = ml + 8 + warp * 16;
  pdl_trigger();
  pdl_wait();
  if (p.qg_ntok[qg] == 0) return;
  const int seq = p.qg_seq[qg], tok = p.qg_tok0[qg], g = h / (p.H / p.G), pos = p.positions[tok];
  for (int c = threadIdx.x; c < p.dp; c += 128) qs[c] = to_f<T>(static_cast<const T*>(p.q)[((size_t)tok * p.H + h) * p.dp + c]);
  __syncthreads();
  float acc[NV], m = -1e30f, l = 0.f;
#pragma unroll
  for (int i = 0; i < NV; ++i) acc[i] = 0.f;
  const int lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const float slope = p.slopes != nullptr ? p.slopes[h] : 0.f;
  for (int pg = (lo >> 4) + warp; pg <= pos >> 4; pg += 4) {
    const int blk = p.block_tables[(size_t)seq * p.max_blocks + pg];
    if (!TI_CHECK(blk, p.num_blocks, p.status)) continue;
    const T* kb = static_cast<const T*>(p.kcache) + (((size_t)blk * p.G + g) * 16 + (lane >> 1)) * p.dp;
    float s = 0.f;
    for (int c = (lane & 1) * 8; c < p.dp; c += 16) {
      float v[8];
      load8(kb + c, v);
#pragma unroll
      for (int i = 0; i < 8; ++i) s = fmaf(v[i], qs[c + i], s);
    }
    s = (s + __shfl_xor_sync(0xffffffffu, s, 1)) * p.scale;
    if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
    const int key = pg * 16 + (lane >> 1);
    s -= slope * (float)(pos - key);
    const bool seen = key <= pos && key >= lo;
    const float mn = fmaxf(m, warp_max(seen ? s : -1e30f));
    const float e = seen ? expf(s - mn) : 0.f, alpha = expf(m - mn);
    l = l * alpha + warp_sum((lane & 1) ? 0.f : e);
    m = mn;
    __syncwarp();
    if ((lane & 1) == 0) ps[lane >> 1] = e;
    __syncwarp();
    const T* vb = static_cast<const T*>(p.vcache) + ((size_t)blk * p.G + g) * p.vp * 16;
    const int last = pos - pg * 16;                        // keys past the query may hold anything: they are not multiplied
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int c = lane + 32 * i;
      if (c >= p.vp) continue;
      float a[8], b[8], t = 0.f;
      load8(vb + (size_t)c * 16, a);
      load8(vb + (size_t)c * 16 + 8, b);
#pragma unroll
      for (int j = 0; j < 8; ++j) {
        if (j <= last) t = fmaf(ps[j], a[j], t);
        if (j + 8 <= last) t = fmaf(ps[j + 8], b[j], t);
      }
      acc[i] = acc[i] * alpha + t;
    }
  }
#pragma unroll
  for (int i = 0; i < NV; ++i)
    if (lane + 32 * i < p.vp) acc_s[warp * p.vp + lane + 32 * i] = acc[i];
  if (lane == 0) { ml[warp] = m; ml[4 + warp] = l; }
  __syncthreads();
  const float M = fmaxf(fmaxf(ml[0], ml[1]), fmaxf(ml[2], ml[3]));
  float w[4], L = 0.f;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    w[i] = expf(ml[i] - M);
    L += w[i] * ml[4 + i];
  }
  float f = p.out_scale / L;
  if (p.head_gate != nullptr) f *= sigmoid_exact(to_f<T>(static_cast<const T*>(p.head_gate)[(size_t)tok * p.ldg + p.gcol + h]));
  T* out = static_cast<T*>(p.out) + (size_t)tok * p.ldo + (size_t)h * p.vp;
  for (int c = threadIdx.x; c < p.vp; c += 128) {
    float o = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) o = fmaf(w[i], acc_s[i * p.vp + c], o);
    if (p.gate != nullptr) o *= sigmoid_exact(to_f<T>(static_cast<const T*>(p.gate)[(size_t)tok * p.ldg + p.gcol + (size_t)h * p.vp + c]));
    out[c] = from_f<T>(o * f);
  }
}

template <typename T>
static int launch_rope(const RopeUnitParams& p, cudaStream_t st) {
  const long long items = (long long)p.T * (p.H + 2 * p.G);
  const dim3 grid((unsigned)((items + 3) / 4));
  const size_t smem = (size_t)4 * p.dp * 4;
  if (p.dp <= 64) launch_kernel(rope_unit_kernel<T, 2>, grid, dim3(128), smem, st, true, p);
  else if (p.dp <= 128) launch_kernel(rope_unit_kernel<T, 4>, grid, dim3(128), smem, st, true, p);
  else if (p.dp <= 256) launch_kernel(rope_unit_kernel<T, 8>, grid, dim3(128), smem, st, true, p);
  else if (p.dp <= 1024) launch_kernel(rope_unit_kernel<T, 32>, grid, dim3(128), smem, st, true, p);
  else return -3;
  return (int)cudaGetLastError();
}

template <typename T>
static int launch_general(const AttnGeneralParams& p, cudaStream_t st) {
  const dim3 grid(p.num_qg, p.H);
  const size_t smem = (size_t)(p.dp + 4 * p.vp + 8 + 64) * 4;
  if (p.vp <= 64) launch_kernel(attn_general_kernel<T, 2>, grid, dim3(128), smem, st, true, p);
  else if (p.vp <= 128) launch_kernel(attn_general_kernel<T, 4>, grid, dim3(128), smem, st, true, p);
  else if (p.vp <= 256) launch_kernel(attn_general_kernel<T, 8>, grid, dim3(128), smem, st, true, p);
  else if (p.vp <= 1024) launch_kernel(attn_general_kernel<T, 32>, grid, dim3(128), smem, st, true, p);
  else return -3;
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_rope_unit_params_size() { return (int)sizeof(ti::RopeUnitParams); }
int ti_norm_rope_params_size() { return (int)sizeof(ti::NormRopeParams); }

int ti_norm_rope(const ti::NormRopeParams* p, int f32, void* stream) {
  if (p->T <= 0) return 0;
  if (p->dp % 8 || p->vp % 8 || p->dim > p->dp || 2 * p->half > p->dim || p->num_blocks < 1 || p->ld % 8 || p->q_col % 8 || p->k_col % 8 || p->v_col % 8 ||
      (((uintptr_t)p->proj | (uintptr_t)p->q_out | (uintptr_t)p->kcache | (uintptr_t)p->q_w | (uintptr_t)p->k_w) & 15))
    return -2;
  // a row in one pass of the block where there are few tokens
  const int vecs = ((p->H + p->G) * p->dp / 8 + 31) / 32 * 32, most = p->T <= 1024 ? 1024 : 256;
  ti::launch_kernel(f32 ? ti::norm_rope_kernel<float> : ti::norm_rope_kernel<ti::bf16>, dim3(p->T), dim3(vecs < most ? vecs : most), (size_t)p->half * 8,
                    (cudaStream_t)stream, true, *p);
  return (int)cudaGetLastError();
}

int ti_attn_general_params_size() { return (int)sizeof(ti::AttnGeneralParams); }

int ti_rope_unit(const ti::RopeUnitParams* p, int f32, void* stream) {
  if (p->T <= 0) return 0;
  if (p->dp % 64 || p->vp % 64 || p->dim > p->dp || 2 * p->half > p->dim || p->num_blocks < 1) return -2;
  return f32 ? ti::launch_rope<float>(*p, (cudaStream_t)stream) : ti::launch_rope<ti::bf16>(*p, (cudaStream_t)stream);
}

int ti_attn_general(const ti::AttnGeneralParams* p, int f32, void* stream) {
  if (p->num_qg <= 0) return 0;
  if (p->dp % 64 || p->vp % 64 || p->H % p->G || p->num_blocks < 1 || p->window < 0 ||
      (((uintptr_t)p->kcache | (uintptr_t)p->vcache) & 15))
    return -2;
  return f32 ? ti::launch_general<float>(*p, (cudaStream_t)stream) : ti::launch_general<ti::bf16>(*p, (cudaStream_t)stream);
}

}  // extern "C"
