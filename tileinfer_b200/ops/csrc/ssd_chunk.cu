// State-space mixer of long portions, in chunks of 64 tokens on the tensor cores.
//
// With L_i the running sum of the log decays inside a chunk (one per head and token) and S the state before it,
//     y_i = exp(L_i) S^T C_i + sum_{j <= i} (C_i . B_j) exp(L_i - L_j) dt_j x_j + D x_i
//     S'  = exp(L_C) S + sum_j exp(L_C - L_j) dt_j B_j x_j^T
// Nothing inside a chunk depends on the state but one multiply-add per state element, so the chunks run in parallel:
//     ssd_chunk_state_kernel   step sizes, L, and what each chunk adds to the state        (chunk, head)
//     ssd_chunk_scan_kernel    S before every chunk, the state after the last, snapshots   (state element, sequence)
//     ssd_chunk_out_kernel     outputs                                                     (chunk, head)
// A decay is one number per head and token, so exp(L_i - L_j) <= 1 multiplies the finished score and needs no factoring.
//
// Step sizes, decays, scores and states are fp32.  Where they enter a tensor-core product they are split into two bf16
// terms (x = hi + lo, about 16 bits); x, B and C are the bf16 outputs of the convolution, exact.
#include "ssd.cuh"
#include "mma_split.cuh"

namespace ti {

constexpr int kC = 64;                  // tokens of a chunk
constexpr int kVP = 64 + 8;             // pitches: rows of the ldmatrix operands start 16 bytes apart modulo 128

template <int NP> struct SsdGeom {
  static constexpr int BP = NP + 8;
  static constexpr int kB = kC * BP * 2, kX = kC * kVP * 2, kS = NP * kVP * 2;
  static constexpr int kOver = kB > 2 * kS ? kB : 2 * kS;          // B, later the state (hi, lo)
  static constexpr size_t kState = (size_t)kB + 2 * kX;
  static constexpr size_t kOut = (size_t)kB + kOver + 3 * kX;      // C | B or state | scores (hi, lo) | x
};

// n rows (the others zero) of 8 * cols8 columns into shared memory
TI_DEVICE void load_rows(bf16* dst, int pitch, const bf16* src, int ld, int n, int cols8) {
  for (int i = threadIdx.x; i < kC * cols8; i += 256) {
    const int j = i / cols8, c = (i - j * cols8) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (j < n) v = *reinterpret_cast<const uint4*>(src + (size_t)j * ld + c);
    *reinterpret_cast<uint4*>(dst + j * pitch + c) = v;
  }
}

// ------------------------------------------------------------------------------------------------ decays, chunk states
template <int NP>
__global__ void __launch_bounds__(256) ssd_chunk_state_kernel(const __grid_constant__ SsdParams p) {
  using M = SsdGeom<NP>;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float cum[kC], dts[kC];
  bf16* B = reinterpret_cast<bf16*>(smem);
  bf16* XH = reinterpret_cast<bf16*>(smem + M::kB);
  bf16* XL = XH + kC * kVP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int ci = blockIdx.x, h = blockIdx.y, tok0 = p.ck_tok0[ci], n = p.ck_ntok[ci], vp = p.vp;
  const size_t ch = (size_t)ci * p.H + h;
  pdl_trigger();
  pdl_wait();
  const bf16* xbc = static_cast<const bf16*>(p.xbc) + (size_t)tok0 * p.ldx;
  float run = 0.f;
  if (tid < kC) {
    float dt = 0.f;
    if (tid < n) dt = ssd_step_size(p, static_cast<const bf16*>(p.proj) + (size_t)(tok0 + tid) * p.ld, h);
    run = p.neg_a[h] * dt * kLog2e;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const float v = __shfl_up_sync(0xffffffffu, run, o);
      if (lane >= o) run += v;
    }
    dts[tid] = dt;
    cum[tid] = run;
  }
  load_rows(B, M::BP, xbc + p.b_col + (h / (p.H / p.G)) * NP, p.ldx, n, NP / 8);
  __syncthreads();
  const float first = cum[31];
  __syncthreads();
  if (tid < kC) {
    if (tid >= 32) cum[tid] = run = run + first;
    p.g_ws[ch * 2 * kC + tid] = run;
    p.g_ws[ch * 2 * kC + kC + tid] = dts[tid];
  }
  // ---- products of B^T with the scaled inputs, 64 columns at a time: warp -> 16 rows of the state (NP 64: half of the
  //      columns as well)
  constexpr int MT = NP / 16 > 8 ? NP / 128 : 1, NT = NP == 64 ? 4 : 8;
  const int m0 = (NP == 64 ? warp & 3 : warp * MT) * 16, n0 = NP == 64 ? (warp >> 2) * 32 : 0;
  const int mi = lane >> 3, row = lane & 7;
  for (int v0 = 0; v0 < vp; v0 += 64) {
    __syncthreads();
    for (int i = tid; i < kC * 8; i += 256) {
      const int j = i >> 3, c = (i & 7) * 8;
      float x[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (j < n) load8(xbc + (size_t)j * p.ldx + p.x_col + h * vp + v0 + c, x);
      const float f = dts[j] * ex2(cum[kC - 1] - cum[j]);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) split2(x[2 * e] * f, x[2 * e + 1] * f, hi[e], lo[e]);
      *reinterpret_cast<uint4*>(XH + j * kVP + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(XL + j * kVP + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
    __syncthreads();
    float acc[MT][NT][4] = {};
#pragma unroll
    for (int kt = 0; kt < kC / 16; ++kt) {
      uint32_t bh[NT / 2][4], bl[NT / 2][4];
#pragma unroll
      for (int c = 0; c < NT / 2; ++c) {
        const int at = (kt * 16 + (mi & 1) * 8 + row) * kVP + n0 + c * 16 + (mi >> 1) * 8;
        ldsm4t(bh[c], XH + at);
        ldsm4t(bl[c], XL + at);
      }
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t a[4];
        ldsm4t(a, B + (kt * 16 + (mi >> 1) * 8 + row) * M::BP + m0 + m * 16 + (mi & 1) * 8);
#pragma unroll
        for (int c = 0; c < NT; ++c) {
          mma(acc[m][c], a, bh[c >> 1][(c & 1) * 2], bh[c >> 1][(c & 1) * 2 + 1]);
          mma(acc[m][c], a, bl[c >> 1][(c & 1) * 2], bl[c >> 1][(c & 1) * 2 + 1]);
        }
      }
    }
    float* out = p.s_ws + ch * NP * vp + v0 + n0 + 2 * t;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int c = 0; c < NT; ++c) {
        const size_t d = m0 + m * 16 + g;
        *reinterpret_cast<float2*>(out + d * vp + c * 8) = make_float2(acc[m][c][0], acc[m][c][1]);
        *reinterpret_cast<float2*>(out + (d + 8) * vp + c * 8) = make_float2(acc[m][c][2], acc[m][c][3]);
      }
  }
}

// ------------------------------------------------------------------------------------------------ scan over the chunks
__global__ void __launch_bounds__(256) ssd_chunk_scan_kernel(const __grid_constant__ SsdParams p, int NP) {
  const int h = blockIdx.y, s = p.long_seq[blockIdx.z], c0 = p.long_ck[blockIdx.z], c1 = p.long_ck[blockIdx.z + 1];
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4;
  const size_t per = (size_t)NP * p.vp;
  if (e >= NP * p.vp) return;
  float* state = p.state + ((size_t)p.slots[s] * p.H + h) * per + e;
  pdl_trigger();
  pdl_wait();
  float4 S = *reinterpret_cast<const float4*>(state);
  constexpr int AHEAD = 8;
  for (int c = c0; c < c1; c += AHEAD) {
    float4 add[AHEAD];
    float f[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (c + i >= c1) break;
      const size_t ch = (size_t)(c + i) * p.H + h;
      add[i] = *reinterpret_cast<const float4*>(p.s_ws + ch * per + e);
      f[i] = p.g_ws[ch * 2 * kC + kC - 1];
    }
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
      if (c + i >= c1) break;
      *reinterpret_cast<float4*>(p.s_ws + ((size_t)(c + i) * p.H + h) * per + e) = S;
      const float a = ex2(f[i]);
      S = make_float4(fmaf(a, S.x, add[i].x), fmaf(a, S.y, add[i].y), fmaf(a, S.z, add[i].z), fmaf(a, S.w, add[i].w));
      const int snap = p.ck_snap[c + i];
      if (snap >= 0) *reinterpret_cast<float4*>(p.snap + ((size_t)snap * p.H + h) * per + e) = S;
    }
  }
  *reinterpret_cast<float4*>(state) = S;
}

// ------------------------------------------------------------------------------------------------ outputs
template <int NP>
__global__ void __launch_bounds__(256) ssd_chunk_out_kernel(const __grid_constant__ SsdParams p) {
  using M = SsdGeom<NP>;
  constexpr int BP = M::BP, VP = kVP;
  extern __shared__ __align__(16) uint8_t smem[];
  __shared__ float cum[kC], dts[kC];
  bf16* Cm = reinterpret_cast<bf16*>(smem);
  bf16* B = reinterpret_cast<bf16*>(smem + M::kB);
  bf16* SH = B;                                            // [NP][VP], over B
  bf16* SL = SH + NP * VP;
  bf16* AH = reinterpret_cast<bf16*>(smem + M::kB + M::kOver);
  bf16* AL = AH + kC * VP;
  bf16* X = AL + kC * VP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int ci = blockIdx.x, h = blockIdx.y, tok0 = p.ck_tok0[ci], n = p.ck_ntok[ci], vp = p.vp;
  const size_t ch = (size_t)ci * p.H + h;
  const int mi = lane >> 3, row = lane & 7;
  pdl_trigger();
  pdl_wait();
  const bf16* xbc = static_cast<const bf16*>(p.xbc) + (size_t)tok0 * p.ldx;
  const int grp = (h / (p.H / p.G)) * NP;
  if (tid < kC) cum[tid] = p.g_ws[ch * 2 * kC + tid];
  else if (tid < 2 * kC) dts[tid - kC] = p.g_ws[ch * 2 * kC + tid];
  load_rows(Cm, BP, xbc + p.c_col + grp, p.ldx, n, NP / 8);
  load_rows(B, BP, xbc + p.b_col + grp, p.ldx, n, NP / 8);
  __syncthreads();
  // ---- scores: warp -> 16 queries, half of the keys
  {
    const int I = warp >> 1, i0 = 16 * I + g, i1 = i0 + 8;
    float acc[2][2][4] = {};
    for (int kt = 0; kt < NP / 16; ++kt) {
      uint32_t a[4];
      ldsm4(a, Cm + (16 * I + (mi & 1) * 8 + row) * BP + kt * 16 + (mi >> 1) * 8);
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        const int J = (warp & 1) * 2 + c;                  // block of 16 keys
        if (J > I) continue;
        uint32_t b[4];
        ldsm4(b, B + (16 * J + (mi >> 1) * 8 + row) * BP + kt * 16 + (mi & 1) * 8);
        mma(acc[c][0], a, b[0], b[1]);
        mma(acc[c][1], a, b[2], b[3]);
      }
    }
#pragma unroll
    for (int c = 0; c < 2; ++c) {
      if ((warp & 1) * 2 + c > I) continue;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j0 = 16 * ((warp & 1) * 2 + c) + 8 * e + 2 * t, j1 = j0 + 1;
        auto m = [&](float s, int i, int j) { return i >= j ? s * ex2(cum[i] - cum[j]) * dts[j] : 0.f; };
        uint32_t hi, lo;
        split2(m(acc[c][e][0], i0, j0), m(acc[c][e][1], i0, j1), hi, lo);
        *reinterpret_cast<uint32_t*>(AH + i0 * VP + j0) = hi;
        *reinterpret_cast<uint32_t*>(AL + i0 * VP + j0) = lo;
        split2(m(acc[c][e][2], i1, j0), m(acc[c][e][3], i1, j1), hi, lo);
        *reinterpret_cast<uint32_t*>(AH + i1 * VP + j0) = hi;
        *reinterpret_cast<uint32_t*>(AL + i1 * VP + j0) = lo;
      }
    }
  }
  // ---- outputs, 64 columns at a time: warp -> 16 tokens, half of the columns
  constexpr int NT = 4, NLD = NP * 16 / 256;
  const int I = warp & 3, i0 = 16 * I, n0 = (warp >> 2) * 32;
  const float* sp = p.s_ws + ch * NP * vp;
  const float e0 = ex2(cum[i0 + g]), e1 = ex2(cum[i0 + g + 8]), D = p.D[h];
  for (int v0 = 0; v0 < vp; v0 += 64) {
    float4 pre[NLD];
#pragma unroll
    for (int i = 0; i < NLD; ++i) pre[i] = *reinterpret_cast<const float4*>(sp + (size_t)((tid + i * 256) >> 4) * vp + v0 + (tid & 15) * 4);
    __syncthreads();                                       // B (or the last columns' state) and x are done with
#pragma unroll
    for (int i = 0; i < NLD; ++i) {
      const int d = (tid + i * 256) >> 4, c = (tid & 15) * 4;
      uint32_t hi[2], lo[2];
      split2(pre[i].x, pre[i].y, hi[0], lo[0]);
      split2(pre[i].z, pre[i].w, hi[1], lo[1]);
      *reinterpret_cast<uint2*>(SH + d * VP + c) = make_uint2(hi[0], hi[1]);
      *reinterpret_cast<uint2*>(SL + d * VP + c) = make_uint2(lo[0], lo[1]);
    }
    load_rows(X, VP, xbc + p.x_col + h * vp + v0, p.ldx, n, 8);
    __syncthreads();
    float acc[NT][4] = {};
#pragma unroll 4
    for (int kt = 0; kt < NP / 16; ++kt) {
      uint32_t a[4];
      ldsm4(a, Cm + (i0 + (mi & 1) * 8 + row) * BP + kt * 16 + (mi >> 1) * 8);
#pragma unroll
      for (int c = 0; c < NT / 2; ++c) {
        uint32_t bh[4], bl[4];
        const int at = (kt * 16 + (mi & 1) * 8 + row) * VP + n0 + c * 16 + (mi >> 1) * 8;
        ldsm4t(bh, SH + at);
        ldsm4t(bl, SL + at);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(acc[2 * c + e], a, bh[2 * e], bh[2 * e + 1]);
          mma(acc[2 * c + e], a, bl[2 * e], bl[2 * e + 1]);
        }
      }
    }
#pragma unroll
    for (int c = 0; c < NT; ++c) {
      acc[c][0] *= e0; acc[c][1] *= e0; acc[c][2] *= e1; acc[c][3] *= e1;
    }
    for (int kt = 0; kt <= I; ++kt) {
      uint32_t ah[4], al[4];
      const int at = (i0 + (mi & 1) * 8 + row) * VP + kt * 16 + (mi >> 1) * 8;
      ldsm4(ah, AH + at);
      ldsm4(al, AL + at);
#pragma unroll
      for (int c = 0; c < NT / 2; ++c) {
        uint32_t b[4];
        ldsm4t(b, X + (kt * 16 + (mi & 1) * 8 + row) * VP + n0 + c * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(acc[2 * c + e], ah, b[2 * e], b[2 * e + 1]);
          mma(acc[2 * c + e], al, b[2 * e], b[2 * e + 1]);
        }
      }
    }
    float* y = p.y + (size_t)(tok0 + i0 + g) * p.H * vp + h * vp + v0 + n0 + 2 * t;
#pragma unroll
    for (int c = 0; c < NT; ++c) {
      const uint32_t x0 = *reinterpret_cast<const uint32_t*>(X + (i0 + g) * VP + n0 + c * 8 + 2 * t);
      const uint32_t x1 = *reinterpret_cast<const uint32_t*>(X + (i0 + g + 8) * VP + n0 + c * 8 + 2 * t);
      if (i0 + g < n) *reinterpret_cast<float2*>(y + c * 8) = make_float2(fmaf(D, bf16lo(x0), acc[c][0]), fmaf(D, bf16hi(x0), acc[c][1]));
      if (i0 + g + 8 < n)
        *reinterpret_cast<float2*>(y + (size_t)8 * p.H * vp + c * 8) = make_float2(fmaf(D, bf16lo(x1), acc[c][2]), fmaf(D, bf16hi(x1), acc[c][3]));
    }
  }
}

template <int NP>
static int launch_chunked(const SsdParams& p, cudaStream_t st) {
  using M = SsdGeom<NP>;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(ssd_chunk_state_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kState);
    cudaFuncSetAttribute(ssd_chunk_out_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kOut);
    configured = true;
  }
  launch_kernel(ssd_chunk_state_kernel<NP>, dim3(p.nc, p.H), dim3(256), M::kState, st, true, p);
  launch_kernel(ssd_chunk_scan_kernel, dim3((NP * p.vp + 1023) / 1024, p.H, p.num_long), dim3(256), 0, st, true, p, NP);
  launch_kernel(ssd_chunk_out_kernel<NP>, dim3(p.nc, p.H), dim3(256), M::kOut, st, true, p);
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_ssd_chunk_size(int Np) { return Np == 64 || Np == 128 || Np == 256 ? ti::kC : 0; }

// y[t, h] and the states of the sequences with chunks (bf16 inputs)
int ti_ssd_chunked(const ti::SsdParams* p, int Np, void* stream) {
  if (p->nc <= 0) return 0;
  if (p->vp % 64 || p->ld % 8 || p->ldx % 8 || p->x_col % 8 || p->b_col % 8 || p->c_col % 8 || p->H % p->G ||
      (((uintptr_t)p->xbc | (uintptr_t)p->y | (uintptr_t)p->state | (uintptr_t)p->g_ws | (uintptr_t)p->s_ws) & 15))
    return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (Np == 64) return ti::launch_chunked<64>(*p, st);
  if (Np == 128) return ti::launch_chunked<128>(*p, st);
  if (Np == 256) return ti::launch_chunked<256>(*p, st);
  return -3;
}

}  // extern "C"
