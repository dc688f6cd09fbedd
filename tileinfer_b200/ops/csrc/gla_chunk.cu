// Gated linear attention of long portions, in chunks of C tokens on the tensor cores.
//
// With G_i the running sum of the log decays inside a chunk (per key channel) and S the state before it,
//     o_i  = (q_i exp(G_i)) S + sum_{j <= i} [sum_d q_id k_jd exp(G_id - G_jd)] v_j
//     S'   = exp(G_C) S + sum_j (k_j exp(G_C - G_j)) v_j^T
// Unlike a delta rule nothing inside a chunk depends on the state, so everything but one multiply-add per state element
// and chunk is parallel over the chunks:
//     gla_chunk_state_kernel   decays, G, and what each chunk adds to the state            (chunk, head)
//     gla_chunk_scan_kernel    S before every chunk, the state after the last, snapshots   (state element, sequence)
//     gla_chunk_out_kernel     outputs                                                     (chunk, head)
//
// exp(G_i - G_j) does not factor safely over a whole chunk (exp(-G_j) overflows under strong decay), so a block of 16 query
// tokens uses the decay from ITS first token as reference: both factors are then at most 1 for every earlier block.  Inside
// the block itself the key's factor exceeds 1; it stays a normal number unless a channel decays by more than 2^80 within 16
// tokens, which is checked per chunk: then the pairs of the block are summed one by one.
//
// Decays, scores and states are fp32.  Where they enter a tensor-core product they are split into two bf16 terms
// (x = hi + lo, about 16 bits); q, k and v are the bf16 projections, exact.
#include "gla.cuh"
#include "mma_split.cuh"

namespace ti {

constexpr float kMaxSpan = 80.f;        // log2 of the decay inside a block of 16 tokens that the products take

// shared-memory pitches: rows of the ldmatrix operands start 16 bytes apart modulo 128
template <int DK> struct GlaGeom {
  static constexpr int C = DK == 256 ? 32 : 64;          // tokens of a chunk
  static constexpr int GP = DK + 4;                      // floats
  static constexpr int KP = DK + 8;                      // bf16
  static constexpr int VP = 64 + 8;
  static constexpr int AP = C + 8;
  static constexpr int kG = C * GP * 4, kK = C * KP * 2, kV = C * VP * 2, kS = DK * VP * 2, kA = C * AP * 2;
  static constexpr int kOver = kG > 2 * kS + kV ? kG : 2 * kS + kV;        // G, later the state (hi, lo) and value tiles
  static constexpr size_t kState = (size_t)kG + 2 * kK + kV;
  static constexpr size_t kOut = (size_t)kOver + 2 * kK + 2 * kA;
};

// ------------------------------------------------------------------------------------------------ decays, chunk states
template <int DK>
__global__ void __launch_bounds__(256) gla_chunk_state_kernel(const __grid_constant__ GlaParams p, int dv) {
  using M = GlaGeom<DK>;
  constexpr int C = M::C, NS = 256 / DK, SEG = C / NS;
  extern __shared__ __align__(16) uint8_t smem[];
  float* G = reinterpret_cast<float*>(smem);
  bf16* KH = reinterpret_cast<bf16*>(smem + M::kG);
  bf16* KL = KH + C * M::KP;
  bf16* V = KL + C * M::KP;
  float* xin = reinterpret_cast<float*>(KH);               // [C][R], until the keys need the space
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int ci = blockIdx.x, h = blockIdx.y, tok0 = p.ck_tok0[ci], n = p.ck_ntok[ci];
  const size_t ch = (size_t)ci * p.H + h;
  pdl_trigger();
  pdl_wait();
  const bf16* proj = static_cast<const bf16*>(p.proj);

  // ---- log2 decays, their running sums: thread = (channel, segment of SEG tokens)
  {
    const int d = tid % DK, seg = tid / DK, col = h * DK + d, cols = p.H * DK;
    float z[SEG];
    const float bias = p.a2_bias[col];
#pragma unroll
    for (int j = 0; j < SEG; ++j) z[j] = bias;
    constexpr int RC = 32;                                 // ranks per pass
    for (int r0 = 0; r0 < p.R; r0 += RC) {
      const int rn = min(RC, p.R - r0);
      __syncthreads();
      for (int i = tid; i < C * rn; i += 256) {
        const int j = i / rn, r = i - j * rn;
        xin[j * RC + r] = j < n ? __bfloat162float(proj[(size_t)(tok0 + j) * p.ld + p.a_col + r0 + r]) : 0.f;
      }
      __syncthreads();
      for (int r = 0; r < rn; ++r) {
        const float a = __ldg(p.a2 + (size_t)(r0 + r) * cols + col);
#pragma unroll
        for (int j = 0; j < SEG; ++j) z[j] = fmaf(a, xin[(seg * SEG + j) * RC + r], z[j]);
      }
    }
    float run = 0.f;
#pragma unroll
    for (int j = 0; j < SEG; ++j) {
      if (seg * SEG + j < n) run += (fminf(z[j], 0.f) - log1pf(expf(-fabsf(z[j])))) * (p.inv_tau * kLog2e);
      z[j] = run;
    }
    float* tot = reinterpret_cast<float*>(V);              // [NS][DK] sums of the segments
    tot[seg * DK + d] = run;
    __syncthreads();
    float base = 0.f;
    for (int s = 0; s < seg; ++s) base += tot[s * DK + d];
    float* gw = p.g_ws + ch * C * DK;
#pragma unroll
    for (int j = 0; j < SEG; ++j) {
      const float v = z[j] + base;
      G[(seg * SEG + j) * M::GP + d] = v;
      gw[(size_t)(seg * SEG + j) * DK + d] = v;
    }
  }
  __syncthreads();
  // ---- k exp(G_C - G_j), split
  for (int i = tid; i < C * DK / 8; i += 256) {
    const int j = i / (DK / 8), d = (i - j * (DK / 8)) * 8;
    float k[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
    if (j < n) load8(proj + (size_t)(tok0 + j) * p.ld + p.k_col + h * DK + d, k);
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int e = 0; e < 8; ++e) k[e] *= ex2(G[(C - 1) * M::GP + d + e] - G[j * M::GP + d + e]);
#pragma unroll
    for (int e = 0; e < 4; ++e) split2(k[2 * e], k[2 * e + 1], hi[e], lo[e]);
    *reinterpret_cast<uint4*>(KH + j * M::KP + d) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4*>(KL + j * M::KP + d) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
  // ---- products with the values, 64 columns at a time: warp -> 16 key channels (DK 64: half of the columns as well)
  constexpr int MT = DK / 16 > 8 ? DK / 128 : 1, NT = DK == 64 ? 4 : 8;
  const int m0 = (DK == 64 ? warp & 3 : warp * MT) * 16, n0 = DK == 64 ? (warp >> 2) * 32 : 0;
  const int mi = lane >> 3, row = lane & 7;
  for (int v0 = 0; v0 < dv; v0 += 64) {
    __syncthreads();
    for (int i = tid; i < C * 8; i += 256) {
      const int j = i >> 3, c = (i & 7) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (j < n) v = *reinterpret_cast<const uint4*>(proj + (size_t)(tok0 + j) * p.ld + p.v_col + h * dv + v0 + c);
      *reinterpret_cast<uint4*>(V + j * M::VP + c) = v;
    }
    __syncthreads();
    float acc[MT][NT][4] = {};
#pragma unroll
    for (int kt = 0; kt < C / 16; ++kt) {
      uint32_t b[NT / 2][4];
#pragma unroll
      for (int c = 0; c < NT / 2; ++c) ldsm4t(b[c], V + (kt * 16 + (mi & 1) * 8 + row) * M::VP + n0 + c * 16 + (mi >> 1) * 8);
#pragma unroll
      for (int m = 0; m < MT; ++m) {
        uint32_t ah[4], al[4];
        const int at = (kt * 16 + (mi >> 1) * 8 + row) * M::KP + m0 + m * 16 + (mi & 1) * 8;
        ldsm4t(ah, KH + at);
        ldsm4t(al, KL + at);
#pragma unroll
        for (int c = 0; c < NT; ++c) {
          mma(acc[m][c], ah, b[c >> 1][(c & 1) * 2], b[c >> 1][(c & 1) * 2 + 1]);
          mma(acc[m][c], al, b[c >> 1][(c & 1) * 2], b[c >> 1][(c & 1) * 2 + 1]);
        }
      }
    }
    float* out = p.s_ws + ch * DK * dv + v0 + n0 + 2 * t;
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int c = 0; c < NT; ++c) {
        const size_t d = m0 + m * 16 + g;
        *reinterpret_cast<float2*>(out + d * dv + c * 8) = make_float2(acc[m][c][0], acc[m][c][1]);
        *reinterpret_cast<float2*>(out + (d + 8) * dv + c * 8) = make_float2(acc[m][c][2], acc[m][c][3]);
      }
  }
}

// ------------------------------------------------------------------------------------------------ scan over the chunks
__global__ void __launch_bounds__(256) gla_chunk_scan_kernel(const __grid_constant__ GlaParams p, int DK, int dv, int C) {
  const int h = blockIdx.y, s = p.long_seq[blockIdx.z], c0 = p.long_ck[blockIdx.z], c1 = p.long_ck[blockIdx.z + 1];
  const int e = (blockIdx.x * 256 + threadIdx.x) * 4, d = e / dv;
  const size_t per = (size_t)DK * dv;
  if (e >= DK * dv) return;
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
      f[i] = p.g_ws[(ch * C + C - 1) * DK + d];
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
template <int DK>
__global__ void __launch_bounds__(256) gla_chunk_out_kernel(const __grid_constant__ GlaParams p, int dv) {
  using M = GlaGeom<DK>;
  constexpr int C = M::C, GP = M::GP, KP = M::KP, VP = M::VP, AP = M::AP;
  extern __shared__ __align__(16) uint8_t smem[];
  float* G = reinterpret_cast<float*>(smem);
  bf16* SH = reinterpret_cast<bf16*>(smem);                // [DK][VP], over G
  bf16* SL = SH + DK * VP;
  bf16* V = SL + DK * VP;
  bf16* Q = reinterpret_cast<bf16*>(smem + M::kOver);      // q, then hi of q exp(G)
  bf16* K = Q + C * KP;                                    // k, then lo of q exp(G)
  bf16* AH = K + C * KP;
  bf16* AL = AH + C * AP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int ci = blockIdx.x, h = blockIdx.y, tok0 = p.ck_tok0[ci], n = p.ck_ntok[ci];
  const size_t ch = (size_t)ci * p.H + h;
  pdl_trigger();
  pdl_wait();
  const bf16* proj = static_cast<const bf16*>(p.proj);
  for (int i = tid; i < C * DK / 4; i += 256) {
    const int j = i / (DK / 4), d = (i - j * (DK / 4)) * 4;
    *reinterpret_cast<float4*>(G + j * GP + d) = *reinterpret_cast<const float4*>(p.g_ws + (ch * C + j) * DK + d);
  }
  for (int i = tid; i < C * DK / 8; i += 256) {
    const int j = i / (DK / 8), d = (i - j * (DK / 8)) * 8;
    uint4 q = make_uint4(0u, 0u, 0u, 0u), k = q;
    if (j < n) {
      const bf16* r = proj + (size_t)(tok0 + j) * p.ld + h * DK + d;
      q = *reinterpret_cast<const uint4*>(r + p.q_col);
      k = *reinterpret_cast<const uint4*>(r + p.k_col);
    }
    *reinterpret_cast<uint4*>(Q + j * KP + d) = q;
    *reinterpret_cast<uint4*>(K + j * KP + d) = k;
  }
  __syncthreads();
  bool wide = false;                                       // some channel decays too far inside a block of 16
  for (int i = tid; i < (C / 16) * DK; i += 256) {
    const int b = i / DK, d = i - b * DK;
    wide |= (b == 0 ? 0.f : G[(16 * b - 1) * GP + d]) - G[(16 * b + 15) * GP + d] > kMaxSpan;
  }
  wide = __syncthreads_or(wide);

  // ---- scores: a warp takes up to three tiles of 8 keys of one block of 16 queries
  {
    constexpr int kI[8] = {0, 1, 1, 2, 2, 3, 3, 3}, kA0[8] = {0, 0, 2, 0, 3, 0, 3, 6}, kA1[8] = {2, 2, 4, 3, 6, 3, 6, 8};
    constexpr int sI[8] = {0, 0, 1, 1, 1, 1, 1, 1}, sA0[8] = {0, 1, 0, 1, 2, 3, 4, 4}, sA1[8] = {1, 2, 1, 2, 3, 4, 4, 4};
    const int I = C == 64 ? kI[warp] : sI[warp], nt0 = C == 64 ? kA0[warp] : sA0[warp], nt1 = C == 64 ? kA1[warp] : sA1[warp];
    const int i0 = 16 * I + g, i1 = i0 + 8;
    float acc[3][4] = {};
    for (int kt = 0; kt < DK / 16; ++kt) {
      uint32_t ah[4], al[4];
      float ref[4];
      const int d0 = 16 * kt + 2 * t;
#pragma unroll
      for (int e = 0; e < 4; ++e) ref[e] = I == 0 ? 0.f : G[(16 * I - 1) * GP + d0 + (e >> 1) * 8 + (e & 1)];
#pragma unroll
      for (int e = 0; e < 4; ++e) {                        // (row i0 / i1, channels d0 / d0 + 8)
        const int i = e & 1 ? i1 : i0, d = d0 + (e >> 1) * 8;
        const uint32_t q = *reinterpret_cast<const uint32_t*>(Q + i * KP + d);
        const float2 gi = *reinterpret_cast<const float2*>(G + i * GP + d);
        split2(bf16lo(q) * p.q_scale * ex2(gi.x - ref[(e >> 1) * 2]), bf16hi(q) * p.q_scale * ex2(gi.y - ref[(e >> 1) * 2 + 1]), ah[e], al[e]);
      }
#pragma unroll
      for (int c = 0; c < 3; ++c) {
        if (nt0 + c >= nt1 || (wide && (nt0 + c) >> 1 == I)) continue;
        const int j = 8 * (nt0 + c) + g;
        uint32_t bh[2], bl[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const uint32_t k = *reinterpret_cast<const uint32_t*>(K + j * KP + d0 + 8 * e);
          const float2 gj = *reinterpret_cast<const float2*>(G + j * GP + d0 + 8 * e);
          split2(bf16lo(k) * ex2(ref[2 * e] - gj.x), bf16hi(k) * ex2(ref[2 * e + 1] - gj.y), bh[e], bl[e]);
        }
        mma(acc[c], ah, bh[0], bh[1]);
        mma(acc[c], al, bh[0], bh[1]);
        mma(acc[c], ah, bl[0], bl[1]);
      }
    }
#pragma unroll
    for (int c = 0; c < 3; ++c) {
      if (nt0 + c >= nt1) continue;
      const int j0 = 8 * (nt0 + c) + 2 * t;
      if (wide && (nt0 + c) >> 1 == I) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = e < 2 ? i0 : i1, j = j0 + (e & 1);
          float s = 0.f;
          if (i >= j)
            for (int d = 0; d < DK; ++d)
              s = fmaf(__bfloat162float(Q[i * KP + d]) * p.q_scale * __bfloat162float(K[j * KP + d]), ex2(G[i * GP + d] - G[j * GP + d]), s);
          acc[c][e] = s;
        }
      }
      uint32_t hi, lo;
      split2(i0 >= j0 ? acc[c][0] : 0.f, i0 >= j0 + 1 ? acc[c][1] : 0.f, hi, lo);
      *reinterpret_cast<uint32_t*>(AH + i0 * AP + j0) = hi;
      *reinterpret_cast<uint32_t*>(AL + i0 * AP + j0) = lo;
      split2(i1 >= j0 ? acc[c][2] : 0.f, i1 >= j0 + 1 ? acc[c][3] : 0.f, hi, lo);
      *reinterpret_cast<uint32_t*>(AH + i1 * AP + j0) = hi;
      *reinterpret_cast<uint32_t*>(AL + i1 * AP + j0) = lo;
    }
  }
  __syncthreads();
  // ---- q exp(G), split, in the place of q and k
  for (int i = tid; i < C * DK / 2; i += 256) {
    const int j = i / (DK / 2), d = (i - j * (DK / 2)) * 2;
    const uint32_t q = *reinterpret_cast<const uint32_t*>(Q + j * KP + d);
    uint32_t hi, lo;
    split2(bf16lo(q) * p.q_scale * ex2(G[j * GP + d]), bf16hi(q) * p.q_scale * ex2(G[j * GP + d + 1]), hi, lo);
    *reinterpret_cast<uint32_t*>(Q + j * KP + d) = hi;
    *reinterpret_cast<uint32_t*>(K + j * KP + d) = lo;
  }
  // ---- outputs, 64 columns at a time: warp -> 16 tokens, a part of the columns.  The state tile of the next columns is
  //      requested before the products of these.
  constexpr int MT = C / 16, NT = MT, NLD = DK * 16 / 256;
  const int I = warp % MT, i0 = 16 * I, n0 = (warp / MT) * (NT * 8);
  const int mi = lane >> 3, row = lane & 7;
  const float* sp = p.s_ws + ch * DK * dv;
  float4 pre[NLD];
#pragma unroll
  for (int i = 0; i < NLD; ++i) pre[i] = *reinterpret_cast<const float4*>(sp + (size_t)((tid + i * 256) >> 4) * dv + (tid & 15) * 4);
  for (int v0 = 0; v0 < dv; v0 += 64) {
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NLD; ++i) {
      const int d = (tid + i * 256) >> 4, c = (tid & 15) * 4;
      uint32_t hi[2], lo[2];
      split2(pre[i].x, pre[i].y, hi[0], lo[0]);
      split2(pre[i].z, pre[i].w, hi[1], lo[1]);
      *reinterpret_cast<uint2*>(SH + d * VP + c) = make_uint2(hi[0], hi[1]);
      *reinterpret_cast<uint2*>(SL + d * VP + c) = make_uint2(lo[0], lo[1]);
    }
    for (int i = tid; i < C * 8; i += 256) {
      const int j = i >> 3, c = (i & 7) * 8;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (j < n) v = *reinterpret_cast<const uint4*>(proj + (size_t)(tok0 + j) * p.ld + p.v_col + h * dv + v0 + c);
      *reinterpret_cast<uint4*>(V + j * VP + c) = v;
    }
    __syncthreads();
    if (v0 + 64 < dv) {
#pragma unroll
      for (int i = 0; i < NLD; ++i) pre[i] = *reinterpret_cast<const float4*>(sp + (size_t)((tid + i * 256) >> 4) * dv + v0 + 64 + (tid & 15) * 4);
    }
    float acc[NT][4] = {};
#pragma unroll 4
    for (int kt = 0; kt < DK / 16; ++kt) {
      uint32_t ah[4], al[4];
      const int at = (i0 + (mi & 1) * 8 + row) * KP + kt * 16 + (mi >> 1) * 8;
      ldsm4(ah, Q + at);
      ldsm4(al, K + at);
#pragma unroll
      for (int c = 0; c < NT / 2; ++c) {
        uint32_t bh[4], bl[4];
        const int bt = (kt * 16 + (mi & 1) * 8 + row) * VP + n0 + c * 16 + (mi >> 1) * 8;
        ldsm4t(bh, SH + bt);
        ldsm4t(bl, SL + bt);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(acc[2 * c + e], ah, bh[2 * e], bh[2 * e + 1]);
          mma(acc[2 * c + e], al, bh[2 * e], bh[2 * e + 1]);
          mma(acc[2 * c + e], ah, bl[2 * e], bl[2 * e + 1]);
        }
      }
    }
    for (int kt = 0; kt <= I; ++kt) {
      uint32_t ah[4], al[4];
      const int at = (i0 + (mi & 1) * 8 + row) * AP + kt * 16 + (mi >> 1) * 8;
      ldsm4(ah, AH + at);
      ldsm4(al, AL + at);
#pragma unroll
      for (int c = 0; c < NT / 2; ++c) {
        uint32_t b[4];
        ldsm4t(b, V + (kt * 16 + (mi & 1) * 8 + row) * VP + n0 + c * 16 + (mi >> 1) * 8);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(acc[2 * c + e], ah, b[2 * e], b[2 * e + 1]);
          mma(acc[2 * c + e], al, b[2 * e], b[2 * e + 1]);
        }
      }
    }
    float* o = p.o + (size_t)(tok0 + i0 + g) * p.H * dv + h * dv + v0 + n0 + 2 * t;
#pragma unroll
    for (int c = 0; c < NT; ++c) {
      if (i0 + g < n) *reinterpret_cast<float2*>(o + c * 8) = make_float2(acc[c][0], acc[c][1]);
      if (i0 + g + 8 < n) *reinterpret_cast<float2*>(o + (size_t)8 * p.H * dv + c * 8) = make_float2(acc[c][2], acc[c][3]);
    }
  }
}

template <int DK>
static int launch_chunked(const GlaParams& p, int dv, cudaStream_t st) {
  using M = GlaGeom<DK>;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(gla_chunk_state_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kState);
    cudaFuncSetAttribute(gla_chunk_out_kernel<DK>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kOut);
    configured = true;
  }
  launch_kernel(gla_chunk_state_kernel<DK>, dim3(p.nc, p.H), dim3(256), M::kState, st, true, p, dv);
  launch_kernel(gla_chunk_scan_kernel, dim3((DK * dv + 1023) / 1024, p.H, p.num_long), dim3(256), 0, st, true, p, DK, dv, (int)M::C);
  launch_kernel(gla_chunk_out_kernel<DK>, dim3(p.nc, p.H), dim3(256), M::kOut, st, true, p, dv);
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_gla_chunk_size(int dk) { return dk == 64 || dk == 128 ? 64 : dk == 256 ? 32 : 0; }

// o[t, h] and the states of the sequences with chunks (projections in bf16)
int ti_gla_chunked(const ti::GlaParams* p, int dk, int dv, void* stream) {
  if (p->nc <= 0) return 0;
  if (dv % 64 || p->ld % 8 || p->q_col % 8 || p->k_col % 8 || p->v_col % 8 || p->R < 1 ||
      (((uintptr_t)p->proj | (uintptr_t)p->o | (uintptr_t)p->state | (uintptr_t)p->g_ws | (uintptr_t)p->s_ws) & 15))
    return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (dk == 64) return ti::launch_chunked<64>(*p, dv, st);
  if (dk == 128) return ti::launch_chunked<128>(*p, dv, st);
  if (dk == 256) return ti::launch_chunked<256>(*p, dv, st);
  return -3;
}

}  // extern "C"
