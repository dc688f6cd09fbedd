// The gated and the general delta rule (delta.cuh) of long portions, in chunks of C tokens on the tensor cores.
//
// With G_t the running sum of the log decays inside a chunk and S the state before it, the reads y_t = u_t^T S_(t-1) solve a
// unit lower triangular system.  Everything that follows is linear in S and in the values, so a chunk is three matrices:
//     S' = (diag(exp G_C) - R) S + E^T V            O = Q S + W V
// general, with  u~ = u exp(G_(t-1)), q~ = q exp(G_t), k^ = k exp(-G_j), p^ = p exp(-G_j)  per key channel:
//     A = (u~ p^T) strictly below,  M = (I + A)^-1,  D = M u~,  N = M (u~ k^T)
//     R = diag(exp G_C) p^T D       E = exp(G_C) (k^ - N^T p^)       Q = q~ - (q~ p^T) D       W = (q~ k^T) - (q~ p^T) N
//   (the decay of a chunk is bounded by the design, so the factors stay far inside the range of a float)
// gated: one decay per token multiplies finished products u u^T and q u^T, which come from the bf16 inputs exactly; with
//     p^ = u exp(G_C - G_j),  M from beta_t exp(G_t - G_j) u_t.u_j,  D = M (beta u exp G),  N = -M diag(beta),  k^ = 0,
//   the same formulas hold (p^ carries exp G_C already).
//
//     delta_chunk_prepare_kernel   the matrices of a chunk                                      (chunk, head)
//     delta_chunk_scan_kernel      S before every chunk, the state after the last, snapshots    (columns of a head, sequence)
//     delta_chunk_out_kernel       outputs                                                      (chunk, head)
//
// Decays, products and states are fp32; where they enter a tensor-core product they are split into two bf16 terms (about 16
// bits).  The decay's part of S' never leaves fp32.  Matrices pass between the kernels in the order of mma fragments: the
// accumulators of one product are the operands of the next, a 16 x 16 tile as one 16-byte word per lane and term.
#include "delta.cuh"
#include "mma_split.cuh"

namespace ti {

template <int DK> struct DeltaGeom {
  static constexpr int C = DK == 256 ? 32 : 64;          // tokens of a chunk
  static constexpr int MT = C / 16, KT = DK / 16;
  static constexpr int KP = DK + 8, AP = C + 8, VP = 64 + 8;       // pitches: ldmatrix rows start 16 bytes apart modulo 128
  static constexpr int GP = DK + 4, FP = C + 4;                    // floats
  static constexpr int kK = C * KP * 2, kA = C * AP * 2, kG = C * GP * 4;
  static constexpr int kSmall = 8 * kA > kG ? 8 * kA : kG;         // the C x C matrices, over the running decays
  static constexpr size_t kScan = (size_t)2 * KT * 128 * 16;
  static constexpr size_t kSmem = (size_t)8 * kK + kSmall + C * VP * 2 + (DK + 4 * C) * 4;
  static_assert(C * FP * 4 <= 2 * kA && (C / 2) * (C / 2) * 4 <= C * VP * 2, "overlays");
};

// 16 x 16 tile as two accumulators -> the word of a lane
TI_DEVICE void pack_tile(const float (&a)[2][4], uint4& hi, uint4& lo) {
  split2(a[0][0], a[0][1], hi.x, lo.x);
  split2(a[0][2], a[0][3], hi.y, lo.y);
  split2(a[1][0], a[1][1], hi.z, lo.z);
  split2(a[1][2], a[1][3], hi.w, lo.w);
}
// two accumulators -> rows i0 + g, i0 + g + 8, columns c0 ..
TI_DEVICE void store_tile(const float (&a)[2][4], bf16* H, bf16* L, int pitch, int i0, int c0, int g, int t) {
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    uint32_t hi, lo;
    split2(a[e >> 1][(e & 1) * 2], a[e >> 1][(e & 1) * 2 + 1], hi, lo);
    const int at = (i0 + g + (e & 1) * 8) * pitch + c0 + (e >> 1) * 8 + 2 * t;
    *reinterpret_cast<uint32_t*>(H + at) = hi;
    *reinterpret_cast<uint32_t*>(L + at) = lo;
  }
}
TI_DEVICE void load_tile(float (&a)[2][4], const bf16* H, const bf16* L, int pitch, int i0, int c0, int g, int t) {
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int at = (i0 + g + (e & 1) * 8) * pitch + c0 + (e >> 1) * 8 + 2 * t;
    const uint32_t hi = *reinterpret_cast<const uint32_t*>(H + at), lo = *reinterpret_cast<const uint32_t*>(L + at);
    a[e >> 1][(e & 1) * 2] = bf16lo(hi) + bf16lo(lo);
    a[e >> 1][(e & 1) * 2 + 1] = bf16hi(hi) + bf16hi(lo);
  }
}
// fragments of a 16 x 16 tile of A stored [row][k], of A stored [k][row], of B stored [k][n], of B stored [n][k]
TI_DEVICE void frag_a(uint32_t (&r)[4], const bf16* p, int pitch, int row0, int k0, int lane) {
  ldsm4(r, p + (row0 + ((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + k0 + (lane >> 4) * 8);
}
TI_DEVICE void frag_at(uint32_t (&r)[4], const bf16* p, int pitch, int row0, int k0, int lane) {
  ldsm4t(r, p + (k0 + (lane >> 4) * 8 + (lane & 7)) * pitch + row0 + ((lane >> 3) & 1) * 8);
}
TI_DEVICE void frag_b(uint32_t (&r)[4], const bf16* p, int pitch, int k0, int n0, int lane) {
  ldsm4t(r, p + (k0 + ((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + n0 + (lane >> 4) * 8);
}
TI_DEVICE void frag_bt(uint32_t (&r)[4], const bf16* p, int pitch, int k0, int n0, int lane) {
  ldsm4(r, p + (n0 + (lane >> 4) * 8 + (lane & 7)) * pitch + k0 + ((lane >> 3) & 1) * 8);
}
// acc += (ah + al) (bh + bl), 16 x 16 x 16, without the product of the small terms
TI_DEVICE void mma3(float (&acc)[2][4], const uint32_t (&ah)[4], const uint32_t (&al)[4], const uint32_t (&bh)[4], const uint32_t (&bl)[4]) {
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    mma(acc[e], ah, bh[2 * e], bh[2 * e + 1]);
    mma(acc[e], al, bh[2 * e], bh[2 * e + 1]);
    mma(acc[e], ah, bl[2 * e], bl[2 * e + 1]);
  }
}

// ------------------------------------------------------------------------------------------------ the matrices of a chunk
constexpr int kPrepWarps = 16, kPrepThreads = 32 * kPrepWarps;

template <int DK, bool GENERAL>
__global__ void __launch_bounds__(kPrepThreads) delta_chunk_prepare_kernel(const __grid_constant__ DeltaParams p, int dv) {
  using M = DeltaGeom<DK>;
  constexpr int C = M::C, MT = M::MT, KT = M::KT, KP = M::KP, AP = M::AP, VP = M::VP, GP = M::GP, FP = M::FP;
  extern __shared__ __align__(16) uint8_t smem[];
  bf16 *UH = reinterpret_cast<bf16*>(smem), *UL = UH + C * KP;     // u~, then D
  bf16 *QH = UL + C * KP, *QL = QH + C * KP;                       // q~
  bf16 *PH = QL + C * KP, *PL = PH + C * KP;                       // p^
  bf16 *KH = PL + C * KP, *KL = KH + C * KP;                       // k^ (gated: the bf16 keys and queries), then E
  uint8_t* small = smem + 8 * M::kK;
  float* G = reinterpret_cast<float*>(small);                      // [C][GP] running log2 decays
  float* F = reinterpret_cast<float*>(small);                      // [C][FP] A, then its inverse
  bf16 *MH = reinterpret_cast<bf16*>(small), *ML = MH + C * AP;    // M
  bf16 *NH = ML + C * AP, *NL = NH + C * AP;                       // u~ k^T, then N
  bf16 *AH = NL + C * AP, *AL = AH + C * AP;                       // q~ p^T
  bf16 *WH = AL + C * AP, *WL = WH + C * AP;                       // q~ k^T, then W
  bf16* V = reinterpret_cast<bf16*>(small + M::kSmall);
  float* tmp = reinterpret_cast<float*>(V);
  float* sc = reinterpret_cast<float*>(V + C * VP);                // [DK] what p^ lacks: exp(G_C), or 1
  float *rk = sc + DK, *rq = rk + C, *cg = rq + C, *bt = cg + C;   // [C] 1 / length of k and q; gated: running log2 decay, beta
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  const int ci = blockIdx.x, h = blockIdx.y, tok0 = p.ck_tok0[ci], n = p.ck_ntok[ci], kh = h / p.rep;
  const size_t ch = (size_t)ci * p.H + h;
  pdl_trigger();
  pdl_wait();
  const bf16 *src = static_cast<const bf16*>(p.src) + (size_t)tok0 * p.lds, *proj = static_cast<const bf16*>(p.proj) + (size_t)tok0 * p.ld;

  // ---- the first value columns, requested now and used last
  const int vj = tid >> 3, vc = (tid & 7) * 8;                     // row and column of a thread's 16 bytes (C 32: half of the threads)
  const bool has_v = vj < n && vj < C;
  const bf16* vsrc = src + (size_t)(has_v ? vj : 0) * p.lds + p.v_col + h * dv + vc;
  uint4 vnext = make_uint4(0u, 0u, 0u, 0u);
  if (has_v) vnext = *reinterpret_cast<const uint4*>(vsrc);
  // ---- lengths, decays and rates of the tokens
  {
    constexpr int NT = C / kPrepWarps;
    float kk[NT], qq[NT], ga[NT], gb[NT];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int j = warp + kPrepWarps * i;
      kk[i] = qq[i] = ga[i] = gb[i] = 0.f;
      if (j >= n) continue;
#pragma unroll
      for (int d = lane * 2; d < DK; d += 64) {
        const uint32_t k = *reinterpret_cast<const uint32_t*>(src + (size_t)j * p.lds + p.k_col + kh * DK + d);
        kk[i] += bf16lo(k) * bf16lo(k) + bf16hi(k) * bf16hi(k);
        if (GENERAL) continue;
        const uint32_t q = *reinterpret_cast<const uint32_t*>(src + (size_t)j * p.lds + p.q_col + kh * DK + d);
        qq[i] += bf16lo(q) * bf16lo(q) + bf16hi(q) * bf16hi(q);
      }
      if (!GENERAL) {
        ga[i] = __bfloat162float(proj[(size_t)j * p.ld + p.a_col + h]);
        gb[i] = __bfloat162float(proj[(size_t)j * p.ld + p.b_col + h]);
      }
    }
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int j = warp + kPrepWarps * i;
      kk[i] = warp_sum(kk[i]);
      if (!GENERAL) qq[i] = warp_sum(qq[i]);
      if (lane == 0) {
        rk[j] = rsqrtf(kk[i] + kUnitEps);
        rq[j] = rsqrtf(qq[i] + kUnitEps) * p.q_scale;
        if (!GENERAL) {
          cg[j] = j < n ? p.neg_a[h] * softplus_exact(ga[i] + p.bias[h]) * kLog2e : 0.f;
          bt[j] = j < n ? sigmoid_exact(gb[i]) : 0.f;
        }
      }
    }
  }
  if (GENERAL) {
    // log2 decays of (channel, segment of SEG tokens), their running sums
    constexpr int NS = kPrepThreads / DK, SEG = C / NS, RC = 32;
    float* xin = reinterpret_cast<float*>(UH);             // [C][RC]
    const int d = tid % DK, seg = tid / DK, col = h * DK + d, cols = p.H * DK;
    float z[SEG];
    const float bias = p.w0[col];
#pragma unroll
    for (int j = 0; j < SEG; ++j) z[j] = bias;
    for (int r0 = 0; r0 < p.R; r0 += RC) {
      const int rn = min(RC, p.R - r0);
      __syncthreads();
      for (int i = tid; i < C * RC; i += kPrepThreads) {
        const int j = i / RC, r = i - j * RC;
        xin[i] = j < n && r < rn ? tanhf(__bfloat162float(proj[(size_t)j * p.ld + p.a_col + r0 + r])) : 0.f;
      }
      __syncthreads();
#pragma unroll 2
      for (int r = 0; r < rn; r += 4) {                    // ranks past the last meet zeros
        float a[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) a[e] = __ldg(p.w2 + (size_t)min(r0 + r + e, p.R - 1) * cols + col);
#pragma unroll
        for (int j = 0; j < SEG; ++j) {
          const float4 x = *reinterpret_cast<const float4*>(xin + (seg * SEG + j) * RC + r);
          z[j] = fmaf(a[0], x.x, fmaf(a[1], x.y, fmaf(a[2], x.z, fmaf(a[3], x.w, z[j]))));
        }
      }
    }
    float run = 0.f;
#pragma unroll
    for (int j = 0; j < SEG; ++j) {
      if (seg * SEG + j < n) run -= p.decay_scale * kLog2e * sigmoid_exact(z[j]);
      z[j] = run;
    }
    tmp[seg * DK + d] = run;                               // [NS][DK] sums of the segments
    __syncthreads();
    float base = 0.f;
    for (int s = 0; s < seg; ++s) base += tmp[s * DK + d];
#pragma unroll
    for (int j = 0; j < SEG; ++j) G[(seg * SEG + j) * GP + d] = z[j] + base;
    if (seg == NS - 1) {
      const float e = ex2(z[SEG - 1] + base);
      sc[d] = e;
      p.f_ws[ch * DK + d] = e;
    }
  }
  __syncthreads();
  if (!GENERAL) {
    if (warp == 0) {                                       // running sum over the tokens
      float c[MT / 2], run = 0.f;
#pragma unroll
      for (int i = 0; i < MT / 2; ++i) {
        c[i] = cg[i * 32 + lane];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float up = __shfl_up_sync(0xffffffffu, c[i], o);
          if (lane >= o) c[i] += up;
        }
        c[i] += run;
        run = __shfl_sync(0xffffffffu, c[i], 31);
        cg[i * 32 + lane] = c[i];
      }
    }
    __syncthreads();
    for (int d = tid; d < DK; d += kPrepThreads) {
      sc[d] = 1.f;
      p.f_ws[ch * DK + d] = ex2(cg[C - 1]);
    }
  }
  // ---- the scaled operands
#pragma unroll
  for (int it = 0; it < C * DK / 8 / kPrepThreads; ++it) {
    const int i = tid + it * kPrepThreads, j = i / (DK / 8), d = (i - j * (DK / 8)) * 8;
    float k[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, q[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f}, a[8], u[8], e[8], f[8];
    uint4 kr = make_uint4(0u, 0u, 0u, 0u), qr = kr;
    if (j < n) {
      kr = *reinterpret_cast<const uint4*>(src + (size_t)j * p.lds + p.k_col + kh * DK + d);
      qr = *reinterpret_cast<const uint4*>(src + (size_t)j * p.lds + p.q_col + kh * DK + d);
      load8(reinterpret_cast<const bf16*>(&kr), k);
      load8(reinterpret_cast<const bf16*>(&qr), q);
    }
    auto put = [&](bf16* H, bf16* L, const float (&v)[8]) {
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int x = 0; x < 4; ++x) split2(v[2 * x], v[2 * x + 1], hi[x], lo[x]);
      *reinterpret_cast<uint4*>(H + j * KP + d) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(L + j * KP + d) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    };
    if (GENERAL) {
      float b[8] = {0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f, 0.f};
      if (j < n) load8(proj + (size_t)j * p.ld + p.b_col + h * DK + d, b);
      load8(p.bias + h * DK + d, a);
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        const float gj = G[j * GP + d + x], gb = j > 0 ? G[(j - 1) * GP + d + x] : 0.f;
        const float unit = k[x] * rk[j], back = ex2(-gj);
        u[x] = unit * ex2(gb);
        q[x] *= ex2(gj);
        e[x] = k[x] * back;
        f[x] = sigmoid_exact(b[x] + a[x]) * unit * back;
      }
      put(KH, KL, e);
    } else {
      const float fu = rk[j] * bt[j] * ex2(cg[j]), fq = rq[j] * ex2(cg[j]), fp = rk[j] * ex2(cg[C - 1] - cg[j]);
#pragma unroll
      for (int x = 0; x < 8; ++x) {
        u[x] = k[x] * fu;
        q[x] *= fq;
        f[x] = k[x] * fp;
      }
      *reinterpret_cast<uint4*>(KH + j * KP + d) = kr;
      *reinterpret_cast<uint4*>(KL + j * KP + d) = qr;
    }
    put(UH, UL, u);
    put(QH, QL, q);
    put(PH, PL, f);
  }
  __syncthreads();

  // ---- the C x C products, blocks of 16 x 16 on and below the diagonal (LB of them): u~ and q~ against p^ and k^, each by
  //      four warps (gated: keys and queries against the keys, each by eight)
  constexpr int LB = MT * (MT + 1) / 2;
  constexpr int kLI[10] = {0, 1, 1, 2, 2, 2, 3, 3, 3, 3}, kLJ[10] = {0, 0, 1, 0, 1, 2, 0, 1, 2, 3};
  for (int i = tid; i < C * C; i += kPrepThreads)          // A is read above its diagonal too
    if (((i % C) >> 4) > (i / C) >> 4) F[(i / C) * FP + i % C] = 0.f;
  {
    constexpr int SHARE = GENERAL ? 4 : 8, NB = (LB + SHARE - 1) / SHARE;
    const bool with_q = warp & 1, with_k = GENERAL && (warp & 2);
    const int first = GENERAL ? warp >> 2 : warp >> 1;
    float acc[NB][2][4] = {};
#pragma unroll 2
    for (int kt = 0; kt < KT; ++kt) {
#pragma unroll
      for (int b = 0; b < NB; ++b) {
        const int at = first + SHARE * b;
        if (at >= LB) continue;
        const int I = kLI[at], J = kLJ[at];
        uint32_t ah[4], al[4], bh[4], bl[4];
        if (GENERAL) {
          frag_a(ah, with_q ? QH : UH, KP, 16 * I, 16 * kt, lane);
          frag_a(al, with_q ? QL : UL, KP, 16 * I, 16 * kt, lane);
          frag_bt(bh, with_k ? KH : PH, KP, 16 * kt, 16 * J, lane);
          frag_bt(bl, with_k ? KL : PL, KP, 16 * kt, 16 * J, lane);
          mma3(acc[b], ah, al, bh, bl);
        } else {
          frag_a(ah, with_q ? KL : KH, KP, 16 * I, 16 * kt, lane);
          frag_bt(bh, KH, KP, 16 * kt, 16 * J, lane);
          mma(acc[b][0], ah, bh[0], bh[1]);
          mma(acc[b][1], ah, bh[2], bh[3]);
        }
      }
    }
#pragma unroll
    for (int b = 0; b < NB; ++b) {
      const int at = first + SHARE * b;
      if (at >= LB) continue;
      const int I = kLI[at], J = kLJ[at];
#pragma unroll
      for (int e = 0; e < 8; ++e) {
        const int i = 16 * I + g + ((e >> 1) & 1) * 8, j = 16 * J + (e >> 2) * 8 + 2 * t + (e & 1);
        float& v = acc[b][e >> 2][e & 3];
        if (!GENERAL) v = i >= j ? v * (with_q ? rq[i] : bt[i] * rk[i]) * rk[j] * ex2(cg[i] - cg[j]) : 0.f;
        if (with_q ? j > i : j >= i) v = 0.f;
        if (!with_q && !with_k) F[i * FP + j] = v;
      }
      if (with_q) store_tile(acc[b], with_k ? WH : AH, with_k ? WL : AL, AP, 16 * I, 16 * J, g, t);
      else if (with_k) store_tile(acc[b], NH, NL, AP, 16 * I, 16 * J, g, t);
    }
  }
  __syncthreads();

  // ---- M = (I + A)^-1 in place: diagonal blocks of 16 by substitution, then two by two
  {
    float x[16];
    const int b = tid >> 4, c = tid & 15;
    if (tid < C) {
      const float* f = F + 16 * b * FP + 16 * b;
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float s = i == c ? 1.f : 0.f;
#pragma unroll
        for (int j = 0; j < i; ++j) s = fmaf(-f[i * FP + j], x[j], s);
        x[i] = i < c ? 0.f : s;
      }
    }
    __syncthreads();
    if (tid < C) {
#pragma unroll
      for (int i = 0; i < 16; ++i) F[(16 * b + i) * FP + 16 * b + c] = x[i];
    }
    __syncthreads();
#pragma unroll
    for (int s = 16; s < C; s *= 2) {                      // [M11 0; -M22 A21 M11, M22]
      const int duos = s * s / 2, pairs = C / (2 * s);
      for (int pass = 0; pass < 2; ++pass) {
        for (int e = tid; e < duos * pairs; e += kPrepThreads) {
          const int pr = e / duos, r = (e - pr * duos) / (s / 2), c0 = ((e - pr * duos) % (s / 2)) * 2, o = pr * 2 * s;
          float2 sum = make_float2(0.f, 0.f);
          const float *a = F + (o + s + r) * FP + (pass == 0 ? o : o + s), *m = pass == 0 ? F + o * FP + o + c0 : tmp + pr * s * s + c0;
          const int mp = pass == 0 ? FP : s;
#pragma unroll 8
          for (int k = 0; k < s; ++k) {
            const float2 v = *reinterpret_cast<const float2*>(m + k * mp);
            const float f = a[k];
            sum.x = fmaf(f, v.x, sum.x);
            sum.y = fmaf(f, v.y, sum.y);
          }
          if (pass == 0) *reinterpret_cast<float2*>(tmp + pr * s * s + r * s + c0) = sum;
          else *reinterpret_cast<float2*>(F + (o + s + r) * FP + o + c0) = make_float2(-sum.x, -sum.y);
        }
        __syncthreads();
      }
    }
    constexpr int NE = C * C / 2 / kPrepThreads;           // pairs of columns per thread
    float2 m[NE];
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int at = (tid + e * kPrepThreads) * 2, i = at / C, j = at % C;
      m[e] = make_float2(j <= i ? F[i * FP + j] : 0.f, j + 1 <= i ? F[i * FP + j + 1] : 0.f);
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < NE; ++e) {
      const int at = (tid + e * kPrepThreads) * 2, i = at / C, j = at % C;
      uint32_t hi, lo;
      split2(m[e].x, m[e].y, hi, lo);
      *reinterpret_cast<uint32_t*>(MH + i * AP + j) = hi;
      *reinterpret_cast<uint32_t*>(ML + i * AP + j) = lo;
      if (!GENERAL) {
        split2(-m[e].x * bt[j], -m[e].y * bt[j + 1], hi, lo);
        *reinterpret_cast<uint32_t*>(NH + i * AP + j) = hi;
        *reinterpret_cast<uint32_t*>(NL + i * AP + j) = lo;
      }
    }
    __syncthreads();
  }

  // tiles of a C x DK product, column tile varies first; blocks on and below the diagonal of a C x C matrix, one per warp
  constexpr int NI = MT * KT / kPrepWarps;
  const bool has_low = warp < LB;
  const int lowI = has_low ? kLI[warp] : 0, lowJ = has_low ? kLJ[warp] : 0;

  // ---- D = M u~, N = M (u~ k^T)
  {
    float acc[NI][2][4] = {}, nn[2][4] = {};
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int id = warp + kPrepWarps * i, c0 = (id % KT) * 16, I = id / KT;
#pragma unroll
      for (int kt = 0; kt < MT; ++kt) {
        if (kt > I) continue;
        uint32_t ah[4], al[4], bh[4], bl[4];
        frag_a(ah, MH, AP, 16 * I, 16 * kt, lane);
        frag_a(al, ML, AP, 16 * I, 16 * kt, lane);
        frag_b(bh, UH, KP, 16 * kt, c0, lane);
        frag_b(bl, UL, KP, 16 * kt, c0, lane);
        mma3(acc[i], ah, al, bh, bl);
      }
    }
    if (GENERAL && has_low) {
      for (int kt = lowJ; kt <= lowI; ++kt) {
        uint32_t ah[4], al[4], bh[4], bl[4];
        frag_a(ah, MH, AP, 16 * lowI, 16 * kt, lane);
        frag_a(al, ML, AP, 16 * lowI, 16 * kt, lane);
        frag_b(bh, NH, AP, 16 * kt, 16 * lowJ, lane);
        frag_b(bl, NL, AP, 16 * kt, 16 * lowJ, lane);
        mma3(nn, ah, al, bh, bl);
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int id = warp + kPrepWarps * i;
      store_tile(acc[i], UH, UL, KP, (id / KT) * 16, (id % KT) * 16, g, t);
    }
    if (GENERAL && has_low) store_tile(nn, NH, NL, AP, 16 * lowI, 16 * lowJ, g, t);
    __syncthreads();
  }

  // ---- Q = q~ - A D into the workspace; E = (k^ - N^T p^) exp(G_C) in the place of k^
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int id = warp + kPrepWarps * i, ct = id % KT, c0 = ct * 16, I = id / KT;
    float acc[2][4] = {}, ee[2][4] = {}, q[2][4];
#pragma unroll
    for (int kt = 0; kt < MT; ++kt) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      if (kt <= I) {
        frag_a(ah, AH, AP, 16 * I, 16 * kt, lane);
        frag_a(al, AL, AP, 16 * I, 16 * kt, lane);
        frag_b(bh, UH, KP, 16 * kt, c0, lane);
        frag_b(bl, UL, KP, 16 * kt, c0, lane);
        mma3(acc, ah, al, bh, bl);
      }
      if (kt >= I) {
        frag_at(ah, NH, AP, 16 * I, 16 * kt, lane);
        frag_at(al, NL, AP, 16 * I, 16 * kt, lane);
        frag_b(bh, PH, KP, 16 * kt, c0, lane);
        frag_b(bl, PL, KP, 16 * kt, c0, lane);
        mma3(ee, ah, al, bh, bl);
      }
    }
    load_tile(q, QH, QL, KP, 16 * I, c0, g, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) q[e >> 2][e & 3] -= acc[e >> 2][e & 3];
    uint4 hi, lo;
    pack_tile(q, hi, lo);
    uint4* dst = p.q_ws + ((ch * MT + I) * KT + ct) * 64 + lane;
    dst[0] = hi;
    dst[32] = lo;
    if (GENERAL) load_tile(q, KH, KL, KP, 16 * I, c0, g, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float s = sc[c0 + (e >> 2) * 8 + 2 * t + (e & 1)];
      q[e >> 2][e & 3] = ((GENERAL ? q[e >> 2][e & 3] : 0.f) - ee[e >> 2][e & 3]) * s;
    }
    store_tile(q, KH, KL, KP, 16 * I, c0, g, t);
  }
  // ---- W = (q~ k^T) - A N in the place of the first
  if (has_low) {
    float acc[2][4] = {}, w[2][4] = {};
    for (int kt = lowJ; kt <= lowI; ++kt) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      frag_a(ah, AH, AP, 16 * lowI, 16 * kt, lane);
      frag_a(al, AL, AP, 16 * lowI, 16 * kt, lane);
      frag_b(bh, NH, AP, 16 * kt, 16 * lowJ, lane);
      frag_b(bl, NL, AP, 16 * kt, 16 * lowJ, lane);
      mma3(acc, ah, al, bh, bl);
    }
    if (GENERAL) load_tile(w, WH, WL, AP, 16 * lowI, 16 * lowJ, g, t);
#pragma unroll
    for (int e = 0; e < 8; ++e) w[e >> 2][e & 3] -= acc[e >> 2][e & 3];
    store_tile(w, WH, WL, AP, 16 * lowI, 16 * lowJ, g, t);
  }
  // ---- -R = -exp(G_C) p^T D into the workspace: a warp takes RUN column tiles of one row tile
  {
    constexpr int RUN = KT * KT / kPrepWarps;
    const int rt = warp % KT, first = (warp / KT) * RUN;
    uint32_t ah[MT][4], al[MT][4];
#pragma unroll
    for (int kt = 0; kt < MT; ++kt) {
      frag_at(ah[kt], PH, KP, 16 * rt, 16 * kt, lane);
      frag_at(al[kt], PL, KP, 16 * rt, 16 * kt, lane);
    }
    const float s0 = -sc[16 * rt + g], s1 = -sc[16 * rt + g + 8];
#pragma unroll 2
    for (int ct = first; ct < first + RUN; ++ct) {
      float acc[2][4] = {};
#pragma unroll
      for (int kt = 0; kt < MT; ++kt) {
        uint32_t bh[4], bl[4];
        frag_b(bh, UH, KP, 16 * kt, 16 * ct, lane);
        frag_b(bl, UL, KP, 16 * kt, 16 * ct, lane);
        mma3(acc, ah[kt], al[kt], bh, bl);
      }
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[e >> 2][e & 3] *= e & 2 ? s1 : s0;
      uint4 hi, lo;
      pack_tile(acc, hi, lo);
      uint4* dst = p.t_ws + ((ch * KT + rt) * KT + ct) * 64 + lane;
      dst[0] = hi;
      dst[32] = lo;
    }
  }
  // ---- E^T V (transposed: rows are value columns) and W V, 64 value columns at a time
  for (int v0 = 0; v0 < dv; v0 += 64) {
    __syncthreads();
    if (vj < C) *reinterpret_cast<uint4*>(V + vj * VP + vc) = vnext;
    if (has_v && v0 + 64 < dv) vnext = *reinterpret_cast<const uint4*>(vsrc + v0 + 64);
    __syncthreads();
    constexpr int NE = 4 * KT / kPrepWarps;
#pragma unroll
    for (int i = 0; i < NE; ++i) {
      const int id = warp + kPrepWarps * i, ct = id % KT, vt = id / KT;
      float acc[2][4] = {};
#pragma unroll
      for (int kt = 0; kt < MT; ++kt) {
        uint32_t a[4], bh[4], bl[4];
        frag_at(a, V, VP, 16 * vt, 16 * kt, lane);
        frag_b(bh, KH, KP, 16 * kt, 16 * ct, lane);
        frag_b(bl, KL, KP, 16 * kt, 16 * ct, lane);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(acc[e], a, bh[2 * e], bh[2 * e + 1]);
          mma(acc[e], a, bl[2 * e], bl[2 * e + 1]);
        }
      }
      float4* dst = p.s_ws + ((ch * (dv / 16) + v0 / 16 + vt) * KT + ct) * 64 + lane;
      dst[0] = make_float4(acc[0][0], acc[0][1], acc[0][2], acc[0][3]);
      dst[32] = make_float4(acc[1][0], acc[1][1], acc[1][2], acc[1][3]);
    }
    if (warp < 4 * MT) {
      const int vt = warp / MT, I = (warp + vt) % MT;      // neighbours share a scheduler: the long rows go to all of them
      float acc[2][4] = {};
      for (int kt = 0; kt <= I; ++kt) {
        uint32_t ah[4], al[4], b[4];
        frag_a(ah, WH, AP, 16 * I, 16 * kt, lane);
        frag_a(al, WL, AP, 16 * I, 16 * kt, lane);
        frag_b(b, V, VP, 16 * kt, 16 * vt, lane);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          mma(acc[e], ah, b[2 * e], b[2 * e + 1]);
          mma(acc[e], al, b[2 * e], b[2 * e + 1]);
        }
      }
      float* o = p.o + (size_t)(tok0 + 16 * I + g) * p.H * dv + h * dv + v0 + 16 * vt + 2 * t;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        if (16 * I + g < n) *reinterpret_cast<float2*>(o + e * 8) = make_float2(acc[e][0], acc[e][1]);
        if (16 * I + g + 8 < n) *reinterpret_cast<float2*>(o + (size_t)8 * p.H * dv + e * 8) = make_float2(acc[e][2], acc[e][3]);
      }
    }
  }
}

// ------------------------------------------------------------------------------------------------ scan over the chunks
// A block owns 16 NV columns of a head's state (transposed: rows are value columns), a warp 16 key channels of it in fp32
// registers.  Per chunk the state goes to shared memory as two bf16 terms, every warp multiplies all of it with its rows of
// -R, and the decay and what the chunk adds come on top in fp32.  The three products of the terms are summed apart, so that
// no chain of products is longer than the keys have tiles.
template <int DK, int NV>
__global__ void __launch_bounds__(DK * 2) delta_chunk_scan_kernel(const __grid_constant__ DeltaParams p, int dv) {
  constexpr int KT = DK / 16, PF = KT == 8 ? 8 : 4;
  extern __shared__ __align__(16) uint8_t smem[];
  uint4 (*sh)[KT][2][NV][32] = reinterpret_cast<uint4 (*)[KT][2][NV][32]>(smem);     // [buffer][key tile][term][16 columns][lane]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int vt0 = blockIdx.x * NV, h = blockIdx.y, s = p.long_seq[blockIdx.z], c0 = p.long_ck[blockIdx.z], c1 = p.long_ck[blockIdx.z + 1];
  float* state = p.state + ((size_t)p.slots[s] * p.H + h) * DK * dv;
  const int key0 = warp * 16 + 2 * t, col0 = vt0 * 16 + g;
  float S[NV][2][4];                                       // [16 columns][8 keys]
#pragma unroll
  for (int v = 0; v < NV; ++v)
#pragma unroll
    for (int e = 0; e < 8; ++e) S[v][e >> 2][e & 3] = state[(size_t)(key0 + (e >> 2) * 8 + (e & 1)) * dv + col0 + v * 16 + (e & 2) * 4];
  pdl_trigger();
  pdl_wait();
  const size_t tstep = (size_t)p.H * KT * KT * 64, sstep = (size_t)p.H * (dv / 16) * KT * 64;
  const uint4* tp = p.t_ws + (((size_t)c0 * p.H + h) * KT + warp) * KT * 64 + lane;
  float4* sp = p.s_ws + ((((size_t)c0 * p.H + h) * (dv / 16) + vt0) * KT + warp) * 64 + lane;
  const float* fp = p.f_ws + ((size_t)c0 * p.H + h) * DK + key0;
  uint4 bh[PF], bl[PF];
  float4 add[NV][2];
  float2 f[2];
  auto fetch_small = [&]() {
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 2; ++e) add[v][e] = sp[v * KT * 64 + e * 32];
    f[0] = *reinterpret_cast<const float2*>(fp);
    f[1] = *reinterpret_cast<const float2*>(fp + 8);
  };
#pragma unroll
  for (int k = 0; k < PF; ++k) {
    bh[k] = tp[k * 64];
    bl[k] = tp[k * 64 + 32];
  }
  fetch_small();
  for (int c = c0; c < c1; ++c) {
    const int b = c & 1;
    uint4 hi[NV], lo[NV];
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      pack_tile(S[v], hi[v], lo[v]);
      sh[b][warp][0][v][lane] = hi[v];
      sh[b][warp][1][v][lane] = lo[v];
    }
    __syncthreads();
#pragma unroll
    for (int v = 0; v < NV; ++v) {
      uint4* dst = reinterpret_cast<uint4*>(sp + v * KT * 64);           // what the chunk added has been read
      dst[0] = hi[v];
      dst[32] = lo[v];
    }
    float acc[NV][2][2][4] = {};                           // the two cross products
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        S[v][e][0] = fmaf(f[e].x, S[v][e][0], add[v][e].x);
        S[v][e][1] = fmaf(f[e].y, S[v][e][1], add[v][e].y);
        S[v][e][2] = fmaf(f[e].x, S[v][e][2], add[v][e].z);
        S[v][e][3] = fmaf(f[e].y, S[v][e][3], add[v][e].w);
      }
    const bool more = c + 1 < c1;
    sp += sstep;
    fp += (size_t)p.H * DK;
    if (more) fetch_small();
#pragma unroll
    for (int k0 = 0; k0 < KT; k0 += PF) {
#pragma unroll
      for (int k = 0; k < PF; ++k) {
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          const uint4 a = sh[b][k0 + k][0][v][lane], z = sh[b][k0 + k][1][v][lane];
          mma_bf16_16816(S[v][0], a.x, a.y, a.z, a.w, bh[k].x, bh[k].z);
          mma_bf16_16816(S[v][1], a.x, a.y, a.z, a.w, bh[k].y, bh[k].w);
          mma_bf16_16816(acc[v][0][0], z.x, z.y, z.z, z.w, bh[k].x, bh[k].z);
          mma_bf16_16816(acc[v][0][1], z.x, z.y, z.z, z.w, bh[k].y, bh[k].w);
          mma_bf16_16816(acc[v][1][0], a.x, a.y, a.z, a.w, bl[k].x, bl[k].z);
          mma_bf16_16816(acc[v][1][1], a.x, a.y, a.z, a.w, bl[k].y, bl[k].w);
        }
        // the word PF tiles ahead: of this chunk, or of the next
        if (k0 + PF < KT || more) {
          const uint4* q = tp + (k0 + PF < KT ? (size_t)(k0 + PF + k) * 64 : tstep + (size_t)k * 64);
          bh[k] = q[0];
          bl[k] = q[32];
        }
      }
    }
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
      for (int e = 0; e < 8; ++e) S[v][e >> 2][e & 3] += acc[v][0][e >> 2][e & 3] + acc[v][1][e >> 2][e & 3];
    tp += tstep;
    const int snap = p.ck_snap[c];
    if (snap >= 0) {
      float* dst = p.snap + ((size_t)snap * p.H + h) * DK * dv;
#pragma unroll
      for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int e = 0; e < 8; ++e) dst[(size_t)(key0 + (e >> 2) * 8 + (e & 1)) * dv + col0 + v * 16 + (e & 2) * 4] = S[v][e >> 2][e & 3];
    }
  }
#pragma unroll
  for (int v = 0; v < NV; ++v)
#pragma unroll
    for (int e = 0; e < 8; ++e) state[(size_t)(key0 + (e >> 2) * 8 + (e & 1)) * dv + col0 + v * 16 + (e & 2) * 4] = S[v][e >> 2][e & 3];
}

// ------------------------------------------------------------------------------------------------ outputs
// o += Q S, a block takes a chunk and up to 128 value columns of a head; a warp 16 tokens and every (8 / MT)-th column tile
template <int DK>
__global__ void __launch_bounds__(256) delta_chunk_out_kernel(const __grid_constant__ DeltaParams p, int dv) {
  using M = DeltaGeom<DK>;
  constexpr int MT = M::MT, KT = M::KT, STEP = 8 / MT;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
  const int ci = blockIdx.x, h = blockIdx.y, tok0 = p.ck_tok0[ci], n = p.ck_ntok[ci], I = warp % MT;
  const size_t ch = (size_t)ci * p.H + h;
  pdl_trigger();
  pdl_wait();
  if (16 * I >= n) return;
  const int vt0 = blockIdx.z * 8, nv = min(8, dv / 16 - vt0);
  const uint4* qp = p.q_ws + (ch * MT + I) * KT * 64 + lane;
  const uint4* sp = reinterpret_cast<const uint4*>(p.s_ws) + (ch * (dv / 16) + vt0) * KT * 64 + lane;
  float acc[MT][2][4] = {};
#pragma unroll 2
  for (int k = 0; k < KT; ++k) {
    const uint4 qh = qp[k * 64], ql = qp[k * 64 + 32];
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const int vt = warp / MT + STEP * i;
      if (vt >= nv) continue;
      const uint4 sh = sp[(vt * KT + k) * 64], sl = sp[(vt * KT + k) * 64 + 32];
      mma_bf16_16816(acc[i][0], qh.x, qh.y, qh.z, qh.w, sh.x, sh.z);
      mma_bf16_16816(acc[i][1], qh.x, qh.y, qh.z, qh.w, sh.y, sh.w);
      mma_bf16_16816(acc[i][0], ql.x, ql.y, ql.z, ql.w, sh.x, sh.z);
      mma_bf16_16816(acc[i][1], ql.x, ql.y, ql.z, ql.w, sh.y, sh.w);
      mma_bf16_16816(acc[i][0], qh.x, qh.y, qh.z, qh.w, sl.x, sl.z);
      mma_bf16_16816(acc[i][1], qh.x, qh.y, qh.z, qh.w, sl.y, sl.w);
    }
  }
#pragma unroll
  for (int i = 0; i < MT; ++i) {
    const int vt = warp / MT + STEP * i;
    if (vt >= nv) continue;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (16 * I + g + 8 * r >= n) continue;
      float* o = p.o + (size_t)(tok0 + 16 * I + g + 8 * r) * p.H * dv + h * dv + (vt0 + vt) * 16 + 2 * t;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float2 w = *reinterpret_cast<const float2*>(o + e * 8);
        *reinterpret_cast<float2*>(o + e * 8) = make_float2(w.x + acc[i][e][2 * r], w.y + acc[i][e][2 * r + 1]);
      }
    }
  }
}

// TI_DELTA_SCAN: the number of blocks up to which the narrow form of the scan runs
static int scan_blocks() {
  static const int n = [] { const char* e = getenv("TI_DELTA_SCAN"); return e == nullptr ? 148 : atoi(e); }();
  return n;
}

template <int DK, bool GENERAL>
static int launch_delta_chunked(const DeltaParams& p, int dv, cudaStream_t st) {
  using M = DeltaGeom<DK>;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(delta_chunk_prepare_kernel<DK, GENERAL>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kSmem);
    cudaFuncSetAttribute(delta_chunk_scan_kernel<DK, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kScan / 2);
    cudaFuncSetAttribute(delta_chunk_scan_kernel<DK, 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)M::kScan);
    configured = true;
  }
  launch_kernel(delta_chunk_prepare_kernel<DK, GENERAL>, dim3(p.nc, p.H), dim3(kPrepThreads), M::kSmem, st, true, p, dv);
  // narrow blocks while they fit the SMs at once; wide ones read a chunk's matrix half as often
  if ((long long)dv / 16 * p.H * p.num_long <= scan_blocks())
    launch_kernel(delta_chunk_scan_kernel<DK, 1>, dim3(dv / 16, p.H, p.num_long), dim3(DK * 2), M::kScan / 2, st, true, p, dv);
  else
    launch_kernel(delta_chunk_scan_kernel<DK, 2>, dim3(dv / 32, p.H, p.num_long), dim3(DK * 2), M::kScan, st, true, p, dv);
  launch_kernel(delta_chunk_out_kernel<DK>, dim3(p.nc, p.H, (dv + 127) / 128), dim3(256), 0, st, true, p, dv);
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_delta_chunk_size(int dk) { return dk == 64 || dk == 128 ? 64 : dk == 256 ? 32 : 0; }

// o[t, h] and the states of the sequences with chunks (inputs in bf16)
int ti_delta_chunked(const ti::DeltaParams* p, int dk, int dv, int general, void* stream) {
  if (p->nc <= 0) return 0;
  if (dv % 64 || p->rep < 1 || p->H % p->rep || p->lds % 8 || p->ld % 8 || p->q_col % 8 || p->k_col % 8 || p->v_col % 8 ||
      (((uintptr_t)p->src | (uintptr_t)p->proj | (uintptr_t)p->o | (uintptr_t)p->state | (uintptr_t)p->t_ws | (uintptr_t)p->q_ws | (uintptr_t)p->s_ws |
        (uintptr_t)p->f_ws) & 15))
    return -2;
  if (general && (p->R < 1 || p->rep != 1 || p->b_col % 8 || ((uintptr_t)p->bias & 15))) return -2;
  // the factors exp(+-G) of a chunk must stay inside the range of a float, with room for the values they multiply
  if (general && !(p->decay_scale >= 0.f && p->decay_scale * ti::kLog2e * (float)ti_delta_chunk_size(dk) < 90.f)) return -4;
  cudaStream_t st = (cudaStream_t)stream;
  if (dk == 64) return general ? ti::launch_delta_chunked<64, true>(*p, dv, st) : ti::launch_delta_chunked<64, false>(*p, dv, st);
  if (dk == 128) return general ? ti::launch_delta_chunked<128, true>(*p, dv, st) : ti::launch_delta_chunked<128, false>(*p, dv, st);
  if (dk == 256) return general ? ti::launch_delta_chunked<256, true>(*p, dv, st) : ti::launch_delta_chunked<256, false>(*p, dv, st);
  return -3;
}

}  // extern "C"
