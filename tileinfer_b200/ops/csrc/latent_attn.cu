// Latent attention over a paged cache of latents, for decode tokens and short portions of prompts.
//
// With W_uk absorbed into the query (q~ = W_uk^T q, one row of R per head) every head attends to the SAME row c of the
// cache, once as key and once as value:  s = scale * q~.c,  o~ = sum p c  (W_uv follows on o~, see latent_ops.cu).  A row
// may carry columns behind the latent that only take part as key (a rotated part that all heads share).  One
// cache row of R values per token serves all heads, so a block takes 16 or 32 heads as the rows of its MMAs and reads
// each latent once from memory.
//
// A layer's mask is a parameter (window = 0: all earlier tokens; otherwise itself and the window - 1 tokens before it),
// and so is the sink: one number per head that joins the denominator without key, value or scale (null: none).
//
// latent_decode.cu (bf16, padded R of 256, 384, 512, 576): the tcgen05 form for the sizes of large models.
// latent_decode_kernel (bf16, other R up to 448): per (query token, head group, split) tiles of 64 keys, two tiles in flight by
// cp.async; S = q~ c^T by mma.sync with the eight warps over (head tile, keys), softmax state in registers of the row's
// threads, O += P c with the eight warps over column slices, the value fragments read from the SAME shared-memory tile
// through ldmatrix.trans.  Splits meet in latent_merge_kernel, which also adds the sink.
// latent_any_kernel (float for 32-bit mode, or bf16 with R above 512): one block per (query token, head).
#include "latent_attn.cuh"

namespace ti {

constexpr int kKeyTile = 64;

TI_DEVICE void cpa16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src) : "memory");
}
TI_DEVICE void cpa_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> TI_DEVICE void cpa_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }
TI_DEVICE void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
TI_DEVICE void ldsm2t(uint32_t (&r)[2], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];\n" : "=r"(r[0]), "=r"(r[1]) : "r"(addr) : "memory");
}

template <int RT, int MT> struct LatentGeom {
  static constexpr int kRp = 64 * RT;
  static constexpr int kRows = 16 * MT;
  static constexpr int kPitch = (kRp + 8) * 2;                    // bytes; 16 mod 128: conflict-free ldmatrix
  static constexpr int kKeyBytes = kKeyTile * kPitch;
  static constexpr int kSPitch = kKeyTile + 4;                    // floats
  static constexpr int kPPitch = (kKeyTile + 8) * 2;              // bytes
  static constexpr int kQOff = 2 * kKeyBytes;
  static constexpr int kSOff = kQOff + kRows * kPitch;
  static constexpr int kPOff = kSOff + kRows * kSPitch * 4;
  static constexpr int kAOff = kPOff + kRows * kPPitch;           // alpha[rows], m[rows], l[rows]
  static constexpr size_t kSmem = kAOff + 3 * kRows * 4;
};

template <int RT, int MT>
__global__ void __launch_bounds__(256) latent_decode_kernel(const __grid_constant__ LatentAttnParams p) {
  using G = LatentGeom<RT, MT>;
  constexpr int Rp = G::kRp, ROWS = G::kRows;
  constexpr int CPR = Rp / 8;                                     // 16-byte chunks of a row
  extern __shared__ __align__(128) uint8_t sm[];
  const uint32_t base = smem_u32(sm);
  float* s_s = reinterpret_cast<float*>(sm + G::kSOff);
  float* alpha_s = reinterpret_cast<float*>(sm + G::kAOff);
  float *m_s = alpha_s + ROWS, *l_s = m_s + ROWS;

  const int qg = blockIdx.x, hg = blockIdx.y, sp = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
  pdl_trigger();
  pdl_wait();
  if (p.qg_ntok[qg] == 0) return;
  const int tok = p.qg_tok0[qg], seq = p.qg_seq[qg];
  const KeyRange kr = key_range(p, tok, kKeyTile);
  const int t0 = sp * kr.tps, t1 = min(kr.ntiles, t0 + kr.tps);
  if (t0 >= t1) return;                                           // inactive split: the merge never reads it
  const int* bt = p.block_tables + (size_t)seq * p.max_blocks;
  const bf16* cache = static_cast<const bf16*>(p.cache);

  auto load_tile = [&](int j, int buf) {
    const uint32_t dst = base + buf * G::kKeyBytes;
    for (int c = tid; c < kKeyTile * CPR; c += 256) {
      const int row = c / CPR, col = c - row * CPR;
      const int page = min(kr.page0 + j * (kKeyTile / 16) + (row >> 4), kr.npages - 1);   // past the end: masked
      const int blk = bt[page];
      if (!TI_CHECK(blk, p.num_blocks, p.status)) continue;
      cpa16(dst + row * G::kPitch + col * 16, cache + ((size_t)blk * 16 + (row & 15)) * Rp + col * 8);
    }
  };
  load_tile(t0, 0);
  cpa_commit();
  {
    const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)tok * p.H + hg * ROWS) * Rp;
    const int nrow = min(ROWS, p.H - hg * ROWS);
    for (int c = tid; c < ROWS * CPR; c += 256) {
      const int row = c / CPR, col = c - row * CPR;
      *reinterpret_cast<uint4*>(sm + G::kQOff + row * G::kPitch + col * 16) =
          row < nrow ? *reinterpret_cast<const uint4*>(q + (size_t)row * Rp + col * 8) : make_uint4(0, 0, 0, 0);
    }
  }
  float o[MT][RT][4];
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int n = 0; n < RT; ++n) o[a][n][0] = o[a][n][1] = o[a][n][2] = o[a][n][3] = 0.f;
  constexpr int TPR = 256 / ROWS, KPT = kKeyTile / TPR;           // threads per row, keys per thread in the softmax
  const int srow = tid / TPR, ssub = tid % TPR;
  float m = kNeg, l = 0.f;
  const float sc = p.scale * kLog2e;

  for (int j = t0; j < t1; ++j) {
    const int buf = (j - t0) & 1;
    if (j + 1 < t1) {
      if (j > t0) __syncthreads();                                // everyone is done with the other buffer
      load_tile(j + 1, buf ^ 1);
      cpa_commit();
      cpa_wait<1>();
    } else {
      cpa_wait<0>();
    }
    __syncthreads();
    const uint32_t kb = base + buf * G::kKeyBytes;
    // ---- S = q~ c^T
    if (MT == 2) {
      const int mt = warp & 1, n0 = (warp >> 1) * 16;
      float d0[4] = {0.f, 0.f, 0.f, 0.f}, d1[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t qa = base + G::kQOff + (mt * 16 + (lane & 15)) * G::kPitch + (lane >> 4) * 16;
      const uint32_t ka = kb + (n0 + ((lane >> 4) & 1) * 8 + (lane & 7)) * G::kPitch + ((lane >> 3) & 1) * 16;
#pragma unroll 4
      for (int k = 0; k < Rp / 16; ++k) {
        uint32_t a[4], b[4];
        ldsm4(a, qa + k * 32);
        ldsm4(b, ka + k * 32);
        mma_bf16_16816(d0, a[0], a[1], a[2], a[3], b[0], b[1]);
        mma_bf16_16816(d1, a[0], a[1], a[2], a[3], b[2], b[3]);
      }
      float* dst = s_s + (mt * 16 + g) * G::kSPitch + n0 + 2 * t;
      *reinterpret_cast<float2*>(dst) = make_float2(d0[0], d0[1]);
      *reinterpret_cast<float2*>(dst + 8) = make_float2(d1[0], d1[1]);
      dst += 8 * G::kSPitch;
      *reinterpret_cast<float2*>(dst) = make_float2(d0[2], d0[3]);
      *reinterpret_cast<float2*>(dst + 8) = make_float2(d1[2], d1[3]);
    } else {
      const int n0 = warp * 8;
      float d0[4] = {0.f, 0.f, 0.f, 0.f}, d1[4] = {0.f, 0.f, 0.f, 0.f};
      const uint32_t qa = base + G::kQOff + (lane & 15) * G::kPitch + (lane >> 4) * 16;
      const uint32_t ka = kb + (n0 + (lane & 7)) * G::kPitch + (lane >> 3) * 16;
#pragma unroll 4
      for (int k = 0; k < Rp / 32; ++k) {
        uint32_t a[4], a2[4], b[4];
        ldsm4(a, qa + k * 64);
        ldsm4(a2, qa + k * 64 + 32);
        ldsm4(b, ka + k * 64);
        mma_bf16_16816(d0, a[0], a[1], a[2], a[3], b[0], b[1]);
        mma_bf16_16816(d1, a2[0], a2[1], a2[2], a2[3], b[2], b[3]);
      }
      float* dst = s_s + g * G::kSPitch + n0 + 2 * t;
      *reinterpret_cast<float2*>(dst) = make_float2(d0[0] + d1[0], d0[1] + d1[1]);
      dst += 8 * G::kSPitch;
      *reinterpret_cast<float2*>(dst) = make_float2(d0[2] + d1[2], d0[3] + d1[3]);
    }
    __syncthreads();
    // ---- softmax over the tile: TPR threads per row
    {
      const int key0 = kr.page0 * 16 + j * kKeyTile + ssub * KPT;
      float s[KPT], mx = kNeg;
      const float* src = s_s + srow * G::kSPitch + ssub * KPT;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        const int key = key0 + i;
        s[i] = (key >= kr.lo && key <= kr.pos) ? src[i] * sc : kNeg;
        mx = fmaxf(mx, s[i]);
      }
#pragma unroll
      for (int w = 1; w < TPR; w <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float mn = fmaxf(m, mx), al = exp2f(m - mn);
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < KPT; ++i) {
        s[i] = s[i] > 0.5f * kNeg ? exp2f(s[i] - mn) : 0.f;
        sum += s[i];
      }
#pragma unroll
      for (int w = 1; w < TPR; w <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, w);
      l = l * al + sum;
      m = mn;
      uint32_t* dst = reinterpret_cast<uint32_t*>(sm + G::kPOff + srow * G::kPPitch + ssub * KPT * 2);
#pragma unroll
      for (int i = 0; i < KPT / 2; ++i) dst[i] = pack_bf16(s[2 * i], s[2 * i + 1]);
      if (ssub == 0) alpha_s[srow] = al;
    }
    __syncthreads();
    // ---- O += P c: this warp's RT * 8 columns
#pragma unroll
    for (int a = 0; a < MT; ++a) {
      const float al0 = alpha_s[a * 16 + g], al1 = alpha_s[a * 16 + g + 8];
#pragma unroll
      for (int n = 0; n < RT; ++n) { o[a][n][0] *= al0; o[a][n][1] *= al0; o[a][n][2] *= al1; o[a][n][3] *= al1; }
    }
#pragma unroll
    for (int kk = 0; kk < kKeyTile / 16; ++kk) {
      uint32_t a[MT][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldsm4(a[i], base + G::kPOff + (i * 16 + (lane & 15)) * G::kPPitch + kk * 32 + (lane >> 4) * 16);
      const uint32_t va = kb + (kk * 16 + (lane & 15)) * G::kPitch + warp * (RT * 16);
#pragma unroll
      for (int n = 0; n < RT; ++n) {
        uint32_t b[2];
        ldsm2t(b, va + n * 16);
#pragma unroll
        for (int i = 0; i < MT; ++i) mma_bf16_16816(o[i][n], a[i][0], a[i][1], a[i][2], a[i][3], b[0], b[1]);
      }
    }
  }
  if (ssub == 0) { m_s[srow] = m; l_s[srow] = l; }
  __syncthreads();
  const int col0 = warp * (RT * 8) + 2 * t;
  if (p.nsplit == 1) {
#pragma unroll
    for (int a = 0; a < MT; ++a)
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int r = a * 16 + g + 8 * h, head = hg * ROWS + r;
        if (head >= p.H) continue;
        const float sk = p.sink == nullptr ? kNeg : p.sink[head] * kLog2e;
        const float M = fmaxf(m_s[r], sk), w = exp2f(m_s[r] - M);
        const float inv = w / (l_s[r] * w + (p.sink == nullptr ? 0.f : exp2f(sk - M)));
        bf16* dst = static_cast<bf16*>(p.out) + ((size_t)tok * p.H + head) * p.Ro + col0;
#pragma unroll
        for (int n = 0; n < RT; ++n)
          if (col0 + n * 8 < p.Ro) *reinterpret_cast<uint32_t*>(dst + n * 8) = pack_bf16(o[a][n][2 * h] * inv, o[a][n][2 * h + 1] * inv);
      }
    return;
  }
  const size_t item = ((size_t)qg * gridDim.y + hg) * p.nsplit + sp;
#pragma unroll
  for (int a = 0; a < MT; ++a)
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const int r = a * 16 + g + 8 * h;
      if (hg * ROWS + r >= p.H) continue;
      float* dst = p.o_part + (item * ROWS + r) * Rp + col0;
#pragma unroll
      for (int n = 0; n < RT; ++n) *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[a][n][2 * h], o[a][n][2 * h + 1]);
    }
  if (tid < ROWS) {
    p.ml_part[(item * ROWS + tid) * 2] = m_s[tid];
    p.ml_part[(item * ROWS + tid) * 2 + 1] = l_s[tid];
  }
}

// Combines the splits of one (query token, head) and adds the sink to the denominator.
__global__ void __launch_bounds__(128) latent_merge_kernel(const __grid_constant__ LatentAttnParams p, int rows, int tile) {
  __shared__ float w_s[kMaxLatentSplit];
  const int qg = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
  pdl_trigger();
  pdl_wait();
  if (p.qg_ntok[qg] == 0) return;
  const int tok = p.qg_tok0[qg];
  const KeyRange kr = key_range(p, tok, tile);
  const int nact = (kr.ntiles + kr.tps - 1) / kr.tps;
  const int groups = (p.H + rows - 1) / rows, hg = head / rows, r = head - hg * rows;
  const size_t item0 = ((size_t)qg * groups + hg) * p.nsplit;
  const float sk = p.sink == nullptr ? kNeg : p.sink[head] * kLog2e;
  float M = sk;
  for (int s = 0; s < nact; ++s) M = fmaxf(M, p.ml_part[((item0 + s) * rows + r) * 2]);
  float L = p.sink == nullptr ? 0.f : exp2f(sk - M);
  for (int s = 0; s < nact; ++s) {
    const float2 ml = *reinterpret_cast<const float2*>(p.ml_part + ((item0 + s) * rows + r) * 2);
    const float w = exp2f(ml.x - M);
    L += w * ml.y;
    if (tid == 0) w_s[s] = w;
  }
  __syncthreads();
  const float inv = 1.f / L;
  bf16* dst = static_cast<bf16*>(p.out) + ((size_t)tok * p.H + head) * p.Ro;
  for (int c = tid * 2; c < p.Ro; c += 256) {
    float a0 = 0.f, a1 = 0.f;
#pragma unroll 4
    for (int s = 0; s < nact; ++s) {
      const float2 v = *reinterpret_cast<const float2*>(p.o_part + ((item0 + s) * rows + r) * p.Rp + c);
      a0 += w_s[s] * v.x;
      a1 += w_s[s] * v.y;
    }
    *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(a0 * inv, a1 * inv);
  }
}

// ---------------------------------------------------------------- any type, any R up to 2048
template <typename T> TI_DEVICE float as_float(T v);
template <> TI_DEVICE float as_float<float>(float v) { return v; }
template <> TI_DEVICE float as_float<bf16>(bf16 v) { return __bfloat162float(v); }
TI_DEVICE void put(float* p, float v) { *p = v; }
TI_DEVICE void put(bf16* p, float v) { *p = __float2bfloat16_rn(v); }

constexpr int kAnyCols = 16;       // columns of O per thread: R <= 128 * 16

template <typename T>
__global__ void __launch_bounds__(128) latent_any_kernel(const __grid_constant__ LatentAttnParams p) {
  extern __shared__ __align__(16) float fsm[];                    // q~ [Rp], scores / weights [64]
  float *q_s = fsm, *s_s = fsm + p.Rp;
  const int qg = blockIdx.x, head = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_trigger();
  pdl_wait();
  if (p.qg_ntok[qg] == 0) return;
  const int tok = p.qg_tok0[qg], seq = p.qg_seq[qg];
  const int pos = p.positions[tok], lo = p.window > 0 ? max(0, pos - p.window + 1) : 0;
  const int* bt = p.block_tables + (size_t)seq * p.max_blocks;
  const T* cache = static_cast<const T*>(p.cache);
  const T* q = static_cast<const T*>(p.q) + ((size_t)tok * p.H + head) * p.Rp;
  for (int c = tid; c < p.Rp; c += 128) q_s[c] = as_float<T>(q[c]) * p.scale;
  float o[kAnyCols];
#pragma unroll
  for (int i = 0; i < kAnyCols; ++i) o[i] = 0.f;
  float m = p.sink == nullptr ? kNeg : p.sink[head], l = p.sink == nullptr ? 0.f : 1.f;   // the sink is the first term
  __syncthreads();
  for (int k0 = lo; k0 <= pos; k0 += 64) {
    for (int i = warp * 16; i < warp * 16 + 16; ++i) {
      const int key = k0 + i;
      float s = kNeg;
      if (key <= pos) {
        const int blk = bt[key >> 4];
        if (TI_CHECK(blk, p.num_blocks, p.status)) {
          const T* c = cache + ((size_t)blk * 16 + (key & 15)) * p.Rp;
          float d = 0.f;
          for (int e = lane; e < p.Rp; e += 32) d = fmaf(q_s[e], as_float<T>(c[e]), d);
          s = warp_sum(d);
        }
      }
      if (lane == 0) s_s[i] = s;
    }
    __syncthreads();
    float mx = m;
    for (int i = 0; i < 64; ++i) mx = fmaxf(mx, s_s[i]);
    const float al = expf(m - mx);
    m = mx;
    __syncthreads();
    if (tid < 64) s_s[tid] = s_s[tid] > 0.5f * kNeg ? expf(s_s[tid] - m) : 0.f;
    __syncthreads();
    l *= al;
#pragma unroll
    for (int i = 0; i < kAnyCols; ++i) o[i] *= al;
    for (int i = 0; i < 64 && k0 + i <= pos; ++i) {
      const float w = s_s[i];
      l += w;
      const int key = k0 + i, blk = bt[key >> 4];
      if (!TI_CHECK(blk, p.num_blocks, p.status)) continue;
      const T* c = cache + ((size_t)blk * 16 + (key & 15)) * p.Rp;
#pragma unroll
      for (int e = 0; e < kAnyCols; ++e)
        if (tid + 128 * e < p.Ro) o[e] = fmaf(w, as_float<T>(c[tid + 128 * e]), o[e]);
    }
    __syncthreads();
  }
  T* dst = static_cast<T*>(p.out) + ((size_t)tok * p.H + head) * p.Ro;
#pragma unroll
  for (int e = 0; e < kAnyCols; ++e)
    if (tid + 128 * e < p.Ro) put(dst + tid + 128 * e, o[e] / l);
}

void launch_latent_merge(const LatentAttnParams& p, int rows, int tile, cudaStream_t st) {
  launch_kernel(latent_merge_kernel, dim3(p.num_qg, p.H), dim3(128), 0, st, true, p, rows, tile);
}

template <int RT, int MT>
static int launch_latent_decode(const LatentAttnParams& p, cudaStream_t st) {
  using G = LatentGeom<RT, MT>;
  auto k = latent_decode_kernel<RT, MT>;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)G::kSmem);
    configured = true;
  }
  const int groups = (p.H + G::kRows - 1) / G::kRows;
  launch_kernel(k, dim3(p.num_qg, groups, p.nsplit), dim3(256), G::kSmem, st, true, p);
  if (p.nsplit > 1) launch_latent_merge(p, G::kRows, kKeyTile, st);
  return (int)cudaGetLastError();
}

}  // namespace ti

extern "C" {

int ti_latent_attn_params_size() { return (int)sizeof(ti::LatentAttnParams); }

// Whether a split kernel takes rows of Rp columns of which Ro are values; others (and fp32) run on the general kernel, unsplit.
int ti_latent_attn_splits(int Rp, int Ro) { return Rp <= 512 || (Rp == 576 && Ro <= 512); }

int ti_latent_attn(const ti::LatentAttnParams* pp, int f32, void* stream) {
  const ti::LatentAttnParams& p = *pp;
  if (p.num_qg <= 0) return 0;
  if (p.Rp % 64 || p.Rp > 128 * ti::kAnyCols || p.H < 1 || p.nsplit < 1 || p.nsplit > ti::kMaxLatentSplit || p.window < 0 ||
      p.Ro < 64 || p.Ro > p.Rp || p.Ro % 64)
    return -2;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32 || !ti_latent_attn_splits(p.Rp, p.Ro)) {
    const size_t smem = (p.Rp + 64) * sizeof(float);
    ti::launch_kernel(f32 ? ti::latent_any_kernel<float> : ti::latent_any_kernel<ti::bf16>, dim3(p.num_qg, p.H), dim3(128), smem,
                      st, true, p);
    return (int)cudaGetLastError();
  }
  const bool two = p.H > 16;
  switch (p.Rp / 64) {
    case 1: return two ? ti::launch_latent_decode<1, 2>(p, st) : ti::launch_latent_decode<1, 1>(p, st);
    case 2: return two ? ti::launch_latent_decode<2, 2>(p, st) : ti::launch_latent_decode<2, 1>(p, st);
    case 3: return two ? ti::launch_latent_decode<3, 2>(p, st) : ti::launch_latent_decode<3, 1>(p, st);
    case 5: return two ? ti::launch_latent_decode<5, 2>(p, st) : ti::launch_latent_decode<5, 1>(p, st);
    case 7: return two ? ti::launch_latent_decode<7, 2>(p, st) : ti::launch_latent_decode<7, 1>(p, st);
    default: return ti::launch_latent_decode_tc(p, st);
  }
}

}  // extern "C"
