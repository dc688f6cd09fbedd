// Variable-length causal GQA attention for prefill chunks on the 5th-generation tensor cores.
//
// Replaces the reference's warp-specialised prefill kernel (kernels/gqa_varlen.py:187-362, mma.sync tiles fed by
// plain loads, shapes fixed at JIT time) together with the gather of the whole cached prefix into a dense K/V
// copy before every later chunk (model/qwen_36.py:1031-1042).  Here a CTA owns 128 query tokens of one head and
// walks the sequence's KV pages in tiles of 128 keys straight out of the paged cache:
//
//   warp 0  TMA producer: Q tile once (4 swizzled 64-column slabs), then per KV tile 8 K pages, each ONE 4-D copy
//           ([16 tokens][D] in the cache -> [2 groups of 8 keys][D/64 slabs][8][64], 128-byte swizzle);
//   warp 6  TMA producer of the 8 V pages per tile ([D][16 tokens] as stored: each page is exactly the B operand
//           of one k = 16 step of P V, 32-byte swizzle); pages are addressed through the block table;
//   warp 1  MMA issuer: S = Q K^T (tcgen05.mma kind::f16, M = N = 128, accumulator in TMEM, two S buffers so the
//           next tile's S is computed while the softmax works on this one), then O += P V (N = D);
//   warps 2-5  softmax: one thread per query row (= TMEM lane) with the 128 scores of a tile in registers: scale, mask,
//           running maximum in the exp2 domain with lazy rescaling (O in TMEM is only touched when the maximum grew by more than 2^8),
//           P written to shared memory as the bf16 A operand of the second product; at the end O / l times the
//           sigmoid output gate goes to [T, hq*D].
//
// TMEM: S0 | S1 | O = 128 + 128 + D columns (512 allocated).  Shared memory at D = 256: Q 64 KB, K 64 KB,
// V 64 KB, P 32 KB; where heads are smaller K and V have two buffers each.  Causal alignment is by absolute position (bottom-right): a chunk that continues a cached
// prefix sees all of it.  Values may be of another size than queries and keys; the gate may be absent, per dimension or per
// head.  A window limits the keys (the walk starts at the page of the first one any row sees), and scores may lose a slope
// per head times the distance of the key.  Scores may be
// capped by cap * tanh(score / cap); where |score / cap| is known to stay small (normalised queries and keys) the tanh is
// its power series and the softmax needs no running maximum at all: exp2 of a bounded score neither overflows nor
// vanishes, so the scores of a tile are read once, two threads can share a query row (eight softmax warps, half of the keys
// of a tile each), and with shared memory for two P tiles the next one is written while P V of this one runs.  Every wait is bounded; on expiry the status word is set, all roles leave their loops
// and TMEM is freed.  No load carries a cluster-multicast qualifier.
#include "tensor_map.cuh"

namespace ti {

struct AttnPrefillParams {
  alignas(64) CUtensorMap map_q;   // bf16 [T][hq*D], box {64, 128}, 128B swizzle
  alignas(64) CUtensorMap map_k;   // bf16 [blocks*hkv*2 groups][D/64 slabs][8 keys][64], box {64, 8, D/64, 2}, 128B swizzle
  alignas(64) CUtensorMap map_v;   // bf16 [blocks*hkv*D][16], box {16, D}, 32B swizzle
  const int* block_tables;         // [S, max_blocks]
  const int* positions;            // [T]
  const int* qt_seq;               // [num_tiles] sequence of the query tile
  const int* qt_tok0;              // [num_tiles] first flat token
  const int* qt_ntok;              // [num_tiles] tokens in the tile (1..128; 0 = padding tile)
  const __nv_bfloat16* gate_src;   // null, or [T, ld]: gates of head h at column gate_col + h * gate_stride
  __nv_bfloat16* out;              // [T, hq*D]
  unsigned* status;
  int hq, hkv, max_blocks, ld;
  float scale_log2e;
  float cap_in, cap_out;           // score = cap_out * tanh(q.k * cap_in), in log2 units
  int window;                      // keys seen, the token itself included (0: all earlier ones)
  const float* slopes;             // BIASED: [hq], taken off a score per token of distance
  const __nv_bfloat16* head_gate;  // null, or [T, ldg]: gate of head h at column gcol + h
  int ldg, gcol, ldo;              // ldo: row pitch of `out`
  float out_scale;
  int gate_col, gate_stride;
};

// How a score follows from q.k: scaled; capped with the series, reference 0 instead of a running maximum; capped; scaled,
// minus a slope times the distance
enum { SCORE_PLAIN = 0, SCORE_SERIES = 1, SCORE_CAPPED = 2, SCORE_BIASED = 3 };
constexpr float kSeriesMax = 0.4f;       // largest |argument| the series serves (error below 1e-7 there)

// Packed pairs of floats
typedef unsigned long long f2;
TI_DEVICE f2 pack2(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};\n" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
TI_DEVICE void unpack2(f2 v, float& a, float& b) { asm("mov.b64 {%0, %1}, %2;\n" : "=f"(a), "=f"(b) : "l"(v)); }
TI_DEVICE f2 fma2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;\n" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
TI_DEVICE f2 mul2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;\n" : "=l"(r) : "l"(a), "l"(b));
  return r;
}
TI_DEVICE float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
// c tanh(k x) = c k x (1 + z (-1/3 + z (2/15 + z (-17/315 + z (62/2835 - z 1382/155925))))) with z = (k x)^2; the powers of
// k are folded into the coefficients.  tanh y = y - y^3/3 + 2 y^5/15 - 17 y^7/315 + ... (Bernoulli numbers).
struct TanhSeries {
  f2 ck, c1, c2, c3, c4, c5;
  TI_DEVICE TanhSeries(float c, float k) {
    const float z = k * k;
    auto two = [](float v) { return pack2(v, v); };
    ck = two(c * k);
    c1 = two(-z / 3.f);
    c2 = two(z * z * (2.f / 15.f));
    c3 = two(z * z * z * (-17.f / 315.f));
    c4 = two(z * z * z * z * (62.f / 2835.f));
    c5 = two(z * z * z * z * z * (-1382.f / 155925.f));
  }
  TI_DEVICE f2 operator()(f2 x) const {
    const f2 a = mul2(x, x);
    f2 u = fma2(c5, a, c4);
    u = fma2(u, a, c3);
    u = fma2(u, a, c2);
    u = fma2(u, a, c1);
    const f2 y = mul2(x, ck);
    return fma2(mul2(u, a), y, y);
  }
};
// `ahead`: slope times (key - query) in log2 units
template <int MODE> TI_DEVICE float prefill_score(const AttnPrefillParams& p, float qk, float ahead) {
  if (MODE == SCORE_BIASED) return fmaf(qk, p.scale_log2e, ahead);
  if (MODE == SCORE_CAPPED) return p.cap_out * (1.f - __fdividef(2.f, 1.f + ex2_approx(qk * p.cap_in * 2.8853900817779268f)));
  return qk * p.scale_log2e;
}

constexpr unsigned long long kAttnWaitNs = 500000000ull;
constexpr int kAttnThreads = 224;        // warp 0: Q/K producer, 1: MMA issuer, 2..5: softmax, 6: V producer
constexpr int kAttnProducerV = 6;
constexpr float kMaskVal = -1e30f;
constexpr float kFirstMax = -1e29f;      // a row may see no key of its first tile: its scores are -inf, its weights 0
constexpr float kRescaleGap = 8.f;       // log2 units the running maximum may lag behind before O is rescaled

template <int D, int DV, int MODE> struct AttnPrefillGeom {
  static constexpr int kSlabs = D / 64;
  static constexpr int kQBytes = kSlabs * 128 * 128;
  static constexpr int kKBytes = kSlabs * 128 * 128;
  static constexpr int kVPage = DV * 32;
  static constexpr int kVBytes = 8 * kVPage;
  static constexpr int kP = 2 * 128 * 128;                          // one P tile
  static constexpr int kBarBytes = 128;
  static constexpr int kPTiles = MODE == SCORE_SERIES && kQBytes + kKBytes + kVBytes + 2 * kP + kBarBytes + 1024 + 1024 <= 227 * 1024 ? 2 : 1;
  static constexpr int kPBytes = kPTiles * kP;
  static constexpr int kStages = kQBytes + 2 * (kKBytes + kVBytes) + kPBytes + kBarBytes + 1024 + 1024 <= 227 * 1024 ? 2 : 1;   // of K and of V
  static constexpr int kHalves = MODE == SCORE_SERIES ? 2 : 1;      // threads that share a query row
  static constexpr int kThreads = MODE == SCORE_SERIES ? 384 : kAttnThreads;
  static constexpr size_t kNeeded = (size_t)kQBytes + kStages * (kKBytes + kVBytes) + kPBytes + kBarBytes + 1024;
  // one CTA per SM (the kernel takes all 512 TMEM columns)
  static constexpr size_t kSmem = kNeeded > 120 * 1024 ? kNeeded : 120 * 1024;
};

// What scales a head's output beside 1 / l
TI_DEVICE float head_factor(const AttnPrefillParams& p, size_t tok, int head) {
  return p.head_gate == nullptr ? p.out_scale : p.out_scale * sigmoid_f(__bfloat162float(p.head_gate[tok * p.ldg + p.gcol + head]));
}

// Gates of 32 output columns of a row, and the request for a whole row of them ahead of its use: the rows of a tile lie far
// apart, and reading them only at the end would cost a memory round trip per 32 columns.
TI_DEVICE void load_gates(const AttnPrefillParams& p, const __nv_bfloat16* gate, int c, uint4 (&g)[4]) {
  if (p.gate_src == nullptr) return;
#pragma unroll
  for (int q = 0; q < 4; ++q) g[q] = *reinterpret_cast<const uint4*>(gate + c * 32 + q * 8);
}
TI_DEVICE void prefetch_gates(const AttnPrefillParams& p, const __nv_bfloat16* gate, int columns) {
  if (p.gate_src == nullptr) return;
  for (int c = 0; c < columns; c += 64) asm volatile("prefetch.global.L2 [%0];\n" ::"l"(gate + c));
}

// 32 output columns of a row: times 1 / l and the sigmoid gate, as bf16
TI_DEVICE void store_rows32(const AttnPrefillParams& p, const uint32_t (&v)[32], float inv, const uint4 (&gates)[4], __nv_bfloat16* dst, int c) {
#pragma unroll
  for (int q4 = 0; q4 < 4; ++q4) {
    float f[8];
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = __uint_as_float(v[q4 * 8 + e]) * inv;
    if (p.gate_src != nullptr) {
      const uint32_t g4[4] = {gates[q4].x, gates[q4].y, gates[q4].z, gates[q4].w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        f[2 * e] *= sigmoid_f(bf16lo(g4[e]));
        f[2 * e + 1] *= sigmoid_f(bf16hi(g4[e]));
      }
    }
    uint32_t o4[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) o4[e] = pack_bf16(f[2 * e], f[2 * e + 1]);
    *reinterpret_cast<uint4*>(dst + c * 32 + q4 * 8) = make_uint4(o4[0], o4[1], o4[2], o4[3]);
  }
}

template <int D, int DV, int MODE>
__global__ void __launch_bounds__((AttnPrefillGeom<D, DV, MODE>::kThreads), 1) attn_prefill_kernel(const __grid_constant__ AttnPrefillParams p) {
  using G = AttnPrefillGeom<D, DV, MODE>;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t q_s = smem_u32(smem), k_s = q_s + G::kQBytes, v_s = k_s + G::kStages * G::kKBytes, p_s = v_s + G::kStages * G::kVBytes;
  const uint32_t bars = p_s + G::kPBytes;
  // two each: k and v one per stage, p one per P tile
  const uint32_t q_full = bars, k_full = bars + 8, k_empty = bars + 24, v_full = bars + 40, v_empty = bars + 56,
                 s_full0 = bars + 72, p_full = bars + 88, p_empty = bars + 104, tmem_slot = bars + 120;
  uint32_t* tmem_slot_ptr = reinterpret_cast<uint32_t*>(smem + (tmem_slot - q_s));
  constexpr int NP = G::kPTiles, NS = G::kStages;
  __shared__ int s_abort;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = blockIdx.x, head = blockIdx.y;
  const int ntok = p.qt_ntok[tile];
  if (ntok <= 0) return;                                   // padding tile (uniform over the CTA)
  const int seq = p.qt_seq[tile], tok0 = p.qt_tok0[tile];
  const int kh = head / (p.hq / p.hkv);
  const int kv_len = p.positions[tok0 + ntok - 1] + 1;
  const int page0 = p.window > 0 ? max(0, p.positions[tok0] - p.window + 1) >> 4 : 0, first = page0 * 16;    // first key of the walk
  const int npages = (kv_len + 15) >> 4;
  const int ntiles = (kv_len - first + 127) >> 7;

  if (threadIdx.x == 0) {
    s_abort = 0;
    mbar_init(q_full, 1);
    for (int i = 0; i < 10; ++i) mbar_init(k_full + 8 * i, 1);       // up to s_full
    for (int i = 0; i < NP; ++i) {
      mbar_init(p_full + 8 * i, 128 * G::kHalves);
      mbar_init(p_empty + 8 * i, 1);
    }
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot_ptr;
  volatile int* abort_flag = &s_abort;

  if (warp == 0 || warp == kAttnProducerV) {
    // ------------------------------------------------------------ TMA producers: warp 0 Q and K, warp 6 V
    // (one thread's wait / expect / copy sequence is slower than the tensor pipe consumes a tile, so K and V are
    // requested by two threads; a K page is ONE 4-D copy: [2 groups of 8 keys][kSlabs][8][64 columns])
    if (elect_one()) {
      const int* bt = p.block_tables + (size_t)seq * p.max_blocks;
      if (warp == 0) {
        mbar_expect_tx(q_full, G::kQBytes);
#pragma unroll
        for (int s = 0; s < G::kSlabs; ++s) tma_load_2d(q_s + s * (128 * 128), &p.map_q, head * D + s * 64, tok0, q_full);
        for (int j = 0; j < ntiles && !*abort_flag; ++j) {
          int blk[8];
#pragma unroll
          for (int g = 0; g < 8; ++g) blk[g] = bt[min(page0 + j * 8 + g, npages - 1)];   // pages past the end repeat the last one (masked)
          const int st = j % NS;
          if (j >= NS && !mbar_wait(k_empty + 8 * st, (uint32_t)((j / NS - 1) & 1), kAttnWaitNs, p.status)) { *abort_flag = 1; break; }
          mbar_expect_tx(k_full + 8 * st, G::kKBytes);
#pragma unroll
          for (int g = 0; g < 8; ++g)
            tma_load_4d(k_s + st * G::kKBytes + g * (G::kSlabs * 2048), &p.map_k, 0, 0, 0, (blk[g] * p.hkv + kh) * 2, k_full + 8 * st);
        }
      } else {
        for (int j = 0; j < ntiles && !*abort_flag; ++j) {
          int blk[8];
#pragma unroll
          for (int g = 0; g < 8; ++g) blk[g] = bt[min(page0 + j * 8 + g, npages - 1)];
          const int st = j % NS;
          if (j >= NS && !mbar_wait(v_empty + 8 * st, (uint32_t)((j / NS - 1) & 1), kAttnWaitNs, p.status)) { *abort_flag = 1; break; }
          mbar_expect_tx(v_full + 8 * st, G::kVBytes);
#pragma unroll
          for (int g = 0; g < 8; ++g) tma_load_2d(v_s + st * G::kVBytes + g * G::kVPage, &p.map_v, 0, (blk[g] * p.hkv + kh) * DV, v_full + 8 * st);
        }
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      constexpr uint32_t idesc_s = idesc_f16_bf16(128, 128), idesc_o = idesc_f16_bf16(128, DV);
      auto issue_qk = [&](int j) {
        const uint32_t d = tmem_base + (uint32_t)(j & 1) * 128u, kb = k_s + (j % NS) * G::kKBytes;
#pragma unroll
        for (int s = 0; s < G::kSlabs; ++s)
#pragma unroll
          for (int ks = 0; ks < 4; ++ks)                     // K: per 8-key group the kSlabs 64-column slabs side by side
            umma_bf16(d, smem_desc_sw128(q_s + s * (128 * 128) + ks * 32),
                      smem_desc_sw128_sbo(kb + s * 1024 + ks * 32, G::kSlabs * 1024), idesc_s, (s | ks) ? 1u : 0u);
        umma_commit(k_empty + 8 * (j % NS));
        umma_commit(s_full0 + 8 * (j & 1));
      };
      bool ok = mbar_wait(q_full, 0, kAttnWaitNs, p.status) && mbar_wait(k_full, 0, kAttnWaitNs, p.status);
      if (ok) {
        tc_fence_after();
        issue_qk(0);
      }
      for (int j = 0; j < ntiles && ok && !*abort_flag; ++j) {
        if (j + 1 < ntiles) {
          ok = mbar_wait(k_full + 8 * ((j + 1) % NS), (uint32_t)(((j + 1) / NS) & 1), kAttnWaitNs, p.status);
          if (!ok) break;
          tc_fence_after();
          issue_qk(j + 1);
        }
        ok = mbar_wait(p_full + 8 * (j % NP), (uint32_t)((j / NP) & 1), kAttnWaitNs, p.status) && mbar_wait(v_full + 8 * (j % NS), (uint32_t)((j / NS) & 1), kAttnWaitNs, p.status);
        if (!ok) break;
        tc_fence_after();
#pragma unroll
        for (int g = 0; g < 8; ++g)
          umma_bf16(tmem_base + 256u, smem_desc_sw128(p_s + (j % NP) * G::kP + (g >> 2) * (128 * 128) + (g & 3) * 32),
                    smem_desc_sw32(v_s + (j % NS) * G::kVBytes + g * G::kVPage), idesc_o, (j | g) ? 1u : 0u);
        umma_commit(v_empty + 8 * (j % NS));
        umma_commit(p_empty + 8 * (j % NP));
      }
      if (!ok) *abort_flag = 1;
    }
  } else if (MODE == SCORE_SERIES) {
    // ------------------------------------------------------------ softmax + epilogue, bounded scores: two threads (in
    // warps 2-5 and 8-11) per query row, each half of the keys of a tile and half of the output columns
    if (warp < 6 || warp >= 8) {
      const int quarter = warp & 3, half = warp >= 8 ? 1 : 0, r = quarter * 32 + lane;
      const bool valid = r < ntok;
      const int pos = p.positions[tok0 + (valid ? r : ntok - 1)];
      const uint32_t lane_base = tmem_base + ((uint32_t)(quarter * 32) << 16);
      const TanhSeries series(p.cap_out, p.cap_in);
      f2 sum2 = pack2(0.f, 0.f);
      const f2 one2 = pack2(1.f, 1.f);
      bool ok = true;
      for (int j = 0; j < ntiles; ++j) {
        ok = ok && !*abort_flag && mbar_wait(s_full0 + 8 * (j & 1), (uint32_t)((j >> 1) & 1), kAttnWaitNs, p.status);
        if (ok && j >= NP) ok = mbar_wait(p_empty + 8 * (j % NP), (uint32_t)((j / NP - 1) & 1), kAttnWaitNs, p.status);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        const uint32_t s_addr = lane_base + (uint32_t)(j & 1) * 128u + (uint32_t)half * 64u;
        const int key0 = j * 128 + half * 64;
        const bool need_mask = key0 + 63 > pos;
        uint32_t v[2][32];
        tmem_ld32(s_addr, v[0]);
        tmem_ld32(s_addr + 32, v[1]);
        tmem_ld_wait();
        const uint32_t row_addr = p_s + (uint32_t)(j % NP) * G::kP + (uint32_t)half * (128 * 128) + (uint32_t)r * 128u;
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          uint32_t pk[16];
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            float s0, s1;
            unpack2(series(pack2(__uint_as_float(v[c][i]), __uint_as_float(v[c][i + 1]))), s0, s1);
            if (need_mask) {
              if (key0 + c * 32 + i > pos) s0 = kMaskVal;
              if (key0 + c * 32 + i + 1 > pos) s1 = kMaskVal;
            }
            const float p0 = ex2_approx(s0), p1 = ex2_approx(s1);
            sum2 = fma2(pack2(p0, p1), one2, sum2);
            pk[i >> 1] = pack_bf16(p0, p1);
          }
#pragma unroll
          for (int q4 = 0; q4 < 4; ++q4) {
            const uint32_t chunk = (uint32_t)(c * 4 + q4) ^ (uint32_t)(r & 7);
            asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};\n" ::"r"(row_addr + chunk * 16u), "r"(pk[4 * q4]),
                         "r"(pk[4 * q4 + 1]), "r"(pk[4 * q4 + 2]), "r"(pk[4 * q4 + 3])
                         : "memory");
          }
        }
        tc_fence_before();
        fence_proxy_async();
        asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(p_full + 8 * (j % NP)) : "memory");
      }
      if (ok) {                                            // every P V has completed: they complete in order
        ok = mbar_wait(p_empty + 8 * ((ntiles - 1) % NP), (uint32_t)(((ntiles - 1) / NP) & 1), kAttnWaitNs, p.status);
        ok = __all_sync(0xffffffffu, ok);
      }
      if (!ok) *abort_flag = 1;
      // the sums of the two halves meet in the idle P tile; a warp that gave up still takes part in the barrier
      float a, b;
      unpack2(sum2, a, b);
      float* l_s = reinterpret_cast<float*>(smem + (p_s - q_s));
      l_s[half * 128 + r] = a + b;
      asm volatile("bar.sync 1, 256;\n" ::: "memory");
      if (ok) {
        tc_fence_after();
        const size_t tok = (size_t)tok0 + (valid ? r : 0);
        const float inv = head_factor(p, tok, head) / (l_s[r] + l_s[128 + r]);
        const __nv_bfloat16* gate = p.gate_src + tok * p.ld + p.gate_col + (size_t)head * p.gate_stride;
        __nv_bfloat16* dst = p.out + tok * (size_t)p.ldo + (size_t)head * DV;
#pragma unroll 1
        for (int c = half * (DV / 64); c < (half + 1) * (DV / 64); ++c) {
          uint32_t v[32];
          tmem_ld32(lane_base + 256u + c * 32, v);
          uint4 gates[4];
          load_gates(p, gate, c, gates);
          tmem_ld_wait();
          if (valid) store_rows32(p, v, inv, gates, dst, c);
        }
      }
      tc_fence_before();
    }
  } else {
    // ------------------------------------------------------------ softmax + epilogue: thread = query row
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const bool valid = r < ntok;
    const int pos = p.positions[tok0 + (valid ? r : ntok - 1)];
    const int lo = p.window > 0 ? pos - p.window + 1 : 0;
    const float slope = MODE == SCORE_BIASED ? p.slopes[head] * 1.4426950408889634f : 0.f;
    const uint32_t lane_base = tmem_base + ((uint32_t)(quarter * 32) << 16);
    const size_t tok = (size_t)tok0 + (valid ? r : 0);
    const __nv_bfloat16* gate = p.gate_src + tok * p.ld + p.gate_col + (size_t)head * p.gate_stride;
    prefetch_gates(p, gate, DV);
    float m_used = kFirstMax, l = 0.f;
    bool ok = true;
    for (int j = 0; j < ntiles; ++j) {
      ok = ok && !*abort_flag && mbar_wait(s_full0 + 8 * (j & 1), (uint32_t)((j >> 1) & 1), kAttnWaitNs, p.status);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t s_addr = lane_base + (uint32_t)(j & 1) * 128u;
      const int key0 = first + j * 128, from = lo - key0, to = pos - key0;       // the row sees keys from .. to of the tile
      // ---- the row's scores (PLAIN: still to be scaled) and their maximum
      uint32_t v[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(s_addr + c * 32, v[c]);
      tmem_ld_wait();
      if (MODE != SCORE_PLAIN) {
        const float ahead = slope * (float)-to;
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            v[c][i] = __float_as_uint(prefill_score<MODE>(p, __uint_as_float(v[c][i]), fmaf(slope, (float)(c * 32 + i), ahead)));
      }
      if (to < 127 || from > 0) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (c * 32 + i > to || c * 32 + i < from) v[c][i] = 0xff800000u;
      }
      float mx = __uint_as_float(0xff800000u);
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(v[c][i]));
      const float factor = MODE == SCORE_PLAIN ? p.scale_log2e : 1.f;
      mx *= factor;
      const float m_new = fmaxf(m_used, mx);
      const bool resc = m_new - m_used > kRescaleGap;
      float alpha = 1.f;
      if (resc) {
        alpha = ex2_approx(m_used - m_new);
        l *= alpha;
        m_used = m_new;
      }
      // ---- P buffer free and O quiescent: the previous tile's P V has completed
      if (j > 0) {
        ok = mbar_wait(p_empty, (uint32_t)((j - 1) & 1), kAttnWaitNs, p.status);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (__any_sync(0xffffffffu, resc)) {
#pragma unroll 1
          for (int c = 0; c < DV / 32; ++c) {
            uint32_t o[32];
            tmem_ld32(lane_base + 256u + c * 32, o);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
            tmem_st32(lane_base + 256u + c * 32, o);
          }
          tmem_st_wait();
        }
      }
      // ---- P = exp2(S - m), row sum, bf16 A operand in the 128-byte-swizzled K-major layout
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float p0 = ex2_approx(fmaf(__uint_as_float(v[c][i]), factor, -m_used)), p1 = ex2_approx(fmaf(__uint_as_float(v[c][i + 1]), factor, -m_used));
          sum += p0 + p1;
          pk[i >> 1] = pack_bf16(p0, p1);
        }
        const uint32_t row_addr = p_s + (uint32_t)(c >> 1) * (128 * 128) + (uint32_t)r * 128u;
#pragma unroll
        for (int q4 = 0; q4 < 4; ++q4) {
          const uint32_t chunk = (uint32_t)((c & 1) * 4 + q4) ^ (uint32_t)(r & 7);
          asm volatile("st.shared.v4.u32 [%0], {%1,%2,%3,%4};\n" ::"r"(row_addr + chunk * 16u), "r"(pk[4 * q4]),
                       "r"(pk[4 * q4 + 1]), "r"(pk[4 * q4 + 2]), "r"(pk[4 * q4 + 3])
                       : "memory");
        }
      }
      l += sum;
      tc_fence_before();
      fence_proxy_async();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(p_full) : "memory");
    }
    // ---- epilogue: O / l * sigmoid(gate) -> bf16
    uint4 gates[4], next[4];
    load_gates(p, gate, 0, gates);
    if (ok) {
      ok = mbar_wait(p_empty, (uint32_t)((ntiles - 1) & 1), kAttnWaitNs, p.status);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (ok) {
      tc_fence_after();
      const float inv = head_factor(p, tok, head) / l;
      __nv_bfloat16* dst = p.out + tok * (size_t)p.ldo + (size_t)head * DV;
#pragma unroll 1
      for (int c = 0; c < DV / 32; ++c) {
        uint32_t v[32];
        tmem_ld32(lane_base + 256u + c * 32, v);
        if (c + 1 < DV / 32) load_gates(p, gate, c + 1, next);
        tmem_ld_wait();
        if (valid) store_rows32(p, v, inv, gates, dst, c);
#pragma unroll
        for (int q = 0; q < 4; ++q) gates[q] = next[q];
      }
    } else {
      *abort_flag = 1;
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem_base, 512);
  }
}

template <int D, int DV, int MODE>
static int launch_mode(const AttnPrefillParams& p, int num_tiles, cudaStream_t st) {
  static bool configured = false;
  auto k = attn_prefill_kernel<D, DV, MODE>;
  if (!configured) {
    cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)AttnPrefillGeom<D, DV, MODE>::kSmem);
    configured = true;
  }
  k<<<dim3(num_tiles, p.hq), AttnPrefillGeom<D, DV, MODE>::kThreads, AttnPrefillGeom<D, DV, MODE>::kSmem, st>>>(p);
  return (int)cudaGetLastError();
}

template <int D, int DV>
static int launch_attn_prefill(const AttnPrefillParams& p, int num_tiles, int mode, cudaStream_t st) {
  if (mode == SCORE_SERIES) return launch_mode<D, DV, SCORE_SERIES>(p, num_tiles, st);
  if (mode == SCORE_CAPPED) return launch_mode<D, DV, SCORE_CAPPED>(p, num_tiles, st);
  if (mode == SCORE_BIASED) return launch_mode<D, DV, SCORE_BIASED>(p, num_tiles, st);
  return launch_mode<D, DV, SCORE_PLAIN>(p, num_tiles, st);
}

}  // namespace ti

extern "C" {

// out[tok, head*DV + d] = softmax(score(q k^T), causal by position) v * sigmoid(gate) for the tokens of the listed query
// tiles (up to 128 consecutive tokens of one sequence each; longest first gives the best balance).
// q: bf16 [T, hq, D] (normalised, rotated); kcache / vcache: the paged cache of this layer, `num_blocks` pages;
// positions: absolute position of every flat token; gate_src: null, or rows [T, ld] with the gates of head h at column
// gate_col + h * gate_stride (stride 0: h*2D + D).
// score(x) = scale x, or with softcap > 0 softcap * tanh(scale x / softcap).  `qk_max`: a bound of |q.k|, or <= 0.  With
// `slopes` [hq] a score loses slopes[h] per token of distance; `window`, `head_gate` [T, ldg], `ldo` (row pitch of out) and
// `out_scale` as in AttnPrefillParams.
int ti_attn_prefill(const void* q, int T, const void* kcache, const void* vcache, int num_blocks, const void* block_tables,
                    const void* positions, const void* qt_seq, const void* qt_tok0, const void* qt_ntok, int num_tiles,
                    const void* gate_src, void* out, int hq, int hkv, int max_blocks, int ld, float scale, int D, int DV,
                    float softcap, float qk_max, int window, const void* slopes, const void* head_gate, int ldg, int gcol, int ldo,
                    float out_scale, int gate_col, int gate_stride, void* status, void* stream) {
  if (num_tiles <= 0) return 0;
  if (hq % hkv || T < 1 || num_blocks < 1 || (gate_src != nullptr && D != DV)) return -2;
  // the gate and the output are read / written 16 bytes at a time: refuse layouts that would make those accesses misaligned
  if ((ld & 7) || (ldo & 7) || (gate_col & 7) || (gate_stride & 7) || (reinterpret_cast<uintptr_t>(gate_src) & 15) || (reinterpret_cast<uintptr_t>(out) & 15)) return -4;
  if (window < 0 || (softcap > 0.f && (window > 0 || slopes != nullptr))) return -2;     // caps come without windows and slopes
  if ((D != 64 && D != 128 && D != 256) || (DV != 64 && DV != 128 && DV != 256)) return -3;
  constexpr float kLog2e = 1.4426950408889634f;
  ti::AttnPrefillParams p = {};
  int mode = slopes != nullptr ? ti::SCORE_BIASED : ti::SCORE_PLAIN;
  if (softcap > 0.f) {
    p.cap_in = scale / softcap;
    p.cap_out = softcap * kLog2e;
    const float y = qk_max * p.cap_in;
    mode = qk_max > 0.f && y > -ti::kSeriesMax && y < ti::kSeriesMax && (y < 0.f ? -y : y) * p.cap_out < 60.f ? ti::SCORE_SERIES : ti::SCORE_CAPPED;
  }
  int rc = ti::bf16_map_2d(&p.map_q, q, (long long)hq * D, T, 64, 128, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = ti::bf16_map_groups(&p.map_k, kcache, D, (long long)num_blocks * hkv * 16, D / 64, 2);
  if (rc) return rc;
  rc = ti::bf16_map_2d(&p.map_v, vcache, 16, (long long)num_blocks * hkv * DV, 16, DV, CU_TENSOR_MAP_SWIZZLE_32B);
  if (rc) return rc;
  p.block_tables = (const int*)block_tables;
  p.positions = (const int*)positions;
  p.qt_seq = (const int*)qt_seq;
  p.qt_tok0 = (const int*)qt_tok0;
  p.qt_ntok = (const int*)qt_ntok;
  p.gate_src = (const __nv_bfloat16*)gate_src;
  p.out = (__nv_bfloat16*)out;
  p.status = (unsigned*)status;
  p.hq = hq;
  p.hkv = hkv;
  p.max_blocks = max_blocks;
  p.ld = ld;
  p.scale_log2e = scale * kLog2e;
  p.window = window;
  p.slopes = (const float*)slopes;
  p.head_gate = (const __nv_bfloat16*)head_gate;
  p.ldg = ldg;
  p.gcol = gcol;
  p.ldo = ldo > 0 ? ldo : hq * DV;
  p.out_scale = out_scale;
  p.gate_stride = gate_stride > 0 ? gate_stride : 2 * D;
  p.gate_col = gate_stride > 0 ? gate_col : D;
  cudaStream_t st = (cudaStream_t)stream;
#define TI_AP(A, B) if (D == A && DV == B) return ti::launch_attn_prefill<A, B>(p, num_tiles, mode, st)
  TI_AP(64, 64); TI_AP(64, 128); TI_AP(64, 256);
  TI_AP(128, 64); TI_AP(128, 128); TI_AP(128, 256);
  TI_AP(256, 64); TI_AP(256, 128); TI_AP(256, 256);
#undef TI_AP
  return -3;
}

}  // extern "C"
