// Latent attention of decode tokens on the 5th-generation tensor cores (bf16, rows of 256, 384, 512 or 576 columns).
//
// All heads of a token attend to the same latents, so the latents are the wide operand and the heads the narrow one:
// per tile of 64 keys   S^T [keys x heads] = C q~^T   and   O^T [R x heads] += C^T P^T,   where C [64 x R] is ONE copy
// of the latents in shared memory: the K-major A operand of the first product, the MN-major A operand of the second.
// N = 16 or 32 heads per block; tensor-core time follows the bytes of C, not the heads that a 128-row tile would waste.
//
//   warp 0     TMA producer: slots of 64 keys x 256 columns (whole rows at R = 384 and 576), one 4-D copy per 16-key page, through the
//              block table
//   warp 1     MMA issuer: S^T of the next tile (two buffers) while the softmax works on this one, then O^T slot by slot,
//              each slot released as soon as it was read
//   warps 2-9  softmax over the keys of a tile (lanes = keys in TMEM; the scores change hands through shared memory so that
//              a thread owns one head and a share of the keys), lazy rescaling of O^T, P^T written as the bf16 B operand
//
// The ring holds two tiles at R = 576, two and a half at 512 and more below.  At R = 576 the last 64 columns are key alone.  Every wait is bounded; on expiry the status word is set, the roles leave and TMEM is freed.
#include "latent_attn.cuh"
#include "tensor_map.cuh"

namespace ti {

constexpr int kDkTile = 64;                      // keys per tile
constexpr int kDkSoftmax = 256;                  // threads of the softmax warps
constexpr int kDkThreads = 64 + kDkSoftmax;
constexpr int kDkMaxSlots = 7;
constexpr unsigned long long kDkWaitNs = 500000000ull;
constexpr float kDkGap = 8.f;                    // log2 units the running maximum may lag behind before O is rescaled

struct LatentDecodeTcParams {
  alignas(64) CUtensorMap map_c;                 // cache rows as [groups of 8][R/64 slabs][8][64], box {64, 8, slabs, 2}
  LatentAttnParams a;
  int slots;                                     // of the ring
};

template <int N> struct DkGeom {                 // N heads per block
  static constexpr int kPitch = N + 1;           // floats per key of the score exchange
  static constexpr int kParts = kDkSoftmax / N;         // threads per head
  static constexpr int kShare = kDkTile / kParts;        // keys per thread in the softmax
  static constexpr size_t fixed(int Rp) {        // everything but the ring
    return (size_t)N * Rp * 2 + 2 * N * 128 + kDkTile * kPitch * 4 + (size_t)(kParts + 2) * N * 4 + 256 + 1024;
  }
};

TI_DEVICE float dk_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}
TI_DEVICE void softmax_bar() { asm volatile("bar.sync 1, 256;\n" ::: "memory"); }
template <int N> TI_DEVICE void tmem_ld_n(uint32_t taddr, float (&v)[N]);
template <> TI_DEVICE void tmem_ld_n<32>(uint32_t taddr, float (&v)[32]) {
  uint32_t r[32];
  tmem_ld32(taddr, r);
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(r[i]);
}
template <> TI_DEVICE void tmem_ld_n<16>(uint32_t taddr, float (&v)[16]) {
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
template <> TI_DEVICE void tmem_ld_n<8>(uint32_t taddr, float (&v)[8]) {
  uint32_t r[8];
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];\n"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
               : "r"(taddr)
               : "memory");
  tmem_ld_wait();
#pragma unroll
  for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[i]);
}
template <int N> TI_DEVICE void tmem_st_n(uint32_t taddr, const float (&v)[N]);
template <> TI_DEVICE void tmem_st_n<32>(uint32_t taddr, const float (&v)[32]) {
  uint32_t r[32];
#pragma unroll
  for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(v[i]);
  tmem_st32(taddr, r);
}
template <> TI_DEVICE void tmem_st_n<16>(uint32_t taddr, const float (&v)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};\n" ::"r"(taddr),
      "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7]), "f"(v[8]), "f"(v[9]), "f"(v[10]),
      "f"(v[11]), "f"(v[12]), "f"(v[13]), "f"(v[14]), "f"(v[15])
      : "memory");
}

// SC: 64-column slabs of a ring slot
template <int N, int SC>
__global__ void __launch_bounds__(kDkThreads, 1) latent_decode_tc_kernel(const __grid_constant__ LatentDecodeTcParams pp) {
  using G = DkGeom<N>;
  const LatentAttnParams& p = pp.a;
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int Rp = p.Rp, np = Rp >> 7, ns = pp.slots;              // 128-row blocks of O^T, slots of the ring
  const int spt = (Rp >> 6) / SC;                                // slots of a tile
  constexpr uint32_t grp = SC * 1024, slot_bytes = 8 * grp;      // an 8-key group, 64 keys
  const uint32_t ring = smem_u32(smem), q_s = ring + ns * slot_bytes, p_s = q_s + N * Rp * 2;
  uint8_t* tail = smem + ns * slot_bytes + N * Rp * 2 + 2 * N * 128;   // two P^T buffers
  float* s_x = reinterpret_cast<float*>(tail);                   // [64 keys][N + 1]
  float* mx_x = s_x + kDkTile * G::kPitch;                           // [parts][N]; at the end the sums
  float* alpha_x = mx_x + G::kParts * N;                         // [N]
  float* ml_x = alpha_x + N;                                     // [N]: factor of O
  const uint32_t bars = smem_u32(ml_x + N);
  const uint32_t full = bars, empty = bars + 8 * kDkMaxSlots, s_full = bars + 16 * kDkMaxSlots, p_empty = s_full + 16,
                 p_full = s_full + 32, q_full = s_full + 48, o_full = s_full + 56, tmem_slot = s_full + 64;
  uint32_t* tmem_slot_ptr = reinterpret_cast<uint32_t*>(smem + (tmem_slot - ring));
  volatile int* abort_flag = reinterpret_cast<int*>(tmem_slot_ptr + 1);

  const int qg = blockIdx.x, hg = blockIdx.y, sp = blockIdx.z;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  pdl_trigger();
  pdl_wait();
  if (p.qg_ntok[qg] == 0) return;
  const int tok = p.qg_tok0[qg], seq = p.qg_seq[qg];
  const KeyRange kr = key_range(p, tok, kDkTile);
  const int t0 = sp * kr.tps, t1 = min(kr.ntiles, t0 + kr.tps);
  if (t0 >= t1) return;                                          // inactive split (uniform over the block)

  if (tid == 0) {
    *abort_flag = 0;
    for (int i = 0; i < 2 * kDkMaxSlots + 4; ++i) mbar_init(bars + 8 * i, 1);
    for (int i = 0; i < 3; ++i) mbar_init(p_full + 8 * i, kDkSoftmax);   // P^T (two buffers), q~
    mbar_init(o_full, 1);
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 256);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot_ptr, o_col = 64;              // S^T at columns 0 and 32, O^T block b at 64 + b * N

  if (warp == 0) {
    // ------------------------------------------------------------ TMA producer: lane g of four copies page g of a tile
    const int* bt = p.block_tables + (size_t)seq * p.max_blocks;
    auto page = [&](int j) {                                     // pages past the end repeat the last one (masked)
      const int blk = bt[min(kr.page0 + j * (kDkTile / 16) + (lane & 3), kr.npages - 1)];
      return TI_CHECK(blk, p.num_blocks, p.status) ? blk : 0;
    };
    int it = 0, blk = page(t0);
    bool ok = true;
    for (int j = t0; j < t1 && ok; ++j) {
      const int next = page(min(j + 1, t1 - 1));
      for (int b = 0; b < spt; ++b, ++it) {
        const int s = it % ns;
        ok = !*abort_flag && (it < ns || mbar_wait(empty + 8 * s, (uint32_t)((it / ns - 1) & 1), kDkWaitNs, p.status));
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        if (lane == 0) mbar_expect_tx(full + 8 * s, slot_bytes);
        __syncwarp();
        if (lane < 4) tma_load_4d(ring + s * slot_bytes + lane * 2 * grp, &pp.map_c, 0, 0, SC * b, blk * 2, full + 8 * s);
      }
      blk = next;
    }
    if (!ok) *abort_flag = 1;
  } else if (warp == 1) {
    // ------------------------------------------------------------ MMA issuer
    if (elect_one()) {
      constexpr uint32_t idesc_s = idesc_f16_bf16(64, N), idesc_o = idesc_f16_bf16_amn(128, N);
      const int nt = t1 - t0;
      auto scores = [&](int j) {                                 // S^T of tile j as its slots land
        for (int b = 0; b < spt; ++b) {
          const int it = j * spt + b, s = it % ns;
          if (*abort_flag || !mbar_wait(full + 8 * s, (uint32_t)((it / ns) & 1), kDkWaitNs, p.status)) return false;
          tc_fence_after();
          // descriptors of one operand differ in the address field alone (units of 16 bytes)
          const uint64_t da = smem_desc_sw128_sbo(ring + s * slot_bytes, grp), db = smem_desc_sw128(q_s + b * SC * (N * 128));
          const uint32_t d = tmem + (j & 1) * 32;
#pragma unroll
          for (int c = 0; c < SC; ++c)
#pragma unroll
            for (int k = 0; k < 4; ++k)
              umma_bf16(d, da + ((c * 1024 + k * 32) >> 4), db + ((c * N * 128 + k * 32) >> 4), idesc_s, (c | k) ? 1u : (b ? 1u : 0u));
        }
        umma_commit(s_full + 8 * (j & 1));
        return true;
      };
      bool ok = mbar_wait(q_full, 0, kDkWaitNs, p.status) && scores(0);
      for (int j = 0; j < nt && ok; ++j) {
        if (j + 1 < nt) ok = scores(j + 1);
        ok = ok && mbar_wait(p_full + 8 * (j & 1), (uint32_t)((j >> 1) & 1), kDkWaitNs, p.status);
        if (!ok) break;
        tc_fence_after();
        const uint64_t db = smem_desc_sw128(p_s + (j & 1) * (N * 128));
        for (int t = 0; t < spt; ++t) {
          const int s = (j * spt + t) % ns;
          const uint64_t da = smem_desc_mn128(ring + s * slot_bytes, 1024, grp);
          const uint32_t d = tmem + o_col + t * (SC / 2) * N;
#pragma unroll
          for (int c = 0; c < SC / 2; ++c)                       // 128 columns of C = 128 rows of O^T
#pragma unroll
            for (int g = 0; g < kDkTile / 16; ++g)
              umma_bf16(d + c * N, da + ((c * 2048 + g * 2 * grp) >> 4), db + ((g * 32) >> 4), idesc_o, g ? 1u : (j ? 1u : 0u));
          umma_commit(empty + 8 * s);
        }
        umma_commit(p_empty + 8 * (j & 1));
      }
      umma_commit(o_full);                                       // O^T complete (or the loop gave up)
      if (!ok) *abort_flag = 1;
    }
  } else {
    // ------------------------------------------------------------ softmax: in TMEM a thread is a key, then a share of a head
    constexpr int NH = N / 2;                                    // two warps per lane quarter share the heads
    const int quarter = warp & 3, half = (warp - 2) >> 2, key_l = quarter * 16 + (lane & 15);   // M = 64: 16 keys in each lane quarter
    const int u = tid - 64, head = u % N, part = u / N;          // head and share of the keys
    const uint32_t lane_base = tmem + ((uint32_t)(quarter * 32) << 16);
    const float sc = p.scale * kLog2e;
    // q~ as the B operand of S^T: per 64-column slab N rows of 128 bytes, 128-byte swizzle; missing heads are zero
    {
      const bf16* q = static_cast<const bf16*>(p.q) + ((size_t)tok * p.H + hg * N) * Rp;
      const int cpr = Rp >> 3, nrow = min(N, p.H - hg * N);
#pragma unroll 4
      for (int i = u; i < N * cpr; i += kDkSoftmax) {
        const int row = i / cpr, c = i - row * cpr;
        const uint4 v = row < nrow ? *reinterpret_cast<const uint4*>(q + (size_t)row * Rp + c * 8) : make_uint4(0, 0, 0, 0);
        *reinterpret_cast<uint4*>(smem + (q_s - ring) + (c >> 3) * (N * 128) + row * 128 + (((c & 7) ^ (row & 7)) << 4)) = v;
      }
      fence_proxy_async();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(q_full) : "memory");
    }
    float m_used = kNeg, l = 0.f;
    bool ok = true;
    for (int j = 0; j < t1 - t0; ++j) {
      ok = !*abort_flag && mbar_wait(s_full + 8 * (j & 1), (uint32_t)((j >> 1) & 1), kDkWaitNs, p.status);
      if (!ok) *abort_flag = 1;
      __syncwarp();
      tc_fence_after();
      float v[NH > G::kShare ? NH : G::kShare];
      {
        float w[NH];
        tmem_ld_n<NH>(lane_base + (j & 1) * 32 + half * NH, w);
#pragma unroll
        for (int i = 0; i < NH; ++i) v[i] = w[i];
      }
      const int key = kr.page0 * 16 + (t0 + j) * kDkTile + key_l;
      const bool seen = ok && key >= kr.lo && key <= kr.pos;
      if (lane < 16) {
#pragma unroll
        for (int i = 0; i < NH; ++i) s_x[key_l * G::kPitch + half * NH + i] = seen ? v[i] * sc : kNeg;
      }
      softmax_bar();
      float mx = kNeg;
#pragma unroll
      for (int i = 0; i < G::kShare; ++i) {
        v[i] = s_x[(part * G::kShare + i) * G::kPitch + head];
        mx = fmaxf(mx, v[i]);
      }
      mx_x[part * N + head] = mx;
      softmax_bar();
#pragma unroll
      for (int i = 0; i < G::kParts; ++i) mx = fmaxf(mx, mx_x[i * N + head]);
      const float m_new = fmaxf(m_used, mx);
      float al = 1.f;
      if (m_new - m_used > kDkGap) {
        al = dk_ex2(m_used - m_new);
        l *= al;
        m_used = m_new;
      }
      if (part == 0) alpha_x[head] = al;
      if (j > 1) {                                               // this P^T buffer is free: the product of tile j - 2 is done
        ok = !*abort_flag && mbar_wait(p_empty + 8 * (j & 1), (uint32_t)(((j >> 1) - 1) & 1), kDkWaitNs, p.status);
        if (!ok) *abort_flag = 1;
        __syncwarp();
        tc_fence_after();
      }
      uint32_t pk[G::kShare / 2];
#pragma unroll
      for (int i = 0; i < G::kShare; i += 2) {                   // masked scores: exp2 of a huge negative number is 0
        const float e0 = dk_ex2(v[i] - m_used), e1 = dk_ex2(v[i + 1] - m_used);
        l += e0 + e1;
        pk[i >> 1] = pack_bf16(e0, e1);
      }
      {
        const int k0 = part * G::kShare;                         // 16-byte chunks of eight keys, swizzled by the row
        uint8_t* dst = smem + (p_s - ring) + (j & 1) * (N * 128) + head * 128 + (((k0 >> 3) ^ (head & 7)) << 4) + (k0 & 7) * 2;
        if constexpr (G::kShare == 8) *reinterpret_cast<uint4*>(dst) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
        else *reinterpret_cast<uint2*>(dst) = make_uint2(pk[0], pk[1]);
      }
      softmax_bar();
      if (j > 0 && __any_sync(0xffffffffu, alpha_x[lane % N] != 1.f)) {
        // O^T quiescent: the product of the last tile is done
        ok = !*abort_flag && mbar_wait(p_empty + 8 * ((j - 1) & 1), (uint32_t)(((j - 1) >> 1) & 1), kDkWaitNs, p.status);
        if (!ok) *abort_flag = 1;
        __syncwarp();
        tc_fence_after();
#pragma unroll 1
        for (int b = half; b < np; b += 2) {
          float o[N];
          tmem_ld_n<N>(lane_base + o_col + b * N, o);
#pragma unroll
          for (int i = 0; i < N; ++i) o[i] *= alpha_x[i];
          tmem_st_n<N>(lane_base + o_col + b * N, o);
        }
        tmem_st_wait();
      }
      tc_fence_before();
      fence_proxy_async();
      asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];\n" ::"r"(p_full + 8 * (j & 1)) : "memory");
    }
    // ---- sums of the parts, then O^T
    mx_x[part * N + head] = l;
    softmax_bar();
    float L = 0.f;
#pragma unroll
    for (int i = 0; i < G::kParts; ++i) L += mx_x[i * N + head];
    ok = mbar_wait(o_full, 0, 2 * kDkWaitNs, p.status) && !*abort_flag;
    __syncwarp();
    tc_fence_after();
    const size_t item = ((size_t)qg * gridDim.y + hg) * p.nsplit + sp;
    const int hglob = hg * N + head;
    if (part == 0) {
      if (p.nsplit == 1) {
        const float sk = p.sink == nullptr || hglob >= p.H ? kNeg : p.sink[hglob] * kLog2e;
        const float M = fmaxf(m_used, sk), w = dk_ex2(m_used - M);
        ml_x[head] = w / (L * w + (sk > 0.5f * kNeg ? dk_ex2(sk - M) : 0.f));
      } else {
        p.ml_part[(item * N + head) * 2] = m_used;
        p.ml_part[(item * N + head) * 2 + 1] = L;
      }
    }
    softmax_bar();
    if (__all_sync(0xffffffffu, ok)) {
      const int nh = min(N, p.H - hg * N);
#pragma unroll 1
      for (int b = half; b < np; b += 2) {
        float o[N];
        tmem_ld_n<N>(lane_base + o_col + b * N, o);
        const int r = b * 128 + quarter * 32 + lane;
        if (r >= p.Ro) continue;
        if (p.nsplit == 1) {
          bf16* dst = static_cast<bf16*>(p.out) + ((size_t)tok * p.H + hg * N) * p.Ro + r;
#pragma unroll
          for (int i = 0; i < N; ++i)
            if (i < nh) dst[(size_t)i * p.Ro] = __float2bfloat16_rn(o[i] * ml_x[i]);
        } else {
          float* dst = p.o_part + item * N * Rp + r;
#pragma unroll
          for (int i = 0; i < N; ++i)
            if (i < nh) dst[(size_t)i * Rp] = o[i];
        }
      }
    }
    tc_fence_before();
  }
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    tmem_dealloc(tmem, 256);
  }
}

template <int N, int SC>
static int launch_dk(LatentDecodeTcParams& p, cudaStream_t st) {
  constexpr size_t kMax = 227 * 1024;
  const size_t fixed = DkGeom<N>::fixed(p.a.Rp);
  const size_t slot = (size_t)SC * 8192;
  p.slots = (int)((kMax - fixed) / slot);
  if (p.slots > kDkMaxSlots) p.slots = kDkMaxSlots;
  if (p.slots < 2 * (p.a.Rp / 64 / SC)) return -2;           // S^T runs one tile ahead of O^T
  auto k = latent_decode_tc_kernel<N, SC>;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kMax);
    configured = true;
  }
  launch_kernel(k, dim3(p.a.num_qg, (p.a.H + N - 1) / N, p.a.nsplit), dim3(kDkThreads), fixed + (size_t)p.slots * slot, st, true, p);
  if (p.a.nsplit > 1) launch_latent_merge(p.a, N, kDkTile, st);
  return (int)cudaGetLastError();
}

int launch_latent_decode_tc(const LatentAttnParams& a, cudaStream_t st) {
  if ((a.Rp != 256 && a.Rp != 384 && a.Rp != 512 && a.Rp != 576) || (a.Rp == 576 && a.Ro > 512) || a.num_blocks < 1) return -2;
  LatentDecodeTcParams p = {};
  p.a = a;
  const int slabs = a.Rp % 256 == 0 ? 4 : a.Rp / 64;
  const int rc = bf16_map_groups(&p.map_c, a.cache, a.Rp, (long long)a.num_blocks * 16, slabs, 2);
  if (rc) return rc;
  if (slabs == 4) return a.H > 16 ? launch_dk<32, 4>(p, st) : launch_dk<16, 4>(p, st);
  if (slabs == 6) return a.H > 16 ? launch_dk<32, 6>(p, st) : launch_dk<16, 6>(p, st);
  return a.H > 16 ? launch_dk<32, 9>(p, st) : launch_dk<16, 9>(p, st);
}

}  // namespace ti
