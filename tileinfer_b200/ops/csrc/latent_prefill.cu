// Windowed attention of prefill query tiles over expanded keys and values on the 5th-generation tensor cores.
//
// For many query tokens it is cheaper to expand the latents in reach once (k = W_uk c, v = W_uv c for all heads: one
// tcgen05 product into rows [K heads | V heads]) than to let every query meet the wider latents, so this kernel works on
// plain per-head keys and values.  A CTA owns 128 consecutive query tokens of one head and walks the keys from the first
// one any of them sees (window) to the last token, in tiles of 128:
//
//   warp 0     TMA producer of Q (once) and K tiles: [128 rows][64 columns] slabs, 128-byte swizzle, K-major
//   warp 6     TMA producer of V tiles: the same slabs, used as the MN-major B operand of P V (no transposition)
//   warp 1     MMA issuer: S = Q K^T (two S buffers in TMEM), then O += P V
//   warps 2-5  softmax: one thread per query row, the 128 scores of a tile in registers, lazy rescaling of O, P written to
//              shared memory as the bf16 A operand; at the end O / l times the head's sigmoid gate
//
// Head sizes are run-time multiples of 64 up to 256; K and V tiles are double-buffered when shared memory allows.  The
// window, the sink (a term of the denominator: the running sum simply starts with it) and the gate are parameters.
// Every wait is bounded; on expiry the status word is set, all roles leave their loops and TMEM is freed.
#include "tensor_map.cuh"

namespace ti {

struct LatentPrefillParams {
  alignas(64) CUtensorMap map_q;   // bf16 [T][ldq], box {64, 128}
  alignas(64) CUtensorMap map_kv;  // bf16 [Nk][ldkv], box {64, 128}
  const int* tiles;                // [5][num_tiles]: first flat token, tokens (1..128), its position, a row of the
                                   // expanded keys, the position that row holds
  const float* sink;               // [H] or null
  const __nv_bfloat16* gate;       // null, or [T, ldg]: gate of head h at column gcol + h
  __nv_bfloat16* out;              // [T, ldo], head h at column h * vp
  unsigned* status;
  int num_tiles, dp, vp, v_col, ldg, gcol, ldo, window, stages;
  float scale_log2e;
};

constexpr unsigned long long kLpWaitNs = 500000000ull;
constexpr int kLpThreads = 224;
constexpr float kLpMask = -1e30f;
constexpr float kLpGap = 8.f;            // log2 units the running maximum may lag behind before O is rescaled
constexpr int kSlabBytes = 128 * 128;    // 128 rows x 64 bf16

TI_DEVICE float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

static size_t latent_prefill_smem(int dp, int vp, int stages) {
  return (size_t)(dp / 64) * kSlabBytes * (1 + stages) + (size_t)(vp / 64) * kSlabBytes * stages + 2 * kSlabBytes + 128 + 1024;
}

__global__ void __launch_bounds__(kLpThreads, 1) latent_prefill_kernel(const __grid_constant__ LatentPrefillParams p) {
  extern __shared__ __align__(1024) uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const int ds = p.dp >> 6, vs = p.vp >> 6, nst = p.stages;
  const uint32_t kbytes = ds * kSlabBytes, vbytes = vs * kSlabBytes;
  const uint32_t q_s = smem_u32(smem), k_s = q_s + kbytes, v_s = k_s + nst * kbytes, p_s = v_s + nst * vbytes;
  const uint32_t bars = p_s + 2 * kSlabBytes;
  // two entries each: k_full, k_empty, v_full, v_empty, s_full
  const uint32_t q_full = bars, k_full = bars + 8, k_empty = bars + 24, v_full = bars + 40, v_empty = bars + 56,
                 s_full = bars + 72, p_full = bars + 88, p_empty = bars + 96, tmem_slot = bars + 104;
  uint32_t* tmem_slot_ptr = reinterpret_cast<uint32_t*>(smem + (tmem_slot - q_s));
  volatile int* abort_flag = reinterpret_cast<int*>(tmem_slot_ptr + 2);     // in dynamic memory: all of it is spoken for

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tile = blockIdx.x, head = blockIdx.y;
  const int tok0 = p.tiles[tile], ntok = p.tiles[p.num_tiles + tile], pos0 = p.tiles[2 * p.num_tiles + tile];
  const int lo = p.window > 0 ? max(0, pos0 - p.window + 1) : 0, hi = pos0 + ntok - 1;
  const int row0 = p.tiles[3 * p.num_tiles + tile] + lo - p.tiles[4 * p.num_tiles + tile];     // row of position lo
  const int ntiles = ((hi - lo) >> 7) + 1;

  if (threadIdx.x == 0) {
    *abort_flag = 0;
    for (int i = 0; i < 11; ++i) mbar_init(bars + 8 * i, 1);
    mbar_init(p_full, 128);
    mbar_init(p_empty, 1);
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
  pdl_trigger();
  pdl_wait();

  if (warp == 0) {
    if (elect_one()) {
      mbar_expect_tx(q_full, kbytes);
      for (int s = 0; s < ds; ++s) tma_load_2d(q_s + s * kSlabBytes, &p.map_q, head * p.dp + s * 64, tok0, q_full);
      for (int j = 0; j < ntiles && !*abort_flag; ++j) {
        const int st = j % nst;
        if (j >= nst && !mbar_wait(k_empty + 8 * st, (uint32_t)((j / nst - 1) & 1), kLpWaitNs, p.status)) { *abort_flag = 1; break; }
        mbar_expect_tx(k_full + 8 * st, kbytes);
        for (int s = 0; s < ds; ++s)
          tma_load_2d(k_s + st * kbytes + s * kSlabBytes, &p.map_kv, head * p.dp + s * 64, row0 + j * 128, k_full + 8 * st);
      }
    }
  } else if (warp == 6) {
    if (elect_one()) {
      for (int j = 0; j < ntiles && !*abort_flag; ++j) {
        const int st = j % nst;
        if (j >= nst && !mbar_wait(v_empty + 8 * st, (uint32_t)((j / nst - 1) & 1), kLpWaitNs, p.status)) { *abort_flag = 1; break; }
        mbar_expect_tx(v_full + 8 * st, vbytes);
        for (int s = 0; s < vs; ++s)
          tma_load_2d(v_s + st * vbytes + s * kSlabBytes, &p.map_kv, p.v_col + head * p.vp + s * 64, row0 + j * 128, v_full + 8 * st);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      const uint32_t idesc_s = idesc_f16_bf16(128, 128), idesc_o = idesc_f16_bf16_bmn(128, p.vp);
      auto issue_qk = [&](int j) {
        const uint32_t d = tmem_base + (uint32_t)(j & 1) * 128u, kb = k_s + (j % nst) * kbytes;
        for (int s = 0; s < ds; ++s)
#pragma unroll
          for (int ks = 0; ks < 4; ++ks)
            umma_bf16(d, smem_desc_sw128(q_s + s * kSlabBytes + ks * 32), smem_desc_sw128(kb + s * kSlabBytes + ks * 32), idesc_s,
                      (s | ks) ? 1u : 0u);
        umma_commit(k_empty + 8 * (j % nst));
        umma_commit(s_full + 8 * (j & 1));
      };
      bool ok = mbar_wait(q_full, 0, kLpWaitNs, p.status) && mbar_wait(k_full, 0, kLpWaitNs, p.status);
      if (ok) {
        tc_fence_after();
        issue_qk(0);
      }
      for (int j = 0; j < ntiles && ok && !*abort_flag; ++j) {
        if (j + 1 < ntiles) {
          ok = mbar_wait(k_full + 8 * ((j + 1) % nst), (uint32_t)(((j + 1) / nst) & 1), kLpWaitNs, p.status);
          if (!ok) break;
          tc_fence_after();
          issue_qk(j + 1);
        }
        ok = mbar_wait(p_full, (uint32_t)(j & 1), kLpWaitNs, p.status) &&
             mbar_wait(v_full + 8 * (j % nst), (uint32_t)((j / nst) & 1), kLpWaitNs, p.status);
        if (!ok) break;
        tc_fence_after();
        const uint32_t vb = v_s + (j % nst) * vbytes;
#pragma unroll
        for (int g = 0; g < 8; ++g)                          // 16 keys each
          umma_bf16(tmem_base + 256u, smem_desc_sw128(p_s + (g >> 2) * kSlabBytes + (g & 3) * 32),
                    smem_desc_mn128(vb + g * 2048, kSlabBytes), idesc_o, (j | g) ? 1u : 0u);
        umma_commit(v_empty + 8 * (j % nst));
        umma_commit(p_empty);
      }
      if (!ok) *abort_flag = 1;
    }
  } else {
    const int quarter = warp & 3;
    const int r = quarter * 32 + lane;
    const bool valid = r < ntok;
    const int pos = pos0 + (valid ? r : ntok - 1);
    const int wlo = p.window > 0 ? pos - p.window + 1 : 0;
    const uint32_t lane_base = tmem_base + ((uint32_t)(quarter * 32) << 16);
    float m_used = p.sink == nullptr ? kLpMask : p.sink[head] * 1.4426950408889634f;
    float l = p.sink == nullptr ? 0.f : 1.f;
    bool ok = true;
    for (int j = 0; j < ntiles; ++j) {
      ok = ok && !*abort_flag && mbar_wait(s_full + 8 * (j & 1), (uint32_t)((j >> 1) & 1), kLpWaitNs, p.status);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      tc_fence_after();
      const uint32_t s_addr = lane_base + (uint32_t)(j & 1) * 128u;
      const int key0 = lo + j * 128;
      uint32_t v[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32(s_addr + c * 32, v[c]);
      tmem_ld_wait();
      if (key0 + 127 > pos || key0 < wlo) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const int key = key0 + c * 32 + i;
            if (key > pos || key < wlo) v[c][i] = __float_as_uint(kLpMask);
          }
      }
      float mx = kLpMask;
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) mx = fmaxf(mx, __uint_as_float(v[c][i]));
      const float m_new = fmaxf(m_used, mx * p.scale_log2e);
      const bool resc = m_new - m_used > kLpGap;
      float alpha = 1.f;
      if (resc) {
        alpha = ex2(m_used - m_new);
        l *= alpha;
        m_used = m_new;
      }
      // P buffer free and O quiescent: the previous tile's P V has completed
      if (j > 0) {
        ok = mbar_wait(p_empty, (uint32_t)((j - 1) & 1), kLpWaitNs, p.status);
        ok = __all_sync(0xffffffffu, ok);
        if (!ok) break;
        tc_fence_after();
        if (__any_sync(0xffffffffu, resc)) {
#pragma unroll 1
          for (int c = 0; c < p.vp / 32; ++c) {
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
      float sum = 0.f;
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t pk[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float p0 = ex2(fmaf(__uint_as_float(v[c][i]), p.scale_log2e, -m_used));
          const float p1 = ex2(fmaf(__uint_as_float(v[c][i + 1]), p.scale_log2e, -m_used));
          sum += p0 + p1;
          pk[i >> 1] = pack_bf16(p0, p1);
        }
        const uint32_t row_addr = p_s + (uint32_t)(c >> 1) * kSlabBytes + (uint32_t)r * 128u;
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
    if (ok) {
      ok = mbar_wait(p_empty, (uint32_t)((ntiles - 1) & 1), kLpWaitNs, p.status);
      ok = __all_sync(0xffffffffu, ok);
    }
    if (ok) {
      tc_fence_after();
      const size_t tok = (size_t)tok0 + (valid ? r : 0);
      const float gv = p.gate == nullptr ? 1.f : sigmoid_f(__bfloat162float(p.gate[tok * p.ldg + p.gcol + head]));
      const float f = gv / l;
      __nv_bfloat16* dst = p.out + tok * (size_t)p.ldo + (size_t)head * p.vp;
#pragma unroll 1
      for (int c = 0; c < p.vp / 32; ++c) {
        uint32_t o[32];
        tmem_ld32(lane_base + 256u + c * 32, o);
        tmem_ld_wait();
        if (valid) {
#pragma unroll
          for (int q4 = 0; q4 < 4; ++q4) {
            uint32_t w[4];
#pragma unroll
            for (int e = 0; e < 4; ++e)
              w[e] = pack_bf16(__uint_as_float(o[q4 * 8 + 2 * e]) * f, __uint_as_float(o[q4 * 8 + 2 * e + 1]) * f);
            *reinterpret_cast<uint4*>(dst + c * 32 + q4 * 8) = make_uint4(w[0], w[1], w[2], w[3]);
          }
        }
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

}  // namespace ti

extern "C" {

// out[t, h] = softmax(scale q.k over the window, sink in the denominator) v * sigmoid(gate) for the tokens of the listed
// query tiles.  q: bf16 [T, ldq], head h at column h * dp; kv: bf16 [Nk, ldkv] expanded rows, keys of head h at column
// h * dp, values at column v_col + h * vp.  Rows of a sequence are consecutive positions.
int ti_latent_prefill(const void* q, int T, int ldq, const void* kv, int Nk, int ldkv, const void* tiles, int num_tiles,
                      const void* sink, const void* gate, int ldg, int gcol, void* out, int ldo, int H, int dp, int vp,
                      int v_col, int window, float scale, void* status, void* stream) {
  if (num_tiles <= 0) return 0;
  if (dp % 64 || vp % 64 || dp < 64 || vp < 64 || dp > 256 || vp > 256 || ldq % 8 || ldkv % 8 || ldo % 8 || v_col % 8 || H < 1 ||
      T < 1 || Nk < 1 || window < 0 || H * dp > ldq || v_col + H * vp > ldkv ||
      (((uintptr_t)q | (uintptr_t)kv | (uintptr_t)out) & 15))
    return -2;
  ti::LatentPrefillParams p = {};
  int rc = ti::bf16_map_2d(&p.map_q, q, ldq, T, 64, 128, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  rc = ti::bf16_map_2d(&p.map_kv, kv, ldkv, Nk, 64, 128, CU_TENSOR_MAP_SWIZZLE_128B);
  if (rc) return rc;
  p.tiles = (const int*)tiles;
  p.sink = (const float*)sink;
  p.gate = (const __nv_bfloat16*)gate;
  p.out = (__nv_bfloat16*)out;
  p.status = (unsigned*)status;
  p.num_tiles = num_tiles;
  p.dp = dp; p.vp = vp; p.v_col = v_col; p.ldg = ldg; p.gcol = gcol; p.ldo = ldo; p.window = window;
  p.stages = ti::latent_prefill_smem(dp, vp, 2) <= 227 * 1024 ? 2 : 1;
  p.scale_log2e = scale * 1.4426950408889634f;
  // one CTA per SM: each takes all 512 TMEM columns, so two must never share one
  size_t smem = ti::latent_prefill_smem(dp, vp, p.stages);
  if (smem < 120 * 1024) smem = 120 * 1024;
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(ti::latent_prefill_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024);
    configured = true;
  }
  ti::launch_kernel(ti::latent_prefill_kernel, dim3(num_tiles, H), dim3(ti::kLpThreads), smem, (cudaStream_t)stream, true, p);
  return (int)cudaGetLastError();
}

}  // extern "C"
