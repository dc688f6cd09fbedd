// Parameters and key ranges shared by the kernels of attention over paged latents (latent_attn.cu, latent_decode.cu).
#pragma once
#include "common.cuh"

namespace ti {

typedef __nv_bfloat16 bf16;

struct LatentAttnParams {
  const void* q;                 // [T][H][Rp] absorbed queries
  const void* cache;             // [num_blocks][16][Rp]
  const int* block_tables;       // [S, max_blocks]
  const int* positions;          // [T]
  const int* qg_seq;             // [num_qg] sequence of the query token
  const int* qg_tok0;            // [num_qg] flat token
  const int* qg_ntok;            // [num_qg] 1, or 0: padding
  const float* sink;             // [H] or null
  float* o_part;                 // [num_qg * head groups * nsplit][rows][Rp]
  float* ml_part;                // [num_qg * head groups * nsplit][rows][2]
  void* out;                     // [T][H][Ro]
  unsigned* status;
  int H, R, Rp, max_blocks, nsplit, num_qg, window, num_blocks;
  float scale;
  int Ro;                        // leading columns of a cache row that are value as well as key (the others are key alone)
};

constexpr float kNeg = -1e30f;
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kMaxLatentSplit = 64;

struct KeyRange { int pos, lo, page0, npages, ntiles, tps; };

// keys of one query token: lo .. pos, walked in tiles of `tile` keys from the start of lo's page; tps tiles per split
TI_DEVICE KeyRange key_range(const LatentAttnParams& p, int tok, int tile) {
  KeyRange r;
  r.pos = p.positions[tok];
  r.lo = p.window > 0 ? max(0, r.pos - p.window + 1) : 0;
  r.page0 = r.lo >> 4;
  r.npages = (r.pos >> 4) + 1;
  r.ntiles = (r.pos - r.page0 * 16) / tile + 1;
  r.tps = (r.ntiles + p.nsplit - 1) / p.nsplit;
  return r;
}

// Splits -> output (latent_attn.cu); `rows` heads per block and `tile` keys per tile of the kernel that made the splits.
void launch_latent_merge(const LatentAttnParams& p, int rows, int tile, cudaStream_t st);
// The tcgen05 form (latent_decode.cu): bf16, Rp 256, 384, 512 or 576 (the last with Ro of at most 512).  Returns a cudaError_t or a negative code.
int launch_latent_decode_tc(const LatentAttnParams& p, cudaStream_t st);

}  // namespace ti
