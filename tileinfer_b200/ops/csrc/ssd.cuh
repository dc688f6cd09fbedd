// Parameters of the state-space mixer (one decay per head and token), shared by the token-serial and the chunked kernels.
#pragma once
#include "row_vec.cuh"

namespace ti {

struct SsdParams {
  const void* xbc;         // [T, ldx]: x (H heads of vp), B and C (G groups of Np each) after convolution and activation
  const void* proj;        // [T, ld]: z (H heads of vp) at z_col, step sizes (H) at dt_col
  const float* dt_bias;    // [H]
  const float* neg_a;      // [H] -exp(A_log)
  const float* D;          // [H]
  const float* norm;       // [H * vp] weights of the group norm (0 in the padding), times the output's factor
  float* state;            // [slots][H][Np][vp]
  const int* slots;        // [S]
  const int* cu;           // [S + 1] token offsets, or null: one token per sequence
  const int* seqs;         // sequences the token-serial kernel takes, or null: all
  float* y;                // [T][H * vp]
  void* out;               // [T][ldo] gated and normed outputs, head h at column h * vp
  const int* snap_rel;     // [S][num_snap] tokens of the step after which a state is copied (<= 0: unused)
  const int* snap_idx;     // [S][num_snap] entry of `snap`
  float* snap;             // [entries][H][Np][vp]
  int ldx, ld, ldo, x_col, b_col, c_col, z_col, dt_col, H, G, V, vp, num_snap, norm_groups;
  float eps;
  // chunked form: chunks of a sequence are consecutive and in order
  const int* ck_seq;       // [nc]
  const int* ck_tok0;      // [nc] first flat token
  const int* ck_ntok;      // [nc]
  const int* ck_snap;      // [nc] entry of `snap` written after the chunk, or -1
  const int* long_seq;     // [num_long] sequences that run in chunks
  const int* long_ck;      // [num_long + 1] their chunk ranges
  float* g_ws;             // [nc][H][2][C] running log2 decay inside the chunk, step sizes
  float* s_ws;             // [nc][H][Np][vp] what the chunk adds to the state, then the state before it
  int nc, num_long;
};

// softplus(dt + bias) of head h; `row`: the token's projection
template <typename T>
TI_DEVICE float ssd_step_size(const SsdParams& p, const T* row, int h) {
  const float z = to_f<T>(row[p.dt_col + h]) + p.dt_bias[h];
  return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z)));
}

}  // namespace ti
