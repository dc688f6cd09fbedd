// Parameters and the decay of gated linear attention, shared by the token-serial and the chunked kernels.
#pragma once
#include "row_vec.cuh"

namespace ti {

struct GlaParams {
  const void* proj;        // [T, ld]: columns of q, k (H heads of dk), v and gate (H heads of dv), inner product of the decay
  const float* a2;         // [R][H * dk] second matrix of the decay, transposed
  const float* a2_bias;    // [H * dk]
  const float* norm;       // [dv]
  float* state;            // [slots][H][dk][dv]
  const int* slots;        // [S]
  const int* cu;           // [S + 1] token offsets, or null: one token per sequence
  const int* seqs;         // sequences the token-serial kernel takes, or null: all
  float* o;                // [T][H * dv] un-normalised outputs
  void* out;               // [T][ldo] gated outputs, head h at column h * dv
  const int* snap_rel;     // [S][num_snap] tokens of the step after which a state is copied (<= 0: unused)
  const int* snap_idx;     // [S][num_snap] entry of `snap`
  float* snap;             // [entries][H][dk][dv]
  int ld, ldo, H, R, q_col, k_col, v_col, g_col, a_col, num_snap, vdim;
  float q_scale, inv_tau, eps;
  // chunked form: chunks of a sequence are consecutive and in order
  const int* ck_seq;       // [nc]
  const int* ck_tok0;      // [nc] first flat token
  const int* ck_ntok;      // [nc]
  const int* ck_snap;      // [nc] entry of `snap` written after the chunk, or -1
  const int* long_seq;     // [num_long] sequences that run in chunks
  const int* long_ck;      // [num_long + 1] their chunk ranges
  float* g_ws;             // [nc][H][C][dk] running log2 decay inside the chunk
  float* s_ws;             // [nc][H][dk][dv] what the chunk adds to the state, then the state before it
  int nc, num_long;
};

// log sigmoid(z)^(1/tau) of one key channel (column c of H * dk = n), z = a2 . inner + bias
template <typename T>
TI_DEVICE float gla_log_decay(const GlaParams& p, const T* row, int c, int n) {
  float z = p.a2_bias[c];
  for (int r = 0; r < p.R; ++r) z = fmaf(to_f<T>(row[p.a_col + r]), __ldg(p.a2 + (size_t)r * n + c), z);
  return (fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * p.inv_tau;
}

}  // namespace ti
