// Parameters of the delta rules, shared by the token-serial and the chunked kernels.
//
// Both rules are one recurrence per head on a state S [dk, dv], with a unit key u_t = k_t / sqrt(sum k_t^2 + 1e-6):
//     S_t = diag(w_t) S_(t-1) - p_t (u_t^T S_(t-1)) + c_t v_t^T          o_t = S_t^T q_t
//   gated:    one decay g_t = exp(-exp(A) softplus(a_t + dt)) and one step beta_t = sigmoid(b_t) per head;
//             w = g, p = beta g u, c = beta u, q a unit vector times q_scale; heads share keys and queries in groups
//   general:  a decay w_t = exp(-scale sigmoid(W_2 tanh(x_t) + w_0)) and a removal rate a_t = sigmoid(. + bias) per key
//             channel; p = a u, c = k as projected, q as projected
#pragma once
#include "row_vec.cuh"

namespace ti {

constexpr float kUnitEps = 1e-6f;        // inside the root of a unit vector's length

struct DeltaParams {
  const void* src;         // [T, lds]: queries at q_col, keys at k_col (H / rep heads of dk), values at v_col (H heads of dv)
  const void* proj;        // [T, ld]: gated: b_t at b_col, a_t at a_col; general: removal logits at b_col, x_t at a_col
  const float* bias;       // gated: [H] added to a_t; general: [H * dk] added to the removal logits
  const float* neg_a;      // gated: [H] -exp(A)
  const float* w2;         // general: [R][H * dk] second matrix of the decay, transposed
  const float* w0;         // general: [H * dk]
  float* state;            // [slots][H][dk][dv]
  const int* slots;        // [S]
  const int* cu;           // [S + 1] token offsets, or null: one token per sequence
  const int* seqs;         // sequences the token-serial kernel takes, or null: all
  float* o;                // [T][H * dv]
  const int* snap_rel;     // [S][num_snap] tokens of the step after which a state is copied (<= 0: unused)
  const int* snap_idx;     // [S][num_snap] entry of `snap`
  float* snap;             // [entries][H][dk][dv]
  int lds, ld, H, rep, R, q_col, k_col, v_col, b_col, a_col, num_snap;
  float q_scale, decay_scale;
  // chunked form: chunks of a sequence are consecutive and in order
  const int* ck_seq;       // [nc]
  const int* ck_tok0;      // [nc] first flat token
  const int* ck_ntok;      // [nc]
  const int* ck_snap;      // [nc] entry of `snap` written after the chunk, or -1
  const int* long_seq;     // [num_long] sequences that run in chunks
  const int* long_ck;      // [num_long + 1] their chunk ranges
  uint4* t_ws;             // [nc][H] what a chunk takes off the state, as a matrix (fragments, two bf16 terms)
  uint4* q_ws;             // [nc][H] queries against the state before the chunk (fragments, two bf16 terms)
  float4* s_ws;            // [nc][H][dk * dv / 4] what a chunk adds to the state; then the state before it (fragments)
  float* f_ws;             // [nc][H][dk] decay over a chunk
  int nc, num_long;
};

TI_DEVICE float softplus_exact(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }

}  // namespace ti
