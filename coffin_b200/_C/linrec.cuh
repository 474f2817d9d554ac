// Arguments shared by the recurrent-state kernels (linrec.cu: token by token; linrec_chunk.cu: prompts in chunks; ssd.cu: both for state-space layers).
#pragma once
#include "act_type.cuh"

enum LinrecKind : int { LINREC_DELTA = 0, LINREC_MLSTM = 1, LINREC_GATED = 3 };      // state-space layers (ssd.cu, 2) have entry points of their own

// Column layout of a projection row: q | k | v | ... ; the first ring_w columns pass the short convolution of the delta
// and state-space layers (channel index == column index).  State-space layers: q = C, k = B, v = x.
struct LinrecArgs {
  // rows
  const void* proj; int64_t ldp;        // q, k, v (and gate / low-rank) columns
  const float* gates; int64_t ldg;      // fp32 gate pre-activations: delta b[H]; mLSTM i[H] | f[H]; ssd dt[H]; gated f[H * dk]
  const float* dec; int64_t ldd;        // delta, optional: decay pre-activations [H * dk] (before dt_bias)
  const void* og; int64_t ldo;          // output-gate pre-activations [H * dv] (null: delta computes them from g1 / g2)
  void* act; int64_t lda;               // result rows [H * dv] (ssd: always fp32, before gate and norm)
  // segments: rows [seg_row[s], seg_row[s + 1]) are consecutive tokens of one sequence from position seg_pos[s],
  // whose state lives in slot seg_slot[s] (< 0: skip).  seg_row null: row s alone.
  const int* seg_row; const int* seg_pos; const int* seg_slot;
  // weights
  const float* conv_w; int taps;        // [conv_width, taps]
  const float* A_log; const float* dt_bias;
  const void* a2; int64_t ra; int64_t a1_col;   // [H * dk, ra]
  const void* g2; int64_t rg; int64_t g1_col;   // [H * dv, rg]
  const float* norm_w;                  // delta, gated [dv]; mLSTM [H * dv]
  const float* gate_b;                  // mLSTM: i.b[H] | f.b[H]; gated: f.b[H * dk]
  // state of this layer
  float* S; float* n; float* m;         // [slots, H, dk, dv], [slots, H, dk], [slots, H]
  void* ring; int ring_mask; int64_t ring_w;    // [slots, ring, ring_w]
  // sizes
  int H, G, dk, dv, jc;
  int64_t k_col, v_col;
  float eps, cap;
  const float* conv_b;                  // ssd: convolution bias [conv_width]
  const float* D;                       // ssd: [H], weight of the value itself in the read-out
  const float* lower;                   // gated: lower bounds of the forget gates [H * dk]
};
// forget gate of a channel with its lower bound, and what it lets in: 1 - f without the cancellation
__device__ __forceinline__ float forget(float z, float low, float* keep_out) {
  const float e = expf(-fabsf(z)), s = 1.f / (1.f + e), c = e * s;         // sigmoid of |z| and of -|z|
  *keep_out = (1.f - low) * (z >= 0.f ? c : s);
  return low + (1.f - low) * (z >= 0.f ? s : c);
}
