// Retention (retention.cu): linear attention with one fixed decay per head; arguments and launchers.
#pragma once
#include "common.cuh"

namespace cb {

constexpr int RET_T = 64;   // tokens per chunk of a multi-token step

struct RetentionArgs {
  // projections, one row of ld floats per (sequence, token): q, k (H heads of Dp) and v, gate (H heads of Ep) at these columns;
  // a multi-token step rotates q and k in place
  float *y = nullptr;
  PartIn pin;                       // single-token steps: the projections may still be split-K partial tiles
  int64_t ld = 0;
  int q_off = 0, k_off = 0, v_off = 0, g_off = 0;
  const float *freq = nullptr;      // [rot_pairs]: dims i and i + rot_pairs turn by position * freq[i]
  int rot_pairs = 0;
  float kscale = 1.0f;              // factor of k
  const float *powers = nullptr;    // [H, RET_T + 1]: decay^0, decay^1, ...
  float *state = nullptr;           // [B, H, Dp, Ep] (key, value)
  float *out = nullptr;             // normed and gated [B * s, out_ld], head h at column h * Ep: fp32, or
  BfOut bf;                         // bf16
  int64_t out_ld = 0;
  float *o = nullptr;               // [B * s, H * Ep]: raw outputs of a multi-token step (values wider than 256 only)
  int B = 0, s = 0, n = 0;          // s tokens per sequence at positions n ..
  const int *d_n = nullptr;         // single-token steps: position on the device
  int H = 0, D = 0, Dp = 0, E = 0, Ep = 0;
  float eps = 0.0f;
};

// Multi-token step: rotation, then the recurrence in chunks, the heads' norm and the gate.
int launch_retention_prep(caten_b200_ctx *ctx, const RetentionArgs &a);
int launch_retention_chunks(caten_b200_ctx *ctx, const RetentionArgs &a);
// Single-token step in one kernel.
int launch_retention_decode(caten_b200_ctx *ctx, const RetentionArgs &a);

}  // namespace cb
