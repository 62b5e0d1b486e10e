// Time mixing with a per-head matrix state and a per-channel, input-dependent decay (wkv.cu).
#pragma once
#include "common.cuh"

namespace cb {

struct WkvArgs {
  // projections, one row of ld floats per (sequence, token): r, k, v, gate (H heads of Dp each) and the decay's
  // low-rank input (w1 floats) at columns 0, gr, 2 gr, 3 gr, 4 gr
  const float *y = nullptr;
  PartIn pin;                       // single-token steps: the projections may still be split-K partial tiles
  int64_t ld = 0;
  int gr = 0, w1 = 0;
  // multi-token steps: the decay's second projection, tanh(low rank) . W2 + w0 (one row of d_ld floats per token;
  // overwritten)
  float *d = nullptr;
  int64_t d_ld = 0;
  // single-token steps form it themselves
  const __nv_bfloat16 *w2 = nullptr;  // [H * Dp, w1]
  const float *w0 = nullptr;          // [H * Dp]
  const float *u = nullptr;           // [H * Dp] bonus of the current token
  const float *norm = nullptr;        // [H * Dp] gain of the heads' norm
  float *state = nullptr;             // [B, H, Dp, Dp] (key, value)
  float *o = nullptr;                 // raw output of the recurrence [rows, o_ld]
  int64_t o_ld = 0;
  float *out = nullptr;               // normed and gated [rows, out_ld]: fp32, or
  BfOut bf;                           // bf16
  int64_t out_ld = 0;
  int B = 0, s = 0, n = 0;
  const int *d_n = nullptr;
  int H = 0, D = 0, Dp = 0;           // head size and its padded storage (zeros, a multiple of 16)
  float eps = 0.0f;
};

// tanh of the decay's low-rank input of every row, as the operand of its second projection; also moves the last
// token's h of every sequence into the carried token-shift state.
int launch_wkv_lowrank(caten_b200_ctx *ctx, const WkvArgs &a, float *t, BfOut tb, const float *h, float *shift, int width_p);
// Recurrence of a multi-token step (raw o), then the heads' norm and the gate.
int launch_wkv_scan(caten_b200_ctx *ctx, const WkvArgs &a);
// Single-token step in one kernel.
int launch_wkv_decode(caten_b200_ctx *ctx, const WkvArgs &a);

}  // namespace cb
