// Grouped-query attention over a ring-buffered cache, optionally limited to a sliding window
// (attn_window.cu, attention_tc.cu): arguments and launchers.
#pragma once
#include "common.cuh"

namespace cb {

struct AttnArgs {
  // projections, one row per (sequence, token): H query heads of Dp, G key heads of Dp, G value heads of Ep floats at
  // these column offsets, and (gate_off >= 0) one output-gate logit per query head
  float *qkv = nullptr;
  int64_t ld = 0, q_off = 0, k_off = 0, v_off = 0, gate_off = -1;
  PartIn pin;                       // single-token steps: the projections may still be split-K partial tiles
  // caches [B, G, cap, Dp] and [B, G, cap, Ep]; position p lives in slot p % cap
  float *kc = nullptr, *vc = nullptr;
  int64_t cap = 0;
  // multi-token steps may find keys and values elsewhere: floats between positions, key/value heads and sequences (ld 0: the
  // caches as above), and the key's columns from kx_from on in rows kx [B, cap, kx_ld] common to the heads
  int64_t k_ld = 0, k_head = 0, k_seq = 0, v_ld = 0, v_head = 0, v_seq = 0;
  const float *kx = nullptr;
  int64_t kx_ld = 0;
  int kx_from = 0;
  float *out = nullptr;             // [B * s, out_ld], head h at column h * Ep: fp32, or
  BfOut bf;                         // bf16
  int64_t out_ld = 0;
  int B = 0, s = 0, n = 0;          // s tokens per sequence at positions n ..
  const int *d_n = nullptr;         // single-token steps: position on the device
  int H = 0, G = 0;
  int D = 0, Dp = 0, E = 0, Ep = 0; // query/key and value head sizes, and their padded storage (zeros, multiples of 16)
  int window = 0;                   // a query sees itself and the window - 1 tokens before it; 0: all of them
  int rot_pairs = 0;                // the first 2 * rot_pairs dims are rotated as interleaved pairs by position * freq[pair]
  const float *freq = nullptr;
  int qk_norm = 0;                  // q and k divided by their root mean square over D after the rotation
  float eps = 0.0f, scale = 1.0f;   // score = q . k * scale

  void fill_strides() {
    if (k_ld == 0) { k_ld = Dp; k_head = cap * Dp; k_seq = G * k_head; }
    if (v_ld == 0) { v_ld = Ep; v_head = cap * Ep; v_seq = G * v_head; }
    if (!kx) kx_from = Dp;
  }
};

// Rotation and q/k norm of a multi-token step: q in place (times scale), k and v into the cache.
int launch_attn_prep(caten_b200_ctx *ctx, const AttnArgs &a);
// Attention of a multi-token step on prepared q (launch_attn_prep); tensor cores when asked for and head sizes allow.
int launch_attn_window_prefill(caten_b200_ctx *ctx, const AttnArgs &a, int tensor_cores);
// Single-token step: rotation, q/k norm, cache append, attention and output gate in one kernel.
int launch_attn_window_decode(caten_b200_ctx *ctx, const AttnArgs &a);
// Tensor-core kernel (attention_tc.cu): Dp, Ep <= 128.  q is multiplied by qscale as it is loaded.
int launch_attention_tc_ex(caten_b200_ctx *ctx, const AttnArgs &a, float qscale);

}  // namespace cb
