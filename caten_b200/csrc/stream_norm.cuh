// Residual-stream kernels (stream_norm.cu): arguments and launchers.
#pragma once
#include "common.cuh"

namespace cb {

enum { SN_EMBED = 0, SN_COPY = 1, SN_ADD = 2, SN_KEEP = 3, SN_SUM = 4 };       // how the stream's row is formed
enum { SN_NORM = 0, SN_SHIFT = 1, SN_CONCAT = 2, SN_NONE = 3, SN_NORM2 = 4 };    // what the next operation reads

struct StreamArgs {
  const float *y = nullptr;      // output of the sublayer's last linear [R, 4 * d4], or
  PartIn pin;                    // its split-K partial tiles
  const float *x = nullptr;      // the stream before
  float *x_out = nullptr;        // the stream after (may be x); NULL: not stored
  float *x0 = nullptr;           // the embedding output
  const __nv_bfloat16 *table = nullptr;  // token embedding [vocab, 4 * d4]
  const int64_t *ids = nullptr;  // row r = (sequence, token): ids[(r / s) * ids_ld + r % s]; an id outside [0, vocab) is a zero row
  int64_t ids_ld = 1, vocab = 0;
  int s = 1;
  float post = 1.0f, pre = 1.0f; // gains of the norm after the sublayer and of the one before the next
  float eps = 0.0f, invd = 0.0f; // 1 / width
  int d4 = 0;                    // padded width / 4
  // SN_SUM: also the outputs of the experts a row used, ye[pos[row * top + k]] (pos NULL: ye[row * top + k])
  const float *ye = nullptr;
  const int *pos = nullptr;
  int top = 0;
  // SN_NORM2: gains per coordinate (zero in the padding); w2 may be NULL
  const float *w1 = nullptr, *w2 = nullptr;
  // SN_NORM2: added to the row first (a pass of a loop starts): [4 * d4], and the embedding output with add_x0
  const float *step = nullptr;
  int add_x0 = 0;
  float *h = nullptr;            // operand of the next linear: fp32, or
  BfOut hb;                      // bf16
  const int *rows = nullptr;     // gather: output row i reads stream row rows[i]
  int64_t src_stride = 1;        // or row (i + 1) * src_stride - 1
  // SN_SHIFT
  const float *mu = nullptr;     // [5, 4 * d4] in the order r, k, v, g, w
  float *shift = nullptr;        // [rows, 4 * d4] the previous token's h
  int64_t plane = 0;             // rows between consecutive mixes (SN_SHIFT) or the two norms (SN_NORM2) in h / hb
  const int *d_n = nullptr;      // position on the device, or
  int n = 0;
};

int launch_stream_norm(caten_b200_ctx *ctx, int in, int out, const StreamArgs &a, int64_t rows);
int launch_token_shift(caten_b200_ctx *ctx, const float *h, const float *shift, const float *mu, int64_t B, int64_t s, int64_t n, int d4,
                       int64_t plane, float *out, BfOut ob);

}  // namespace cb
