// Latent attention (latent.cu): queries, keys and values of all heads come from low-rank latents, and the cache
// holds one normed latent and one rotated key part per token.  Arguments and launchers.
#pragma once
#include "common.cuh"

namespace cb {

struct LatentArgs {
  int H = 0, D = 0, Dp = 0, P = 0, Pp = 0, E = 0, Ep = 0;   // heads; unrotated and rotated query/key dims, value dims, and their storage (p16)
  int K = 0, Kp = 0, Kr = 0;        // latent size, its storage in the cache (p16) and as a linear's input (p64)
  int Q = 0, Qr = 0;                // query latent size, and as a linear's input (p64)
  const float *freq = nullptr;      // [P / 2]: rotated dims i and i + P / 2 turn by position * freq[i]
  const float *q_norm = nullptr, *kv_norm = nullptr;   // [Qr], [Kp] gains of the latents (zero in the padding)
  float eps = 0.0f, scale = 1.0f;   // score = (q . k) * scale
  // cache of `cap` rows per sequence: latent (Kp), rotated key part (Pp).  fp32, or bf16, row after row; or (tiled, bf16, at most 576
  // columns, cap a multiple of 128) tiles of 128 rows laid out as the shared-memory operand tiles of the decode kernel: blocks
  // of 64 columns, rows of 128 bytes with the 128-byte swizzle; a last block that holds up to 32 columns of the key part alone has
  // rows of 64 bytes with the 64-byte swizzle
  void *cache = nullptr;
  bool cache_bf16 = false, tiled = false;
  int64_t cap = 0;
  int B = 0, s = 0, n = 0;          // s tokens per sequence at positions n ..
  const int *d_n = nullptr;         // single-token steps: position on the device

  __host__ __device__ int KC() const { return Kp + Pp; }
  int Dq() const { return Dp + Pp; }
  __host__ __device__ int blocks() const { return (KC() + 63) / 64; }
  __host__ __device__ bool narrow() const { return KC() % 64 != 0 && KC() % 64 <= 32 && (KC() / 64) * 64 >= Kp; }
  __host__ __device__ int tile_elems() const { return blocks() * 128 * 64 - (narrow() ? 128 * 32 : 0); }
  __host__ __device__ int64_t seq_elems() const { return tiled ? cap / 128 * tile_elems() : cap * KC(); }
  // where column c of a sequence's row is; 8 columns from a multiple of 8 on are contiguous
  __host__ __device__ int64_t at(int64_t seq, int64_t row, int c) const {
    if (!tiled) return (seq * cap + row) * KC() + c;
    const int r = (int)(row & 127), b = c >> 6, chunk = (c & 63) >> 3;
    const int64_t tile = seq * seq_elems() + (row >> 7) * tile_elems() + b * 8192 + (c & 7);
    if (narrow() && b == blocks() - 1) return tile + r * 32 + ((chunk ^ ((r >> 1) & 3)) << 3);
    return tile + r * 64 + ((chunk ^ (r & 7)) << 3);
  }
};

// Rows of the projection [query latent (Qr) | latent (Kp) | key part (Pp)] (y, or its split-K partial tiles): the normed query
// latent [rows, Qr] as the next linear's input, the normed latent and the rotated key part into the cache.
int launch_latent_prep(caten_b200_ctx *ctx, const LatentArgs &a, const float *y, PartIn pin, int64_t ld, float *cq, BfOut cq_bf);
// Queries [rows, ld], head h at column h * Dq, for the expanded form: rotated and scaled in place.
int launch_latent_q_expanded(caten_b200_ctx *ctx, const LatentArgs &a, float *q, int64_t ld);
// Queries (or their partial tiles) for the absorbed form: unrotated parts as planes [H][plane][p64(D)] (input of the product with
// W_uk^T), rotated parts into qcat [rows, H, Kp + Pp] from column Kp on.
int launch_latent_q_absorbed(caten_b200_ctx *ctx, const LatentArgs &a, const float *q, PartIn pin, int64_t ld, int64_t plane, float *qn, BfOut qn_bf,
                             float *qcat, BfOut qcat_bf);
// The same and the product with W_uk^T (BF16 [H * Kp, p64(D)]) in one kernel, into all of qcat; with launch_latent_down for
// the rows of latent_fused, above which the per-head products are better off on the tensor cores.
inline bool latent_fused(const LatentArgs &a, int64_t rows) { return rows <= (a.Kr <= 128 ? 256 : 32); }
int launch_latent_up(caten_b200_ctx *ctx, const LatentArgs &a, const caten_b200_weight *uk, const float *q, PartIn pin, int64_t ld, float *qcat, BfOut qcat_bf);
// Cached rows [0, t) of sequences b0 .. b0 + nb: latents [nb * t, Kr] as a linear's input, key parts [nb * t, Pp] in fp32.
int launch_latent_gather(caten_b200_ctx *ctx, const LatentArgs &a, int b0, int nb, int t, float *c, BfOut c_bf, float *kr);

struct LatentAbsorbed {
  const float *qcat = nullptr;      // [rows, H, Kp + Pp] fp32, or
  BfOut qcat_bf;                    // bf16
  float *o = nullptr;               // planes [H][plane][Kr]: sum_j p_j c_j per head; fp32, or
  BfOut o_bf;                       // bf16
  int64_t plane = 0;
  float *part = nullptr, *ml = nullptr;   // several splits: [splits, rows, H, Kr] and [splits, rows, H, 2]
  int splits = 1;
  bool combine = true;              // several splits: merge the parts into the planes (otherwise launch_latent_down does)
  bool early = false;               // cache and position are complete before the kernel in front of this one starts
};
// Key splits of a launch over `rows` rows that may see `keys` keys.
int latent_splits(const caten_b200_ctx *ctx, const LatentArgs &a, int64_t rows, int64_t keys);
// Softmax attention of every row (sequence, token) over its cached latents.
int launch_latent_absorbed(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x);
// Its result, in fp32 planes or still in parts, times W_uv (BF16 [H * Ep, Kr]) per head: out [rows, ld], head h at column h * Ep.
int launch_latent_down(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x, const caten_b200_weight *uv, float *out, BfOut bf, int64_t ld);

}  // namespace cb
