// Latent attention.  Per token the cache holds c (a normed latent of K values) and r (one rotated key part of P values
// for all heads).  With q = [q_n, q_r] per head the scores are (q_n . W_uk c + q_r . r) * scale and the output is
// sum_j p_j W_uv c_j.  Two forms:
//   absorbed   (q_n W_uk) . c and W_uv (sum_j p_j c_j): the cache is read as it is, once for all heads of a CTA.  Decoding
//              and very short portions.
//   expanded   keys and values of all heads are formed from the cached latents by one linear and go through the
//              ordinary prompt attention (attention_tc.cu, attn_window.cu).  Longer portions.
//
// latent_attn_tc_kernel (bf16 models): tcgen05.  A CTA serves NH = 16 or 32 heads of one row; keys go in tiles of 128, and both
// products have the keys' or the latent's dims, not the heads, as the 128 lanes of tensor memory, so that few heads waste nothing:
//   warp 8      bulk copies: a tile of 128 cached rows, stored in device memory as the operand tiles it becomes (LatentArgs::cache), two
//               64-column blocks to a barrier.  The same blocks are the K-major A operand of S^T = C.Q^T and the MN-major A operand
//               of O^T += C^T.P^T
//   warps 9, 10 tcgen05.mma: one warp issues the scores of tile after tile, as soon as a tile has arrived and its score columns have
//               been read, the other the outputs.  With few heads a product takes less time than issuing it, so the two streams
//               of issues run side by side, and a tile is given back as soon as its output is formed
//   warps 0..7  one key and half of the heads per thread: a head's reference maximum moves lazily (as in attention_tc.cu: only when a
//               score exceeds it by LA_TAU; one vote per tile finds out), p = hi + lo in bf16 goes to shared memory as the 2 NH rows
//               of the second product's B operand (hi of all heads, then lo), so p keeps 16 bits; the two halves of O are added at
//               the end
// Keys may be split over CTAs; latent_combine_kernel then merges the parts.
// Every mbarrier wait is bounded: when one runs out the CTA records it in the status word, leaves its loops, waits for its
// copies in flight, frees tensor memory and writes no output.
#include "latent.cuh"
#include "tcgen05.cuh"

namespace cb {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ void st1(float *out, BfOut bf, int64_t at, float v) {
  if (bf.hi) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    bf.hi[at] = h;
    if (bf.lo) bf.lo[at] = __float2bfloat16_rn(v - __bfloat162float(h));
  } else {
    out[at] = v;
  }
}
__device__ __forceinline__ float ld_cache(const void *cache, bool bf16, int64_t at) {
  return bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16 *>(cache)[at]) : reinterpret_cast<const float *>(cache)[at];
}
__device__ __forceinline__ void st_cache(void *cache, bool bf16, int64_t at, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16 *>(cache)[at] = __float2bfloat16_rn(v);
  else reinterpret_cast<float *>(cache)[at] = v;
}

}  // namespace

// ---------------------------------------------------------------------------------------------
// Before and after the linears
// ---------------------------------------------------------------------------------------------
constexpr int LP_THREADS = 256;

__global__ void __launch_bounds__(LP_THREADS) latent_prep_kernel(const LatentArgs a, const float *__restrict__ y, const PartIn pin, int64_t ld,
                                                                 float *__restrict__ cq, BfOut cq_bf) {
  extern __shared__ __align__(16) float row[];   // [Qr + Kp + Pp]
  __shared__ float red[2][LP_THREADS / 32];
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int pos = (a.d_n ? *a.d_n : a.n) + (int)(r % a.s);
  const int cols = a.Qr + a.Kp + a.Pp;
  float sq = 0.0f, sc = 0.0f;   // (padding is zero)
  for (int c = 4 * tid; c < cols; c += 4 * LP_THREADS) {
    const float4 v = pin.splits > 0 ? partin_load4(pin, r, c) : *reinterpret_cast<const float4 *>(y + r * ld + c);
    *reinterpret_cast<float4 *>(row + c) = v;
    const float ss = (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
    if (c < a.Qr) sq += ss;
    else if (c < a.Qr + a.Kp) sc += ss;
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if (lane == 0) { red[0][warp] = sq; red[1][warp] = sc; }
  __syncthreads();
  sq = sc = 0.0f;
#pragma unroll
  for (int w = 0; w < LP_THREADS / 32; ++w) { sq += red[0][w]; sc += red[1][w]; }
  const float rq = 1.0f / sqrtf(sq / (float)a.Q + a.eps), rc = 1.0f / sqrtf(sc / (float)a.K + a.eps);
  for (int c = tid; c < a.Qr; c += LP_THREADS) st1(cq, cq_bf, r * a.Qr + c, row[c] * rq * a.q_norm[c]);
  const int64_t seq = r / a.s;
  const float *lat = row + a.Qr, *key = lat + a.Kp;
  for (int c = tid; c < a.Kp; c += LP_THREADS) st_cache(a.cache, a.cache_bf16, a.at(seq, pos, c), lat[c] * rc * a.kv_norm[c]);
  const int half = a.P / 2;
  for (int i = tid; i < a.Pp; i += LP_THREADS) {
    float v = 0.0f;
    if (i < a.P) {
      const int f = i < half ? i : i - half;
      float sn, cs;
      sincosf((float)pos * a.freq[f], &sn, &cs);
      v = i < half ? key[i] * cs - key[i + half] * sn : key[i] * cs + key[f] * sn;
    }
    st_cache(a.cache, a.cache_bf16, a.at(seq, pos, a.Kp + i), v);
  }
}

static int check_latent(caten_b200_ctx *ctx, const LatentArgs &a) {
  if (a.H <= 0 || a.D <= 0 || a.E <= 0 || a.K <= 0 || a.Q <= 0 || a.P < 0 || a.P % 2 || a.Dp % 16 || a.Pp % 16 || a.Ep % 16 || a.Kp % 16 || a.Kr % 64 || a.Qr % 64 || a.n < 0 || a.cap <= 0 ||
      (a.tiled && (!a.cache_bf16 || a.cap % 128)))
    return fail(ctx, CATEN_B200_EINVAL, "latent attention: bad shape");
  if (a.K > 1024 || a.P > 256 || a.Q > 8192 || a.H > 4096) return fail(ctx, CATEN_B200_EUNSUPPORTED, "latent attention: latent of %d or rotated part of %d", a.K, a.P);
  if (!a.d_n && (int64_t)a.n + a.s > a.cap) return fail(ctx, CATEN_B200_EINVAL, "latent attention: %lld tokens in a cache of %lld", (long long)a.n + a.s, (long long)a.cap);
  if ((int64_t)a.B * a.s > 0x7fffffff) return fail(ctx, CATEN_B200_EUNSUPPORTED, "latent attention: too many rows");
  return 0;
}

int launch_latent_prep(caten_b200_ctx *ctx, const LatentArgs &a, const float *y, PartIn pin, int64_t ld, float *cq, BfOut cq_bf) {
  if (int rc = check_latent(ctx, a)) return rc;
  const size_t smem = (size_t)(a.Qr + a.KC()) * sizeof(float);
  launch_k(ctx, latent_prep_kernel, dim3((unsigned)(a.B * a.s)), dim3(LP_THREADS), smem, a, y, pin, ld, cq, cq_bf);
  CB_LAUNCH_CHECK(ctx, "latent_prep_kernel");
  return 0;
}

// one CTA per row; a thread keeps one pair's angle for several heads
__global__ void __launch_bounds__(256) latent_q_expanded_kernel(const LatentArgs a, float *__restrict__ q, int64_t ld) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int pos = a.n + (int)(r % a.s), tid = threadIdx.x, half = a.P / 2, Dq = a.Dp + a.Pp;
  float *row = q + r * ld;
  const int d4 = a.Dp / 4;
  for (int i = tid; i < a.H * d4; i += 256) {
    float4 *x = reinterpret_cast<float4 *>(row + (int64_t)(i / d4) * Dq) + i % d4;
    *x = make_float4(x->x * a.scale, x->y * a.scale, x->z * a.scale, x->w * a.scale);
  }
  if (half == 0) return;
  const int lanes = 256 / half;   // (at least 2)
  const int i = tid % half;
  if (tid / half >= lanes) return;
  float sn, cs;
  sincosf((float)pos * a.freq[i], &sn, &cs);
  for (int h = tid / half; h < a.H; h += lanes) {
    float *x = row + (int64_t)h * Dq + a.Dp + i;
    const float u = x[0], v = x[half];
    x[0] = (u * cs - v * sn) * a.scale;
    x[half] = (v * cs + u * sn) * a.scale;
  }
}

int launch_latent_q_expanded(caten_b200_ctx *ctx, const LatentArgs &a, float *q, int64_t ld) {
  if (int rc = check_latent(ctx, a)) return rc;
  launch_k(ctx, latent_q_expanded_kernel, dim3((unsigned)(a.B * a.s)), dim3(256), 0, a, q, ld);
  CB_LAUNCH_CHECK(ctx, "latent_q_expanded_kernel");
  return 0;
}

// grid (row, part of the heads)
__global__ void __launch_bounds__(256) latent_q_absorbed_kernel(const LatentArgs a, const float *__restrict__ q, const PartIn pin, int64_t ld, int64_t plane,
                                                                int heads_per_cta, float *__restrict__ qn, BfOut qn_bf, float *__restrict__ qcat, BfOut qcat_bf) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int pos = (a.d_n ? *a.d_n : a.n) + (int)(r % a.s), tid = threadIdx.x, half = a.P / 2, Dq = a.Dp + a.Pp, KC = a.Kp + a.Pp;
  const int h0 = blockIdx.y * heads_per_cta, hn = min(heads_per_cta, a.H - h0);
  const int Dr = (a.Dp + 63) / 64 * 64, d4 = Dr / 4;
  for (int i = tid; i < hn * d4; i += 256) {
    const int h = h0 + i / d4, c = i % d4 * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < a.Dp) v = pin.splits > 0 ? partin_load4(pin, r, h * Dq + c) : *reinterpret_cast<const float4 *>(q + r * ld + (int64_t)h * Dq + c);
    const int64_t at = ((int64_t)h * plane + r) * Dr + c;
    if (qn_bf.hi) {
      *reinterpret_cast<uint2 *>(qn_bf.hi + at) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      if (qn_bf.lo) *reinterpret_cast<uint2 *>(qn_bf.lo + at) = make_uint2(pack_bf16(bf16_lo(v.x), bf16_lo(v.y)), pack_bf16(bf16_lo(v.z), bf16_lo(v.w)));
    } else {
      *reinterpret_cast<float4 *>(qn + at) = v;
    }
  }
  for (int i = tid; i < hn * a.Pp; i += 256) {
    const int h = h0 + i / a.Pp, j = i % a.Pp;
    float v = 0.0f;
    if (j < a.P) {
      const int f = j < half ? j : j - half;
      auto at = [&](int d) { const int c = h * Dq + a.Dp + d; return pin.splits > 0 ? partin_load1(pin, r, c) : q[r * ld + c]; };
      const float u = at(f), w = at(f + half);
      float sn, cs;
      sincosf((float)pos * a.freq[f], &sn, &cs);
      v = j < half ? u * cs - w * sn : w * cs + u * sn;
    }
    st1(qcat, qcat_bf, (r * a.H + h) * KC + a.Kp + j, v);
  }
}

int launch_latent_q_absorbed(caten_b200_ctx *ctx, const LatentArgs &a, const float *q, PartIn pin, int64_t ld, int64_t plane, float *qn, BfOut qn_bf,
                             float *qcat, BfOut qcat_bf) {
  if (int rc = check_latent(ctx, a)) return rc;
  const int rows = a.B * a.s;
  int per = a.H;   // enough CTAs for the GPU: a row's heads are split when there are few rows
  while (per > 1 && (int64_t)rows * ((a.H + per - 1) / per) < ctx->sm_count) per = (per + 1) / 2;
  launch_k(ctx, latent_q_absorbed_kernel, dim3((unsigned)rows, (unsigned)((a.H + per - 1) / per)), dim3(256), 0, a, q, pin, ld, plane, per, qn, qn_bf, qcat, qcat_bf);
  CB_LAUNCH_CHECK(ctx, "latent_q_absorbed_kernel");
  return 0;
}

// grid (head, 16 rows, 64 latent dims): the head's queries, rotated, and their product with W_uk^T.  Four neighbouring threads
// share a latent dim and take its row of weights in turn, 16 bytes each; the rows' queries are in shared memory.
constexpr int LU_ROWS = 16, LU_DIMS = 64, LU_AHEAD = 4;

__global__ void __launch_bounds__(256) latent_up_kernel(const LatentArgs a, const __nv_bfloat16 *__restrict__ uk, const float *__restrict__ q, const PartIn pin, int64_t ld,
                                                        int64_t rows, float *__restrict__ qcat, BfOut qcat_bf) {
  extern __shared__ __align__(16) float qs[];   // [LU_ROWS][Dp]
  const int h = blockIdx.x, tid = threadIdx.x, half = a.P / 2, Dq = a.Dp + a.Pp, KC = a.KC(), Dr = (a.Dp + 63) / 64 * 64;
  const int64_t r0 = (int64_t)blockIdx.y * LU_ROWS;
  const int rn = (int)(rows - r0 < LU_ROWS ? rows - r0 : LU_ROWS);
  const int k = blockIdx.z * LU_DIMS + (tid >> 2), part = tid & 3, nv = a.Dp / 8;
  const bool on = k < a.Kp;
  const uint4 *w = reinterpret_cast<const uint4 *>(uk + ((int64_t)h * a.Kp + (on ? k : 0)) * Dr);
  uint4 x[LU_AHEAD];   // the first weights depend on no other kernel
#pragma unroll
  for (int u = 0; u < LU_AHEAD; ++u) x[u] = on && part + 4 * u < nv ? w[part + 4 * u] : make_uint4(0u, 0u, 0u, 0u);
  pdl_enter();
  const int d4 = a.Dp / 4;
  for (int i = tid; i < LU_ROWS * d4; i += 256) {
    const int r = i / d4, c = i % d4 * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < rn) v = pin.splits > 0 ? partin_load4(pin, r0 + r, h * Dq + c) : *reinterpret_cast<const float4 *>(q + (r0 + r) * ld + (int64_t)h * Dq + c);
    *reinterpret_cast<float4 *>(qs + r * a.Dp + c) = v;
  }
  if (blockIdx.z == 0) {
    const int n = a.d_n ? *a.d_n : a.n;
    for (int i = tid; i < rn * a.Pp; i += 256) {
      const int r = i / a.Pp, j = i % a.Pp;
      float v = 0.0f;
      if (j < a.P) {
        const int f = j < half ? j : j - half;
        auto at = [&](int d) { const int c = h * Dq + a.Dp + d; return pin.splits > 0 ? partin_load1(pin, r0 + r, c) : q[(r0 + r) * ld + c]; };
        const float u = at(f), y = at(f + half);
        float sn, cs;
        sincosf((float)(n + (int)((r0 + r) % a.s)) * a.freq[f], &sn, &cs);
        v = j < half ? u * cs - y * sn : y * cs + u * sn;
      }
      st1(qcat, qcat_bf, ((r0 + r) * a.H + h) * KC + a.Kp + j, v);
    }
  }
  __syncthreads();
  float acc[LU_ROWS];
#pragma unroll
  for (int r = 0; r < LU_ROWS; ++r) acc[r] = 0.0f;
  for (int i0 = part; i0 < nv; i0 += 4 * LU_AHEAD) {
#pragma unroll
    for (int u = 0; u < LU_AHEAD; ++u) {
      const int d = 8 * (i0 + 4 * u);
      if (d >= a.Dp) continue;
      const uint32_t b[4] = {x[u].x, x[u].y, x[u].z, x[u].w};
      float f[8];
#pragma unroll
      for (int e = 0; e < 4; ++e) { f[2 * e] = __uint_as_float(b[e] << 16); f[2 * e + 1] = __uint_as_float(b[e] & 0xFFFF0000u); }
#pragma unroll
      for (int r = 0; r < LU_ROWS; ++r) {
        if (r < rn) {
          const float4 x0 = *reinterpret_cast<const float4 *>(qs + r * a.Dp + d), x1 = *reinterpret_cast<const float4 *>(qs + r * a.Dp + d + 4);
          acc[r] = fmaf(f[0], x0.x, fmaf(f[1], x0.y, fmaf(f[2], x0.z, fmaf(f[3], x0.w, acc[r]))));
          acc[r] = fmaf(f[4], x1.x, fmaf(f[5], x1.y, fmaf(f[6], x1.z, fmaf(f[7], x1.w, acc[r]))));
        }
      }
    }
    if (i0 + 4 * LU_AHEAD < nv) {
#pragma unroll
      for (int u = 0; u < LU_AHEAD; ++u) x[u] = on && i0 + 4 * (LU_AHEAD + u) < nv ? w[i0 + 4 * (LU_AHEAD + u)] : make_uint4(0u, 0u, 0u, 0u);
    }
  }
  // the four threads' sums: each exchange halves the rows a thread carries
  const bool hi2 = (tid & 2) != 0, hi1 = (tid & 1) != 0;
#pragma unroll
  for (int r = 0; r < 8; ++r) acc[r] = (hi2 ? acc[r + 8] : acc[r]) + __shfl_xor_sync(0xffffffffu, hi2 ? acc[r] : acc[r + 8], 2);
#pragma unroll
  for (int r = 0; r < 4; ++r) acc[r] = (hi1 ? acc[r + 4] : acc[r]) + __shfl_xor_sync(0xffffffffu, hi1 ? acc[r] : acc[r + 4], 1);
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = (hi2 ? 8 : 0) + (hi1 ? 4 : 0) + i;
    if (on && r < rn) st1(qcat, qcat_bf, ((r0 + r) * a.H + h) * KC + k, acc[i]);
  }
}

int launch_latent_up(caten_b200_ctx *ctx, const LatentArgs &a, const caten_b200_weight *uk, const float *q, PartIn pin, int64_t ld, float *qcat, BfOut qcat_bf) {
  if (int rc = check_latent(ctx, a)) return rc;
  const int64_t rows = (int64_t)a.B * a.s;
  if (rows <= 0) return 0;
  if (uk->type != CATEN_B200_BF16) return fail(ctx, CATEN_B200_EUNSUPPORTED, "latent attention: W_uk must be BF16");
  const size_t smem = (size_t)LU_ROWS * a.Dp * sizeof(float);
  launch_k(ctx, latent_up_kernel, dim3((unsigned)a.H, (unsigned)((rows + LU_ROWS - 1) / LU_ROWS), (unsigned)((a.Kp + LU_DIMS - 1) / LU_DIMS)), dim3(256), smem, a,
           (const __nv_bfloat16 *)uk->qs, q, pin, ld, rows, qcat, qcat_bf);
  CB_LAUNCH_CHECK(ctx, "latent_up_kernel");
  return 0;
}

// one warp per cached row
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentArgs a, int b0, int t, int64_t rows, float *__restrict__ c, BfOut c_bf, float *__restrict__ kr) {
  pdl_enter();
  const int64_t r = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int lane = threadIdx.x & 31;
  const int64_t seq = b0 + r / t, row = r % t;
  for (int j = 8 * lane; j < a.Kr; j += 256) {   // 8 columns a lane
    const int64_t to = r * a.Kr + j, from = a.at(seq, row, j);
    if (a.cache_bf16 && c_bf.hi) {
      *reinterpret_cast<uint4 *>(c_bf.hi + to) = j < a.Kp ? *reinterpret_cast<const uint4 *>(reinterpret_cast<const __nv_bfloat16 *>(a.cache) + from) : make_uint4(0u, 0u, 0u, 0u);
    } else {
      for (int e = 0; e < 8; ++e) st1(c, c_bf, to + e, j < a.Kp ? ld_cache(a.cache, a.cache_bf16, from + e) : 0.0f);
    }
  }
  for (int j = lane; j < a.Pp; j += 32) kr[r * a.Pp + j] = ld_cache(a.cache, a.cache_bf16, a.at(seq, row, a.Kp + j));
}

int launch_latent_gather(caten_b200_ctx *ctx, const LatentArgs &a, int b0, int nb, int t, float *c, BfOut c_bf, float *kr) {
  const int64_t rows = (int64_t)nb * t;
  if (rows <= 0) return 0;
  if (t > a.cap || b0 + nb > a.B) return fail(ctx, CATEN_B200_EINVAL, "latent attention: %d cached rows of %lld", t, (long long)a.cap);
  launch_k(ctx, latent_gather_kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, a, b0, t, rows, c, c_bf, kr);
  CB_LAUNCH_CHECK(ctx, "latent_gather_kernel");
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Absorbed attention on the CUDA cores (fp32 caches, and shapes the tensor-core kernel does not take): LS_H heads of
// one row per CTA, keys in blocks of 32 (a warp takes four), running maximum and sum.
// ---------------------------------------------------------------------------------------------
constexpr int LS_H = 4, LS_KEYS = 32, LS_THREADS = 256, LS_COLS = 4;   // a thread owns latent columns tid + 256 i, i < LS_COLS

// where a CTA's result goes: the planes (one split) or the partial buffers
struct LatentOut {
  float *o, *part, *ml;
  BfOut o_bf;
  int64_t plane, rows;
  int Kr, H, splits;
};

__global__ void __launch_bounds__(LS_THREADS) latent_attn_simt_kernel(const LatentArgs a, const float *__restrict__ qcat, BfOut qcat_bf, const LatentOut out) {
  extern __shared__ __align__(16) float sm[];
  const int KC = a.Kp + a.Pp;
  float *q = sm, *p = q + LS_H * KC, *stat = p + LS_H * LS_KEYS;   // stat: [LS_H] rescale, [LS_H] max, [LS_H] sum
  pdl_enter();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h0 = blockIdx.x * LS_H, split = blockIdx.z;
  const int64_t r = blockIdx.y;
  const int t = (a.d_n ? *a.d_n : a.n) + (int)(r % a.s) + 1;
  const int blocks = (t + LS_KEYS - 1) / LS_KEYS, per = (blocks + out.splits - 1) / out.splits;
  const int jb = split * per * LS_KEYS, je = min(t, (split + 1) * per * LS_KEYS);
  const int64_t seq = r / a.s;
  for (int i = tid; i < LS_H * KC; i += LS_THREADS) {
    const int h = h0 + i / KC;
    const int64_t at = (r * a.H + h) * KC + i % KC;
    q[i] = h >= a.H ? 0.0f : (qcat_bf.hi ? __bfloat162float(qcat_bf.hi[at]) + (qcat_bf.lo ? __bfloat162float(qcat_bf.lo[at]) : 0.0f) : qcat[at]) * a.scale;
  }
  if (tid < LS_H) { stat[LS_H + tid] = -INFINITY; stat[2 * LS_H + tid] = 0.0f; }
  float acc[LS_H][LS_COLS];
#pragma unroll
  for (int h = 0; h < LS_H; ++h)
#pragma unroll
    for (int i = 0; i < LS_COLS; ++i) acc[h][i] = 0.0f;
  __syncthreads();
  for (int j0 = jb; j0 < je; j0 += LS_KEYS) {
#pragma unroll
    for (int k = 0; k < LS_KEYS / 8; ++k) {
      const int j = j0 + warp * (LS_KEYS / 8) + k;
      float s[LS_H];
#pragma unroll
      for (int h = 0; h < LS_H; ++h) s[h] = 0.0f;
      if (j < je)
        for (int c = lane; c < KC; c += 32) {
          const float x = ld_cache(a.cache, a.cache_bf16, a.at(seq, j, c));
#pragma unroll
          for (int h = 0; h < LS_H; ++h) s[h] = fmaf(q[h * KC + c], x, s[h]);
        }
#pragma unroll
      for (int h = 0; h < LS_H; ++h) {
        s[h] = warp_sum(s[h]);
        if (lane == 0) p[h * LS_KEYS + warp * (LS_KEYS / 8) + k] = j < je ? s[h] : -INFINITY;
      }
    }
    __syncthreads();
    if (warp < LS_H) {   // one warp per head
      const float x = p[warp * LS_KEYS + lane], m_old = stat[LS_H + warp];
      float m = x;
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      m = fmaxf(m, m_old);
      const float e = exp2f((x - m) * kLog2e), f = exp2f((m_old - m) * kLog2e), ss = warp_sum(e);
      p[warp * LS_KEYS + lane] = e;
      if (lane == 0) {
        stat[warp] = f;
        stat[LS_H + warp] = m;
        stat[2 * LS_H + warp] = stat[2 * LS_H + warp] * f + ss;
      }
    }
    __syncthreads();
    const int jn = min(LS_KEYS, je - j0);
#pragma unroll
    for (int h = 0; h < LS_H; ++h)
#pragma unroll
      for (int i = 0; i < LS_COLS; ++i) acc[h][i] *= stat[h];
    for (int j = 0; j < jn; ++j) {
#pragma unroll
      for (int i = 0; i < LS_COLS; ++i) {
        const int c = tid + LS_THREADS * i;
        if (c < a.Kp) {
          const float x = ld_cache(a.cache, a.cache_bf16, a.at(seq, j0 + j, c));
#pragma unroll
          for (int h = 0; h < LS_H; ++h) acc[h][i] = fmaf(p[h * LS_KEYS + j], x, acc[h][i]);
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int h = 0; h < LS_H; ++h) {
    if (h0 + h >= a.H) break;
    const float l = stat[2 * LS_H + h];
#pragma unroll
    for (int i = 0; i < LS_COLS; ++i) {
      const int c = tid + LS_THREADS * i;
      if (c >= out.Kr) continue;
      const float v = c < a.Kp ? acc[h][i] : 0.0f;
      if (out.splits == 1) st1(out.o, out.o_bf, ((int64_t)(h0 + h) * out.plane + r) * out.Kr + c, v / l);
      else out.part[(((int64_t)split * out.rows + r) * a.H + h0 + h) * out.Kr + c] = v;
    }
    if (out.splits > 1 && tid == 0) {
      float *ml = out.ml + (((int64_t)split * out.rows + r) * a.H + h0 + h) * 2;
      ml[0] = stat[LS_H + h] * kLog2e;
      ml[1] = l;
    }
  }
}

// parts of the key splits -> planes; grid (head, row)
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentOut out) {
  pdl_enter();
  const int h = blockIdx.x;
  const int64_t r = blockIdx.y, step = out.rows * out.H, at = r * out.H + h;
  float m = -INFINITY;
  for (int z = 0; z < out.splits; ++z)
    if (out.ml[(z * step + at) * 2 + 1] > 0.0f) m = fmaxf(m, out.ml[(z * step + at) * 2]);
  float l = 0.0f;
  for (int z = 0; z < out.splits; ++z) {
    const float lz = out.ml[(z * step + at) * 2 + 1];
    if (lz > 0.0f) l = fmaf(exp2f(out.ml[(z * step + at) * 2] - m), lz, l);
  }
  for (int c = threadIdx.x; c < out.Kr; c += 128) {
    float o = 0.0f;
    for (int z = 0; z < out.splits; ++z)   // fixed order; a part without keys counts nothing
      if (out.ml[(z * step + at) * 2 + 1] > 0.0f) o = fmaf(exp2f(out.ml[(z * step + at) * 2] - m), out.part[(z * step + at) * out.Kr + c], o);
    st1(out.o, out.o_bf, ((int64_t)h * out.plane + r) * out.Kr + c, o / l);
  }
}

// grid (head, 8 rows, part of the outputs): the rows' sums over the latents (merged from the key splits' parts), then W_uv.  `lanes` neighbouring
// threads share an output and take its row of weights in turn, 16 bytes each.
constexpr int LD_ROWS = 8, LD_MAX_SPLITS = 32;

__global__ void __launch_bounds__(256) latent_down_kernel(const LatentArgs a, const LatentOut in, const __nv_bfloat16 *__restrict__ uv, int lanes, int per, float *__restrict__ out, BfOut bf,
                                                          int64_t ld) {
  extern __shared__ __align__(16) float os[];   // [LD_ROWS][Kr]
  __shared__ float part_f[LD_ROWS][LD_MAX_SPLITS];
  const int h = blockIdx.x, tid = threadIdx.x, Kr = in.Kr, S = in.splits;
  const int64_t r0 = (int64_t)blockIdx.y * LD_ROWS;
  const int rn = (int)(in.rows - r0 < LD_ROWS ? in.rows - r0 : LD_ROWS);
  const int e0 = blockIdx.z * per + tid / lanes, e1 = min(a.Ep, (int)(blockIdx.z + 1) * per), es = 256 / lanes, ks = tid % lanes, nv = Kr / 8;
  // the first weights depend on no other kernel
  uint4 ahead[4];
#pragma unroll
  for (int u = 0; u < 4; ++u)
    ahead[u] = e0 < e1 && ks + lanes * u < nv ? reinterpret_cast<const uint4 *>(uv + ((int64_t)h * a.Ep + e0) * Kr)[ks + lanes * u] : make_uint4(0u, 0u, 0u, 0u);
  pdl_enter();
  const int64_t step = in.rows * in.H;
  if (S > 1) {   // one warp per row, one lane per part
    const int r = tid >> 5, z = tid & 31;
    float2 ml = make_float2(-INFINITY, 0.0f);
    if (r < rn && z < S) ml = *reinterpret_cast<const float2 *>(in.ml + (z * step + (r0 + r) * in.H + h) * 2);
    float m = ml.y > 0.0f ? ml.x : -INFINITY;   // (a part without keys counts nothing)
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    const float f = ml.y > 0.0f ? exp2f(ml.x - m) : 0.0f, l = warp_sum(f * ml.y);
    part_f[r][z] = f / l;
    __syncthreads();
  }
  const int k4 = Kr / 4;
  for (int i = tid; i < LD_ROWS * k4; i += 256) {
    const int r = i / k4, c = i % k4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (r < rn) {
      if (S == 1) {
        v = reinterpret_cast<const float4 *>(in.o + ((int64_t)h * in.plane + r0 + r) * Kr)[c];
      } else {
        const float4 *p = reinterpret_cast<const float4 *>(in.part + ((r0 + r) * in.H + h) * Kr) + c;
        for (int z0 = 0; z0 < S; z0 += 4) {   // fixed order, four parts requested together
          float4 x[4];
#pragma unroll
          for (int u = 0; u < 4; ++u)
            if (z0 + u < S) x[u] = p[(z0 + u) * step * k4];
#pragma unroll
          for (int u = 0; u < 4; ++u)
            if (z0 + u < S) {
              const float f = part_f[r][z0 + u];
              v = make_float4(fmaf(f, x[u].x, v.x), fmaf(f, x[u].y, v.y), fmaf(f, x[u].z, v.z), fmaf(f, x[u].w, v.w));
            }
        }
      }
    }
    *reinterpret_cast<float4 *>(os + r * Kr + 4 * c) = v;
  }
  __syncthreads();
  for (int e = e0; e - tid / lanes < e1; e += es) {   // (whole warps: the lanes of an output exchange their sums)
    const bool on = e < e1;
    const uint4 *w = reinterpret_cast<const uint4 *>(uv + ((int64_t)h * a.Ep + (on ? e : 0)) * Kr);
    float acc[LD_ROWS];
#pragma unroll
    for (int r = 0; r < LD_ROWS; ++r) acc[r] = 0.0f;
    for (int i = ks; i < nv; i += 4 * lanes) {
      uint4 x[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) x[u] = e == e0 && i == ks ? ahead[u] : on && i + lanes * u < nv ? w[i + lanes * u] : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int k = 8 * (i + lanes * u);
        if (k >= Kr) continue;
        const uint32_t b[4] = {x[u].x, x[u].y, x[u].z, x[u].w};
        float f[8];
#pragma unroll
        for (int j = 0; j < 4; ++j) { f[2 * j] = __uint_as_float(b[j] << 16); f[2 * j + 1] = __uint_as_float(b[j] & 0xFFFF0000u); }
#pragma unroll
        for (int r = 0; r < LD_ROWS; ++r) {
          if (r < rn) {
            const float4 x0 = *reinterpret_cast<const float4 *>(os + r * Kr + k), x1 = *reinterpret_cast<const float4 *>(os + r * Kr + k + 4);
            acc[r] = fmaf(f[0], x0.x, fmaf(f[1], x0.y, fmaf(f[2], x0.z, fmaf(f[3], x0.w, acc[r]))));
            acc[r] = fmaf(f[4], x1.x, fmaf(f[5], x1.y, fmaf(f[6], x1.z, fmaf(f[7], x1.w, acc[r]))));
          }
        }
      }
    }
#pragma unroll
    for (int r = 0; r < LD_ROWS; ++r) {
      for (int m = lanes >> 1; m > 0; m >>= 1) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], m);
      if (on && ks == 0 && r < rn) st1(out, bf, (r0 + r) * ld + (int64_t)h * a.Ep + e, acc[r]);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Absorbed attention on the tensor cores
// ---------------------------------------------------------------------------------------------
constexpr int LA_KEYS = 128;              // cached rows per tile
constexpr int LA_SOFT = 256;              // softmax threads
constexpr int LA_THREADS = LA_SOFT + 96;
constexpr int LA_MAX_BLOCKS = 9;          // 64-column blocks of a cached row: up to 576 columns
constexpr int LA_MAX_STAGES = 4, LA_MAX_PAIRS = 10, LA_BARS = 2 * LA_MAX_PAIRS + 6;   // full, empty of the ring's pairs; s, p, o (two each); then q
constexpr uint32_t LA_BLOCK = LA_KEYS * 128;   // bytes
constexpr float LA_TAU = 11.5f;           // slack of the reference maximum, in powers of two

__device__ __forceinline__ uint32_t la_sw128(int row, int chunk) { return (uint32_t)((row >> 3) * 1024 + (row & 7) * 128 + ((chunk ^ (row & 7)) << 4)); }
__device__ __forceinline__ float la_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));   // results below 2^-126 flush to zero
  return y;
}
__device__ __forceinline__ void la_sync() { asm volatile("bar.sync 1, %0;" ::"n"(LA_SOFT) : "memory"); }
__device__ __forceinline__ bool la_any(bool x) {   // over the softmax threads
  uint32_t r;
  asm volatile("{\n\t.reg .pred p, q;\n\tsetp.ne.u32 p, %1, 0;\n\tbarrier.cta.red.or.pred q, 1, %2, p;\n\tselp.u32 %0, 1, 0, q;\n\t}"
               : "=r"(r) : "r"(x ? 1u : 0u), "n"(LA_SOFT) : "memory");
  return r != 0;
}
// N values per lane, reduced over the warp: each exchange halves the values a lane carries; afterwards red[i] holds value i's.
template <int N, bool MAX>
__device__ __forceinline__ void la_reduce(const float *x, int lane, float *red) {
  float v[N];
#pragma unroll
  for (int i = 0; i < N; ++i) v[i] = x[i];
  int which = 0, step = 16;
#pragma unroll
  for (int n = N; n > 1; n >>= 1, step >>= 1) {
    const bool up = (lane & step) != 0;
#pragma unroll
    for (int i = 0; i < n / 2; ++i) {
      const float give = up ? v[i] : v[i + n / 2], keep = up ? v[i + n / 2] : v[i];
      const float got = __shfl_xor_sync(0xffffffffu, give, step);
      v[i] = MAX ? fmaxf(keep, got) : keep + got;
    }
    which += up ? n / 2 : 0;
  }
#pragma unroll
  for (int o = 16 / N; o > 0; o >>= 1) {   // the lanes that hold the same value
    const float got = __shfl_xor_sync(0xffffffffu, v[0], o);
    v[0] = MAX ? fmaxf(v[0], got) : v[0] + got;
  }
  if ((lane & (32 / N - 1)) == 0) red[which] = v[0];
}
template <int N> __device__ __forceinline__ void la_ld(uint32_t taddr, uint32_t *r) {
  if (N == 8) tmem_ld8(taddr, r);
  else tmem_ld16(taddr, r);
}
template <int N> __device__ __forceinline__ void la_st(uint32_t taddr, const uint32_t *r) {
  if (N == 8) tmem_st8(taddr, r);
  else tmem_st16(taddr, r);
}

// MN-major operand, 128-byte swizzle: 64-element blocks LA_BLOCK bytes apart, groups of 8 along k 1024 bytes apart
__device__ __forceinline__ uint64_t la_desc_mn(uint32_t saddr) { return umma_desc(saddr) - ((uint64_t)1 << 16) + ((uint64_t)(LA_BLOCK >> 4) << 16); }
// K-major operand with rows of 64 bytes, 64-byte swizzle, 8-row groups 512 bytes apart
__device__ __forceinline__ uint64_t la_desc_narrow(uint32_t saddr) {
  return (uint64_t)((saddr >> 4) & 0x3FFF) | (uint64_t)1 << 16 | (uint64_t)(512 >> 4) << 32 | (uint64_t)1 << 46 | (uint64_t)4 << 61;
}

template <int NH>
__global__ void __launch_bounds__(LA_THREADS, 1) latent_attn_tc_kernel(const LatentArgs a, const float *__restrict__ qcat, const __nv_bfloat16 *__restrict__ qcat_hi,
                                                                       const LatentOut out, const int stages, const int early, const uint32_t tmem_cols, const uint32_t idesc_s,
                                                                       const uint32_t idesc_pv, int *status) {
  extern __shared__ unsigned char la_raw[];
  unsigned char *sm = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(la_raw) + 1023) & ~(uintptr_t)1023);
  constexpr int HT = NH / 2;   // heads of a softmax thread
  constexpr uint32_t QB = NH * 128, PB = 2 * 2 * NH * 128;   // bytes of a Q block; of a P buffer (two blocks of 64 keys, 2 NH rows)
  const int KC = a.KC(), nkc = a.blocks(), np = (nkc + 1) / 2, ksteps = KC / 16, npv = (out.Kr / 64 + 1) / 2;
  const uint32_t tile_bytes = (uint32_t)a.tile_elems() * 2u;
  unsigned char *kv = sm, *qs = kv + (size_t)stages * tile_bytes, *ps = qs + nkc * QB;
  uint64_t *bars = reinterpret_cast<uint64_t *>(ps + 2 * PB);
  float *red = reinterpret_cast<float *>(bars + LA_BARS + 1);   // [4][NH]: a row per quadrant of keys
  const uint32_t bar0 = smem_u32(bars);
  auto full = [&](int s, int p) { return bar0 + 8u * (s * np + p); };
  auto empty = [&](int s, int p) { return bar0 + 8u * (LA_MAX_PAIRS + s * np + p); };
  auto s_full = [&](int b) { return bar0 + 8u * (2 * LA_MAX_PAIRS + b); };
  auto p_full = [&](int b) { return bar0 + 8u * (2 * LA_MAX_PAIRS + 2 + b); };
  auto o_done = [&](int b) { return bar0 + 8u * (2 * LA_MAX_PAIRS + 4 + b); };
  const uint32_t q_full = bar0 + 8u * LA_BARS;
  __shared__ uint32_t tmem_slot;
  __shared__ volatile int flags[2];   // [0] a wait ran out; [1] never set
  volatile int *abort_flag = flags;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h0 = blockIdx.x * NH, hn = min(NH, a.H - h0), split = blockIdx.z;
  const int64_t r = blockIdx.y;

  if (tid == 0) {
    for (int i = 0; i < stages * np; ++i) {
      mbar_init(bar0 + 8u * i, 1);
      mbar_init(bar0 + 8u * (LA_MAX_PAIRS + i), 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(s_full(b), 1);
      mbar_init(p_full(b), LA_SOFT / 32);
      mbar_init(o_done(b), 1);
    }
    mbar_init(q_full, LA_SOFT / 32);
    flags[0] = flags[1] = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 9) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(tmem_cols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = tmem_slot, col_s = (uint32_t)npv * 2 * NH;   // O: npv x 2 NH columns, then two score tiles of NH
  // `early`: the cache and the position were complete before the kernel in front of this one started; only Q comes from it
  if (warp != 8 || !early) pdl_wait();
  pdl_launch_dependents();
  const int t = (a.d_n ? *a.d_n : a.n) + (int)(r % a.s) + 1;   // keys this row sees
  const int tiles = (t + LA_KEYS - 1) / LA_KEYS, per = (tiles + out.splits - 1) / out.splits;
  const int tile0 = min(split * per, tiles), nt = min(tile0 + per, tiles) - tile0;
  auto give_up = [&](int where) {
    if (!*abort_flag) { *abort_flag = 1; atomicCAS(status, 0, DEV_WAIT_TIMEOUT); status[1] = where; }
  };

  bool ok = true;
  if (warp == 8) {
    if (lane == 0) {
      int issued = 0, s = 0;
      uint32_t ph = 1;
      const unsigned char *src = reinterpret_cast<const unsigned char *>(a.cache) + (r / a.s) * a.seq_elems() * 2 + (int64_t)tile0 * tile_bytes;
      for (int i = 0; i < nt && ok; ++i, src += tile_bytes) {
        for (int p = 0; p < np; ++p) {
          if (!mbar_wait(empty(s, p), ph, abort_flag)) { give_up(30); ok = false; break; }
          const uint32_t at = (uint32_t)p * 2 * LA_BLOCK, bytes = min(2 * LA_BLOCK, tile_bytes - at);
          mbar_expect_tx(full(s, p), bytes);
          bulk_load(smem_u32(kv) + s * tile_bytes + at, src + at, bytes, full(s, p));
          ++issued;
        }
        if (++s == stages) { s = 0; ph ^= 1u; }
      }
      if (*abort_flag)   // copies in flight land before the CTA's shared memory is released
        for (int i = issued > stages * np ? issued - stages * np : 0; i < issued; ++i)
          mbar_wait(full(i / np % stages, i % np), (uint32_t)(i / np / stages) & 1u, abort_flag + 1);
    }
    __syncwarp();
  } else if (warp == 9) {
    const uint64_t dq = umma_desc(smem_u32(qs)), dk0 = umma_desc(smem_u32(kv)), dn0 = la_desc_narrow(smem_u32(kv));
    const int narrow = a.narrow() ? nkc - 1 : -1;
    ok = nt == 0 || mbar_wait(q_full, 0, abort_flag);
    if (!ok && lane == 0) give_up(31);
    int s = 0;
    uint32_t ph = 0;
    for (int i = 0; i < nt && ok; ++i) {
      // the scores of tile i - 2 in these columns have been read
      if (i >= 2 && !(ok = mbar_wait(p_full(i & 1), (uint32_t)((i - 2) >> 1) & 1u, abort_flag))) {
        if (lane == 0) give_up(38);
        break;
      }
      for (int p = 0; p < np && ok; ++p) {
        if (!(ok = mbar_wait(full(s, p), ph, abort_flag))) {
          if (lane == 0) give_up(32);
          break;
        }
        tc_fence_after();
        if (elect_one()) {
          const uint64_t at = (uint64_t)((s * tile_bytes + (uint32_t)p * 2 * LA_BLOCK) >> 4), db = dq + (uint64_t)(2 * p * (int)(QB >> 4));
          const int left = ksteps - 8 * p;
#pragma unroll
          for (int k = 0; k < 8; ++k)   // 16 columns = 32 bytes = 2 descriptor units
            if (k < left)
              umma_bf16(tmem_base + col_s + NH * (i & 1), (2 * p + (k >> 2) == narrow ? dn0 : dk0) + at + (uint64_t)((k >> 2) * (LA_BLOCK >> 4) + 2 * (k & 3)),
                        db + (uint64_t)((k >> 2) * (QB >> 4) + 2 * (k & 3)), idesc_s, p > 0 || k > 0 ? 1u : 0u);
          if (p == np - 1) umma_commit(s_full(i & 1));
        }
        __syncwarp();
      }
      if (++s == stages) { s = 0; ph ^= 1u; }
    }
  } else if (warp == 10) {
    const uint64_t dm = la_desc_mn(smem_u32(kv)), dp = umma_desc(smem_u32(ps));
    int s = 0;
    for (int i = 0; i < nt; ++i) {
      if (!(ok = mbar_wait(p_full(i & 1), (uint32_t)(i >> 1) & 1u, abort_flag))) {
        if (lane == 0) give_up(33);
        break;
      }
      tc_fence_after();
      if (elect_one()) {
        const uint64_t db = dp + (uint64_t)((i & 1) * (int)(PB >> 4));
        for (int j = 0; j < npv; ++j) {
          const uint64_t da = dm + (uint64_t)((s * tile_bytes + (uint32_t)j * 2 * LA_BLOCK) >> 4);
          const uint32_t acc = tmem_base + (uint32_t)j * 2 * NH;
#pragma unroll
          for (int k = 0; k < LA_KEYS / 16; ++k)   // A: 16 keys = 16 rows of 128 bytes = 128 descriptor units
            umma_bf16(acc, da + (uint64_t)(128 * k), db + (uint64_t)((k >> 2) * (PB >> 5) + 2 * (k & 3)), idesc_pv, (i > 0 || k > 0) ? 1u : 0u);
          umma_commit(empty(s, j));
        }
        // (the tile's scores, which also read it, were complete before its probabilities were formed)
        for (int p = npv; p < np; ++p) umma_commit(empty(s, p));
        umma_commit(o_done(i & 1));
      }
      __syncwarp();
      if (++s == stages) s = 0;
    }
  } else {
    // ---- softmax: thread = (key of the tile = lane of tensor memory, half of the heads) ----
    const int quad = warp & 3, hh = (warp >> 2) * HT, key = quad * 32 + lane;
    const uint32_t tlane = tmem_base + ((uint32_t)(quad * 32) << 16);
    {
      const int pieces = KC / 8, all = NH * nkc * 8;   // 16-byte pieces of the heads' rows, three per thread requested together
      for (int i0 = tid; i0 < all; i0 += 3 * LA_SOFT) {
        uint4 v[3];
#pragma unroll
        for (int u = 0; u < 3; ++u) {
          const int i = i0 + LA_SOFT * u, row = i / (nkc * 8), c = i % (nkc * 8);
          v[u] = make_uint4(0u, 0u, 0u, 0u);
          if (i < all && row < hn && c < pieces) {
            const int64_t at = (r * a.H + h0 + row) * KC + 8 * c;
            if (qcat_hi) {
              v[u] = *reinterpret_cast<const uint4 *>(qcat_hi + at);
            } else {
              const float4 x = *reinterpret_cast<const float4 *>(qcat + at), y = *reinterpret_cast<const float4 *>(qcat + at + 4);
              v[u] = make_uint4(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w), pack_bf16(y.x, y.y), pack_bf16(y.z, y.w));
            }
          }
        }
#pragma unroll
        for (int u = 0; u < 3; ++u) {
          const int i = i0 + LA_SOFT * u, row = i / (nkc * 8), c = i % (nkc * 8);
          if (i < all) *reinterpret_cast<uint4 *>(qs + (c >> 3) * QB + la_sw128(row, c & 7)) = v[u];
        }
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(q_full);
    }
    const float f = a.scale * kLog2e;
    float m[HT], l[HT];   // in powers of two, the same for every key; this key's share of the sum
#pragma unroll
    for (int h = 0; h < HT; ++h) { m[h] = -INFINITY; l[h] = 0.0f; }
    // (a warp that gives up stays in the loop, without waiting for anything, so that all warps reach the same block barriers)
    auto wait = [&](uint32_t bar, uint32_t parity, int where) {
      if (!ok) return;
      ok = __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag));
      if (!ok && lane == 0) give_up(where);
    };
    for (int i = 0; i < nt; ++i) {
      wait(s_full(i & 1), (uint32_t)(i >> 1) & 1u, 34);
      float v[HT];
      bool above = false;
      if (ok) {
        tc_fence_after();
        uint32_t raw[HT];
        la_ld<HT>(tlane + col_s + NH * (i & 1) + hh, raw);
        tmem_ld_wait();
        const bool visible = (tile0 + i) * LA_KEYS + key < t;
#pragma unroll
        for (int h = 0; h < HT; ++h) {
          v[h] = visible ? __uint_as_float(raw[h]) * f : -INFINITY;
          above |= v[h] > m[h] + LA_TAU;   // (every score at the first visible key: m = -inf)
        }
      }
      if (la_any(above || !ok)) {
        if (ok) la_reduce<HT, true>(v, lane, red + quad * NH + hh);
        la_sync();
        if (i > 0) wait(o_done((i - 1) & 1), (uint32_t)((i - 1) >> 1) & 1u, 35);
        tc_fence_after();
        float g[HT];
#pragma unroll
        for (int h = 0; h < HT; ++h) {
          const float *x = red + hh + h;
          const float mx = fmaxf(fmaxf(x[0], x[NH]), fmaxf(x[2 * NH], x[3 * NH]));
          const bool move = mx > m[h] + LA_TAU;
          g[h] = move ? exp2f(m[h] - mx) : 1.0f;
          if (move) m[h] = mx;
          l[h] *= g[h];
        }
        if (ok && i > 0)
          for (int c = hh; c < npv * 2 * NH; c += NH) {   // this thread's heads in the hi and lo columns of every block
            uint32_t o[HT];
            la_ld<HT>(tlane + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < HT; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * g[e]);
            la_st<HT>(tlane + c, o);
          }
        tmem_st_wait();
      }
      if (i >= 2) wait(o_done(i & 1), (uint32_t)((i - 2) >> 1) & 1u, 36);   // this P buffer has been read
      unsigned char *pb = ps + (i & 1) * PB + (key >> 6) * (PB / 2) + (key & 7) * 2;
      const int chunk = (key & 63) >> 3;
      if (ok) {
#pragma unroll
        for (int h = 0; h < HT; ++h) {
          const float p = la_ex2(v[h] - m[h]);   // (a hidden key: 2^-inf = 0)
          l[h] += p;
          const __nv_bfloat16 hi = __float2bfloat16_rn(p);
          *reinterpret_cast<__nv_bfloat16 *>(pb + la_sw128(hh + h, chunk)) = hi;
          *reinterpret_cast<__nv_bfloat16 *>(pb + la_sw128(NH + hh + h, chunk)) = __float2bfloat16_rn(p - __bfloat162float(hi));
        }
        fence_proxy_async();
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(p_full(i & 1));
      }
    }
    if (nt > 0) wait(o_done((nt - 1) & 1), (uint32_t)((nt - 1) >> 1) & 1u, 37);   // the last product (and so all of them) is complete
    tc_fence_after();
    la_sync();
    la_reduce<HT, false>(l, lane, red + quad * NH + hh);
    la_sync();
    if (__all_sync(0xffffffffu, ok && !*abort_flag)) {
      float inv[HT];
#pragma unroll
      for (int h = 0; h < HT; ++h) {
        const float *x = red + hh + h;
        l[h] = x[0] + x[NH] + x[2 * NH] + x[3 * NH];
        inv[h] = out.splits == 1 ? 1.0f / l[h] : 1.0f;
      }
      // this thread's first head in this row, and from one head to the next
      const int hb = h0 + hh;
      const int64_t first = out.splits == 1 ? ((int64_t)hb * out.plane + r) * out.Kr : (((int64_t)split * out.rows + r) * a.H + hb) * out.Kr;
      const int64_t step = out.splits == 1 ? out.plane * out.Kr : out.Kr;
      float *of = out.splits == 1 ? out.o : out.part;
      const BfOut ob = out.splits == 1 ? out.o_bf : BfOut();
      for (int j = 0; j < npv; ++j) {
        const int c = 128 * j + key;   // this lane's column of the latent (columns past it belong to the key part)
        uint32_t hi[HT], lo[HT];
        if (nt > 0) {
          la_ld<HT>(tlane + j * 2 * NH + hh, hi);
          la_ld<HT>(tlane + j * 2 * NH + NH + hh, lo);
          tmem_ld_wait();
        }
        const bool in = nt > 0 && c < a.Kp;
        if (c < out.Kr) {
          int64_t at = first + c;
#pragma unroll
          for (int h = 0; h < HT; ++h, at += step)
            if (hb + h < a.H) st1(of, ob, at, in ? (__uint_as_float(hi[h]) + __uint_as_float(lo[h])) * inv[h] : 0.0f);
        }
      }
      if (out.splits > 1 && key == 0)
#pragma unroll
        for (int h = 0; h < HT; ++h)
          if (hb + h < a.H) {
            float *ml = out.ml + (((int64_t)split * out.rows + r) * a.H + hb + h) * 2;
            ml[0] = m[h];
            ml[1] = l[h];
          }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 9) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(tmem_cols) : "memory");
  }
}

// ---- host ---------------------------------------------------------------------------------------

static bool latent_tc(const caten_b200_ctx *ctx, const LatentArgs &a) {
  return a.tiled && ctx->attn_tc && a.KC() <= 64 * LA_MAX_BLOCKS;
}
static int latent_heads(const LatentArgs &a) { return a.H <= 16 ? 16 : 32; }   // per CTA
static int64_t latent_ctas(const LatentArgs &a, bool tc, int64_t rows) {
  const int per = tc ? latent_heads(a) : LS_H;
  return (a.H + per - 1) / per * rows;
}

int latent_splits(const caten_b200_ctx *ctx, const LatentArgs &a, int64_t rows, int64_t keys) {
  const bool tc = latent_tc(ctx, a);
  const int kt = tc ? LA_KEYS : LS_KEYS, fixed = tc ? 2 : 6;   // what a CTA costs besides its tiles, in tiles
  const int64_t tiles = (keys + kt - 1) / kt, ctas = latent_ctas(a, tc, rows), slots = (int64_t)ctx->sm_count * (tc ? 1 : 4);
  int best = 1;
  int64_t cost = INT64_MAX;
  for (int S = 1; S <= 32 && S <= tiles; S = S < 4 ? S + 1 : S + S / 4) {
    // waves x (tiles of a CTA + its fixed part), and merging the parts
    const int64_t c = (ctas * S + slots - 1) / slots * ((tiles + S - 1) / S + fixed) + (S > 1 ? 2 : 0);
    if (c < cost) { cost = c; best = S; }
  }
  return best;
}

template <int NH>
static int launch_tc(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x, const LatentOut &out, dim3 grid) {
  const int nkc = a.blocks(), np = (nkc + 1) / 2, npv = (a.Kr / 64 + 1) / 2;
  const size_t stage = (size_t)a.tile_elems() * 2, rest = (size_t)nkc * NH * 128 + 2 * 4 * NH * 128 + (LA_BARS + 1) * 8 + 4 * NH * sizeof(float);
  int stages = (int)((224 * 1024 - rest) / stage);
  if (stages > LA_MAX_STAGES) stages = LA_MAX_STAGES;
  while (stages * np > LA_MAX_PAIRS) --stages;
  // (beside a pair of a single block the second product's operand reaches into what follows, at least 16 KB: rows of O nobody reads)
  const size_t smem = 1024 + stage * stages + rest;
  uint32_t cols = 32;
  while (cols < (uint32_t)(npv * 2 * NH + 2 * NH)) cols *= 2;
  const uint32_t base = (1u << 4) | (1u << 7) | (1u << 10) | (8u << 24);   // fp32 accumulate, bf16 x bf16, M = 128
  const uint32_t idesc_s = base | ((uint32_t)(NH >> 3) << 17), idesc_pv = base | ((uint32_t)(2 * NH >> 3) << 17) | (1u << 15);   // second product: A MN-major
  CB_CUDA(ctx, cudaFuncSetAttribute(latent_attn_tc_kernel<NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_k(ctx, latent_attn_tc_kernel<NH>, grid, dim3(LA_THREADS), smem, a, x.qcat_bf.hi ? nullptr : x.qcat, x.qcat_bf.hi, out, stages, x.early ? 1 : 0, cols, idesc_s,
           idesc_pv, ctx->d_status);
  CB_LAUNCH_CHECK(ctx, "latent_attn_tc_kernel");
  return 0;
}

static LatentOut latent_out(const LatentArgs &a, const LatentAbsorbed &x) {
  LatentOut out;
  out.o = x.o; out.o_bf = x.o_bf; out.part = x.part; out.ml = x.ml; out.plane = x.plane; out.rows = (int64_t)a.B * a.s; out.Kr = a.Kr; out.H = a.H; out.splits = x.splits;
  return out;
}

int launch_latent_down(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x, const caten_b200_weight *uv, float *out, BfOut bf, int64_t ld) {
  if (int rc = check_latent(ctx, a)) return rc;
  const LatentOut in = latent_out(a, x);
  if (in.rows <= 0) return 0;
  if (uv->type != CATEN_B200_BF16 || x.splits > LD_MAX_SPLITS || (x.splits == 1 && x.o_bf.hi)) return fail(ctx, CATEN_B200_EINVAL, "latent attention: W_uv takes fp32 sums and BF16 weights");
  // few rows: a head's outputs are split over CTAs (each merges the parts again)
  const int64_t ctas = (in.rows + LD_ROWS - 1) / LD_ROWS * a.H;
  int pieces = 1;
  while (pieces < 4 && 2 * pieces * ctas <= ctx->sm_count && a.Ep / (2 * pieces) >= 16) pieces *= 2;
  const int per = (a.Ep + pieces - 1) / pieces;
  int lanes = 1;   // threads per output
  while (lanes < 32 && 2 * lanes * per <= 256) lanes *= 2;
  launch_k(ctx, latent_down_kernel, dim3((unsigned)a.H, (unsigned)((in.rows + LD_ROWS - 1) / LD_ROWS), (unsigned)pieces), dim3(256), (size_t)LD_ROWS * a.Kr * sizeof(float), a, in,
           (const __nv_bfloat16 *)uv->qs, lanes, per, out, bf, ld);
  CB_LAUNCH_CHECK(ctx, "latent_down_kernel");
  return 0;
}

int launch_latent_absorbed(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x) {
  const int64_t rows = (int64_t)a.B * a.s;
  if (rows <= 0) return 0;
  if (int rc = check_latent(ctx, a)) return rc;
  if (rows > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "latent attention: %lld rows", (long long)rows);
  if (x.splits > 1 && (!x.part || !x.ml)) return fail(ctx, CATEN_B200_EINVAL, "latent attention: key splits need their buffers");
  const LatentOut out = latent_out(a, x);
  if (latent_tc(ctx, a)) {
    const dim3 grid((unsigned)(latent_ctas(a, true, 1)), (unsigned)rows, (unsigned)x.splits);
    if (int rc = latent_heads(a) == 16 ? launch_tc<16>(ctx, a, x, out, grid) : launch_tc<32>(ctx, a, x, out, grid)) return rc;
  } else {
    const size_t smem = (size_t)(LS_H * (a.KC() + LS_KEYS) + 3 * LS_H) * sizeof(float);
    launch_k(ctx, latent_attn_simt_kernel, dim3((unsigned)((a.H + LS_H - 1) / LS_H), (unsigned)rows, (unsigned)x.splits), dim3(LS_THREADS), smem, a, x.qcat, x.qcat_bf, out);
    CB_LAUNCH_CHECK(ctx, "latent_attn_simt_kernel");
  }
  if (x.splits > 1 && x.combine) {
    launch_k(ctx, latent_combine_kernel, dim3((unsigned)a.H, (unsigned)rows), dim3(128), 0, out);
    CB_LAUNCH_CHECK(ctx, "latent_combine_kernel");
  }
  return 0;
}

}  // namespace cb
