// Latent attention.  Per token the cache holds c (a normed latent of K values) and r (one rotated key part of P values
// for all heads).  With q = [q_n, q_r] per head the scores are (q_n . W_uk c + q_r . r) * scale and the output is
// sum_j p_j W_uv c_j.  Two forms:
//   absorbed   (q_n W_uk) . c and W_uv (sum_j p_j c_j): the cache is read as it is, once for all heads of a CTA.  Decoding
//              and very short portions.
//   expanded   keys and values of all heads are formed from the cached latents by one linear and go through the
//              ordinary prompt attention (attention_tc.cu, attn_window.cu).  Longer portions.
//
// latent_attn_tc_kernel (bf16 models): tcgen05.  A CTA serves up to 64 heads of one row: the 128 lanes of tensor memory hold every
// head twice, so that both halves find the same scores and probabilities, and the upper half stores the high, the lower half the
// low bf16 part of p as the A operand of the second product: p keeps 16 bits and the two partial outputs are added at the end.
//   warp 4      TMA: tiles of KT cached rows, all columns, as 64-column blocks with the 128-byte swizzle.  The same tile is the K-major B
//               operand of S = Q.C^T and the MN-major B operand of O += P.C
//   warp 5      tcgen05.mma: S of the next tile is issued before O of this one, so that it runs during the softmax
//   warps 0..3  one score row per thread: lazily moved reference maximum (as in attention_tc.cu), p to tensor memory
// Value columns go in blocks of 256 per CTA, keys may be split over CTAs; latent_combine_kernel then merges the parts.
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
  const int64_t at = ((r / a.s) * a.cap + pos) * (a.Kp + a.Pp);
  const float *lat = row + a.Qr, *key = lat + a.Kp;
  for (int c = tid; c < a.Kp; c += LP_THREADS) st_cache(a.cache, a.cache_bf16, at + c, lat[c] * rc * a.kv_norm[c]);
  const int half = a.P / 2;
  for (int i = tid; i < a.Pp; i += LP_THREADS) {
    float v = 0.0f;
    if (i < a.P) {
      const int f = i < half ? i : i - half;
      float sn, cs;
      sincosf((float)pos * a.freq[f], &sn, &cs);
      v = i < half ? key[i] * cs - key[i + half] * sn : key[i] * cs + key[f] * sn;
    }
    st_cache(a.cache, a.cache_bf16, at + a.Kp + i, v);
  }
}

static int check_latent(caten_b200_ctx *ctx, const LatentArgs &a) {
  if (a.H <= 0 || a.D <= 0 || a.E <= 0 || a.K <= 0 || a.Q <= 0 || a.P < 0 || a.P % 2 || a.Dp % 16 || a.Pp % 16 || a.Ep % 16 || a.Kp % 16 || a.Kr % 64 || a.Qr % 64 || a.n < 0 || a.cap <= 0)
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

// one warp per cached row
__global__ void __launch_bounds__(256) latent_gather_kernel(const LatentArgs a, int b0, int t, int64_t rows, float *__restrict__ c, BfOut c_bf, float *__restrict__ kr) {
  pdl_enter();
  const int64_t r = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= rows) return;
  const int lane = threadIdx.x & 31, KC = a.Kp + a.Pp;
  const int64_t from = ((int64_t)(b0 + r / t) * a.cap + r % t) * KC;
  for (int j = lane; j < a.Kr; j += 32) {
    if (a.cache_bf16 && c_bf.hi) c_bf.hi[r * a.Kr + j] = j < a.Kp ? reinterpret_cast<const __nv_bfloat16 *>(a.cache)[from + j] : __float2bfloat16_rn(0.0f);
    else st1(c, c_bf, r * a.Kr + j, j < a.Kp ? ld_cache(a.cache, a.cache_bf16, from + j) : 0.0f);
  }
  for (int j = lane; j < a.Pp; j += 32) kr[r * a.Pp + j] = ld_cache(a.cache, a.cache_bf16, from + a.Kp + j);
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
  const int64_t base = (r / a.s) * a.cap * KC;
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
          const float x = ld_cache(a.cache, a.cache_bf16, base + (int64_t)j * KC + c);
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
          const float x = ld_cache(a.cache, a.cache_bf16, base + (int64_t)(j0 + j) * KC + c);
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
      ml[0] = stat[LS_H + h];
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
    if (lz > 0.0f) l = fmaf(exp2f((out.ml[(z * step + at) * 2] - m) * kLog2e), lz, l);
  }
  for (int c = threadIdx.x; c < out.Kr; c += 128) {
    float o = 0.0f;
    for (int z = 0; z < out.splits; ++z)   // fixed order; a part without keys counts nothing
      if (out.ml[(z * step + at) * 2 + 1] > 0.0f) o = fmaf(exp2f((out.ml[(z * step + at) * 2] - m) * kLog2e), out.part[(z * step + at) * out.Kr + c], o);
    st1(out.o, out.o_bf, ((int64_t)h * out.plane + r) * out.Kr + c, o / l);
  }
}

// ---------------------------------------------------------------------------------------------
// Absorbed attention on the tensor cores
// ---------------------------------------------------------------------------------------------
constexpr int LA_H = 64;                // heads per CTA
constexpr int LA_THREADS = 192;
constexpr int LA_MAX_STAGES = 4, LA_MAX_BLOCKS = 9;   // 64-column blocks of a cached row: up to 576 columns
constexpr int LA_VBLOCKS = 4;           // value blocks per CTA
constexpr float LA_TAU = 8.0f;          // slack of the reference maximum, in units of the score
constexpr uint32_t LA_COL_O = 0, LA_COL_S = 256, LA_COL_P = 384;   // two score tiles of 64 columns, two P tiles of 32
constexpr int LA_OLD = 260;             // row pitch (floats) of the output exchange buffer

__device__ __forceinline__ uint32_t la_sw128(int row, int chunk) { return (uint32_t)((row >> 3) * 1024 + (row & 7) * 128 + ((chunk ^ (row & 7)) << 4)); }
__device__ __forceinline__ float la_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));   // results below 2^-126 flush to zero
  return y;
}

// KT: cached rows per tile
template <int KT>
__global__ void __launch_bounds__(LA_THREADS, 1) latent_attn_tc_kernel(const __grid_constant__ CUtensorMap map, const LatentArgs a, const float *__restrict__ qcat,
                                                                       const __nv_bfloat16 *__restrict__ qcat_hi, const LatentOut out, const int stages,
                                                                       const uint32_t idesc_s, const uint32_t idesc_pv, int *status) {
  extern __shared__ unsigned char la_raw[];
  unsigned char *sm = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(la_raw) + 1023) & ~(uintptr_t)1023);
  const int KC = a.Kp + a.Pp, nkc = (KC + 63) / 64, ksteps = KC / 16;
  const uint32_t stage_bytes = (uint32_t)nkc * KT * 128;
  unsigned char *qs = sm, *kv = sm + nkc * 16384;
  // (the tiles become the output exchange buffer at the end)
  uint64_t *bars = reinterpret_cast<uint64_t *>(sm + max((size_t)nkc * 16384 + (size_t)stages * stage_bytes, (size_t)LA_H * LA_OLD * 4));
  const uint32_t bar0 = smem_u32(bars);
  auto full = [&](int s) { return bar0 + 8u * s; };
  auto empty = [&](int s) { return bar0 + 8u * (LA_MAX_STAGES + s); };
  auto s_full = [&](int b) { return bar0 + 8u * (2 * LA_MAX_STAGES + b); };
  auto p_full = [&](int b) { return bar0 + 8u * (2 * LA_MAX_STAGES + 2 + b); };
  auto o_done = [&](int b) { return bar0 + 8u * (2 * LA_MAX_STAGES + 4 + b); };
  const uint32_t q_full = bar0 + 8u * (2 * LA_MAX_STAGES + 6);
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 2 * LA_MAX_STAGES + 7);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(tmem_slot + 1);   // [0] a wait ran out; [1] never set
  float *lsum = reinterpret_cast<float *>(tmem_slot + 4);                       // [LA_H]

  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int vparts = (out.Kr / 64 + LA_VBLOCKS - 1) / LA_VBLOCKS;
  const int h0 = blockIdx.x / vparts * LA_H, vb0 = blockIdx.x % vparts * LA_VBLOCKS, nvb = min(LA_VBLOCKS, out.Kr / 64 - vb0);
  const int hn = min(LA_H, a.H - h0), split = blockIdx.z;
  const int64_t r = blockIdx.y;

  if (tid == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(full(s), 1);
      mbar_init(empty(s), 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(s_full(b), 1);
      mbar_init(p_full(b), 4);
      mbar_init(o_done(b), 1);
    }
    mbar_init(q_full, 4);
    abort_flag[0] = abort_flag[1] = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 5) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(512u) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  if (warp == 4 && lane == 0) tma_prefetch_map(&map);
  pdl_enter();
  const int t = (a.d_n ? *a.d_n : a.n) + (int)(r % a.s) + 1;   // keys this row sees
  const int tiles = (t + KT - 1) / KT, per = (tiles + out.splits - 1) / out.splits;
  const int tile0 = min(split * per, tiles), nt = min(tile0 + per, tiles) - tile0;
  auto give_up = [&](int where) {
    if (!*abort_flag) { *abort_flag = 1; atomicCAS(status, 0, DEV_WAIT_TIMEOUT); status[1] = where; }
  };

  float m = -INFINITY, l = 0.0f;   // softmax threads
  bool ok = true;
  if (warp == 4) {
    if (lane == 0) {
      int issued = 0, s = 0;
      uint32_t ph = 1;
      const int row0 = (int)(r / a.s * a.cap);
      for (int i = 0; i < nt; ++i) {
        if (!mbar_wait(empty(s), ph, abort_flag)) { give_up(30); break; }
        mbar_expect_tx(full(s), stage_bytes);
        for (int c = 0; c < nkc; ++c)
          tma_load_2d(smem_u32(kv) + s * stage_bytes + (uint32_t)c * KT * 128, &map, full(s), c * 64, row0 + (tile0 + i) * KT);
        issued = i + 1;
        if (++s == stages) { s = 0; ph ^= 1u; }
      }
      if (*abort_flag)   // copies in flight land before the CTA's shared memory is released
        for (int i = issued > stages ? issued - stages : 0; i < issued; ++i) mbar_wait(full(i % stages), (uint32_t)(i / stages) & 1u, abort_flag + 1);
    }
    __syncwarp();
  } else if (warp == 5) {
    const uint64_t dq = umma_desc(smem_u32(qs)), dk0 = umma_desc(smem_u32(kv));
    const uint32_t stage16 = stage_bytes >> 4;
    ok = nt == 0 || mbar_wait(q_full, 0, abort_flag);
    if (!ok && lane == 0) give_up(31);
    tc_fence_after();
    auto scores = [&](int i) {   // S(i) into its tile
      if (!mbar_wait(full(i % stages), (uint32_t)(i / stages) & 1u, abort_flag)) {
        if (lane == 0) give_up(32);
        return false;
      }
      tc_fence_after();
      if (elect_one()) {
        const uint64_t dk = dk0 + (uint64_t)(i % stages) * stage16;
        for (int k = 0; k < ksteps; ++k)   // 16 columns = 32 bytes = 2 descriptor units; a Q block has 1024 units, a tile's block KT * 8
          umma_bf16(tmem_base + LA_COL_S + 64 * (i & 1), dq + (uint64_t)((k >> 2) * 1024 + 2 * (k & 3)), dk + (uint64_t)((k >> 2) * (KT * 8) + 2 * (k & 3)), idesc_s, k > 0 ? 1u : 0u);
        umma_commit(s_full(i & 1));
      }
      __syncwarp();
      return true;
    };
    if (ok && nt > 0) ok = scores(0);
    for (int i = 0; i < nt && ok; ++i) {
      // (tile i + 1's scores overwrite those of i - 1, which the softmax has read: its P(i - 1) was waited for)
      if (i + 1 < nt && !(ok = scores(i + 1))) break;
      if (!mbar_wait(p_full(i & 1), (uint32_t)(i >> 1) & 1u, abort_flag)) {
        if (lane == 0) give_up(33);
        ok = false;
        break;
      }
      tc_fence_after();
      if (elect_one()) {
        const uint64_t dv = dk0 + (uint64_t)(i % stages) * stage16 + (uint64_t)(vb0 * KT * 8);
        for (int w = 0; w < nvb; ++w)
#pragma unroll
          for (int k4 = 0; k4 < KT / 16; ++k4)   // 16 keys = 16 rows of 128 bytes = 128 descriptor units
            umma_bf16_ts(tmem_base + LA_COL_O + 64 * w, tmem_base + LA_COL_P + 32 * (i & 1) + 8 * k4, dv + (uint64_t)(w * KT * 8 + 128 * k4), idesc_pv, (i > 0 || k4 > 0) ? 1u : 0u);
        umma_commit(o_done(i & 1));
        umma_commit(empty(i % stages));
      }
      __syncwarp();
    }
  } else {
    // ---- softmax: thread = lane of tensor memory; head h0 + (tid & 63), high part of p in lanes 0..63, low part in 64..127 ----
    const uint32_t tlane = tmem_base + ((uint32_t)(warp * 32) << 16);
    {
      const int pieces = KC / 8;
      for (int i = tid; i < 64 * nkc * 8; i += 128) {   // 16-byte pieces, both copies of the head's row
        const int row = i / (nkc * 8), c = i % (nkc * 8);
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (row < hn && c < pieces) {
          const int64_t at = (r * a.H + h0 + row) * KC + 8 * c;
          if (qcat_hi) {
            v = *reinterpret_cast<const uint4 *>(qcat_hi + at);
          } else {
            const float4 x = *reinterpret_cast<const float4 *>(qcat + at), y = *reinterpret_cast<const float4 *>(qcat + at + 4);
            v = make_uint4(pack_bf16(x.x, x.y), pack_bf16(x.z, x.w), pack_bf16(y.x, y.y), pack_bf16(y.z, y.w));
          }
        }
        *reinterpret_cast<uint4 *>(qs + (c >> 3) * 16384 + la_sw128(row, c & 7)) = v;
        *reinterpret_cast<uint4 *>(qs + (c >> 3) * 16384 + la_sw128(64 + row, c & 7)) = v;
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(q_full);
    }
    const float f = a.scale;
    for (int i = 0; i < nt; ++i) {
      ok = __all_sync(0xffffffffu, mbar_wait(s_full(i & 1), (uint32_t)(i >> 1) & 1u, abort_flag));
      if (!ok) { if (lane == 0) give_up(34); break; }
      tc_fence_after();
      uint32_t sc[KT];
#pragma unroll
      for (int c = 0; c < KT; c += 16) tmem_ld16(tlane + LA_COL_S + 64 * (i & 1) + c, sc + c);
      tmem_ld_wait();
      const int lim = t - 1 - (tile0 + i) * KT;   // key e of the tile is visible iff e <= lim
      float mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < KT; ++e) {
        const float v = e <= lim ? __uint_as_float(sc[e]) * f : -INFINITY;
        sc[e] = __float_as_uint(v);
        mx = fmaxf(mx, v);
      }
      const bool move = mx > m + LA_TAU;   // also at the first tile (m = -inf)
      const float m_new = move ? mx : m;
      if (i > 0 && __any_sync(0xffffffffu, move)) {
        ok = __all_sync(0xffffffffu, mbar_wait(o_done((i - 1) & 1), (uint32_t)((i - 1) >> 1) & 1u, abort_flag));
        if (!ok) { if (lane == 0) give_up(35); break; }
        tc_fence_after();
        const float g = move ? exp2f((m - m_new) * kLog2e) : 1.0f;
        l *= g;
        for (int c = 0; c < 64 * nvb; c += 16) {
          uint32_t o[16];
          tmem_ld16(tlane + LA_COL_O + c, o);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * g);
          tmem_st16(tlane + LA_COL_O + c, o);
        }
      }
      m = m_new;
      if (i >= 2) {   // this P tile has been read
        ok = __all_sync(0xffffffffu, mbar_wait(o_done(i & 1), (uint32_t)((i - 2) >> 1) & 1u, abort_flag));
        if (!ok) { if (lane == 0) give_up(36); break; }
        tc_fence_after();
      }
#pragma unroll
      for (int c = 0; c < KT; c += 16) {
        float p[16];
        uint32_t w[8];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          p[e] = la_ex2((__uint_as_float(sc[c + e]) - m) * kLog2e);   // (hidden keys: 2^-inf = 0)
          l += p[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) w[e] = warp < 2 ? pack_bf16(p[2 * e], p[2 * e + 1]) : pack_bf16(bf16_lo(p[2 * e]), bf16_lo(p[2 * e + 1]));
        tmem_st8(tlane + LA_COL_P + 32 * (i & 1) + c / 2, w);
      }
      tmem_st_wait();
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full(i & 1));
    }
    if (ok && nt > 0) {   // the last product (and so all of them) is complete
      ok = __all_sync(0xffffffffu, mbar_wait(o_done((nt - 1) & 1), (uint32_t)((nt - 1) >> 1) & 1u, abort_flag));
      if (!ok && lane == 0) give_up(37);
      tc_fence_after();
    }
  }
  ok = __syncthreads_and(ok ? 1 : 0) != 0 && !*abort_flag;   // nothing reads the tiles any more: they become the exchange buffer
  float *ex = reinterpret_cast<float *>(sm);                 // [LA_H][LA_OLD]
  if (ok && warp < 4) {
    const uint32_t tlane = tmem_base + ((uint32_t)(warp * 32) << 16);
    float *mine = ex + (tid & 63) * LA_OLD;
    if (tid < LA_H) lsum[tid] = l;
    auto part = [&](bool add) {
      for (int c = 0; c < 64 * nvb; c += 16) {
        uint32_t o[16];
        if (nt > 0) {
          tmem_ld16(tlane + LA_COL_O + c, o);
          tmem_ld_wait();
        } else {
#pragma unroll
          for (int e = 0; e < 16; ++e) o[e] = 0u;
        }
#pragma unroll
        for (int e = 0; e < 16; e += 4) {
          float4 v = make_float4(__uint_as_float(o[e]), __uint_as_float(o[e + 1]), __uint_as_float(o[e + 2]), __uint_as_float(o[e + 3]));
          float4 *dst = reinterpret_cast<float4 *>(mine + c + e);
          if (add) { const float4 x = *dst; v = make_float4(x.x + v.x, x.y + v.y, x.z + v.z, x.w + v.w); }
          *dst = v;
        }
      }
    };
    if (warp >= 2) part(false);
    asm volatile("bar.sync 1, 128;" ::: "memory");
    if (warp < 2) part(true);
    if (out.splits > 1 && vb0 == 0 && tid < hn) {
      float *ml = out.ml + (((int64_t)split * out.rows + r) * a.H + h0 + tid) * 2;
      ml[0] = m;
      ml[1] = l;
    }
  }
  tc_fence_before();
  __syncthreads();
  if (ok) {
    const int cols = 64 * nvb, c0 = 64 * vb0;
    for (int i = tid; i < hn * cols; i += LA_THREADS) {
      const int h = i / cols, c = i % cols;
      const float v = c0 + c < a.Kp ? ex[h * LA_OLD + c] : 0.0f;   // (columns past the latent belong to the key part)
      if (out.splits == 1) st1(out.o, out.o_bf, ((int64_t)(h0 + h) * out.plane + r) * out.Kr + c0 + c, v / lsum[h]);
      else out.part[(((int64_t)split * out.rows + r) * a.H + h0 + h) * out.Kr + c0 + c] = v;
    }
  }
  if (warp == 5) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(512u) : "memory");
  }
}

// ---- host ---------------------------------------------------------------------------------------

static bool latent_tc(const caten_b200_ctx *ctx, const LatentArgs &a) {
  return a.cache_bf16 && ctx->attn_tc && ctx->encode_tiled && a.KC() <= 64 * LA_MAX_BLOCKS;
}
static int latent_tile(const LatentArgs &a) { return a.KC() <= 320 ? 64 : 32; }   // a ring of at least two tiles beside Q
static int64_t latent_ctas(const LatentArgs &a, bool tc, int64_t rows) {
  if (!tc) return (a.H + LS_H - 1) / LS_H * rows;
  return (int64_t)((a.H + LA_H - 1) / LA_H) * ((a.Kr / 64 + LA_VBLOCKS - 1) / LA_VBLOCKS) * rows;
}

int latent_splits(const caten_b200_ctx *ctx, const LatentArgs &a, int64_t rows, int64_t keys) {
  const bool tc = latent_tc(ctx, a);
  const int kt = tc ? latent_tile(a) : LS_KEYS;
  const int64_t tiles = (keys + kt - 1) / kt, ctas = latent_ctas(a, tc, rows), slots = (int64_t)ctx->sm_count * (tc ? 1 : 4);
  int best = 1;
  int64_t cost = INT64_MAX;
  for (int S = 1; S <= 32 && (S == 1 || tiles >= 2 * S); S = S < 4 ? S + 1 : S + S / 4) {
    // waves x (tiles of a CTA + what a CTA costs besides), and merging the parts
    const int64_t c = (ctas * S + slots - 1) / slots * ((tiles + S - 1) / S + 6) + (S > 1 ? 6 : 0);
    if (c < cost) { cost = c; best = S; }
  }
  return best;
}

typedef CUresult (*EncodeTiledFn)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *, const cuuint64_t *, const cuuint32_t *, const cuuint32_t *,
                                  CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

template <int KT>
static int launch_tc(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x, const LatentOut &out, dim3 grid) {
  const int KC = a.KC(), nkc = (KC + 63) / 64;
  const cuuint64_t dims[2] = {(cuuint64_t)KC, (cuuint64_t)(a.B * a.cap)}, strides[1] = {(cuuint64_t)KC * 2};
  const cuuint32_t box[2] = {64, KT}, estr[2] = {1, 1};
  CUtensorMap map;
  const CUresult e = ((EncodeTiledFn)ctx->encode_tiled)(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                                                        CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (e != CUDA_SUCCESS) return fail(ctx, CATEN_B200_ECUDA, "cuTensorMapEncodeTiled failed (%d)", (int)e);
  const size_t stage = (size_t)nkc * KT * 128, q = (size_t)nkc * 16384, tail = (2 * LA_MAX_STAGES + 7) * 8 + 16 + LA_H * 4;
  int stages = (int)((224 * 1024 - q) / stage);
  if (stages > LA_MAX_STAGES) stages = LA_MAX_STAGES;
  size_t tiles = q + stage * stages;
  if (tiles < (size_t)LA_H * LA_OLD * 4) tiles = (size_t)LA_H * LA_OLD * 4;
  const size_t smem = 1024 + tiles + tail;
  const uint32_t base = (1u << 4) | (1u << 7) | (1u << 10) | (8u << 24);   // fp32 accumulate, bf16 x bf16, M = 128
  const uint32_t idesc_s = base | ((uint32_t)(KT >> 3) << 17), idesc_pv = base | ((uint32_t)(64 >> 3) << 17) | (1u << 16);
  CB_CUDA(ctx, cudaFuncSetAttribute(latent_attn_tc_kernel<KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_k(ctx, latent_attn_tc_kernel<KT>, grid, dim3(LA_THREADS), smem, map, a, x.qcat_bf.hi ? nullptr : x.qcat, x.qcat_bf.hi, out, stages, idesc_s, idesc_pv, ctx->d_status);
  CB_LAUNCH_CHECK(ctx, "latent_attn_tc_kernel");
  return 0;
}

int launch_latent_absorbed(caten_b200_ctx *ctx, const LatentArgs &a, const LatentAbsorbed &x) {
  const int64_t rows = (int64_t)a.B * a.s;
  if (rows <= 0) return 0;
  if (int rc = check_latent(ctx, a)) return rc;
  if (rows > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "latent attention: %lld rows", (long long)rows);
  if (x.splits > 1 && (!x.part || !x.ml)) return fail(ctx, CATEN_B200_EINVAL, "latent attention: key splits need their buffers");
  LatentOut out;
  out.o = x.o; out.o_bf = x.o_bf; out.part = x.part; out.ml = x.ml; out.plane = x.plane; out.rows = rows; out.Kr = a.Kr; out.H = a.H; out.splits = x.splits;
  if (latent_tc(ctx, a)) {
    const dim3 grid((unsigned)(latent_ctas(a, true, 1)), (unsigned)rows, (unsigned)x.splits);
    if (int rc = latent_tile(a) == 64 ? launch_tc<64>(ctx, a, x, out, grid) : launch_tc<32>(ctx, a, x, out, grid)) return rc;
  } else {
    const size_t smem = (size_t)(LS_H * (a.KC() + LS_KEYS) + 3 * LS_H) * sizeof(float);
    launch_k(ctx, latent_attn_simt_kernel, dim3((unsigned)((a.H + LS_H - 1) / LS_H), (unsigned)rows, (unsigned)x.splits), dim3(LS_THREADS), smem, a, x.qcat, x.qcat_bf, out);
    CB_LAUNCH_CHECK(ctx, "latent_attn_simt_kernel");
  }
  if (x.splits > 1) {
    launch_k(ctx, latent_combine_kernel, dim3((unsigned)a.H, (unsigned)rows), dim3(128), 0, out);
    CB_LAUNCH_CHECK(ctx, "latent_combine_kernel");
  }
  return 0;
}

}  // namespace cb
