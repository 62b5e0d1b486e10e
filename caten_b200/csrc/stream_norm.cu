// The residual stream of a decoder with RMS norms before and after every sublayer, one kernel per
// sublayer boundary.  A row (one CTA of 256 threads, the row in registers) goes through two stages:
//
//   in    how the stream's row is formed
//           EMBED  a row of the token embedding (kept in x0 as well when a later stage needs it)
//           COPY   the output y of a linear
//           ADD    x + y * post / rms(y)          (norm of the sublayer's output, then the residual sum)
//           SUM    x + y [+ the outputs of the row's experts]
//           KEEP   x as it is
//   out   what the next operation reads
//           NORM   x * pre / rms(x)
//           NORM2  x * w1 / rms(x) and x * w2 / rms(x), a gain per coordinate (mixer and feed-forward side by side);
//                  before that the row may get the step vector of a loop pass and the embedding output
//           SHIFT  NORM, then the five token-shift mixes h + (h_prev - h) * mu of a time-mixing layer
//                  (single-token steps: h_prev comes from the carried state, which becomes h)
//           CONCAT [x ; x0]
//           NONE   nothing: the row is only stored
//
// rms(v) = sqrt(mean(v^2) + eps).  y may still be the split-K partial tiles of the linear that
// produced it (PartIn).  x, norms and sums are fp32; the operand of the next linear is written as
// bf16 (hi, lo) or fp32.  Rows are `width` long in buffers padded with zeros to 4 * d4 floats.
#include "common.cuh"
#include "stream_norm.cuh"

namespace cb {

constexpr int SN_THREADS = 256;

__device__ __forceinline__ float sn_block_sum(float v, float *red) {
  v = warp_sum(v);
  __syncthreads();  // protects `red` from the previous use
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = red[0];
#pragma unroll
  for (int w = 1; w < SN_THREADS / 32; ++w) t += red[w];
  return t;
}

__device__ __forceinline__ float sq4(float4 v) { return (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w); }

// operand element group c (float4) at offset `at4` (in float4) of the output
__device__ __forceinline__ void sn_store(float *h, BfOut hb, int64_t at4, float4 v) {
  if (hb.hi) {
    reinterpret_cast<uint2 *>(hb.hi)[at4] = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    if (hb.lo)
      reinterpret_cast<uint2 *>(hb.lo)[at4] = make_uint2(pack_bf16(bf16_lo(v.x), bf16_lo(v.y)), pack_bf16(bf16_lo(v.z), bf16_lo(v.w)));
  } else {
    reinterpret_cast<float4 *>(h)[at4] = v;
  }
}

__device__ __forceinline__ float4 mix4(float4 h, float4 p, float4 mu) {
  return make_float4(fmaf(p.x - h.x, mu.x, h.x), fmaf(p.y - h.y, mu.y, h.y), fmaf(p.z - h.z, mu.z, h.z), fmaf(p.w - h.w, mu.w, h.w));
}

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 mul4(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }

template <int IN, int OUT, int MAXV>
__global__ void __launch_bounds__(SN_THREADS) stream_norm_kernel(const StreamArgs a) {
  __shared__ float red[SN_THREADS / 32];
  pdl_enter();
  const int64_t row = blockIdx.x;
  const int64_t src = a.rows ? a.rows[row] : (a.src_stride > 1 ? (row + 1) * a.src_stride - 1 : row);
  const int d4 = a.d4;
  float4 v[MAXV];
  if (IN == SN_EMBED) {
    const int64_t tok = a.ids[(src / a.s) * a.ids_ld + src % a.s];
    const bool ok = tok >= 0 && tok < a.vocab;
    const uint2 *e = reinterpret_cast<const uint2 *>(a.table) + (ok ? tok : 0) * d4;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) {
        const uint2 w = ok ? e[c] : make_uint2(0u, 0u);
        v[i] = make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xFFFF0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xFFFF0000u));
      }
    }
  } else if (IN == SN_KEEP) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) v[i] = reinterpret_cast<const float4 *>(a.x)[src * d4 + c];
    }
  } else {
    // v holds y first; the partial tiles of a split-K linear are fetched together (the kernel is a chain of latencies)
    float4 xr[MAXV];
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) {
        if (IN == SN_ADD || IN == SN_SUM) xr[i] = reinterpret_cast<const float4 *>(a.x)[src * d4 + c];
        v[i] = a.pin.splits > 0 ? partin_load4(a.pin, src, 4 * c) : reinterpret_cast<const float4 *>(a.y)[src * d4 + c];
      }
    }
    if (IN == SN_ADD) {
      float sq = 0.0f;
#pragma unroll
      for (int i = 0; i < MAXV; ++i)
        if (threadIdx.x + SN_THREADS * i < d4) sq += sq4(v[i]);
      const float rs = a.post / sqrtf(sn_block_sum(sq, red) * a.invd + a.eps);
#pragma unroll
      for (int i = 0; i < MAXV; ++i) {
        if (threadIdx.x + SN_THREADS * i < d4) {
          v[i].x = fmaf(v[i].x, rs, xr[i].x);
          v[i].y = fmaf(v[i].y, rs, xr[i].y);
          v[i].z = fmaf(v[i].z, rs, xr[i].z);
          v[i].w = fmaf(v[i].w, rs, xr[i].w);
        }
      }
    }
    if (IN == SN_SUM) {
      for (int k = 0; k < a.top; ++k) {
        const int64_t p = a.pos ? a.pos[src * a.top + k] : src * a.top + k;
#pragma unroll
        for (int i = 0; i < MAXV; ++i) {
          const int c = threadIdx.x + SN_THREADS * i;
          if (c < d4) v[i] = add4(v[i], reinterpret_cast<const float4 *>(a.ye)[p * d4 + c]);
        }
      }
#pragma unroll
      for (int i = 0; i < MAXV; ++i)
        if (threadIdx.x + SN_THREADS * i < d4) v[i] = add4(xr[i], v[i]);
    }
  }
  if (IN == SN_EMBED && a.x_out && a.x0) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) reinterpret_cast<float4 *>(a.x0)[src * d4 + c] = v[i];
    }
  }
  if (OUT == SN_NORM2 && a.step) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) {
        if (a.add_x0) v[i] = add4(v[i], reinterpret_cast<const float4 *>(a.x0)[src * d4 + c]);
        v[i] = add4(v[i], reinterpret_cast<const float4 *>(a.step)[c]);
      }
    }
  }
  if ((IN != SN_KEEP || (OUT == SN_NORM2 && a.step)) && a.x_out) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) reinterpret_cast<float4 *>(a.x_out)[src * d4 + c] = v[i];
    }
  }
  if (OUT == SN_NORM || OUT == SN_SHIFT) {
    float sq = 0.0f;
#pragma unroll
    for (int i = 0; i < MAXV; ++i)
      if (threadIdx.x + SN_THREADS * i < d4) sq += sq4(v[i]);
    const float rs = a.pre / sqrtf(sn_block_sum(sq, red) * a.invd + a.eps);
    const bool fresh = OUT == SN_SHIFT && (a.d_n ? *a.d_n : a.n) == 0;  // first token: the one before it is zero
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) {
        const float4 h = make_float4(v[i].x * rs, v[i].y * rs, v[i].z * rs, v[i].w * rs);
        if (OUT == SN_NORM) {
          sn_store(a.h, a.hb, row * d4 + c, h);
        } else {
          float4 *st = reinterpret_cast<float4 *>(a.shift) + row * d4 + c;
          const float4 p = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *st;
          *st = h;
#pragma unroll
          for (int j = 0; j < 5; ++j) {
            const float4 mu = reinterpret_cast<const float4 *>(a.mu)[j * d4 + c];
            sn_store(a.h, a.hb, (j * a.plane + row) * d4 + c, mix4(h, p, mu));
          }
        }
      }
    }
  }
  if (OUT == SN_NORM2) {
    float sq = 0.0f;
#pragma unroll
    for (int i = 0; i < MAXV; ++i)
      if (threadIdx.x + SN_THREADS * i < d4) sq += sq4(v[i]);
    const float rs = 1.0f / sqrtf(sn_block_sum(sq, red) * a.invd + a.eps);
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) {
        const float4 u = make_float4(v[i].x * rs, v[i].y * rs, v[i].z * rs, v[i].w * rs);
        sn_store(a.h, a.hb, row * d4 + c, mul4(u, reinterpret_cast<const float4 *>(a.w1)[c]));
        if (a.w2) sn_store(a.h, a.hb, (a.plane + row) * d4 + c, mul4(u, reinterpret_cast<const float4 *>(a.w2)[c]));
      }
    }
  }
  if (OUT == SN_CONCAT) {
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
      const int c = threadIdx.x + SN_THREADS * i;
      if (c < d4) {
        sn_store(a.h, a.hb, row * 2 * d4 + c, v[i]);
        const float4 e = IN == SN_EMBED ? v[i] : reinterpret_cast<const float4 *>(a.x0)[src * d4 + c];
        sn_store(a.h, a.hb, row * 2 * d4 + d4 + c, e);
      }
    }
  }
}

template <int IN, int OUT>
static int launch_sn(caten_b200_ctx *ctx, const StreamArgs &a, int64_t rows) {
  const dim3 g((unsigned)rows), b(SN_THREADS);
  if (a.d4 <= SN_THREADS) launch_k(ctx, stream_norm_kernel<IN, OUT, 1>, g, b, 0, a);
  else if (a.d4 <= 2 * SN_THREADS) launch_k(ctx, stream_norm_kernel<IN, OUT, 2>, g, b, 0, a);
  else if (a.d4 <= 4 * SN_THREADS) launch_k(ctx, stream_norm_kernel<IN, OUT, 4>, g, b, 0, a);
  else launch_k(ctx, stream_norm_kernel<IN, OUT, 8>, g, b, 0, a);
  CB_LAUNCH_CHECK(ctx, "stream_norm_kernel");
  return 0;
}

template <int IN>
static int launch_sn_in(caten_b200_ctx *ctx, int out, const StreamArgs &a, int64_t rows) {
  switch (out) {
    case SN_NORM: return launch_sn<IN, SN_NORM>(ctx, a, rows);
    case SN_SHIFT: return launch_sn<IN, SN_SHIFT>(ctx, a, rows);
    case SN_CONCAT: return launch_sn<IN, SN_CONCAT>(ctx, a, rows);
    default: return launch_sn<IN, SN_NONE>(ctx, a, rows);
  }
}

int launch_stream_norm(caten_b200_ctx *ctx, int in, int out, const StreamArgs &a, int64_t rows) {
  if (rows <= 0) return 0;
  if (a.d4 < 1 || a.d4 > 8 * SN_THREADS) return fail(ctx, CATEN_B200_EUNSUPPORTED, "stream_norm: width %d (at most 8192)", 4 * a.d4);
  if (rows > 0x7fffffff) return fail(ctx, CATEN_B200_EUNSUPPORTED, "stream_norm: too many rows");
  if (out == SN_NORM2 || in == SN_SUM) {   // the pairs a decoder with parallel sublayers uses
    if (out == SN_NORM2 && in == SN_EMBED) return launch_sn<SN_EMBED, SN_NORM2>(ctx, a, rows);
    if (out == SN_NORM2 && in == SN_KEEP) return launch_sn<SN_KEEP, SN_NORM2>(ctx, a, rows);
    if (out == SN_NORM2 && in == SN_SUM) return launch_sn<SN_SUM, SN_NORM2>(ctx, a, rows);
    if (out == SN_NONE && in == SN_SUM) return launch_sn<SN_SUM, SN_NONE>(ctx, a, rows);
    return fail(ctx, CATEN_B200_EUNSUPPORTED, "stream_norm: stages %d, %d", in, out);
  }
  switch (in) {
    case SN_EMBED: return launch_sn_in<SN_EMBED>(ctx, out, a, rows);
    case SN_COPY: return launch_sn_in<SN_COPY>(ctx, out, a, rows);
    case SN_ADD: return launch_sn_in<SN_ADD>(ctx, out, a, rows);
    default: return launch_sn_in<SN_KEEP>(ctx, out, a, rows);
  }
}

// Token-shift mixes of a multi-token step: row r = (sequence, token i) of h mixes with the row before it; token 0 with
// the state carried from the step before (zeros when the sequence starts here).
__global__ void __launch_bounds__(SN_THREADS) token_shift_kernel(const float *__restrict__ h, const float *__restrict__ shift,
                                                                 const float *__restrict__ mu, int s, int n, int d4, int64_t plane,
                                                                 float *__restrict__ out, BfOut ob) {
  pdl_enter();
  const int64_t row = blockIdx.x;
  const int i = (int)(row % s);
  const float4 *hr = reinterpret_cast<const float4 *>(h) + row * d4;
  const float4 *pr = i > 0 ? hr - d4 : (n > 0 ? reinterpret_cast<const float4 *>(shift) + (row / s) * d4 : nullptr);
  for (int c = threadIdx.x; c < d4; c += SN_THREADS) {
    const float4 v = hr[c], p = pr ? pr[c] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < 5; ++j) sn_store(out, ob, (j * plane + row) * d4 + c, mix4(v, p, reinterpret_cast<const float4 *>(mu)[j * d4 + c]));
  }
}

int launch_token_shift(caten_b200_ctx *ctx, const float *h, const float *shift, const float *mu, int64_t B, int64_t s, int64_t n, int d4,
                       int64_t plane, float *out, BfOut ob) {
  if (B * s <= 0) return 0;
  if (B * s > 0x7fffffff) return fail(ctx, CATEN_B200_EUNSUPPORTED, "token_shift: too many rows");
  launch_k(ctx, token_shift_kernel, dim3((unsigned)(B * s)), dim3(SN_THREADS), 0, h, shift, mu, (int)s, (int)n, d4, plane, out, ob);
  CB_LAUNCH_CHECK(ctx, "token_shift_kernel");
  return 0;
}

}  // namespace cb
