// Time mixing of RWKV kind: per head a matrix state S[key, value] in fp32,
//   o_t[j] = sum_i r_t[i] (S[i, j] + u[i] k_t[i] v_t[j]),     S[i, j] = w_t[i] S[i, j] + k_t[i] v_t[j]
//   w_t    = exp(-exp(d_t)),  d_t = W2 tanh(low rank) + w0
// then o is divided by its root mean square over the head, times a gain and silu(gate).
// The state starts at zero with the sequence (position 0) and is carried from step to step.
//
// Multi-token steps walk the tokens in order (fp32, no reordering of the recurrence), which is
// parallel over sequences, heads, value columns and keys: a thread keeps 4 KQ keys x CPT value
// columns of the state in registers, so a token costs three fused multiply-adds per element and one
// exchange over the few lanes that share a column, which is off the chain from token to token.
#include "wkv.cuh"

namespace cb {

namespace {

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float decay(float d) { return expf(-expf(d)); }

__device__ __forceinline__ void st_out(float *out, BfOut bf, int64_t at, float v) {
  if (bf.hi) {
    const __nv_bfloat16 h = __float2bfloat16_rn(v);
    bf.hi[at] = h;
    if (bf.lo) bf.lo[at] = __float2bfloat16_rn(v - __bfloat162float(h));
  } else {
    out[at] = v;
  }
}

__device__ __forceinline__ void cp16(float *dst, const float *src, bool ok) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}

}  // namespace

__global__ void __launch_bounds__(128) wkv_lowrank_kernel(const WkvArgs a, float *__restrict__ t, BfOut tb, const float *__restrict__ h,
                                                          float *__restrict__ shift, int w4) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const float *src = a.y + r * a.ld + 4 * (int64_t)a.gr;
  for (int j = threadIdx.x; j < a.w1; j += 128) st_out(t, tb, r * a.w1 + j, tanhf(src[j]));
  if (h && (int)(r % a.s) == a.s - 1) {
    const float4 *hr = reinterpret_cast<const float4 *>(h) + r * w4;
    float4 *st = reinterpret_cast<float4 *>(shift) + (r / a.s) * w4;
    for (int c = threadIdx.x; c < w4; c += 128) st[c] = hr[c];
  }
}

int launch_wkv_lowrank(caten_b200_ctx *ctx, const WkvArgs &a, float *t, BfOut tb, const float *h, float *shift, int width_p) {
  const int64_t rows = (int64_t)a.B * a.s;
  if (rows <= 0) return 0;
  if (rows > 0x7fffffff) return fail(ctx, CATEN_B200_EUNSUPPORTED, "wkv: too many rows");
  launch_k(ctx, wkv_lowrank_kernel, dim3((unsigned)rows), dim3(128), 0, a, t, tb, h, shift, width_p / 4);
  CB_LAUNCH_CHECK(ctx, "wkv_lowrank_kernel");
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Scan.  Grid (value column block, head, sequence), 128 threads: KS lanes share a column's keys (lane
// ks holds the float4 key groups ks, ks + KS, ...).  Tokens are staged TCH at a time in shared memory
// by cp.async, one chunk ahead; r, k and the decay are laid out [token][KS * 4 KQ] with zeros past the
// head's keys.
// ---------------------------------------------------------------------------------------------
constexpr int WS_THREADS = 128, WS_TCH = 16;

template <int KQ, int CPT>
__global__ void __launch_bounds__(WS_THREADS) wkv_scan_kernel(const WkvArgs a, const int KS) {
  extern __shared__ __align__(16) float sm[];
  const int KC = KS * 4 * KQ;                       // key capacity (>= Dp)
  const int VC = WS_THREADS / KS * CPT;             // value columns of this CTA
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int ks = tid % KS, vc = tid / KS * CPT;
  const int v0 = blockIdx.x * VC, h = blockIdx.y, b = blockIdx.z;
  const int Dp = a.Dp, s = a.s;
  const int vw = min(VC, Dp - v0);                  // a multiple of 4 (Dp % 16 == 0, VC % 4 == 0)
  // two buffers of r, k, decay [TCH][KC] and v [TCH][VC]; then u [KC] and sum_i r u k per token [TCH]
  const int buf_floats = WS_TCH * (3 * KC + VC);
  float *us = sm + 2 * buf_floats, *ruk = us + KC;
  pdl_enter();
  for (int i = tid; i < 2 * buf_floats; i += WS_THREADS) sm[i] = 0.0f;  // the pads stay zero
  for (int i = tid; i < KC; i += WS_THREADS) us[i] = i < Dp ? a.u[(int64_t)h * Dp + i] : 0.0f;
  __syncthreads();
  const int64_t row0 = (int64_t)b * s;
  const int d4 = Dp / 4, v4 = vw / 4, per_tok = 3 * d4 + v4;
  auto stage = [&](int t0, int buf) {
    float *base = sm + buf * buf_floats;
    for (int e = tid; e < WS_TCH * per_tok; e += WS_THREADS) {
      const int t = e / per_tok, c = e % per_tok;
      const bool ok = t0 + t < s;
      const int64_t row = row0 + (ok ? t0 + t : 0);
      const float *y = a.y + row * a.ld + (int64_t)h * Dp;
      if (c < d4) cp16(base + t * KC + 4 * c, y + 4 * c, ok);
      else if (c < 2 * d4) cp16(base + WS_TCH * KC + t * KC + 4 * (c - d4), y + a.gr + 4 * (c - d4), ok);
      else if (c < 3 * d4) cp16(base + 2 * WS_TCH * KC + t * KC + 4 * (c - 2 * d4), a.d + row * a.d_ld + (int64_t)h * Dp + 4 * (c - 2 * d4), ok);
      else cp16(base + 3 * WS_TCH * KC + t * VC + 4 * (c - 3 * d4), y + 2 * (int64_t)a.gr + v0 + 4 * (c - 3 * d4), ok);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  stage(0, 0);

  float S[CPT][4 * KQ];
  float *st = a.state + ((int64_t)b * a.H + h) * Dp * Dp + v0;
#pragma unroll
  for (int q = 0; q < KQ; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = 4 * (ks + KS * q) + e;
#pragma unroll
      for (int c = 0; c < CPT; ++c) S[c][4 * q + e] = a.n > 0 && key < Dp && vc + c < vw ? st[(int64_t)key * Dp + vc + c] : 0.0f;
    }

  for (int t0 = 0, buf = 0; t0 < s; t0 += WS_TCH, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // chunk staged; the other buffer has been consumed
    float *rs = sm + buf * buf_floats, *kk = rs + WS_TCH * KC, *ws = kk + WS_TCH * KC, *vs = ws + WS_TCH * KC;
    if (t0 + WS_TCH < s) stage(t0 + WS_TCH, buf ^ 1);
    for (int e = tid; e < WS_TCH * KC; e += WS_THREADS) ws[e] = decay(ws[e]);
    for (int t = warp; t < WS_TCH; t += WS_THREADS / 32) {
      float x = 0.0f;
      for (int i = lane; i < KC; i += 32) x = fmaf(rs[t * KC + i] * us[i], kk[t * KC + i], x);
      x = warp_sum(x);
      if (lane == 0) ruk[t] = x;
    }
    __syncthreads();
    const int tn = min(WS_TCH, s - t0);
#pragma unroll 4
    for (int t = 0; t < tn; ++t) {
      float o[CPT], v[CPT];
#pragma unroll
      for (int c = 0; c < CPT; ++c) {
        o[c] = 0.0f;
        v[c] = vs[t * VC + vc + c];
      }
#pragma unroll
      for (int q = 0; q < KQ; ++q) {
        const int at = t * KC + 4 * (ks + KS * q);
        const float4 r4 = *reinterpret_cast<const float4 *>(rs + at), k4 = *reinterpret_cast<const float4 *>(kk + at), w4 = *reinterpret_cast<const float4 *>(ws + at);
        const float rr[4] = {r4.x, r4.y, r4.z, r4.w}, kv[4] = {k4.x, k4.y, k4.z, k4.w}, ww[4] = {w4.x, w4.y, w4.z, w4.w};
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
          for (int c = 0; c < CPT; ++c) {
            o[c] = fmaf(rr[e], S[c][4 * q + e], o[c]);
            S[c][4 * q + e] = fmaf(ww[e], S[c][4 * q + e], kv[e] * v[c]);
          }
      }
#pragma unroll
      for (int c = 0; c < CPT; ++c)
        for (int m = KS >> 1; m > 0; m >>= 1) o[c] += __shfl_xor_sync(0xffffffffu, o[c], m);
      if (ks == 0) {
        float *op = a.o + (row0 + t0 + t) * a.o_ld + (int64_t)h * Dp + v0 + vc;
#pragma unroll
        for (int c = 0; c < CPT; ++c)
          if (vc + c < vw) op[c] = fmaf(v[c], ruk[t], o[c]);
      }
    }
    __syncthreads();  // ruk and this buffer are free
  }
#pragma unroll
  for (int q = 0; q < KQ; ++q)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = 4 * (ks + KS * q) + e;
#pragma unroll
      for (int c = 0; c < CPT; ++c)
        if (key < Dp && vc + c < vw) st[(int64_t)key * Dp + vc + c] = S[c][4 * q + e];
    }
}

// heads' norm and gate of one row: one warp per head
__global__ void __launch_bounds__(256) wkv_gate_kernel(const WkvArgs a) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int Dp = a.Dp;
  for (int h = warp; h < a.H; h += 8) {
    const float *o = a.o + r * a.o_ld + (int64_t)h * Dp, *g = a.y + r * a.ld + 3 * (int64_t)a.gr + (int64_t)h * Dp, *w = a.norm + (int64_t)h * Dp;
    float v[8], ss = 0.0f;
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = lane + 32 * i;
      v[i] = c < Dp ? o[c] : 0.0f;
      ss += v[i] * v[i];
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.D + a.eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = lane + 32 * i;
      if (c < Dp) st_out(a.out, a.bf, r * a.out_ld + (int64_t)h * Dp + c, v[i] * inv * w[c] * silu(g[c]));
    }
  }
}

static int check_wkv(caten_b200_ctx *ctx, const WkvArgs &a) {
  if (a.H <= 0 || a.D <= 0 || a.D > a.Dp || a.Dp % 16 || a.gr < a.H * a.Dp || a.n < 0) return fail(ctx, CATEN_B200_EINVAL, "wkv: bad shape");
  if (a.Dp > 256) return fail(ctx, CATEN_B200_EUNSUPPORTED, "wkv: head size above 256");
  if (a.H > 65535 || a.B > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "wkv: B or H > 65535");
  return 0;
}

template <int KQ, int CPT>
static int launch_scan_t(caten_b200_ctx *ctx, const WkvArgs &a) {
  int KS = 1;
  while (KS * 4 * KQ < a.Dp) KS *= 2;
  const int KC = KS * 4 * KQ, VC = WS_THREADS / KS * CPT;
  const size_t smem = ((size_t)2 * WS_TCH * (3 * KC + VC) + KC + WS_TCH) * sizeof(float);
  if (smem > 48 * 1024) CB_CUDA(ctx, cudaFuncSetAttribute(wkv_scan_kernel<KQ, CPT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_k(ctx, wkv_scan_kernel<KQ, CPT>, dim3((unsigned)((a.Dp + VC - 1) / VC), (unsigned)a.H, (unsigned)a.B), dim3(WS_THREADS), smem, a, KS);
  CB_LAUNCH_CHECK(ctx, "wkv_scan_kernel");
  return 0;
}

int launch_wkv_scan(caten_b200_ctx *ctx, const WkvArgs &a) {
  if (a.B <= 0 || a.s <= 0) return 0;
  if (int rc = check_wkv(ctx, a)) return rc;
  // few heads and sequences: fewer keys per thread, so that more warps share the work of a token
  const int64_t warps = (int64_t)a.B * a.H * ((a.Dp * a.Dp + 511) / 512);  // of 16 keys x 1 column per thread
  int rc;
  if (warps >= 16ll * ctx->sm_count) rc = launch_scan_t<4, 2>(ctx, a);
  else if (warps >= 4ll * ctx->sm_count) rc = launch_scan_t<4, 1>(ctx, a);
  else rc = launch_scan_t<2, 1>(ctx, a);
  if (rc) return rc;
  launch_k(ctx, wkv_gate_kernel, dim3((unsigned)((int64_t)a.B * a.s)), dim3(256), 0, a);
  CB_LAUNCH_CHECK(ctx, "wkv_gate_kernel");
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Single-token step: one CTA per (head, sequence) reads and writes the head's state once.  The first
// state rows are requested before the decay is formed.
// ---------------------------------------------------------------------------------------------
constexpr int WD_THREADS = 256, WD_U = 4;

__global__ void __launch_bounds__(WD_THREADS) wkv_decode_kernel(const WkvArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int Dp = a.Dp, h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *r = sm, *k = r + Dp, *v = k + Dp, *w = v + Dp, *g = w + Dp, *t = g + Dp, *red = t + a.w1, *part = red + 8;
  const int d4 = Dp / 4, RP = WD_THREADS / d4;    // state rows per pass
  const int vq = tid % d4, kr = tid / d4;
  const bool on = kr < RP;
  float4 *st = reinterpret_cast<float4 *>(a.state + ((int64_t)b * a.H + h) * Dp * Dp);
  pdl_enter();
  const bool fresh = (a.d_n ? *a.d_n : a.n) == 0;
  float4 s[WD_U];
  auto load = [&](int base) {
#pragma unroll
    for (int i = 0; i < WD_U; ++i) {
      const int key = base + kr + RP * i;
      s[i] = on && key < Dp && !fresh ? st[(int64_t)key * d4 + vq] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(0);
  auto proj = [&](int col) { return a.pin.splits > 0 ? partin_load1(a.pin, b, col) : a.y[(int64_t)b * a.ld + col]; };
  for (int i = tid; i < 4 * Dp; i += WD_THREADS) {
    const int which = i / Dp, c = i - which * Dp;
    (which == 0 ? r : which == 1 ? k : which == 2 ? v : g)[c] = proj(which * a.gr + h * Dp + c);
  }
  for (int j = tid; j < a.w1; j += WD_THREADS) t[j] = tanhf(proj(4 * a.gr + j));
  __syncthreads();
  // decay: eight lanes per channel, each 8 weights (16 bytes) at a time
  for (int c = tid >> 3; c < Dp; c += WD_THREADS / 8) {
    const __nv_bfloat16 *wr = a.w2 + ((int64_t)h * Dp + c) * a.w1;
    float x = 0.0f;
    for (int j = (tid & 7) * 8; j < a.w1; j += 64) {
      const uint4 q = *reinterpret_cast<const uint4 *>(wr + j);
      const uint32_t qq[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        x = fmaf(__uint_as_float(qq[e] << 16), t[j + 2 * e], x);
        x = fmaf(__uint_as_float(qq[e] & 0xFFFF0000u), t[j + 2 * e + 1], x);
      }
    }
    x += __shfl_xor_sync(0xffffffffu, x, 4);
    x += __shfl_xor_sync(0xffffffffu, x, 2);
    x += __shfl_xor_sync(0xffffffffu, x, 1);
    if ((tid & 7) == 0) w[c] = decay(x + a.w0[(int64_t)h * Dp + c]);
  }
  float x = 0.0f;
  for (int i = tid; i < Dp; i += WD_THREADS) x = fmaf(r[i] * a.u[(int64_t)h * Dp + i], k[i], x);
  x = warp_sum(x);
  if (lane == 0) red[warp] = x;
  __syncthreads();
  float ruk = red[0];
#pragma unroll
  for (int i = 1; i < WD_THREADS / 32; ++i) ruk += red[i];
  float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 vv = on ? reinterpret_cast<const float4 *>(v)[vq] : o;
  for (int base = 0; base < Dp; base += WD_U * RP) {
    if (base) load(base);
#pragma unroll
    for (int i = 0; i < WD_U; ++i) {
      const int key = base + kr + RP * i;
      if (on && key < Dp) {
        const float rk = r[key], kk = k[key], wk = w[key];
        o.x = fmaf(rk, s[i].x, o.x); o.y = fmaf(rk, s[i].y, o.y); o.z = fmaf(rk, s[i].z, o.z); o.w = fmaf(rk, s[i].w, o.w);
        st[(int64_t)key * d4 + vq] = make_float4(fmaf(wk, s[i].x, kk * vv.x), fmaf(wk, s[i].y, kk * vv.y), fmaf(wk, s[i].z, kk * vv.z), fmaf(wk, s[i].w, kk * vv.w));
      }
    }
  }
  if (on) reinterpret_cast<float4 *>(part + kr * Dp)[vq] = o;
  __syncthreads();
  float ov = 0.0f;
  if (tid < Dp) {
    for (int i = 0; i < RP; ++i) ov += part[i * Dp + tid];
    ov = fmaf(v[tid], ruk, ov);
  }
  float ss = warp_sum(ov * ov);  // threads past the head hold zero
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = red[0];
#pragma unroll
  for (int i = 1; i < WD_THREADS / 32; ++i) ss += red[i];
  if (tid < Dp) {
    const float inv = 1.0f / sqrtf(ss / (float)a.D + a.eps);
    st_out(a.out, a.bf, (int64_t)b * a.out_ld + (int64_t)h * Dp + tid, ov * inv * a.norm[(int64_t)h * Dp + tid] * silu(g[tid]));
  }
}

int launch_wkv_decode(caten_b200_ctx *ctx, const WkvArgs &a) {
  if (a.B <= 0) return 0;
  if (int rc = check_wkv(ctx, a)) return rc;
  if (a.w1 % 8) return fail(ctx, CATEN_B200_EINVAL, "wkv: the decay's low-rank width must be padded to a multiple of 8");
  const int RP = WD_THREADS / (a.Dp / 4);
  const size_t smem = ((size_t)5 * a.Dp + a.w1 + 8 + (size_t)RP * a.Dp) * sizeof(float);
  if (smem > 48 * 1024) CB_CUDA(ctx, cudaFuncSetAttribute(wkv_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_k(ctx, wkv_decode_kernel, dim3((unsigned)a.H, (unsigned)a.B), dim3(WD_THREADS), smem, a);
  CB_LAUNCH_CHECK(ctx, "wkv_decode_kernel");
  return 0;
}

}  // namespace cb

using namespace cb;

extern "C" int caten_b200_wkv(caten_b200_ctx *ctx, const caten_b200_wkv_desc *c, const float *d_y, float *d_state, float *d_out, int64_t B,
                              int64_t s, int64_t n, int precision) {
  if (!ctx) return fail(nullptr, CATEN_B200_EINVAL, "wkv: ctx is NULL");
  cudaSetDevice(ctx->device);
  if (!c || !d_y || !d_state || !d_out || !c->w0 || !c->u || !c->norm || !c->w2) return fail(ctx, CATEN_B200_EINVAL, "wkv: NULL argument");
  WkvArgs a;
  a.H = c->heads; a.D = c->dim; a.Dp = (c->dim + 15) / 16 * 16;
  const int64_t hd = ((int64_t)a.H * a.Dp + 63) / 64 * 64;
  if (B < 0 || s < 0 || n < 0 || n + s > 0x7fffffff || c->heads <= 0 || c->dim <= 0 || c->group_rows % 4 || c->low_rank <= 0 || c->low_rank % 64 || c->w2->type != CATEN_B200_BF16 ||
      c->w2->rows != hd || c->w2->cols != c->low_rank)
    return fail(ctx, CATEN_B200_EINVAL, "wkv: bad shape");
  if (precision < CATEN_B200_PREC_FP32 || precision > CATEN_B200_PREC_BF16X3) return fail(ctx, CATEN_B200_EINVAL, "wkv: unknown precision %d", precision);
  if (B == 0 || s == 0) return 0;
  a.y = d_y; a.gr = c->group_rows; a.w1 = c->low_rank; a.ld = 4ll * a.gr + a.w1;
  a.w2 = (const __nv_bfloat16 *)c->w2->qs; a.w0 = c->w0; a.u = c->u; a.norm = c->norm; a.eps = c->eps;
  a.state = d_state; a.out = d_out; a.out_ld = hd;
  a.B = (int)B; a.s = (int)s; a.n = (int)n;
  if (s == 1) {
    ProfScope prof(ctx, CATEN_B200_K_WKV);
    return launch_wkv_decode(ctx, a);
  }
  const int64_t R = B * s;
  const size_t t_b = (size_t)(R * a.w1) * 4, d_b = (size_t)(R * hd) * 4;
  auto al = [](size_t b) { return (b + 255) / 256 * 256; };
  if (int rc = scratch_reserve(ctx, &ctx->wkv_tmp, al(t_b) + 2 * al(d_b) + al((size_t)hd * 4))) return rc;
  uint8_t *base = (uint8_t *)ctx->wkv_tmp.ptr;
  float *t = (float *)base, *d = (float *)(base + al(t_b)), *o = (float *)(base + al(t_b) + al(d_b)), *w0 = (float *)(base + al(t_b) + 2 * al(d_b));
  CB_CUDA(ctx, cudaMemsetAsync(w0, 0, (size_t)hd * 4, ctx->stream));
  CB_CUDA(ctx, cudaMemcpyAsync(w0, c->w0, (size_t)a.H * a.Dp * 4, cudaMemcpyDeviceToDevice, ctx->stream));
  if (int rc = launch_wkv_lowrank(ctx, a, t, BfOut(), nullptr, nullptr, 0)) return rc;
  if (int rc = model_linear(ctx, precision, c->w2, t, BfOut(), w0, nullptr, CATEN_B200_ACT_NONE, d, BfOut(), R)) return rc;
  a.d = d; a.d_ld = hd; a.o = o; a.o_ld = hd;
  ProfScope prof(ctx, CATEN_B200_K_WKV);
  return launch_wkv_scan(ctx, a);
}
