// Time mixing of RWKV kind: per head a matrix state S[key, value] in fp32,
//   o_t[j] = sum_i r_t[i] (S[i, j] + u[i] k_t[i] v_t[j]),     S[i, j] = w_t[i] S[i, j] + k_t[i] v_t[j]
//   w_t    = exp(-exp(d_t)),  d_t = W2 tanh(low rank) + w0
// then o is divided by its root mean square over the head, times a gain and silu(gate).
// The state starts at zero with the sequence (position 0) and is carried from step to step.
//
// Prompts (heads up to 64) are computed in chunks of 64 tokens, all of them at once: within a chunk the
// output is a causal matrix product and the state's contribution another, so only the chunk states form a
// chain.  Everything stays fp32, and every decay factor is the exponential of a sum of non-positive
// numbers (never a quotient of two cumulative products, which could underflow).
//
// Short multi-token steps, and wider heads, walk the tokens in order: a thread keeps 4 KQ keys x CPT value
// columns of the state in registers, so a token costs three fused multiply-adds per element and one
// exchange over the few lanes that share a column, which is off the chain from token to token.
#include "wkv.cuh"

namespace cb {

namespace {

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

// ---------------------------------------------------------------------------------------------
// Chunked form.  With e = -log w, subchunks of 16 tokens, and for token t of subchunk a
//   P_t = sum of e before t in a,  Q_t = sum of e after t in a,  tot_a = sum of e in a:
//   out from earlier tokens s of subchunk b < a:  sum_i r_t k_s exp(-P_t - Q_s - tot_{b+1} - .. - tot_{a-1})
//   out from earlier tokens of the same subchunk: the same with segments of 8, 4 and 2 tokens in place of
//     subchunks (every pair of tokens is split by exactly one level's segment boundary)
//   out from the state before the chunk:          r_t exp(-P_t - tot_0 - .. - tot_{a-1}) . S
//   the chunk's contribution to the state:        k_s exp(-Q_s - tot_{b+1} - .. - tot_3) v_s
// wkv_chunk_kernel: the first two, the contribution U, and exp(-sum tot); leaves the scaled r in d.
// wkv_states_kernel: walks the chunks, replacing U by the state before the chunk.
// wkv_out_kernel: adds the state's part, then the head's norm and the gate.
// ---------------------------------------------------------------------------------------------
constexpr int WC_T = 64, WC_D = 64, WC_LD = 68, WC_THREADS = 256;   // tokens per chunk, head size, row pitch in shared memory
constexpr size_t WC_SMEM = (size_t)(6 * WC_T * WC_LD + 2 * 4 * WC_D) * sizeof(float);

__device__ __forceinline__ float exp_neg(float x) { return exp2f(-1.4426950408889634f * x); }

__device__ __forceinline__ float dot_rows(const float *p, const float *q) {
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < WC_D; i += 4) {
    const float4 x = *reinterpret_cast<const float4 *>(p + i), y = *reinterpret_cast<const float4 *>(q + i);
    acc.x = fmaf(x.x, y.x, acc.x); acc.y = fmaf(x.y, y.y, acc.y); acc.z = fmaf(x.z, y.z, acc.z); acc.w = fmaf(x.w, y.w, acc.w);
  }
  return (acc.x + acc.y) + (acc.z + acc.w);
}

// One subchunk's channel at segment length 2 M: tokens of a segment's first half carry k decayed to its middle, those of
// the second half r decayed from it (16 tokens, e in registers).
template <int M>
__device__ __forceinline__ void split_level(const float *ev, const float *r, const float *k, float *x) {
#pragma unroll
  for (int seg = 0; seg < 16; seg += 2 * M) {
    float sum = 0.0f;
#pragma unroll
    for (int j = seg + M - 1; j >= seg; --j) {
      x[j * WC_LD] = k[j * WC_LD] * exp_neg(sum);
      sum += ev[j];
    }
    sum = 0.0f;
#pragma unroll
    for (int j = seg + M; j < seg + 2 * M; ++j) {
      x[j * WC_LD] = r[j * WC_LD] * exp_neg(sum);
      sum += ev[j];
    }
  }
}

__global__ void __launch_bounds__(WC_THREADS, 2) wkv_chunk_kernel(const WkvArgs a, float *__restrict__ U, float *__restrict__ decays) {
  extern __shared__ __align__(16) float sm[];
  float *rs = sm, *ks = rs + WC_T * WC_LD, *vs = ks + WC_T * WC_LD, *ws = vs + WC_T * WC_LD, *xs = ws + WC_T * WC_LD, *As = xs + WC_T * WC_LD;
  float *tot = As + WC_T * WC_LD;   // [4][WC_D] sums of e per subchunk
  float *g = tot + 4 * WC_D;        // [4][WC_D] exp(-tot)
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, Dp = a.Dp;
  const int t0 = c * WC_T, tn = min(WC_T, a.s - t0);
  const int64_t row0 = (int64_t)b * a.s + t0;
  pdl_enter();
  // tokens past the end and channels past the head: r = k = v = 0 and no decay
  for (int e = tid; e < 4 * WC_T * (WC_D / 4); e += WC_THREADS) {
    const int which = e >> 10, t = (e >> 4) & 63, c4 = e & 15;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool ok = t < tn && 4 * c4 < Dp;
    if (ok) {
      const float *src = which < 3 ? a.y + (row0 + t) * a.ld + (int64_t)which * a.gr + (int64_t)h * Dp : a.d + (row0 + t) * a.d_ld + (int64_t)h * Dp;
      v = reinterpret_cast<const float4 *>(src)[c4];
      if (which == 3) v = make_float4(expf(v.x), expf(v.y), expf(v.z), expf(v.w));
    }
    *reinterpret_cast<float4 *>((which == 0 ? rs : which == 1 ? ks : which == 2 ? vs : ws) + t * WC_LD + 4 * c4) = v;
  }
  __syncthreads();
  const int sub = tid >> 6, ch = tid & 63;   // this thread's subchunk and channel in the element-wise passes
  const float *rc = rs + 16 * sub * WC_LD + ch, *kc = ks + 16 * sub * WC_LD + ch;
  float ev[16];
  {
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      ev[j] = ws[(16 * sub + j) * WC_LD + ch];
      sum += ev[j];
    }
    tot[sub * WC_D + ch] = sum;
    g[sub * WC_D + ch] = exp_neg(sum);
    split_level<8>(ev, rc, kc, ws + 16 * sub * WC_LD + ch);   // (a thread's own elements of ws)
    split_level<4>(ev, rc, kc, xs + 16 * sub * WC_LD + ch);
  }
  __syncthreads();
  // ---- same subchunk, one pair of tokens (t, s < t) per thread and level ----
  {
    const int bl = tid >> 6, t8 = (tid >> 3) & 7, s8 = tid & 7;
    As[(16 * bl + 8 + t8) * WC_LD + 16 * bl + s8] = dot_rows(ws + (16 * bl + 8 + t8) * WC_LD, ws + (16 * bl + s8) * WC_LD);
    if (tid < 128) {
      const int base = 8 * (tid >> 4), t = base + 4 + ((tid >> 2) & 3), s_ = base + (tid & 3);
      As[t * WC_LD + s_] = dot_rows(xs + t * WC_LD, xs + s_ * WC_LD);
    } else if (tid < 192) {   // the token itself, with the bonus
      const int t = tid - 128;
      float acc = 0.0f;
#pragma unroll 4
      for (int i = 0; i < Dp; i += 4) {
        const float4 k4 = *reinterpret_cast<const float4 *>(ks + t * WC_LD + i), r4 = *reinterpret_cast<const float4 *>(rs + t * WC_LD + i);
        const float4 u4 = *reinterpret_cast<const float4 *>(a.u + (int64_t)h * Dp + i);
        acc = fmaf(r4.x * u4.x, k4.x, fmaf(r4.y * u4.y, k4.y, fmaf(r4.z * u4.z, k4.z, fmaf(r4.w * u4.w, k4.w, acc))));
      }
      As[t * WC_LD + t] = acc;
      for (int s_ = t + 1; s_ < (t | 15) + 1; ++s_) As[t * WC_LD + s_] = 0.0f;   // later tokens of the subchunk do not reach back
    } else if (tid < 224) {   // neighbours: nothing decays in between
      const int s_ = 2 * (tid - 192);
      As[(s_ + 1) * WC_LD + s_] = dot_rows(rs + (s_ + 1) * WC_LD, ks + s_ * WC_LD);
    }
  }
  __syncthreads();
  split_level<2>(ev, rc, kc, ws + 16 * sub * WC_LD + ch);
  __syncthreads();
  if (tid < 64) {
    const int base = 4 * (tid >> 2), t = base + 2 + ((tid >> 1) & 1), s_ = base + (tid & 1);
    As[t * WC_LD + s_] = dot_rows(ws + t * WC_LD, ws + s_ * WC_LD);
  }
  // ---- r_t exp(-P_t), k_t exp(-Q_t) ----
  {
    float sum = 0.0f;
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      rs[(16 * sub + j) * WC_LD + ch] *= exp_neg(sum);
      sum += ev[j];
    }
    sum = 0.0f;
#pragma unroll
    for (int j = 15; j >= 0; --j) {
      ks[(16 * sub + j) * WC_LD + ch] *= exp_neg(sum);
      sum += ev[j];
    }
  }
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  // ---- earlier subchunks: thread (ty, tx) owns (token ty of subchunk a, token tx of subchunk b) for all a > b ----
  {
    float a10 = 0.f, a21 = 0.f, a32 = 0.f, a20 = 0.f, a31 = 0.f, a30 = 0.f;
#pragma unroll 4
    for (int i = 0; i < WC_D; i += 4) {
      const float4 g1 = *reinterpret_cast<const float4 *>(g + WC_D + i), g2 = *reinterpret_cast<const float4 *>(g + 2 * WC_D + i);
      float4 r[4], k[3];
#pragma unroll
      for (int j = 1; j < 4; ++j) r[j] = *reinterpret_cast<const float4 *>(rs + (ty + 16 * j) * WC_LD + i);
#pragma unroll
      for (int j = 0; j < 3; ++j) k[j] = *reinterpret_cast<const float4 *>(ks + (tx + 16 * j) * WC_LD + i);
#define WC_DOT(acc, R, K) acc = fmaf((R).x, (K).x, fmaf((R).y, (K).y, fmaf((R).z, (K).z, fmaf((R).w, (K).w, acc))))
      WC_DOT(a10, r[1], k[0]);
      WC_DOT(a21, r[2], k[1]);
      WC_DOT(a32, r[3], k[2]);
      k[0].x *= g1.x; k[0].y *= g1.y; k[0].z *= g1.z; k[0].w *= g1.w;
      k[1].x *= g2.x; k[1].y *= g2.y; k[1].z *= g2.z; k[1].w *= g2.w;
      WC_DOT(a20, r[2], k[0]);
      WC_DOT(a31, r[3], k[1]);
      k[0].x *= g2.x; k[0].y *= g2.y; k[0].z *= g2.z; k[0].w *= g2.w;
      WC_DOT(a30, r[3], k[0]);
#undef WC_DOT
    }
    As[(ty + 16) * WC_LD + tx] = a10;
    As[(ty + 32) * WC_LD + tx] = a20;
    As[(ty + 48) * WC_LD + tx] = a30;
    As[(ty + 32) * WC_LD + tx + 16] = a21;
    As[(ty + 48) * WC_LD + tx + 16] = a31;
    As[(ty + 48) * WC_LD + tx + 32] = a32;
  }
  __syncthreads();
  // ---- scale r for the state before the chunk (written over d) and k for the state after it ----
  {
    float fr = 1.0f, fk = 1.0f, all = 1.0f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float f = g[j * WC_D + ch];
      if (j < sub) fr *= f;
      if (j > sub) fk *= f;
      all *= f;
    }
#pragma unroll
    for (int j = 0; j < 16; ++j) {
      const int t = 16 * sub + j;
      ks[t * WC_LD + ch] *= fk;
      if (t < tn && ch < Dp) a.d[(row0 + t) * a.d_ld + (int64_t)h * Dp + ch] = rs[t * WC_LD + ch] * fr;
    }
    if (sub == 0) decays[(((int64_t)b * a.H + h) * gridDim.x + c) * WC_D + ch] = all;
  }
  // ---- outputs from within the chunk: tokens ty + 16 j, columns 4 tx .. 4 tx + 3 ----
  {
    float4 o[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) o[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int sb = 0; sb < 4; ++sb) {
#pragma unroll
      for (int s4 = 0; s4 < 16; s4 += 4) {
        const int s = 16 * sb + s4;
        float4 v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = *reinterpret_cast<const float4 *>(vs + (s + e) * WC_LD + 4 * tx);
#pragma unroll
        for (int j = sb; j < 4; ++j) {
          const float4 A = *reinterpret_cast<const float4 *>(As + (ty + 16 * j) * WC_LD + s);
          o[j].x = fmaf(A.x, v[0].x, fmaf(A.y, v[1].x, fmaf(A.z, v[2].x, fmaf(A.w, v[3].x, o[j].x))));
          o[j].y = fmaf(A.x, v[0].y, fmaf(A.y, v[1].y, fmaf(A.z, v[2].y, fmaf(A.w, v[3].y, o[j].y))));
          o[j].z = fmaf(A.x, v[0].z, fmaf(A.y, v[1].z, fmaf(A.z, v[2].z, fmaf(A.w, v[3].z, o[j].z))));
          o[j].w = fmaf(A.x, v[0].w, fmaf(A.y, v[1].w, fmaf(A.z, v[2].w, fmaf(A.w, v[3].w, o[j].w))));
        }
      }
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int t = ty + 16 * j;
      if (t < tn && 4 * tx < Dp) *reinterpret_cast<float4 *>(a.o + (row0 + t) * a.o_ld + (int64_t)h * Dp + 4 * tx) = o[j];
    }
  }
  __syncthreads();  // k is scaled
  // ---- contribution to the state: keys 4 ty .. + 3, values 4 tx .. + 3 ----
  {
    float4 acc[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < WC_T; ++s) {
      const float4 k = *reinterpret_cast<const float4 *>(ks + s * WC_LD + 4 * ty), v = *reinterpret_cast<const float4 *>(vs + s * WC_LD + 4 * tx);
      const float kk[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        acc[j].x = fmaf(kk[j], v.x, acc[j].x);
        acc[j].y = fmaf(kk[j], v.y, acc[j].y);
        acc[j].z = fmaf(kk[j], v.z, acc[j].z);
        acc[j].w = fmaf(kk[j], v.w, acc[j].w);
      }
    }
    float *dst = U + (((int64_t)b * a.H + h) * gridDim.x + c) * (WC_D * WC_D);
#pragma unroll
    for (int j = 0; j < 4; ++j) *reinterpret_cast<float4 *>(dst + (4 * ty + j) * WC_D + 4 * tx) = acc[j];
  }
}

// one thread per four values of a state row: U[c] <- S; S <- exp(-sum tot_c) S + U[c]
__global__ void __launch_bounds__(256) wkv_states_kernel(const WkvArgs a, float *__restrict__ U, const float *__restrict__ decays, int chunks) {
  pdl_enter();
  const int h = blockIdx.y, b = blockIdx.z, Dp = a.Dp;
  const int e = blockIdx.x * 256 + threadIdx.x, key = e >> 4, v4 = (e & 15) * 4;   // of WC_D x WC_D
  const int64_t bh = (int64_t)b * a.H + h;
  float4 *u = reinterpret_cast<float4 *>(U + bh * chunks * (WC_D * WC_D)) + e;
  const float *w = decays + bh * chunks * WC_D + key;
  float4 *st = reinterpret_cast<float4 *>(a.state + (bh * Dp + key) * Dp + v4);
  const bool in = key < Dp && v4 < Dp;
  float4 S = in && a.n > 0 ? *st : make_float4(0.f, 0.f, 0.f, 0.f);
  for (int c0 = 0; c0 < chunks; c0 += 8) {
    float4 uc[8];
    float wc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < chunks) {
        uc[j] = u[(int64_t)(c0 + j) * (WC_D * WC_D / 4)];
        wc[j] = w[(int64_t)(c0 + j) * WC_D];
      }
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < chunks) {
        u[(int64_t)(c0 + j) * (WC_D * WC_D / 4)] = S;
        S.x = fmaf(wc[j], S.x, uc[j].x); S.y = fmaf(wc[j], S.y, uc[j].y); S.z = fmaf(wc[j], S.z, uc[j].z); S.w = fmaf(wc[j], S.w, uc[j].w);
      }
  }
  if (in) *st = S;
}

__global__ void __launch_bounds__(WC_THREADS) wkv_out_kernel(const WkvArgs a, const float *__restrict__ U) {
  __shared__ __align__(16) float rs[WC_T * WC_LD], S[WC_D * WC_LD];
  const int c = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, Dp = a.Dp;
  const int t0 = c * WC_T, tn = min(WC_T, a.s - t0);
  const int64_t row0 = (int64_t)b * a.s + t0;
  pdl_enter();
  const float4 *src = reinterpret_cast<const float4 *>(U + (((int64_t)b * a.H + h) * gridDim.x + c) * (WC_D * WC_D));
  for (int e = tid; e < WC_T * 16; e += WC_THREADS) {
    const int t = e >> 4, c4 = e & 15;
    float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
    if (t < tn && 4 * c4 < Dp) r = reinterpret_cast<const float4 *>(a.d + (row0 + t) * a.d_ld + (int64_t)h * Dp)[c4];
    *reinterpret_cast<float4 *>(rs + t * WC_LD + 4 * c4) = r;
    *reinterpret_cast<float4 *>(S + t * WC_LD + 4 * c4) = src[e];
  }
  __syncthreads();
  const int tx = tid & 15, ty = tid >> 4;
  float4 o[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int t = ty + 16 * j;
    o[j] = t < tn && 4 * tx < Dp ? *reinterpret_cast<const float4 *>(a.o + (row0 + t) * a.o_ld + (int64_t)h * Dp + 4 * tx) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
#pragma unroll 4
  for (int i = 0; i < WC_D; i += 4) {
    float4 v[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = *reinterpret_cast<const float4 *>(S + (i + e) * WC_LD + 4 * tx);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float4 r = *reinterpret_cast<const float4 *>(rs + (ty + 16 * j) * WC_LD + i);
      o[j].x = fmaf(r.x, v[0].x, fmaf(r.y, v[1].x, fmaf(r.z, v[2].x, fmaf(r.w, v[3].x, o[j].x))));
      o[j].y = fmaf(r.x, v[0].y, fmaf(r.y, v[1].y, fmaf(r.z, v[2].y, fmaf(r.w, v[3].y, o[j].y))));
      o[j].z = fmaf(r.x, v[0].z, fmaf(r.y, v[1].z, fmaf(r.z, v[2].z, fmaf(r.w, v[3].z, o[j].z))));
      o[j].w = fmaf(r.x, v[0].w, fmaf(r.y, v[1].w, fmaf(r.z, v[2].w, fmaf(r.w, v[3].w, o[j].w))));
    }
  }
  const float4 nw = 4 * tx < Dp ? *reinterpret_cast<const float4 *>(a.norm + (int64_t)h * Dp + 4 * tx) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    float ss = (o[j].x * o[j].x + o[j].y * o[j].y) + (o[j].z * o[j].z + o[j].w * o[j].w);
#pragma unroll
    for (int m = 8; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    const int t = ty + 16 * j;
    if (t < tn && 4 * tx < Dp) {
      const float inv = 1.0f / sqrtf(ss / (float)a.D + a.eps);
      const float4 z = *reinterpret_cast<const float4 *>(a.y + (row0 + t) * a.ld + 3 * (int64_t)a.gr + (int64_t)h * Dp + 4 * tx);
      const float4 v = make_float4(o[j].x * inv * nw.x * silu(z.x), o[j].y * inv * nw.y * silu(z.y), o[j].z * inv * nw.z * silu(z.z), o[j].w * inv * nw.w * silu(z.w));
      const int64_t at = (row0 + t) * a.out_ld + (int64_t)h * Dp + 4 * tx;
      if (a.bf.hi) {
        *reinterpret_cast<uint2 *>(a.bf.hi + at) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
        if (a.bf.lo) *reinterpret_cast<uint2 *>(a.bf.lo + at) = make_uint2(pack_bf16(bf16_lo(v.x), bf16_lo(v.y)), pack_bf16(bf16_lo(v.z), bf16_lo(v.w)));
      } else {
        *reinterpret_cast<float4 *>(a.out + at) = v;
      }
    }
  }
}

static int check_wkv(caten_b200_ctx *ctx, const WkvArgs &a) {
  if (a.H <= 0 || a.D <= 0 || a.D > a.Dp || a.Dp % 16 || a.gr < a.H * a.Dp || a.n < 0) return fail(ctx, CATEN_B200_EINVAL, "wkv: bad shape");
  if (a.Dp > 256) return fail(ctx, CATEN_B200_EUNSUPPORTED, "wkv: head size above 256");
  if (a.H > 65535 || a.B > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "wkv: B or H > 65535");
  return 0;
}

static int launch_chunked(caten_b200_ctx *ctx, const WkvArgs &a) {
  const int chunks = (a.s + WC_T - 1) / WC_T;
  const size_t n = (size_t)a.B * a.H * chunks;
  if (int rc = scratch_reserve(ctx, &ctx->chunk_states, n * (WC_D * WC_D + WC_D) * sizeof(float))) return rc;
  float *U = (float *)ctx->chunk_states.ptr, *decays = U + n * (WC_D * WC_D);
  const dim3 grid((unsigned)chunks, (unsigned)a.H, (unsigned)a.B);
  CB_CUDA(ctx, cudaFuncSetAttribute(wkv_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)WC_SMEM));
  launch_k(ctx, wkv_chunk_kernel, grid, dim3(WC_THREADS), WC_SMEM, a, U, decays);
  CB_LAUNCH_CHECK(ctx, "wkv_chunk_kernel");
  launch_k(ctx, wkv_states_kernel, dim3(WC_D * WC_D / 4 / 256, (unsigned)a.H, (unsigned)a.B), dim3(256), 0, a, U, decays, chunks);
  CB_LAUNCH_CHECK(ctx, "wkv_states_kernel");
  launch_k(ctx, wkv_out_kernel, grid, dim3(WC_THREADS), 0, a, U);
  CB_LAUNCH_CHECK(ctx, "wkv_out_kernel");
  return 0;
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
  if (a.Dp <= WC_D && a.s >= 32) return launch_chunked(ctx, a);
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
constexpr int WD_THREADS = 128, WD_U = 8, WD_P = 4;   // WD_P: passes over the channels of a 64-wide head


__global__ void __launch_bounds__(WD_THREADS, 6) wkv_decode_kernel(const WkvArgs a) {
  extern __shared__ __align__(16) float sm[];
  const int Dp = a.Dp, h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *r = sm, *k = r + Dp, *v = k + Dp, *w = v + Dp, *g = w + Dp, *t = g + Dp, *red = t + a.w1, *part = red + 8;
  const int d4 = Dp / 4, RP = WD_THREADS / d4;    // state rows per pass
  const int vq = tid % d4, kr = tid / d4;
  const bool on = kr < RP;
  float4 *st = reinterpret_cast<float4 *>(a.state + ((int64_t)b * a.H + h) * Dp * Dp);
  // parameters first (they depend on no other kernel): this thread's share of the decay's second projection, when a few
  // passes of one 16-byte piece cover it
  const bool ahead = a.w1 == 64 && Dp <= WD_THREADS / 8 * WD_P;
  uint4 wq[WD_P];
#pragma unroll
  for (int p = 0; p < WD_P; ++p) {
    const int c = (tid >> 3) + WD_THREADS / 8 * p;
    wq[p] = ahead && c < Dp ? *reinterpret_cast<const uint4 *>(a.w2 + ((int64_t)h * Dp + c) * 64 + (tid & 7) * 8) : make_uint4(0u, 0u, 0u, 0u);
  }
  pdl_enter();
  float4 s[WD_U];
  auto load = [&](int base) {
#pragma unroll
    for (int i = 0; i < WD_U; ++i) {
      const int key = base + kr + RP * i;
      s[i] = on && key < Dp ? __ldcs(st + (int64_t)key * d4 + vq) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  };
  load(0);   // (discarded at position 0; waiting for the position first would put its latency before the state's)
  const bool fresh = (a.d_n ? *a.d_n : a.n) == 0;
  // r, k, v, gate of this head and the low-rank input, four values per thread and request
  const int items = 4 * d4 + a.w1 / 4;
  for (int i = tid; i < items; i += WD_THREADS) {
    const bool lr = i >= 4 * d4;
    const int which = i / d4, c = lr ? 4 * (i - 4 * d4) : 4 * (i - which * d4);
    const int col = lr ? 4 * a.gr + c : which * a.gr + h * Dp + c;
    float4 p = a.pin.splits > 0 ? partin_load4(a.pin, b, col) : *reinterpret_cast<const float4 *>(a.y + (int64_t)b * a.ld + col);
    if (lr) p = make_float4(tanhf(p.x), tanhf(p.y), tanhf(p.z), tanhf(p.w));
    *reinterpret_cast<float4 *>((lr ? t : which == 0 ? r : which == 1 ? k : which == 2 ? v : g) + c) = p;
  }
  __syncthreads();
  // decay: eight lanes per channel, each 8 weights (16 bytes) at a time
  auto dot8 = [&](uint4 q, int j) {
    const uint32_t qq[4] = {q.x, q.y, q.z, q.w};
    float x = 0.0f;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      x = fmaf(__uint_as_float(qq[e] << 16), t[j + 2 * e], x);
      x = fmaf(__uint_as_float(qq[e] & 0xFFFF0000u), t[j + 2 * e + 1], x);
    }
    return x;
  };
  auto channel = [&](int c, float x) {
    x += __shfl_xor_sync(0xffffffffu, x, 4);
    x += __shfl_xor_sync(0xffffffffu, x, 2);
    x += __shfl_xor_sync(0xffffffffu, x, 1);
    if ((tid & 7) == 0) w[c] = decay(x + a.w0[(int64_t)h * Dp + c]);
  };
  if (ahead) {
#pragma unroll
    for (int p = 0; p < WD_P; ++p) {
      const int c = (tid >> 3) + WD_THREADS / 8 * p;
      if (c < Dp) channel(c, dot8(wq[p], (tid & 7) * 8));   // (whole warps: Dp is a multiple of 4)
    }
  } else {
    for (int c = tid >> 3; c < Dp; c += WD_THREADS / 8) {
      const __nv_bfloat16 *wr = a.w2 + ((int64_t)h * Dp + c) * a.w1;
      float x = 0.0f;
      for (int j = (tid & 7) * 8; j < a.w1; j += 64) x += dot8(*reinterpret_cast<const uint4 *>(wr + j), j);
      channel(c, x);
    }
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
      if (fresh) s[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (on && key < Dp) {
        const float rk = r[key], kk = k[key], wk = w[key];
        o.x = fmaf(rk, s[i].x, o.x); o.y = fmaf(rk, s[i].y, o.y); o.z = fmaf(rk, s[i].z, o.z); o.w = fmaf(rk, s[i].w, o.w);
        st[(int64_t)key * d4 + vq] = make_float4(fmaf(wk, s[i].x, kk * vv.x), fmaf(wk, s[i].y, kk * vv.y), fmaf(wk, s[i].z, kk * vv.z), fmaf(wk, s[i].w, kk * vv.w));
      }
    }
  }
  if (on) reinterpret_cast<float4 *>(part + kr * Dp)[vq] = o;
  __syncthreads();
  constexpr int OC = 256 / WD_THREADS;   // output columns per thread at the widest head
  float ov[OC], ss = 0.0f;
#pragma unroll
  for (int p = 0; p < OC; ++p) {
    const int c = tid + WD_THREADS * p;
    ov[p] = 0.0f;
    if (c < Dp) {
      for (int i = 0; i < RP; ++i) ov[p] += part[i * Dp + c];
      ov[p] = fmaf(v[c], ruk, ov[p]);
    }
    ss += ov[p] * ov[p];
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = red[0];
#pragma unroll
  for (int i = 1; i < WD_THREADS / 32; ++i) ss += red[i];
  const float inv = 1.0f / sqrtf(ss / (float)a.D + a.eps);
#pragma unroll
  for (int p = 0; p < OC; ++p) {
    const int c = tid + WD_THREADS * p;
    if (c < Dp) st_out(a.out, a.bf, (int64_t)b * a.out_ld + (int64_t)h * Dp + c, ov[p] * inv * a.norm[(int64_t)h * Dp + c] * silu(g[c]));
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
