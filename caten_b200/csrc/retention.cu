// Retention: per head a matrix state S[key, value] in fp32 with a fixed decay g,
//   S_t = g S_{t-1} + k_t v_t^T,   o_t = S_t^T q_t
// q and k are rotated by position (dims i and i + rot_pairs), k carries a constant factor.  Then o is divided by
// its root mean square over the head and multiplied with silu(gate).  The state starts at zero with the sequence
// (position 0) and is carried from step to step.
//
// Multi-token steps go in chunks of 64 tokens, all of them at once (everything fp32; decay^j from a table):
//   retention_state_kernel   U_c = sum_s g^(T-1-s) k_s v_s^T of every chunk
//   retention_scan_kernel    walks the chunks: U_c <- S, S <- g^T S + U_c
//   retention_out_kernel     o_t = g^(t+1) q_t S_c + sum_{s <= t} g^(t-s) (q_t . k_s) v_s, norm, gate
#include "retention.cuh"

namespace cb {

namespace {

constexpr int RT_LD = RET_T + 4, RT_THREADS = 256;

__device__ __forceinline__ void st4(float *out, BfOut bf, int64_t at, float4 v) {
  if (bf.hi) {
    *reinterpret_cast<uint2 *>(bf.hi + at) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    if (bf.lo) *reinterpret_cast<uint2 *>(bf.lo + at) = make_uint2(pack_bf16(bf16_lo(v.x), bf16_lo(v.y)), pack_bf16(bf16_lo(v.z), bf16_lo(v.w)));
  } else {
    *reinterpret_cast<float4 *>(out + at) = v;
  }
}
__device__ __forceinline__ float4 zero4() { return make_float4(0.f, 0.f, 0.f, 0.f); }
__device__ __forceinline__ float4 axpy4(float a, float4 x, float4 y) { return make_float4(fmaf(a, x.x, y.x), fmaf(a, x.y, y.y), fmaf(a, x.z, y.z), fmaf(a, x.w, y.w)); }
__device__ __forceinline__ float dot4(float4 a, float4 b, float c) { return fmaf(a.x, b.x, fmaf(a.y, b.y, fmaf(a.z, b.z, fmaf(a.w, b.w, c)))); }

}  // namespace

// one CTA per row; a thread keeps one pair's angle for several heads
__global__ void __launch_bounds__(RT_THREADS) retention_prep_kernel(const RetentionArgs a) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int pos = a.n + (int)(r % a.s), tid = threadIdx.x, np = a.rot_pairs;
  float *row = a.y + r * a.ld;
  if (np > 0) {
    const int lanes = RT_THREADS / np > 0 ? RT_THREADS / np : 1;
    for (int i = tid % np; i < np && tid / np < lanes; i += RT_THREADS) {
      float sn, cs;
      sincosf((float)pos * a.freq[i], &sn, &cs);
      for (int h = tid / np; h < 2 * a.H; h += lanes) {
        const bool is_k = h >= a.H;
        float *x = row + (is_k ? a.k_off + (int64_t)(h - a.H) * a.Dp : a.q_off + (int64_t)h * a.Dp) + i;
        const float u = x[0], v = x[np], f = is_k ? a.kscale : 1.0f;
        x[0] = (u * cs - v * sn) * f;
        x[np] = (v * cs + u * sn) * f;
      }
    }
  }
  const int rest = a.D - 2 * np;   // dims of k that do not turn
  for (int i = tid; i < a.H * rest; i += RT_THREADS) row[a.k_off + (int64_t)(i / rest) * a.Dp + 2 * np + i % rest] *= a.kscale;
}

// Rows [r0, r0 + 64) x columns [c0, c0 + 4 * W4) of a matrix into shared memory, zeros outside [0, rows) x [0, cols); asynchronous.
template <int W4>
__device__ __forceinline__ void load_tile(float *dst, int ld, const float *src, int64_t src_ld, int r0, int rows, int c0, int cols, int tid) {
#pragma unroll 4
  for (int e = tid; e < 64 * W4; e += RT_THREADS) {
    const int r = e / W4, c = (e % W4) * 4;
    const bool in = r0 + r < rows && c0 + c < cols;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst + r * ld + c)),
                 "l"(src + (in ? (int64_t)(r0 + r) * src_ld + c0 + c : 0)), "r"(in ? 16 : 0) : "memory");
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
}
// all tiles but the `N` last ones have arrived
template <int N> __device__ __forceinline__ void tiles_ready() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
  __syncthreads();
}

// U of one chunk: a tile of 64 keys x 64 NEB values per CTA; grid (chunk, head x key tiles x value tiles, sequence)
template <int NEB>
__global__ void __launch_bounds__(RT_THREADS) retention_state_kernel(const RetentionArgs a, float *__restrict__ U) {
  extern __shared__ __align__(16) float sm[];
  constexpr int VLD = 64 * NEB + 4;
  float *ks = sm, *vs = ks + RET_T * RT_LD;   // [token][key], [token][value]
  const int nd = (a.Dp + 63) / 64, ne = (a.Ep + 64 * NEB - 1) / (64 * NEB);
  const int c = blockIdx.x, b = blockIdx.z, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int h = blockIdx.y / (nd * ne), d0 = blockIdx.y / ne % nd * 64, e0 = blockIdx.y % ne * 64 * NEB;
  const int tn = min(RET_T, a.s - c * RET_T);
  const int64_t row0 = (int64_t)b * a.s + c * RET_T;
  const float *pw = a.powers + (int64_t)h * (RET_T + 1);
  pdl_enter();
  load_tile<16>(ks, RT_LD, a.y + row0 * a.ld + a.k_off + (int64_t)h * a.Dp, a.ld, 0, tn, d0, a.Dp, tid);
  load_tile<16 * NEB>(vs, VLD, a.y + row0 * a.ld + a.v_off + (int64_t)h * a.Ep, a.ld, 0, tn, e0, a.Ep, tid);
  tiles_ready<0>();
  float4 acc[4][NEB];
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) acc[j][nb] = zero4();
#pragma unroll 4
  for (int t = 0; t < tn; ++t) {
    const float f = pw[tn - 1 - t];
    float4 k = *reinterpret_cast<const float4 *>(ks + t * RT_LD + 4 * ty);
    k = make_float4(k.x * f, k.y * f, k.z * f, k.w * f);
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) {
      const float4 v = *reinterpret_cast<const float4 *>(vs + t * VLD + 64 * nb + 4 * tx);
      acc[0][nb] = axpy4(k.x, v, acc[0][nb]);
      acc[1][nb] = axpy4(k.y, v, acc[1][nb]);
      acc[2][nb] = axpy4(k.z, v, acc[2][nb]);
      acc[3][nb] = axpy4(k.w, v, acc[3][nb]);
    }
  }
  float *dst = U + (((int64_t)b * a.H + h) * gridDim.x + c) * a.Dp * a.Ep;
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) {
      const int key = d0 + 4 * ty + j, col = e0 + 64 * nb + 4 * tx;
      if (key < a.Dp && col < a.Ep) *reinterpret_cast<float4 *>(dst + (int64_t)key * a.Ep + col) = acc[j][nb];
    }
}

// one thread per four values of a state row
__global__ void __launch_bounds__(256) retention_scan_kernel(const RetentionArgs a, float *__restrict__ U, int chunks) {
  pdl_enter();
  const int h = blockIdx.y, b = blockIdx.z, per = a.Dp * a.Ep / 4, e = blockIdx.x * 256 + threadIdx.x;
  if (e >= per) return;
  const float *pw = a.powers + (int64_t)h * (RET_T + 1);
  const float w = pw[RET_T], w_last = pw[a.s - (chunks - 1) * RET_T];
  float4 *u = reinterpret_cast<float4 *>(U) + ((int64_t)b * a.H + h) * chunks * per + e;
  float4 *st = reinterpret_cast<float4 *>(a.state) + ((int64_t)b * a.H + h) * per + e;
  float4 S = a.n > 0 ? *st : zero4();
  for (int c0 = 0; c0 < chunks; c0 += 8) {
    float4 uc[8];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < chunks) uc[j] = u[(int64_t)(c0 + j) * per];
#pragma unroll
    for (int j = 0; j < 8; ++j)
      if (c0 + j < chunks) {
        u[(int64_t)(c0 + j) * per] = S;
        S = axpy4(c0 + j == chunks - 1 ? w_last : w, S, uc[j]);
      }
  }
  *st = S;
}

// grid (chunk, head x value tiles, sequence): 64 tokens x 64 NEB value columns.  Thread (ty, tx) owns tokens ty + 16 j and
// columns 4 tx + 64 nb; of the token pairs (ty + 16 j, tx + 16 i).
template <int NEB>
__global__ void __launch_bounds__(RT_THREADS, 2) retention_out_kernel(const RetentionArgs a, const float *__restrict__ U) {
  extern __shared__ __align__(16) float sm[];
  constexpr int VLD = 64 * NEB + 4;
  __shared__ float pw[RET_T + 1];
  float *qs = sm, *ks = qs + RET_T * RT_LD, *vs = ks + RET_T * RT_LD;
  const int ne = (a.Ep + 64 * NEB - 1) / (64 * NEB);
  const int c = blockIdx.x, b = blockIdx.z, tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int h = blockIdx.y / ne, e0 = blockIdx.y % ne * 64 * NEB;
  const int tn = min(RET_T, a.s - c * RET_T);
  const int64_t row0 = (int64_t)b * a.s + c * RET_T;
  pdl_enter();
  if (tid <= RET_T) pw[tid] = a.powers[(int64_t)h * (RET_T + 1) + tid];
  const float *qg = a.y + row0 * a.ld + a.q_off + (int64_t)h * a.Dp, *kg = a.y + row0 * a.ld + a.k_off + (int64_t)h * a.Dp;
  const float *S = U + (((int64_t)b * a.H + h) * gridDim.x + c) * a.Dp * a.Ep;
  float *as = ks;   // [token][earlier token], once the products are formed
  {
    float A[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) A[j][i] = 0.0f;
    for (int d0 = 0; d0 < a.Dp; d0 += 64) {
      __syncthreads();
      load_tile<16>(qs, RT_LD, qg, a.ld, 0, tn, d0, a.Dp, tid);
      load_tile<16>(ks, RT_LD, kg, a.ld, 0, tn, d0, a.Dp, tid);
      if (d0 == 0) {   // the first block of the state arrives during the products
        load_tile<16 * NEB>(vs, VLD, S, a.Ep, 0, a.Dp, e0, a.Ep, tid);
        tiles_ready<1>();
      } else {
        tiles_ready<0>();
      }
      const int dn = min(64, a.Dp - d0);
      for (int d = 0; d < dn; d += 4) {
        float4 q[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) q[j] = *reinterpret_cast<const float4 *>(qs + (ty + 16 * j) * RT_LD + d);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const float4 k = *reinterpret_cast<const float4 *>(ks + (tx + 16 * i) * RT_LD + d);
#pragma unroll
          for (int j = i; j < 4; ++j) A[j][i] = dot4(q[j], k, A[j][i]);   // (pairs with i > j are never used)
        }
      }
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = ty + 16 * j, s = tx + 16 * i;
        as[t * RT_LD + s] = s <= t ? A[j][i] * pw[t - s] : 0.0f;
      }
  }
  float4 o[4][NEB];
#pragma unroll
  for (int j = 0; j < 4; ++j)
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) o[j][nb] = zero4();
  for (int d0 = 0; d0 < a.Dp; d0 += 64) {
    __syncthreads();
    if (a.Dp > 64) load_tile<16>(qs, RT_LD, qg, a.ld, 0, tn, d0, a.Dp, tid);   // (a single block is still there)
    if (d0 > 0) load_tile<16 * NEB>(vs, VLD, S, a.Ep, d0, a.Dp, e0, a.Ep, tid);
    tiles_ready<0>();
    const int dn = min(64, a.Dp - d0);
    for (int d = 0; d < dn; d += 4) {
      float4 q[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) q[j] = *reinterpret_cast<const float4 *>(qs + (ty + 16 * j) * RT_LD + d);
#pragma unroll
      for (int nb = 0; nb < NEB; ++nb) {
        float4 v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = *reinterpret_cast<const float4 *>(vs + (d + e) * VLD + 64 * nb + 4 * tx);
#pragma unroll
        for (int j = 0; j < 4; ++j) o[j][nb] = axpy4(q[j].x, v[0], axpy4(q[j].y, v[1], axpy4(q[j].z, v[2], axpy4(q[j].w, v[3], o[j][nb]))));
      }
    }
  }
  __syncthreads();
  load_tile<16 * NEB>(vs, VLD, a.y + row0 * a.ld + a.v_off + (int64_t)h * a.Ep, a.ld, 0, tn, e0, a.Ep, tid);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float f = pw[ty + 16 * j + 1];
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) o[j][nb] = make_float4(o[j][nb].x * f, o[j][nb].y * f, o[j][nb].z * f, o[j][nb].w * f);
  }
  tiles_ready<0>();
#pragma unroll
  for (int sb = 0; sb < 4; ++sb) {
#pragma unroll 2
    for (int s4 = 0; s4 < 16; s4 += 4) {
      const int s = 16 * sb + s4;
      float4 w[4];
#pragma unroll
      for (int j = sb; j < 4; ++j) w[j] = *reinterpret_cast<const float4 *>(as + (ty + 16 * j) * RT_LD + s);
#pragma unroll
      for (int nb = 0; nb < NEB; ++nb) {
        float4 v[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = *reinterpret_cast<const float4 *>(vs + (s + e) * VLD + 64 * nb + 4 * tx);
#pragma unroll
        for (int j = sb; j < 4; ++j) o[j][nb] = axpy4(w[j].x, v[0], axpy4(w[j].y, v[1], axpy4(w[j].z, v[2], axpy4(w[j].w, v[3], o[j][nb]))));
      }
    }
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int t = ty + 16 * j;
    float ss = 0.0f;
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) ss += (o[j][nb].x * o[j][nb].x + o[j][nb].y * o[j][nb].y) + (o[j][nb].z * o[j][nb].z + o[j][nb].w * o[j][nb].w);
#pragma unroll
    for (int m = 8; m > 0; m >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, m);
    if (t >= tn) continue;
    const float inv = 1.0f / sqrtf(ss / (float)a.E + a.eps);
#pragma unroll
    for (int nb = 0; nb < NEB; ++nb) {
      const int col = e0 + 64 * nb + 4 * tx;
      if (col >= a.Ep) continue;
      if (ne > 1) {   // the head's norm needs the other tiles too
        *reinterpret_cast<float4 *>(a.o + ((row0 + t) * a.H + h) * a.Ep + col) = o[j][nb];
      } else {
        const float4 z = *reinterpret_cast<const float4 *>(a.y + (row0 + t) * a.ld + a.g_off + (int64_t)h * a.Ep + col), v = o[j][nb];
        st4(a.out, a.bf, (row0 + t) * a.out_ld + (int64_t)h * a.Ep + col,
            make_float4(v.x * inv * silu(z.x), v.y * inv * silu(z.y), v.z * inv * silu(z.z), v.w * inv * silu(z.w)));
      }
    }
  }
}

// heads' norm and gate of one row: one warp per head
__global__ void __launch_bounds__(256) retention_gate_kernel(const RetentionArgs a) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int lane = threadIdx.x & 31, e4 = a.Ep / 4;
  for (int h = threadIdx.x >> 5; h < a.H; h += 8) {
    const float4 *o = reinterpret_cast<const float4 *>(a.o + (r * a.H + h) * a.Ep), *g = reinterpret_cast<const float4 *>(a.y + r * a.ld + a.g_off + (int64_t)h * a.Ep);
    float ss = 0.0f;
    for (int c = lane; c < e4; c += 32) ss += (o[c].x * o[c].x + o[c].y * o[c].y) + (o[c].z * o[c].z + o[c].w * o[c].w);
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.E + a.eps);
    for (int c = lane; c < e4; c += 32) {
      const float4 v = o[c], z = g[c];
      st4(a.out, a.bf, r * a.out_ld + (int64_t)h * a.Ep + 4 * c, make_float4(v.x * inv * silu(z.x), v.y * inv * silu(z.y), v.z * inv * silu(z.z), v.w * inv * silu(z.w)));
    }
  }
}

static int check_retention(caten_b200_ctx *ctx, const RetentionArgs &a) {
  if (a.H <= 0 || a.D <= 0 || a.E <= 0 || a.D > a.Dp || a.E > a.Ep || a.Dp % 16 || a.Ep % 16 || 2 * a.rot_pairs > a.D || a.n < 0) return fail(ctx, CATEN_B200_EINVAL, "retention: bad shape");
  if (a.Dp > 512 || a.Ep > 1024) return fail(ctx, CATEN_B200_EUNSUPPORTED, "retention: heads of %d x %d (at most 512 x 1024)", a.D, a.E);
  const int64_t tiles = (int64_t)a.H * ((a.Dp + 63) / 64) * ((a.Ep + 63) / 64);
  if (tiles > 65535 || a.B > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "retention: too many heads or sequences");
  return 0;
}

int launch_retention_prep(caten_b200_ctx *ctx, const RetentionArgs &a) {
  const int64_t rows = (int64_t)a.B * a.s;
  if (rows <= 0) return 0;
  if (int rc = check_retention(ctx, a)) return rc;
  if (rows > 0x7fffffff) return fail(ctx, CATEN_B200_EUNSUPPORTED, "retention: too many rows");
  launch_k(ctx, retention_prep_kernel, dim3((unsigned)rows), dim3(RT_THREADS), 0, a);
  CB_LAUNCH_CHECK(ctx, "retention_prep_kernel");
  return 0;
}

template <int NEB>
static int launch_chunks_t(caten_b200_ctx *ctx, const RetentionArgs &a, float *U, int chunks) {
  constexpr int NS = NEB > 2 ? 2 : NEB;   // value tile of the state kernel
  const size_t s_smem = (size_t)(RET_T * RT_LD + RET_T * (64 * NS + 4)) * sizeof(float), o_smem = (size_t)(2 * RET_T * RT_LD + RET_T * (64 * NEB + 4)) * sizeof(float);
  const int nd = (a.Dp + 63) / 64, ns = (a.Ep + 64 * NS - 1) / (64 * NS), ne = (a.Ep + 64 * NEB - 1) / (64 * NEB);
  CB_CUDA(ctx, cudaFuncSetAttribute(retention_state_kernel<NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s_smem));
  launch_k(ctx, retention_state_kernel<NS>, dim3((unsigned)chunks, (unsigned)(a.H * nd * ns), (unsigned)a.B), dim3(RT_THREADS), s_smem, a, U);
  CB_LAUNCH_CHECK(ctx, "retention_state_kernel");
  launch_k(ctx, retention_scan_kernel, dim3((unsigned)((a.Dp * a.Ep / 4 + 255) / 256), (unsigned)a.H, (unsigned)a.B), dim3(256), 0, a, U, chunks);
  CB_LAUNCH_CHECK(ctx, "retention_scan_kernel");
  CB_CUDA(ctx, cudaFuncSetAttribute(retention_out_kernel<NEB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)o_smem));
  launch_k(ctx, retention_out_kernel<NEB>, dim3((unsigned)chunks, (unsigned)(a.H * ne), (unsigned)a.B), dim3(RT_THREADS), o_smem, a, U);
  CB_LAUNCH_CHECK(ctx, "retention_out_kernel");
  if (ne > 1) {
    launch_k(ctx, retention_gate_kernel, dim3((unsigned)((int64_t)a.B * a.s)), dim3(256), 0, a);
    CB_LAUNCH_CHECK(ctx, "retention_gate_kernel");
  }
  return 0;
}

int launch_retention_chunks(caten_b200_ctx *ctx, const RetentionArgs &a) {
  if (a.B <= 0 || a.s <= 0) return 0;
  if (int rc = check_retention(ctx, a)) return rc;
  if (a.Ep > 256 && !a.o) return fail(ctx, CATEN_B200_EINVAL, "retention: values above 256 need a buffer for the raw outputs");
  const int chunks = (a.s + RET_T - 1) / RET_T;
  if (int rc = scratch_reserve(ctx, &ctx->chunk_states, (size_t)a.B * a.H * chunks * a.Dp * a.Ep * sizeof(float))) return rc;
  float *U = (float *)ctx->chunk_states.ptr;
  if (a.Ep <= 64) return launch_chunks_t<1>(ctx, a, U, chunks);
  if (a.Ep <= 128) return launch_chunks_t<2>(ctx, a, U, chunks);
  return launch_chunks_t<4>(ctx, a, U, chunks);
}

// ---------------------------------------------------------------------------------------------
// Single-token step: one CTA per (head, sequence) reads and writes the head's state once.  The first
// state rows are requested before the projections are summed.
// ---------------------------------------------------------------------------------------------
constexpr int RD_THREADS = 256, RD_U = 8;

__global__ void __launch_bounds__(RD_THREADS, 3) retention_decode_kernel(const RetentionArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[RD_THREADS / 32];
  const int Dp = a.Dp, Ep = a.Ep, h = blockIdx.x, b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *q = sm, *k = q + Dp, *v = k + Dp, *g = v + Ep, *part = g + Ep;
  const int e4 = Ep / 4, RP = RD_THREADS / e4;    // state rows per pass
  const int vq = tid % e4, kr = tid / e4;
  const bool on = kr < RP;
  float4 *st = reinterpret_cast<float4 *>(a.state + ((int64_t)b * a.H + h) * Dp * Ep);
  const float decay = a.powers[(int64_t)h * (RET_T + 1) + 1];
  pdl_enter();
  float4 s[RD_U];
  auto load = [&](int base) {
#pragma unroll
    for (int i = 0; i < RD_U; ++i) {
      const int key = base + kr + RP * i;
      s[i] = on && key < Dp ? __ldcs(st + (int64_t)key * e4 + vq) : zero4();
    }
  };
  load(0);   // (discarded at position 0; waiting for the position first would put its latency before the state's)
  const int n = a.d_n ? *a.d_n : a.n;
  const bool fresh = n == 0;
  const int d4 = Dp / 4;
  for (int i = tid; i < 2 * d4 + 2 * e4; i += RD_THREADS) {
    const bool qk = i < 2 * d4;
    const int which = qk ? i / d4 : (i - 2 * d4) / e4, c = 4 * (qk ? i - which * d4 : i - 2 * d4 - which * e4);
    const int col = qk ? (which ? a.k_off : a.q_off) + h * Dp + c : (which ? a.g_off : a.v_off) + h * Ep + c;
    *reinterpret_cast<float4 *>((qk ? (which ? k : q) : (which ? g : v)) + c) =
        a.pin.splits > 0 ? partin_load4(a.pin, b, col) : *reinterpret_cast<const float4 *>(a.y + (int64_t)b * a.ld + col);
  }
  __syncthreads();
  for (int i = tid; i < a.rot_pairs; i += RD_THREADS) {
    float sn, cs;
    sincosf((float)n * a.freq[i], &sn, &cs);
    const int j = i + a.rot_pairs;
    const float qu = q[i], qv = q[j], ku = k[i], kv = k[j];
    q[i] = qu * cs - qv * sn;
    q[j] = qv * cs + qu * sn;
    k[i] = ku * cs - kv * sn;
    k[j] = kv * cs + ku * sn;
  }
  __syncthreads();
  float4 o = zero4();
  const float4 vv = on ? reinterpret_cast<const float4 *>(v)[vq] : o;
  for (int base = 0; base < Dp; base += RD_U * RP) {
    if (base) load(base);
#pragma unroll
    for (int i = 0; i < RD_U; ++i) {
      const int key = base + kr + RP * i;
      if (fresh) s[i] = zero4();
      if (on && key < Dp) {
        const float kk = k[key] * a.kscale;
        const float4 x = make_float4(fmaf(decay, s[i].x, kk * vv.x), fmaf(decay, s[i].y, kk * vv.y), fmaf(decay, s[i].z, kk * vv.z), fmaf(decay, s[i].w, kk * vv.w));
        st[(int64_t)key * e4 + vq] = x;
        o = axpy4(q[key], x, o);
      }
    }
  }
  if (on) reinterpret_cast<float4 *>(part + kr * Ep)[vq] = o;
  __syncthreads();
  float4 ov = zero4();
  float ss = 0.0f;
  if (tid < e4) {
    for (int i = 0; i < RP; ++i) {
      const float4 p = reinterpret_cast<const float4 *>(part + i * Ep)[tid];
      ov = make_float4(ov.x + p.x, ov.y + p.y, ov.z + p.z, ov.w + p.w);
    }
    ss = (ov.x * ov.x + ov.y * ov.y) + (ov.z * ov.z + ov.w * ov.w);
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = red[0];
#pragma unroll
  for (int i = 1; i < RD_THREADS / 32; ++i) ss += red[i];
  const float inv = 1.0f / sqrtf(ss / (float)a.E + a.eps);
  if (tid < e4) {
    const float4 z = reinterpret_cast<const float4 *>(g)[tid];
    st4(a.out, a.bf, (int64_t)b * a.out_ld + (int64_t)h * Ep + 4 * tid,
        make_float4(ov.x * inv * silu(z.x), ov.y * inv * silu(z.y), ov.z * inv * silu(z.z), ov.w * inv * silu(z.w)));
  }
}

int launch_retention_decode(caten_b200_ctx *ctx, const RetentionArgs &a) {
  if (a.B <= 0) return 0;
  if (int rc = check_retention(ctx, a)) return rc;
  const int RP = RD_THREADS / (a.Ep / 4);
  const size_t smem = ((size_t)2 * a.Dp + 2 * a.Ep + (size_t)RP * a.Ep) * sizeof(float);
  launch_k(ctx, retention_decode_kernel, dim3((unsigned)a.H, (unsigned)a.B), dim3(RD_THREADS), smem, a);
  CB_LAUNCH_CHECK(ctx, "retention_decode_kernel");
  return 0;
}

}  // namespace cb
