// fp32 GEMM on the CUDA cores with in-kernel dequantisation:
//   y[m, o] = act(sum_k x[m,k] * W[o,k] + bias[o]) + res[m, o]
// This is the CATEN_B200_PREC_FP32 path for more than a few rows.  Each output is accumulated
// as `acc = acc + x*w` with k ascending, a rounded multiply followed by a rounded add — the same
// order and roundings as the C loop BACKEND=CLANG renders for !matmul (source/byoc/clang.lisp:58-111,
// api/high-level-ops.lisp:85-86) when gcc targets baseline x86-64 (no FMA contraction).
#include "common.cuh"
#include "blocks32.cuh"

namespace cb {


constexpr int SG_BM = 64, SG_BN = 64, SG_BK = 32, SG_LD = 68;

// where a tile's outputs go and, with experts, which rows it covers
struct SgMap {
  int64_t group_rows, xplane, ygroup, ldy;
  int tiles_per_group;    // 64-row tiles of a group
  ExpertRows er;          // EXPERTS: sorted rows; group = expert
};

template <int WT, bool EXPERTS = false>
__global__ void __launch_bounds__(256) gemm_simt_kernel(const void *__restrict__ qs, const __half *__restrict__ d,
                                                        const __half *__restrict__ mins, const uint32_t *__restrict__ qh5,
                                                        const float *__restrict__ x, const float *__restrict__ bias,
                                                        const float *res, float *y, int act, int64_t M, int64_t N,
                                                        int64_t K, int64_t nkb, const SgMap map) {
  __shared__ __align__(16) float Xs[SG_BK * SG_LD];  // [k][m]
  __shared__ __align__(16) float Ws[SG_BK * SG_LD];  // [k][n]
  pdl_enter();
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  const int lrow = tid & 63, part = tid >> 6;
  int64_t m0 = (int64_t)blockIdx.y * SG_BM, g = blockIdx.x / map.tiles_per_group;
  const int64_t in_group = (int64_t)(blockIdx.x % map.tiles_per_group) * SG_BN;
  if (EXPERTS) {   // blockIdx.y counts the row tiles of all experts
    int left = blockIdx.y, e = 0, lo = 0, hi = 0;
    for (; e < map.er.experts; ++e) {
      lo = map.er.offsets[e]; hi = map.er.offsets[e + 1];
      const int t = (hi - lo + SG_BM - 1) / SG_BM;
      if (left < t) break;
      left -= t;
    }
    if (e == map.er.experts) return;
    g = e;
    m0 = lo + (int64_t)left * SG_BM;
    M = hi;
  }
  const int64_t n0 = g * map.group_rows + in_group;
  const int64_t n_end = N < (g + 1) * map.group_rows ? N : (g + 1) * map.group_rows;
  const int64_t shift = EXPERTS ? g * map.group_rows : g * (map.group_rows - map.ygroup);   // output column = row of W - shift
  if (!EXPERTS) x += g * map.xplane * K;  // the input plane of this tile's output rows
  const int64_t xrow = m0 + lrow < M ? (EXPERTS && map.er.src ? map.er.src[m0 + lrow] : m0 + lrow) : 0;
  float acc[4][4];
#pragma unroll
  for (int a = 0; a < 4; ++a)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[a][e] = 0.0f;
  for (int kb = 0; kb < (int)(K / 32); ++kb) {
    float xv[8], wv[8];
    if (m0 + lrow < M) {
      const float4 *p = reinterpret_cast<const float4 *>(x + xrow * K + (int64_t)kb * 32 + part * 8);
      const float4 a = p[0], b = p[1];
      xv[0] = a.x; xv[1] = a.y; xv[2] = a.z; xv[3] = a.w; xv[4] = b.x; xv[5] = b.y; xv[6] = b.z; xv[7] = b.w;
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) xv[e] = 0.0f;
    }
    if (WT == WT_F32_T) {
      // b[k, n]: thread reads 8 consecutive k for its column (coalesced across the 64 columns)
#pragma unroll
      for (int e = 0; e < 8; ++e)
        wv[e] = n0 + lrow < N ? ((const float *)qs)[((int64_t)kb * 32 + part * 8 + e) * N + n0 + lrow] : 0.0f;
    } else {
      load_w8<WT>(qs, d, mins, qh5, n0 + lrow, N, K, nkb, kb, part, wv);
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      Xs[(part * 8 + e) * SG_LD + lrow] = xv[e];
      Ws[(part * 8 + e) * SG_LD + lrow] = wv[e];
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_BK; ++k) {
      const float4 xa = *reinterpret_cast<const float4 *>(Xs + k * SG_LD + 4 * ty);
      const float4 wa = *reinterpret_cast<const float4 *>(Ws + k * SG_LD + 4 * tx);
      const float xr[4] = {xa.x, xa.y, xa.z, xa.w}, wr[4] = {wa.x, wa.y, wa.z, wa.w};
#pragma unroll
      for (int a = 0; a < 4; ++a)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[a][e] = acc[a][e] + xr[a] * wr[e];  // rounded mul, rounded add
    }
  }
#pragma unroll
  for (int a = 0; a < 4; ++a) {
    const int64_t m = m0 + 4 * ty + a;
    if (m >= M) continue;
    if (EXPERTS && map.er.weight) {
      const float wt = map.er.weight[m];
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[a][e] = acc[a][e] * wt;
    }
    if (act_is_glu(act)) {
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int64_t o = n0 + 4 * tx + e;
        if (o < n_end) y[m * map.ldy + (o - shift) / 2] = glu(act, acc[a][e] + (bias ? bias[o] : 0.0f), acc[a][e + 1] + (bias ? bias[o + 1] : 0.0f));
      }
      continue;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int64_t o = n0 + 4 * tx + e;
      if (o >= n_end) continue;
      float v = acc[a][e];
      if (bias) v = v + bias[o];
      v = apply_act(v, act);
      const int64_t at = m * map.ldy + o - shift;
      if (res) v = res[at] + v;
      y[at] = v;
    }
  }
}

template <int WT>
static int launch_simt(caten_b200_ctx *ctx, const void *qs, const __half *d, const __half *mins, const uint32_t *qh5, const float *x,
                       const float *bias, const float *res, int act, float *y, int64_t M, int64_t N, int64_t K, LinGroups grp = LinGroups()) {
  if (K % 32) return fail(ctx, CATEN_B200_EUNSUPPORTED, "gemm: inner dimension %lld is not a multiple of 32", (long long)K);
  SgMap map;
  map.group_rows = grp.group_rows > 0 ? grp.group_rows : N;
  map.xplane = grp.xplane;
  map.ygroup = grp.ygroup ? grp.ygroup : map.group_rows;
  map.ldy = grp.ldy ? grp.ldy : act_is_glu(act) ? N / 2 : N;
  map.tiles_per_group = (int)((map.group_rows + SG_BN - 1) / SG_BN);
  const int64_t gx = (N + map.group_rows - 1) / map.group_rows * map.tiles_per_group, gy = (M + SG_BM - 1) / SG_BM;
  if (gy > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "gemm: too many rows for one launch (%lld)", (long long)M);
  launch_k(ctx, gemm_simt_kernel<WT>, dim3((unsigned)gx, (unsigned)gy), dim3(256), 0, qs, d, mins, qh5, x, bias, res, y, act, M, N, K, K / 32, map);
  CB_LAUNCH_CHECK(ctx, "gemm_simt_kernel");
  return 0;
}

int launch_gemm_simt(caten_b200_ctx *ctx, const caten_b200_weight *w, const float *x, const float *bias,
                     const float *res, int act, float *y, int64_t M, LinGroups grp) {
  if (M <= 0) return 0;
#define SIMT_CASE(T) \
  case T: return launch_simt<T>(ctx, w->qs, w->d, w->m, w->qh, x, bias, res, act, y, M, w->rows, w->cols, grp)
  switch (w->type) {
    SIMT_CASE(CATEN_B200_F32);
    SIMT_CASE(CATEN_B200_F16);
    SIMT_CASE(CATEN_B200_BF16);
    SIMT_CASE(CATEN_B200_Q8_0);
    SIMT_CASE(CATEN_B200_Q4_0);
    SIMT_CASE(CATEN_B200_Q4_1);
    SIMT_CASE(CATEN_B200_Q5_0);
    SIMT_CASE(CATEN_B200_Q5_1);
  }
#undef SIMT_CASE
  return fail(ctx, CATEN_B200_EUNSUPPORTED, "gemm: weight type %d", w->type);
}

int launch_gemm_simt_experts(caten_b200_ctx *ctx, const caten_b200_weight *w, const ExpertRows &er, const float *x, const int *src, int act, float *y) {
  if (er.pairs <= 0) return 0;
  if (w->type != CATEN_B200_BF16 || w->cols % 32 || w->rows % er.experts) return fail(ctx, CATEN_B200_EUNSUPPORTED, "gemm: experts take BF16 weights");
  SgMap map;
  map.er = er;
  map.er.src = src;
  map.group_rows = w->rows / er.experts;
  map.xplane = 0;
  map.ygroup = map.group_rows;
  map.ldy = act_is_glu(act) ? map.group_rows / 2 : map.group_rows;
  map.tiles_per_group = (int)((map.group_rows + SG_BN - 1) / SG_BN);
  // row tiles: every expert with rows has at most one that is not full
  const int64_t gy = er.pairs / SG_BM + (er.pairs < er.experts ? er.pairs : er.experts);
  if (gy > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "gemm: too many rows for one launch (%lld)", (long long)er.pairs);
  launch_k(ctx, gemm_simt_kernel<CATEN_B200_BF16, true>, dim3((unsigned)map.tiles_per_group, (unsigned)gy), dim3(256), 0, (const void *)w->qs, w->d, w->m, w->qh, x, nullptr, nullptr, y,
           act, er.pairs, w->rows, w->cols, w->cols / 32, map);
  CB_LAUNCH_CHECK(ctx, "gemm_simt_kernel");
  return 0;
}

int launch_relu_matmul_simt(caten_b200_ctx *ctx, const float *a, const float *b, float *c, int64_t M, int64_t K, int64_t N) {
  if (M <= 0 || N <= 0) return 0;
  return launch_simt<WT_F32_T>(ctx, b, nullptr, nullptr, nullptr, a, nullptr, nullptr, CATEN_B200_ACT_RELU, c, M, N, K);
}

}  // namespace cb
