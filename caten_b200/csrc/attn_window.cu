// Grouped-query softmax attention with an optional sliding window: query i sees the keys j with
// 0 <= i - j < window.  The cache of a sequence is a ring of `cap` positions (slot = position % cap),
// so a windowed layer keeps window + one prompt portion whatever the sequence's length.
//
//   q, k   rotated on their first 2 * rot_pairs dims (interleaved pairs, angle = position * freq),
//          then divided by their root mean square over the head (optional)
//   out    softmax(q . k * scale) . v, times sigmoid(gate) per head (optional)
//
// Keys are cached rotated and normalised; everything here is fp32.
#include "attn_window.cuh"
#include "tcgen05.cuh"

namespace cb {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float sigmoidf(float z) { return 1.0f / (1.0f + expf(-z)); }

// One warp, one head of up to 256 dims: lane holds the pairs lane, lane + 32, ...
struct HeadPairs {
  float2 p[4];
};
__device__ __forceinline__ void rotate_pairs(HeadPairs &h, const float *__restrict__ freq, int rot_pairs, int pos, int lane) {
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int i = lane + 32 * j;
    if (i < rot_pairs) {
      float sn, cs;
      sincosf((float)pos * freq[i], &sn, &cs);
      const float u = h.p[j].x, v = h.p[j].y;
      h.p[j].x = u * cs - v * sn;
      h.p[j].y = v * cs + u * sn;
    }
  }
}
// A head of row m whose linear left split-K partial tiles: every pair's partial values are requested together, two
// splits at a time, and added in split order.
__device__ __forceinline__ void load_pairs_pending(HeadPairs &h, const PartIn &pin, int m, int off, int np, int lane) {
  const float *src[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int o = off + 2 * (lane + 32 * j);
    const long long tile = (long long)(m / pin.bnx) * pin.tiles_x + (o >> 7);
    src[j] = pin.part + (tile * pin.bnx + m % pin.bnx) * 128 + (o & 127);
    h.p[j] = make_float2(0.f, 0.f);
  }
  for (int z = 0; z < pin.splits; z += 2) {
    float2 t[2][4];
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (lane + 32 * j < np && z + u < pin.splits) t[u][j] = __ldcs(reinterpret_cast<const float2 *>(src[j] + (long long)(z + u) * pin.zstride));
#pragma unroll
    for (int u = 0; u < 2; ++u)
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (lane + 32 * j < np && z + u < pin.splits) { h.p[j].x += t[u][j].x; h.p[j].y += t[u][j].y; }
  }
  if (pin.bias)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (lane + 32 * j < np) {
        h.p[j].x += pin.bias[off + 2 * (lane + 32 * j)];
        h.p[j].y += pin.bias[off + 2 * (lane + 32 * j) + 1];
      }
}
__device__ __forceinline__ float pairs_inv_rms(const HeadPairs &h, int D, float eps) {
  float ss = 0.0f;
#pragma unroll
  for (int j = 0; j < 4; ++j) ss += h.p[j].x * h.p[j].x + h.p[j].y * h.p[j].y;  // padding is zero
  return 1.0f / sqrtf(warp_sum(ss) / (float)D + eps);
}

}  // namespace

// ---------------------------------------------------------------------------------------------
// Multi-token step: one CTA per row, one warp per head.
// ---------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) attn_prep_kernel(const AttnArgs a) {
  pdl_enter();
  const int64_t r = blockIdx.x;
  const int b = (int)(r / a.s), pos = a.n + (int)(r % a.s);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float *row = a.qkv + r * a.ld;
  const int64_t slot = pos % a.cap;
  for (int hd = warp; hd < a.H + 2 * a.G; hd += 8) {
    const bool is_q = hd < a.H, is_k = !is_q && hd < a.H + a.G;
    const int g = is_q ? 0 : (is_k ? hd - a.H : hd - a.H - a.G);
    float *src = row + (is_q ? a.q_off + (int64_t)hd * a.Dp : is_k ? a.k_off + (int64_t)g * a.Dp : a.v_off + (int64_t)g * a.Ep);
    const int np = (is_q || is_k ? a.Dp : a.Ep) / 2;
    HeadPairs h;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = lane + 32 * j;
      h.p[j] = i < np ? reinterpret_cast<const float2 *>(src)[i] : make_float2(0.f, 0.f);
    }
    float mul = 1.0f;
    float *dst = src;
    if (is_q || is_k) {
      rotate_pairs(h, a.freq, a.rot_pairs, pos, lane);
      if (a.qk_norm) mul = pairs_inv_rms(h, a.D, a.eps);
    }
    if (is_q) mul *= a.scale;
    else if (is_k) dst = a.kc + (((int64_t)b * a.G + g) * a.cap + slot) * a.Dp;
    else dst = a.vc + (((int64_t)b * a.G + g) * a.cap + slot) * a.Ep;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int i = lane + 32 * j;
      if (i < np) reinterpret_cast<float2 *>(dst)[i] = make_float2(h.p[j].x * mul, h.p[j].y * mul);
    }
  }
}

int launch_attn_prep(caten_b200_ctx *ctx, const AttnArgs &a) {
  const int64_t rows = (int64_t)a.B * a.s;
  if (rows <= 0) return 0;
  if (rows > 0x7fffffff || a.Dp > 256 || a.Ep > 256) return fail(ctx, CATEN_B200_EUNSUPPORTED, "attention: head size above 256");
  launch_k(ctx, attn_prep_kernel, dim3((unsigned)rows), dim3(256), 0, a);
  CB_LAUNCH_CHECK(ctx, "attn_prep_kernel");
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Multi-token step on the CUDA cores, any head size up to 256: 32 queries of one head per CTA, keys
// in blocks of 32, running maximum and sum.  Thread (ty, tx) of a 16 x 16 grid owns the scores of
// queries 2 ty, 2 ty + 1 with keys tx, tx + 16, and of the same queries the value columns
// 4 tx + 64 j .. + 3.
// ---------------------------------------------------------------------------------------------
constexpr int AW_T = 32;

__global__ void __launch_bounds__(256) attn_window_simt_kernel(const AttnArgs a) {
  extern __shared__ __align__(16) float sm[];
  pdl_enter();
  const int ldk = a.Dp + 4, ldv = a.Ep + 4;
  float *Qs = sm, *Ks = Qs + AW_T * ldk, *Vs = Ks + AW_T * ldk, *Ps = Vs + AW_T * ldv;
  const int q0 = blockIdx.x * AW_T, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const int tx = tid & 15, ty = tid >> 4;
  const int g = h / (a.H / a.G), t = a.n + a.s;
  const float *kb = a.kc + b * a.k_seq + g * a.k_head;
  const float *vb = a.vc + b * a.v_seq + g * a.v_head;
  const float *kx = a.kx + (a.kx ? b * a.cap * a.kx_ld : 0);
  const int d4 = a.Dp / 4, e4 = a.Ep / 4;
  for (int e = tid; e < AW_T * d4; e += 256) {
    const int i = e / d4, c = e % d4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (q0 + i < a.s) v = reinterpret_cast<const float4 *>(a.qkv + ((int64_t)b * a.s + q0 + i) * a.ld + a.q_off + (int64_t)h * a.Dp)[c];
    *reinterpret_cast<float4 *>(Qs + i * ldk + 4 * c) = v;
  }
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  float4 o[2][4];
#pragma unroll
  for (int q = 0; q < 2; ++q)
#pragma unroll
    for (int j = 0; j < 4; ++j) o[q][j] = make_float4(0.f, 0.f, 0.f, 0.f);
  const int W = a.window > 0 ? a.window : 0x3fffffff;
  const int first = a.n + q0 - W + 1;
  const int jbeg = first > 0 ? first / AW_T * AW_T : 0;
  const int jend = min(t, a.n + q0 + AW_T);
  for (int j0 = jbeg; j0 < jend; j0 += AW_T) {
    __syncthreads();
    for (int e = tid; e < AW_T * d4; e += 256) {
      const int i = e / d4, c = e % d4;
      const int64_t slot = (j0 + i) % a.cap;
      *reinterpret_cast<float4 *>(Ks + i * ldk + 4 * c) =
          j0 + i >= t ? make_float4(0.f, 0.f, 0.f, 0.f)
                      : *reinterpret_cast<const float4 *>(4 * c < a.kx_from ? kb + slot * a.k_ld + 4 * c : kx + slot * a.kx_ld + 4 * c - a.kx_from);
    }
    for (int e = tid; e < AW_T * e4; e += 256) {
      const int i = e / e4, c = e % e4;
      *reinterpret_cast<float4 *>(Vs + i * ldv + 4 * c) =
          j0 + i < t ? reinterpret_cast<const float4 *>(vb + (int64_t)((j0 + i) % a.cap) * a.v_ld)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    __syncthreads();
    float sc[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
    for (int c = 0; c < d4; ++c) {
      const float4 qa = *reinterpret_cast<const float4 *>(Qs + (2 * ty) * ldk + 4 * c), qb = *reinterpret_cast<const float4 *>(Qs + (2 * ty + 1) * ldk + 4 * c);
      const float4 ka = *reinterpret_cast<const float4 *>(Ks + tx * ldk + 4 * c), kc2 = *reinterpret_cast<const float4 *>(Ks + (tx + 16) * ldk + 4 * c);
      sc[0][0] = fmaf(qa.x, ka.x, fmaf(qa.y, ka.y, fmaf(qa.z, ka.z, fmaf(qa.w, ka.w, sc[0][0]))));
      sc[0][1] = fmaf(qa.x, kc2.x, fmaf(qa.y, kc2.y, fmaf(qa.z, kc2.z, fmaf(qa.w, kc2.w, sc[0][1]))));
      sc[1][0] = fmaf(qb.x, ka.x, fmaf(qb.y, ka.y, fmaf(qb.z, ka.z, fmaf(qb.w, ka.w, sc[1][0]))));
      sc[1][1] = fmaf(qb.x, kc2.x, fmaf(qb.y, kc2.y, fmaf(qb.z, kc2.z, fmaf(qb.w, kc2.w, sc[1][1]))));
    }
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      const int i = a.n + q0 + 2 * ty + q;  // the query's position
      float mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = j0 + tx + 16 * e;
        if (j > i || i - j >= W) sc[q][e] = -INFINITY;
        mx = fmaxf(mx, sc[q][e]);
      }
#pragma unroll
      for (int w = 8; w > 0; w >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, w));
      const float mn = fmaxf(m[q], mx), mu = mn == -INFINITY ? 0.0f : mn;  // nothing visible yet: keep the differences defined
      const float corr = exp2f((m[q] - mu) * kLog2e);
      float rs = 0.0f;
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const float p = exp2f((sc[q][e] - mu) * kLog2e);
        Ps[(2 * ty + q) * (AW_T + 1) + tx + 16 * e] = p;
        rs += p;
      }
#pragma unroll
      for (int w = 8; w > 0; w >>= 1) rs += __shfl_xor_sync(0xffffffffu, rs, w);
      l[q] = l[q] * corr + rs;
      m[q] = mn;
#pragma unroll
      for (int j = 0; j < 4; ++j) { o[q][j].x *= corr; o[q][j].y *= corr; o[q][j].z *= corr; o[q][j].w *= corr; }
    }
    __syncthreads();
    for (int k = 0; k < AW_T; ++k) {
      const float p0 = Ps[(2 * ty) * (AW_T + 1) + k], p1 = Ps[(2 * ty + 1) * (AW_T + 1) + k];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (4 * tx + 64 * j < a.Ep) {
          const float4 v = *reinterpret_cast<const float4 *>(Vs + k * ldv + 4 * tx + 64 * j);
          o[0][j].x = fmaf(p0, v.x, o[0][j].x); o[0][j].y = fmaf(p0, v.y, o[0][j].y);
          o[0][j].z = fmaf(p0, v.z, o[0][j].z); o[0][j].w = fmaf(p0, v.w, o[0][j].w);
          o[1][j].x = fmaf(p1, v.x, o[1][j].x); o[1][j].y = fmaf(p1, v.y, o[1][j].y);
          o[1][j].z = fmaf(p1, v.z, o[1][j].z); o[1][j].w = fmaf(p1, v.w, o[1][j].w);
        }
      }
    }
  }
#pragma unroll
  for (int q = 0; q < 2; ++q) {
    const int qi = q0 + 2 * ty + q;
    if (qi >= a.s) continue;
    const int64_t r = (int64_t)b * a.s + qi;
    float inv = 1.0f / l[q];
    if (a.gate_off >= 0) inv *= sigmoidf(a.qkv[r * a.ld + a.gate_off + h]);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = 4 * tx + 64 * j;
      if (c >= a.Ep) continue;
      const float4 v = make_float4(o[q][j].x * inv, o[q][j].y * inv, o[q][j].z * inv, o[q][j].w * inv);
      const int64_t at = r * a.out_ld + (int64_t)h * a.Ep + c;
      if (a.bf.hi) {
        *reinterpret_cast<uint2 *>(a.bf.hi + at) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
        if (a.bf.lo) *reinterpret_cast<uint2 *>(a.bf.lo + at) = make_uint2(pack_bf16(bf16_lo(v.x), bf16_lo(v.y)), pack_bf16(bf16_lo(v.z), bf16_lo(v.w)));
      } else {
        *reinterpret_cast<float4 *>(a.out + at) = v;
      }
    }
  }
}

static int check_attn(caten_b200_ctx *ctx, const AttnArgs &a) {
  if (a.H <= 0 || a.G <= 0 || a.H % a.G || a.D <= 0 || a.E <= 0 || a.Dp % 16 || a.Ep % 16 || a.D > a.Dp || a.E > a.Ep || a.cap <= 0 || a.n < 0)
    return fail(ctx, CATEN_B200_EINVAL, "attention: bad shape");
  if (a.Dp > 256 || a.Ep > 256) return fail(ctx, CATEN_B200_EUNSUPPORTED, "attention: head size above 256");
  if (a.H > 65535 || a.B > 65535) return fail(ctx, CATEN_B200_EUNSUPPORTED, "attention: B or H > 65535");
  return 0;
}

int launch_attn_window_prefill(caten_b200_ctx *ctx, const AttnArgs &args, int tensor_cores) {
  AttnArgs a = args;
  a.fill_strides();
  if (a.B <= 0 || a.s <= 0) return 0;
  if (int rc = check_attn(ctx, a)) return rc;
  // every key the step's queries may see is still in the ring
  const int64_t span = a.window > 0 && (int64_t)a.window - 1 < a.n ? (int64_t)a.window - 1 + a.s : (int64_t)a.n + a.s;
  if (span > a.cap) return fail(ctx, CATEN_B200_EINVAL, "attention: %lld live positions in a ring of %lld", (long long)span, (long long)a.cap);
  if (tensor_cores && a.Dp <= 128 && a.Ep <= 128) return launch_attention_tc_ex(ctx, a, 1.0f);
  const size_t smem = ((size_t)2 * AW_T * (a.Dp + 4) + (size_t)AW_T * (a.Ep + 4) + (size_t)AW_T * (AW_T + 1)) * sizeof(float);
  CB_CUDA(ctx, cudaFuncSetAttribute(attn_window_simt_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_k(ctx, attn_window_simt_kernel, dim3((unsigned)((a.s + AW_T - 1) / AW_T), (unsigned)a.H, (unsigned)a.B), dim3(256), smem, a);
  CB_LAUNCH_CHECK(ctx, "attn_window_simt_kernel");
  return 0;
}

// ---------------------------------------------------------------------------------------------
// Single-token step.  One CTA serves HPC query heads of one key/value head of one sequence, so a K / V
// row is read once for all of them; with few sequences a thread-block cluster splits the keys and its
// CTAs combine their (maximum, sum, output) through distributed shared memory.
//   producer warp   streams the history in chunks of CH rows, all of K and then all of V, into a ring of
//                   shared-memory stages (one bulk copy per chunk, two where it crosses the ring's end);
//                   V arrives while the last scores and the softmax are computed
//   prologue        the step's q, k, v (from the projection or its split-K partial tiles), rotated and
//                   normalised by one warp each; the k / v row is appended to the cache
//   scores          KL lanes x NV float4 per K row; the HPC x U dot products of a lane group are reduced
//                   together (each exchange halves the values a lane carries)
//   softmax         two passes over the CTA's scores in shared memory
//   output          P.V, summed over the row groups, rescaled over the cluster, gated
// Every mbarrier wait is bounded; when one runs out the CTA records it in the status word, leaves its
// loops, waits for its copies in flight, takes part in the cluster barriers and writes no output.
// ---------------------------------------------------------------------------------------------
constexpr int AD_WORK = 256, AD_THREADS = AD_WORK + 32, AD_MIN_STAGES = 3, AD_MAX_STAGES = 8;

__device__ __forceinline__ void work_sync() { asm volatile("bar.sync 1, %0;" ::"n"(AD_WORK) : "memory"); }
__device__ __forceinline__ void bulk_hint(const void *src, uint32_t bytes) {
  asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(src), "r"(bytes) : "memory");
}

template <int R>
__device__ __forceinline__ float group_reduce(float *v, int lane, int lanes) {
  int step = lanes >> 1;
#pragma unroll
  for (int r = R; r > 1; r >>= 1, step >>= 1) {
    const bool up = (lane & step) != 0;
#pragma unroll
    for (int i = 0; i < r / 2; ++i) {
      const float give = up ? v[i] : v[i + r / 2], keep = up ? v[i + r / 2] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, step);
    }
  }
  for (; step > 0; step >>= 1) v[0] += __shfl_xor_sync(0xffffffffu, v[0], step);
  return v[0];
}

template <int KL, int NV> struct AdShape {
  static constexpr int GROUPS = AD_WORK / KL;             // rows per load
  static constexpr int U = NV == 2 ? 2 : 4;               // loads per lane and chunk
  static constexpr int CH = GROUPS * U;                   // rows per chunk: 16 KB at the widest head of the class
};

template <int KL, int NV, int HPC>
__global__ void __launch_bounds__(AD_THREADS, NV == 1 ? 3 : 1) attn_window_decode_kernel(const AttnArgs a, const int S, const int stages, const int per_max, const long long hint_bytes,
                                                                        int *status) {
  constexpr int GROUPS = AdShape<KL, NV>::GROUPS, U = AdShape<KL, NV>::U, CH = AdShape<KL, NV>::CH;
  constexpr int R = U * HPC;                    // dot products reduced together (<= KL)
  static_assert(R <= KL, "one value per lane after the exchanges");
  constexpr int TPH = AD_WORK / HPC;            // threads per head in the softmax
  extern __shared__ __align__(16) float sm[];
  const int Dp = a.Dp, Ep = a.Ep, wide = Dp > Ep ? Dp : Ep;
  float *ring = sm;                             // [stages][CH][wide]; afterwards the row groups' outputs [GROUPS][HPC][Ep]
  float *q = ring + stages * CH * wide;      // [HPC][Dp]
  float *kn = q + HPC * Dp;                     // the step's key
  float *vn = kn + Dp;                          // and value
  float *gate = vn + Ep;                        // [4]
  float *ml = gate + 4;                         // [HPC] max, [HPC] sum (read by the other CTAs of the cluster): 8
  float *red = ml + 8;                          // 8
  float *ol = red + 8;                          // [HPC][Ep] this CTA's output
  uint64_t *bars = reinterpret_cast<uint64_t *>(ol + HPC * Ep);  // full, empty: [AD_MAX_STAGES] each
  volatile int *abort_flag = reinterpret_cast<volatile int *>(bars + 2 * AD_MAX_STAGES);  // [0] a wait ran out; [1] never set; 4 words
  float *sc = reinterpret_cast<float *>(bars + 2 * AD_MAX_STAGES + 2);  // [per_max][HPC]
  const uint32_t bar0 = smem_u32(bars);
  auto full = [&](int s) { return bar0 + 8u * s; };
  auto empty = [&](int s) { return bar0 + 8u * (AD_MAX_STAGES + s); };
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h0 = blockIdx.x * HPC, b = blockIdx.y, rank = blockIdx.z;
  const int rep = a.H / a.G, g = h0 / rep, cap = (int)a.cap;
  float *kb = a.kc + ((int64_t)b * a.G + g) * a.cap * Dp;
  float *vb = a.vc + ((int64_t)b * a.G + g) * a.cap * Ep;
  // this CTA's keys of the step at position n: [jb, je), of which [jb, hb) are history
  auto range = [&](int n, int &jb, int &je) {
    const int t0 = a.window > 0 && n - a.window + 1 > 0 ? n - a.window + 1 : 0;
    const int count = n + 1 - t0, per = (count + S - 1) / S;
    jb = t0 + min(rank * per, count);
    je = t0 + min((rank + 1) * per, count);
  };
  if (tid == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(full(s), 1);
      mbar_init(empty(s), AD_WORK / 32);
    }
    abort_flag[0] = abort_flag[1] = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  // While the kernels before this one still run, the first CTAs ask for their history to be brought into L2 (see
  // attn_decode_kernel: a hint, limited to what fits L2; a stale position only changes what is asked for).
  if (warp == AD_WORK / 32) {
    int jb, je, n = a.d_n ? *reinterpret_cast<const volatile int *>(a.d_n) : a.n;
    n = n < 0 ? 0 : n > 0x3fffffff ? 0x3fffffff : n;
    range(n, jb, je);
    const int hb = min(je, n);
    const long long bytes = (long long)(hb - jb) * (Dp + Ep) * 4;
    const long long index = ((long long)b * gridDim.x + blockIdx.x) * S + rank;
    if (hb > jb && hb - jb <= cap && (index + 1) * bytes <= hint_bytes) {
      const int which = lane & 1, piece = lane >> 1, w = which ? Ep : Dp;   // 16 pieces each of K and V
      const int rows = (hb - jb + 15) / 16, s0 = (jb + piece * rows) % cap, r = min(rows, hb - jb - piece * rows);
      if (r > 0) bulk_hint((which ? vb : kb) + (int64_t)s0 * w, (uint32_t)(min(r, cap - s0) * w) * 4u);
    }
  }
  __syncthreads();
  pdl_enter();
  const int n = a.d_n ? *a.d_n : a.n;
  int jb, je;
  range(n, jb, je);
  const int hb = min(je, n), hist = hb - jb, nc = (hist + CH - 1) / CH;
  const bool own_new = je == n + 1 && je > jb;   // the step's own key is in this CTA's range
  const int cnt = hist + (own_new ? 1 : 0);

  if (warp == AD_WORK / 32) {
    if (lane == 0) {
      int issued = 0, s = 0;
      uint32_t ph = 1;   // (a fresh barrier's previous phase counts as complete)
      for (int i = 0; i < 2 * nc; ++i) {
        if (!mbar_wait(empty(s), ph, abort_flag)) {
          if (!*abort_flag) { *abort_flag = 1; atomicCAS(status, 0, DEV_WAIT_TIMEOUT); status[1] = 20; }
          break;
        }
        const bool isv = i >= nc;
        const int c = isv ? i - nc : i, w = isv ? Ep : Dp;
        const int rows = min(CH, hist - c * CH), s0 = (jb + c * CH) % cap, r0 = min(rows, cap - s0);
        const float *base = isv ? vb : kb;
        const uint32_t dst = smem_u32(ring + s * CH * wide);
        mbar_expect_tx(full(s), (uint32_t)(rows * w) * 4u);
        bulk_load(dst, base + (int64_t)s0 * w, (uint32_t)(r0 * w) * 4u, full(s));
        if (r0 < rows) bulk_load(dst + (uint32_t)(r0 * w) * 4u, base, (uint32_t)((rows - r0) * w) * 4u, full(s));
        issued = i + 1;
        if (++s == stages) { s = 0; ph ^= 1u; }
      }
      if (*abort_flag)  // copies in flight land before the CTA's shared memory is released
        for (int i = issued > stages ? issued - stages : 0; i < issued; ++i) mbar_wait(full(i % stages), (uint32_t)(i / stages) & 1u, abort_flag + 1);
    }
    __syncwarp();
  } else {
    if (warp < HPC + 2) {
      const bool is_q = warp < HPC, is_k = warp == HPC;
      const int64_t off = is_q ? a.q_off + (int64_t)(h0 + warp) * Dp : is_k ? a.k_off + (int64_t)g * Dp : a.v_off + (int64_t)g * Ep;
      const int np = (is_q || is_k ? Dp : Ep) / 2;
      HeadPairs h;
      if (a.pin.splits > 0) {
        load_pairs_pending(h, a.pin, b, (int)off, np, lane);
      } else {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int i = lane + 32 * j;
          h.p[j] = i < np ? reinterpret_cast<const float2 *>(a.qkv + (int64_t)b * a.ld + off)[i] : make_float2(0.f, 0.f);
        }
      }
      float mul = 1.0f;
      if (is_q || is_k) {
        rotate_pairs(h, a.freq, a.rot_pairs, n, lane);
        if (a.qk_norm) mul = pairs_inv_rms(h, a.D, a.eps);
      }
      if (is_q) mul *= a.scale;
      float *dst = is_q ? q + warp * Dp : is_k ? kn : vn;
      float *row = is_k ? kb + (int64_t)(n % cap) * Dp : vb + (int64_t)(n % cap) * Ep;
      const bool append = !is_q && rank == 0 && h0 % rep == 0;  // one CTA per key/value head
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int i = lane + 32 * j;
        if (i < np) {
          const float2 v = make_float2(h.p[j].x * mul, h.p[j].y * mul);
          reinterpret_cast<float2 *>(dst)[i] = v;
          if (append) reinterpret_cast<float2 *>(row)[i] = v;
        }
      }
    } else if (warp == 7 && lane < HPC && a.gate_off >= 0) {
      const int col = (int)a.gate_off + h0 + lane;
      gate[lane] = sigmoidf(a.pin.splits > 0 ? partin_load1(a.pin, b, col) : a.qkv[(int64_t)b * a.ld + col]);
    }
    work_sync();
    const int gi = tid / KL, gl = tid % KL;
    if (own_new && warp < HPC) {
      float x = 0.0f;
      for (int i = lane; i < Dp; i += 32) x = fmaf(q[warp * Dp + i], kn[i], x);
      x = warp_sum(x);
      if (lane == 0) sc[hist * HPC + warp] = x;
    }
    bool ok = true;
    int s = 0;           // stage and phase of the chunk being consumed
    uint32_t ph = 0;
    {
      float4 q4[HPC][NV];
#pragma unroll
      for (int h = 0; h < HPC; ++h)
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          const int c = gl + KL * v;
          q4[h][v] = 4 * c < Dp ? reinterpret_cast<const float4 *>(q + h * Dp)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
        }
      for (int i = 0; i < nc && ok; ++i) {
        ok = __all_sync(0xffffffffu, mbar_wait(full(s), ph, abort_flag));
        if (!ok) break;
        const float *st = ring + s * CH * wide;
        float d[R];
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const int row = u * GROUPS + gi;
          float4 k4[NV];
#pragma unroll
          for (int v = 0; v < NV; ++v) {
            const int c = gl + KL * v;
            k4[v] = i * CH + row < hist && 4 * c < Dp ? reinterpret_cast<const float4 *>(st + row * Dp)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
          for (int h = 0; h < HPC; ++h) {
            float x = 0.0f;
#pragma unroll
            for (int v = 0; v < NV; ++v) x = fmaf(q4[h][v].x, k4[v].x, fmaf(q4[h][v].y, k4[v].y, fmaf(q4[h][v].z, k4[v].z, fmaf(q4[h][v].w, k4[v].w, x))));
            d[u * HPC + h] = x;
          }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(empty(s));
        if (++s == stages) { s = 0; ph ^= 1u; }
        const float x = group_reduce<R>(d, gl, KL);
        if (gl % (KL / R) == 0) {
          const int idx = gl / (KL / R), row = i * CH + (idx / HPC) * GROUPS + gi;
          if (row < hist) sc[row * HPC + idx % HPC] = x;
        }
      }
    }
    if (!ok && lane == 0 && !*abort_flag) { *abort_flag = 1; atomicCAS(status, 0, DEV_WAIT_TIMEOUT); status[1] = 21; }
    work_sync();
    {
      const int h = tid / TPH, i0 = tid % TPH;
      float m = -INFINITY;
      for (int i = i0; i < cnt; i += TPH) m = fmaxf(m, sc[i * HPC + h]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      if (lane == 0) red[warp] = m;
      work_sync();
      m = red[h * (8 / HPC)];
#pragma unroll
      for (int w = 1; w < 8 / HPC; ++w) m = fmaxf(m, red[h * (8 / HPC) + w]);
      float ss = 0.0f;
      for (int i = i0; i < cnt; i += TPH) {
        const float e = exp2f((sc[i * HPC + h] - m) * kLog2e);
        sc[i * HPC + h] = e;
        ss += e;
      }
      ss = warp_sum(ss);
      work_sync();
      if (lane == 0) red[warp] = ss;
      work_sync();
      if (i0 == 0) {
        ss = 0.0f;
#pragma unroll
        for (int w = 0; w < 8 / HPC; ++w) ss += red[h * (8 / HPC) + w];
        ml[h] = m;
        ml[4 + h] = ss;
      }
    }
    float4 acc[HPC][NV];
#pragma unroll
    for (int h = 0; h < HPC; ++h)
#pragma unroll
      for (int v = 0; v < NV; ++v) {
        const int c = gl + KL * v;
        const float p = own_new && gi == 0 ? sc[hist * HPC + h] : 0.0f;
        const float4 x = 4 * c < Ep ? reinterpret_cast<const float4 *>(vn)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
        acc[h][v] = make_float4(p * x.x, p * x.y, p * x.z, p * x.w);
      }
    for (int i = nc; i < 2 * nc && ok; ++i) {
      ok = __all_sync(0xffffffffu, mbar_wait(full(s), ph, abort_flag));
      if (!ok) break;
      const float *st = ring + s * CH * wide;
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int row = u * GROUPS + gi, key = (i - nc) * CH + row;
        if (key < hist) {
          float p[HPC];
          if (HPC == 4) *reinterpret_cast<float4 *>(p) = *reinterpret_cast<const float4 *>(sc + key * HPC);
          else
#pragma unroll
            for (int h = 0; h < HPC; ++h) p[h] = sc[key * HPC + h];
#pragma unroll
          for (int v = 0; v < NV; ++v) {
            const int c = gl + KL * v;
            const float4 x = 4 * c < Ep ? reinterpret_cast<const float4 *>(st + row * Ep)[c] : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int h = 0; h < HPC; ++h) {
              acc[h][v].x = fmaf(p[h], x.x, acc[h][v].x);
              acc[h][v].y = fmaf(p[h], x.y, acc[h][v].y);
              acc[h][v].z = fmaf(p[h], x.z, acc[h][v].z);
              acc[h][v].w = fmaf(p[h], x.w, acc[h][v].w);
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) mbar_arrive(empty(s));
      if (++s == stages) { s = 0; ph ^= 1u; }
    }
    if (!ok && lane == 0 && !*abort_flag) { *abort_flag = 1; atomicCAS(status, 0, DEV_WAIT_TIMEOUT); status[1] = 22; }
    work_sync();  // every chunk has been consumed: the ring becomes the exchange buffer of the row groups
    if (!*abort_flag) {
      float *part = ring;
#pragma unroll
      for (int h = 0; h < HPC; ++h)
#pragma unroll
        for (int v = 0; v < NV; ++v) {
          const int c = gl + KL * v;
          if (4 * c < Ep) reinterpret_cast<float4 *>(part + (gi * HPC + h) * Ep)[c] = acc[h][v];
        }
    }
    work_sync();
    if (!*abort_flag)
      for (int i = tid; i < HPC * Ep; i += AD_WORK) {
        float o = 0.0f;
#pragma unroll
        for (int w = 0; w < GROUPS; ++w) o += ring[w * HPC * Ep + i];
        ol[i] = o;
      }
  }
  auto finish = [&](int i, float o, float l) {
    const int h = i / Ep;
    o = o / l;
    if (a.gate_off >= 0) o *= gate[h];
    const int64_t at = (int64_t)b * a.out_ld + (int64_t)(h0 + h) * Ep + (i - h * Ep);
    if (a.bf.hi) {
      const __nv_bfloat16 hh = __float2bfloat16_rn(o);
      a.bf.hi[at] = hh;
      if (a.bf.lo) a.bf.lo[at] = __float2bfloat16_rn(o - __bfloat162float(hh));
    } else {
      a.out[at] = o;
    }
  };
  if (S == 1) {
    __syncthreads();
    if (!*abort_flag)
      for (int i = tid; i < HPC * Ep; i += AD_THREADS) finish(i, ol[i], ml[4 + i / Ep]);
    return;
  }
  // combine over the cluster; both barriers are reached by every thread of every CTA
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
  const uint32_t ml0 = smem_u32(ml), ol0 = smem_u32(ol);
  auto remote = [&](uint32_t local, int z) {
    uint32_t addr;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(addr) : "r"(local), "r"(z));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(addr) : "memory");
    return v;
  };
  if (!*abort_flag)
    for (int i = rank + S * tid; i < HPC * Ep; i += S * AD_THREADS) {
      // all CTAs' values are requested together: S <= 8 loads in flight instead of a chain of round trips
      const uint32_t h4 = 4u * (uint32_t)(i / Ep);
      float mz[8], lz[8], oz[8];
#pragma unroll
      for (int z = 0; z < 8; ++z)
        if (z < S) {
          mz[z] = remote(ml0 + h4, z);
          lz[z] = remote(ml0 + 16u + h4, z);
          oz[z] = remote(ol0 + 4u * (uint32_t)i, z);
        }
      float m = -INFINITY, l = 0.0f, o = 0.0f;
#pragma unroll
      for (int z = 0; z < 8; ++z)
        if (z < S) m = fmaxf(m, mz[z]);
#pragma unroll
      for (int z = 0; z < 8; ++z)
        if (z < S) {  // fixed order
          const float f = exp2f((mz[z] - m) * kLog2e);  // a CTA without keys has maximum -inf and adds nothing
          l = fmaf(f, lz[z], l);
          o = fmaf(f, oz[z], o);
        }
      finish(i, o, l);
    }
  asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}

template <int KL, int NV, int HPC>
static int launch_decode_t(caten_b200_ctx *ctx, const AttnArgs &a, int S, int stages, int per_max, size_t smem) {
  if (smem > 48 * 1024) CB_CUDA(ctx, cudaFuncSetAttribute(attn_window_decode_kernel<KL, NV, HPC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((unsigned)(a.H / HPC), (unsigned)a.B, (unsigned)S);
  cfg.blockDim = dim3(AD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = ctx->stream;
  cudaLaunchAttribute at[2];
  int na = 0;
  if (take_pdl(ctx)) {
    at[na].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[na].val.programmaticStreamSerializationAllowed = 1;
    ++na;
  }
  if (S > 1) {
    at[na].id = cudaLaunchAttributeClusterDimension;
    at[na].val.clusterDim.x = 1;
    at[na].val.clusterDim.y = 1;
    at[na].val.clusterDim.z = (unsigned)S;
    ++na;
  }
  cfg.attrs = at;
  cfg.numAttrs = na;
  CB_CUDA(ctx, cudaLaunchKernelEx(&cfg, attn_window_decode_kernel<KL, NV, HPC>, a, S, stages, per_max, ctx->attn_prefetch_bytes, ctx->d_status));
  CB_LAUNCH_CHECK(ctx, "attn_window_decode_kernel");
  return 0;
}

int launch_attn_window_decode(caten_b200_ctx *ctx, const AttnArgs &a) {
  if (a.B <= 0) return 0;
  if (a.s != 1) return fail(ctx, CATEN_B200_EINVAL, "attention: the decode kernel takes one token per sequence");
  if (int rc = check_attn(ctx, a)) return rc;
  // the most keys a query may see (with a device-side position: what the cache allows)
  int64_t keys = a.d_n ? a.cap : (int64_t)a.n + 1;
  if (a.window > 0 && a.window < keys) keys = a.window;
  if (keys > a.cap) return fail(ctx, CATEN_B200_EINVAL, "attention: %lld live positions in a ring of %lld", (long long)keys, (long long)a.cap);
  const int rep = a.H / a.G;
  int hpc = rep % 4 == 0 ? 4 : rep % 2 == 0 ? 2 : 1;
  const int wide = a.Dp > a.Ep ? a.Dp : a.Ep;
  if (wide > 128 && hpc == 4) hpc = 2;  // registers
  // few sequences: split the keys over the CTAs of a cluster (8 = portable size), at least 32 keys each
  auto ctas = [&](int h, int s) { return (int64_t)a.B * (a.H / h) * s; };
  int S = 1;
  while (S < 8 && ctas(hpc, S) < ctx->sm_count && keys / (2 * S) >= 32) S *= 2;
  // a little more than one wave (3 CTAs per SM): halves even out the second
  if (S == 1 && ctas(hpc, 1) > 3 * ctx->sm_count && ctas(hpc, 1) < 6 * ctx->sm_count && keys >= 256) S = 2;
  while (hpc > 1 && ctas(hpc, S) * 2 <= ctx->sm_count) hpc /= 2;
  const int kl = wide <= 64 ? 16 : 32, nv = wide <= 128 ? 1 : 2;
  const int ch = AD_WORK / kl * (nv == 2 ? 2 : 4);
  size_t smem = 0;
  int64_t per_max = 0;
  for (;;) {
    per_max = (keys + S - 1) / S;
    // (the row groups' outputs, hpc / 4 of [ch][4][Ep] / U floats, fit the ring they reuse)
    smem = ((size_t)AD_MIN_STAGES * ch * wide + (size_t)hpc * a.Dp + a.Dp + a.Ep + 20 + (size_t)hpc * a.Ep + (size_t)hpc * per_max) * sizeof(float) +
           (2 * AD_MAX_STAGES + 2) * 8;
    if (smem <= 200 * 1024) break;
    if (S < 8) S *= 2;
    else if (hpc > 1) hpc /= 2;
    else return fail(ctx, CATEN_B200_EUNSUPPORTED, "attention: context too long for the decode kernel");
  }
  // a small grid leaves shared memory for a deeper ring: at most as many stages as there are chunks, and about 200 KB per SM
  int stages = AD_MIN_STAGES;
  // (a large cluster is placed inside one group of SMs: its CTAs share SMs even when the grid alone would not need to)
  const size_t stage = (size_t)ch * wide * sizeof(float);
  size_t per_sm = (size_t)((ctas(hpc, S) + ctx->sm_count - 1) / ctx->sm_count);
  if (S >= 4 && per_sm < 2) per_sm = 2;
  while (stages < AD_MAX_STAGES && stages < 2 * ((per_max + ch - 1) / ch) && (smem + stage) * per_sm <= 200 * 1024) { ++stages; smem += stage; }
#define AD_CASE(KL, NV)                                                                                    \
  (hpc == 4 ? launch_decode_t<KL, NV, 4>(ctx, a, S, stages, (int)per_max, smem)                                    \
   : hpc == 2 ? launch_decode_t<KL, NV, 2>(ctx, a, S, stages, (int)per_max, smem) : launch_decode_t<KL, NV, 1>(ctx, a, S, stages, (int)per_max, smem))
  if (kl == 16) return AD_CASE(16, 1);
  if (nv == 1) return AD_CASE(32, 1);
  return AD_CASE(32, 2);
#undef AD_CASE
}

}  // namespace cb

using namespace cb;

extern "C" int caten_b200_attn_window(caten_b200_ctx *ctx, const caten_b200_attn_desc *c, float *d_qkv, int64_t ld, float *d_kcache,
                                      float *d_vcache, int64_t cap, float *d_out, int64_t B, int64_t s, int64_t n, int precision) {
  if (!ctx) return fail(nullptr, CATEN_B200_EINVAL, "attn_window: ctx is NULL");
  cudaSetDevice(ctx->device);
  if (!c || !d_qkv || !d_kcache || !d_vcache || !d_out) return fail(ctx, CATEN_B200_EINVAL, "attn_window: NULL argument");
  if (B < 0 || s < 0 || n < 0 || cap <= 0 || cap % 64 || cap > 0x3fffffff || n + s > 0x3fffffff || c->heads <= 0 || c->kv_heads <= 0 || c->heads % c->kv_heads || c->dim <= 0 || c->vdim <= 0 ||
      c->window < 0 || c->rot_dims < 0 || c->rot_dims % 2 || c->rot_dims > c->dim || (c->rot_dims && !c->rot_freq))
    return fail(ctx, CATEN_B200_EINVAL, "attn_window: bad shape");
  if (precision < CATEN_B200_PREC_FP32 || precision > CATEN_B200_PREC_BF16X3) return fail(ctx, CATEN_B200_EINVAL, "attn_window: unknown precision %d", precision);
  AttnArgs a;
  a.H = c->heads; a.G = c->kv_heads;
  a.D = c->dim; a.Dp = (c->dim + 15) / 16 * 16; a.E = c->vdim; a.Ep = (c->vdim + 15) / 16 * 16;
  a.qkv = d_qkv; a.ld = ld;
  a.k_off = (int64_t)a.H * a.Dp; a.v_off = a.k_off + (int64_t)a.G * a.Dp;
  a.gate_off = c->gated ? a.v_off + (int64_t)a.G * a.Ep : -1;
  if (ld % 4 || ld < a.v_off + (int64_t)a.G * a.Ep + (c->gated ? a.H : 0)) return fail(ctx, CATEN_B200_EINVAL, "attn_window: ld=%lld", (long long)ld);
  a.kc = d_kcache; a.vc = d_vcache; a.cap = cap;
  a.out = d_out; a.out_ld = (int64_t)a.H * a.Ep;
  a.B = (int)B; a.s = (int)s; a.n = (int)n;
  a.window = c->window; a.rot_pairs = c->rot_dims / 2; a.freq = c->rot_freq; a.qk_norm = c->qk_norm; a.eps = c->eps; a.scale = c->scale;
  if (B == 0 || s == 0) return 0;
  ProfScope prof(ctx, s == 1 ? CATEN_B200_K_ATTN_DECODE : CATEN_B200_K_ATTN_PREFILL);
  if (s == 1) return launch_attn_window_decode(ctx, a);
  // checked before the append, which writes the ring
  const int64_t live = c->window > 0 && c->window - 1 < n ? c->window - 1 + s : n + s;
  if (live > cap) return fail(ctx, CATEN_B200_EINVAL, "attn_window: %lld live positions in a ring of %lld", (long long)live, (long long)cap);
  if (int rc = launch_attn_prep(ctx, a)) return rc;
  return launch_attn_window_prefill(ctx, a, precision != CATEN_B200_PREC_FP32);
}
