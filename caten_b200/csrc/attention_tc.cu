// Prefill attention (s > 1) on the 5th-generation tensor cores over an fp32 KV cache, for head sizes up
// to 128 (NQ / NE = 64-wide blocks of the query/key / value head), grouped query heads, an optional
// sliding window and a ring-buffered cache (attn_window.cuh).  GPT-2 (head dim 64, a cache
// [B, H, T, 64] that never wraps, no window) is the PLAIN case of NQ = NE = 1.  Same semantics as the SIMT kernels in attention.cu
// (external/llm/layers.lisp:3-5,19-51: S = (q.K^T) * 0.125 + causal mask; P = softmax(S) with
// exp(x) = exp2(x * 1/ln2), two passes: row maximum first, then exp and sum; O = P.V), with both
// contractions as bf16 hi/lo split products accumulated in fp32 (every operand x = x_hi + x_lo;
// q.K^T keeps all four products, P.V drops only lo*lo), so the result stays within about 2^-16
// of the fp32 one.
//
// One CTA = 128 queries of one (sequence, head) = the 128 lanes of tensor memory; keys go in
// steps of 64 (with a window: from the step that holds the first key any of the tile's queries sees).
// With NQ = NE = 1 a CTA uses 256 of the 512 TMEM columns and under half of the shared memory, so two
// CTAs share an SM and one's MMAs overlap the other's softmax.  Per step:
//   all 8 warps  copy the NEXT step's K (and V) rows from the cache into a staging buffer in shared
//                memory (cp.async, 16 bytes per thread, coalesced; in flight during this step's
//                MMAs and softmax), and split the current step's staged rows into bf16 hi/lo,
//                stored as 128-byte-swizzled K-major tiles in shared memory:
//                K tiles  = 64 keys x 64 dims, hi and lo, per block  (K-major B operands of S = Q.K^T)
//                V tiles  = 64 keys x 64 dims, hi and lo, per block  (MN-major B operands of O += P.V)
//   one thread   issues S[128 x 64] = (Q_hi + Q_lo) . (K_hi + K_lo)^T as four MMAs per 16 dims into
//                the same 64 columns (Q tile in shared memory)
//   all 8 warps  read their query's scores from tensor memory (warps w and w+4 share lanes and
//                take 32 keys each), mask, and
//                p = exp2((s - max)/ln2), accumulate the row sum, split p into bf16 hi/lo and
//                write it back to tensor memory as the A operand of the second product
//   one thread   issues O[128 x 64] += P_hi.V_hi + P_lo.V_hi + P_hi.V_lo, accumulating over the
//                key steps in tensor memory
// The softmax is single-pass with a lazily moved reference maximum: each step exchanges the
// maximum of its visible scores between the row's two threads; the reference only moves (and O and
// the row sum are rescaled, O by a TMEM load / multiply / store) when a step exceeds it by more
// than AT_TAU, which in causal attention happens in the first steps and then rarely.  Softmax is
// invariant to the reference, so this equals the reference's two-pass form up to rounding.  The
// phases of a step are sequential within the CTA (block-wide barriers + one mbarrier the MMAs
// commit to).
// TMEM columns: [0,64) S, [128,192) P (hi 32, lo 32), [192, 192 + 64 NE) O.
//
// The mbarrier waits are bounded; when one runs out the CTA records it in the context's status
// word, skips the remaining work and its output, frees its tensor memory and returns.
#include "attn_window.cuh"
#include "tcgen05.cuh"

namespace cb {

namespace {

constexpr float kAtInvLn2 = 1.0f / 0.6931472f;  // (/ (log 2)) in single float, api/function.lisp:437-440
constexpr int AT_Q = 128;                        // queries per CTA (MMA M)
constexpr int AT_K = 64;                         // keys per step
constexpr float AT_TAU = 8.0f;                   // slack of the running maximum, in units of the score
constexpr uint32_t AT_COL_S = 0, AT_COL_P = 128, AT_COL_O = 192;
template <int NQ, int NE> struct AtLayout {
  static constexpr uint32_t COLS = NE == 1 ? 256 : 512;  // TMEM columns per CTA (a power of two)
  // Q: per block 128 rows hi, 128 rows lo (16 KB each); K, V: per block 64 rows hi, 64 rows lo (8 KB each)
  static constexpr uint32_t OFF_Q = 0, OFF_K = NQ * 32768, OFF_V = OFF_K + NQ * 16384, OFF_SK = OFF_V + NE * 16384;
  // staging of the raw fp32 rows: 256 bytes per block and row, padded by 16, so that threads reading one
  // row each (16 bytes at a time) spread over all banks
  static constexpr uint32_t LD_K = NQ * 256 + 16, LD_V = NE * 256 + 16;
  static constexpr uint32_t OFF_SV = OFF_SK + AT_K * LD_K, OFF_MISC = OFF_SV + AT_K * LD_V;
  // tiles + staging + exchange buffer + barrier / TMEM slot / abort flag + alignment slack
  static constexpr size_t SMEM = OFF_MISC + 1024 + 64 + 1024;
  static constexpr int CTAS = NQ == 1 && NE == 1 ? 2 : 1;  // per SM
};
static_assert(2 * (AtLayout<1, 1>::SMEM + 1024) <= 227 * 1024, "two CTAs per SM");
static_assert(AtLayout<2, 2>::SMEM <= 227 * 1024, "one CTA per SM");

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src, uint32_t src_bytes) {  // src_bytes 0: zero fill
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(src_bytes) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

// byte offset of 16-byte chunk `chunk` (0..7) of row `row` in a K-major tile with 128-byte rows
// and the 128-byte swizzle (8-row groups of 1024 bytes)
__device__ __forceinline__ uint32_t sw128(int row, int chunk) {
  return (uint32_t)((row >> 3) * 1024 + (row & 7) * 128 + ((chunk ^ (row & 7)) << 4));
}

__device__ __forceinline__ uint4 pack8(const float4 a, const float4 b) {
  return make_uint4(pack_bf16(a.x, a.y), pack_bf16(a.z, a.w), pack_bf16(b.x, b.y), pack_bf16(b.z, b.w));
}
__device__ __forceinline__ uint4 pack8_lo(const float4 a, const float4 b) {
  return make_uint4(pack_bf16(bf16_lo(a.x), bf16_lo(a.y)), pack_bf16(bf16_lo(a.z), bf16_lo(a.w)),
                    pack_bf16(bf16_lo(b.x), bf16_lo(b.y)), pack_bf16(bf16_lo(b.z), bf16_lo(b.w)));
}
// 8 consecutive fp32 of one row -> one chunk of the hi row and one of the lo row
__device__ __forceinline__ void st_split8(unsigned char *tile, int row_hi, int row_lo, int chunk, const float4 a, const float4 b) {
  *reinterpret_cast<uint4 *>(tile + sw128(row_hi, chunk)) = pack8(a, b);
  *reinterpret_cast<uint4 *>(tile + sw128(row_lo, chunk)) = pack8_lo(a, b);
}

// 2^x by one PTX ex2.approx instruction; results below 2^-126 flush to zero (such probabilities do not
// register in a row sum >= 1/e^8)
__device__ __forceinline__ float ex2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

template <int N> struct IntC { static constexpr int value = N; };

__device__ __forceinline__ float4 scale4(float4 v, float c) { return make_float4(v.x * c, v.y * c, v.z * c, v.w * c); }

}  // namespace

// PLAIN: heads of exactly 64, no window, a cache that never wraps (GPT-2): the masks' lower ends, the ring arithmetic and
// the zero-filled head columns compile away.
template <int NQ, int NE, bool PLAIN>
__global__ void __launch_bounds__(256, AtLayout<NQ, NE>::CTAS) attn_prefill_tc_kernel(const AttnArgs p, float qscale, int *status, uint32_t idesc_n64) {
  using Lay = AtLayout<NQ, NE>;
  constexpr uint32_t AT_OFF_Q = Lay::OFF_Q, AT_OFF_K = Lay::OFF_K, AT_OFF_V = Lay::OFF_V, AT_OFF_SK = Lay::OFF_SK, AT_OFF_SV = Lay::OFF_SV, AT_OFF_MISC = Lay::OFF_MISC;
  extern __shared__ unsigned char at_raw[];
  unsigned char *sm = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(at_raw) + 1023) & ~(uintptr_t)1023);
  float *red = reinterpret_cast<float *>(sm + AT_OFF_MISC);
  const uint32_t bar = smem_u32(sm + AT_OFF_MISC + 1024);
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(sm + AT_OFF_MISC + 1024 + 8);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(sm + AT_OFF_MISC + 1024 + 12);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int quad = warp & 3;  // 32-lane quadrant of tensor memory this warp may access
  const int hf = warp >> 2;   // which half (of a step's keys / of a block's head dims) this thread takes
  const int r = quad * 32 + lane;  // query row within the tile = TMEM lane
  const int ck = tid & 63, cq = tid >> 6;  // conversion: key row of the step, and which 16 of a block's 64 dims
  const int q0 = (int)(gridDim.x - 1 - blockIdx.x) * AT_Q;  // tiles with the longest history first
  const int h = blockIdx.y, b = blockIdx.z;
  const int s = p.s, n = p.n, t = n + s;

  if (tid == 0) {
    mbar_init(bar, 1);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 0) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(Lay::COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tlane = tmem_base + ((uint32_t)(quad * 32) << 16);
  pdl_enter();

  const int Dp = PLAIN ? 64 : p.Dp, Ep = PLAIN ? 64 : p.Ep;
  const int64_t head = (int64_t)b * p.G + (PLAIN ? h : h / (p.H / p.G));  // the key/value head this query head reads
  const int64_t kv_head = head - (int64_t)b * p.G;
  const float *kb = PLAIN ? p.kc + head * p.cap * 64 : p.kc + b * p.k_seq + kv_head * p.k_head;
  const float *vb = PLAIN ? p.vc + head * p.cap * 64 : p.vc + b * p.v_seq + kv_head * p.v_head;
  const float *kx = !PLAIN && p.kx ? p.kx + b * p.cap * p.kx_ld - p.kx_from : nullptr;   // column c of the key, c >= kx_from
  const int W = !PLAIN && p.window > 0 ? p.window : 0x3fffffff;
  const int kend = min(t, n + q0 + AT_Q);  // keys beyond the last query of this tile are masked
  const int kfirst = PLAIN ? 0 : n + q0 - W + 1;       // first key the tile's first query sees
  const int kbeg = kfirst > 0 ? kfirst / AT_K * AT_K : 0;
  const int nblk = (kend - kbeg + AT_K - 1) / AT_K;
  const int qi = min(q0 + r, s - 1);  // rows past the end of the step mask like the last row (their output is dropped)
  const int jmax = n + qi;            // last visible key of this query (< t)
  const int jmin = jmax - W + 1;      // first visible key (may be negative)

  const uint64_t dq = umma_desc(smem_u32(sm + AT_OFF_Q)), dk = umma_desc(smem_u32(sm + AT_OFF_K)), dv = umma_desc(smem_u32(sm + AT_OFF_V));
  const uint32_t idesc_pv = idesc_n64 | (1u << 16);  // B operand MN-major: V rows (keys) with the dims contiguous
  const int ksteps = Dp / 16;
  uint32_t ph = 0;
  int ok = 1;

  // copy the 64 rows [j0, j0+64) of one head's K or V history into a staging buffer; rows past
  // the end of the context and columns past the head are zero-filled
  auto prefetch = [&](const float *base, int64_t ld, int j0, uint32_t stage_off, auto nb, int width, bool key) {
    constexpr int NB = decltype(nb)::value;
    const int slot0 = PLAIN ? j0 : (int)(j0 % p.cap);
#pragma unroll
    for (int i = 0; i < 4 * NB; ++i) {
      const int piece = tid + 256 * i, row = piece / (16 * NB), c16 = piece % (16 * NB);
      const bool okk = j0 + row < t && (PLAIN || c16 * 4 < width);
      int slot = slot0 + row;
      if (!PLAIN && slot >= (int)p.cap) slot -= (int)p.cap;
      const float *src = base + (okk ? (int64_t)slot * (PLAIN ? 64 : ld) + c16 * 4 : 0);
      if (!PLAIN && key && okk && c16 * 4 >= p.kx_from) src = kx + (int64_t)slot * p.kx_ld + c16 * 4;
      cp_async16(smem_u32(sm + stage_off + row * (NB * 256 + 16) + c16 * 16), src, okk ? 16u : 0u);
    }
  };
  auto staged_row = [&](uint32_t row_off, int block, float4 *v) {  // this thread's 16 dims of its key row
    const float4 *src = reinterpret_cast<const float4 *>(sm + row_off + 256 * block + 64 * cq);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = src[i];
  };
  // one warp polls the mbarrier; the others park at the block barrier instead of spinning (their
  // issue slots go to the other CTA of the SM)
  auto wait_mma = [&]() {
    if (warp == 0 && !mbar_wait(bar, ph, abort_flag)) {
      ok = 0;
      *abort_flag = 1;
    }
    ph ^= 1u;
    ok = __syncthreads_and(ok);
  };

  prefetch(kb, p.k_ld, kbeg, AT_OFF_SK, IntC<NQ>(), Dp, true);
  prefetch(vb, p.v_ld, kbeg, AT_OFF_SV, IntC<NE>(), Ep, false);
  cp_async_commit();
  // Q tiles: rows [0,128) hi, [128,256) lo per block; GPT-2's 1/8 score scale is folded in (a power of two: exact)
  {
    const bool okq = q0 + r < s;
    const float4 *src = reinterpret_cast<const float4 *>(p.qkv + ((int64_t)b * s + (okq ? q0 + r : 0)) * p.ld + p.q_off + (int64_t)h * Dp);
#pragma unroll
    for (int kb_ = 0; kb_ < NQ; ++kb_) {
      float4 v[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int c4 = 16 * kb_ + 8 * hf + i;
        v[i] = okq && (PLAIN || 4 * c4 < Dp) ? scale4(src[c4], qscale) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int c = 0; c < 4; ++c) st_split8(sm + AT_OFF_Q + kb_ * 32768, r, 128 + r, 4 * hf + c, v[2 * c], v[2 * c + 1]);
    }
  }
  cp_async_wait_all();
  __syncthreads();  // step 0 of K and V is staged (and the Q tile is written)

  // ---- key steps: scores, running maximum, probabilities, row sums, O ---------------------------------
  float m = -INFINITY;  // the row's reference maximum: the same value in both threads of a row
  float lsum = 0.0f;    // this thread's part of the row sum, relative to m
  for (int blk = 0; blk < nblk && ok; ++blk) {
    const int j0 = kbeg + blk * AT_K;
    {
      // split this thread's part of the staged rows in registers, then (once the previous step's
      // P.V has read the V^T tile and P) store it into the tiles
      uint4 khi[NQ][2], klo[NQ][2], vhi[NE][2], vlo[NE][2];
#pragma unroll
      for (int w = 0; w < NQ; ++w) {
        float4 kv[4];
        staged_row(AT_OFF_SK + ck * Lay::LD_K, w, kv);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          khi[w][c] = pack8(kv[2 * c], kv[2 * c + 1]);
          klo[w][c] = pack8_lo(kv[2 * c], kv[2 * c + 1]);
        }
      }
#pragma unroll
      for (int w = 0; w < NE; ++w) {
        float4 vv[4];
        staged_row(AT_OFF_SV + ck * Lay::LD_V, w, vv);
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          vhi[w][c] = pack8(vv[2 * c], vv[2 * c + 1]);
          vlo[w][c] = pack8_lo(vv[2 * c], vv[2 * c + 1]);
        }
      }
      if (blk > 0) wait_mma();
#pragma unroll
      for (int w = 0; w < NQ; ++w)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          *reinterpret_cast<uint4 *>(sm + AT_OFF_K + w * 16384 + sw128(ck, 2 * cq + c)) = khi[w][c];
          *reinterpret_cast<uint4 *>(sm + AT_OFF_K + w * 16384 + sw128(64 + ck, 2 * cq + c)) = klo[w][c];
        }
      // V tiles (hi, then lo): rows = keys, 64 dims contiguous: the MMA reads them as an MN-major B operand
#pragma unroll
      for (int w = 0; w < NE; ++w)
#pragma unroll
        for (int c = 0; c < 2; ++c) {
          *reinterpret_cast<uint4 *>(sm + AT_OFF_V + w * 16384 + sw128(ck, 2 * cq + c)) = vhi[w][c];
          *reinterpret_cast<uint4 *>(sm + AT_OFF_V + w * 16384 + 8192 + sw128(ck, 2 * cq + c)) = vlo[w][c];
        }
    }
    fence_proxy_async();
    tc_fence_before();
    ok = __syncthreads_and(ok);  // tiles complete, staging buffers free
    if (!ok) break;
    if (warp == 0) {  // converged warp, one elected lane: the descriptors stay in uniform registers
      tc_fence_after();
      if (elect_one()) {
#pragma unroll
        for (int k = 0; k < 4 * NQ; ++k) {
          if (NQ == 1 || k < ksteps) {
            // 16 bf16 = 32 bytes = 2 descriptor units; a Q block is 32 KB = 2048 units, a K block 16 KB = 1024
            const uint64_t aq = dq + (uint64_t)((k >> 2) * 2048 + 2 * (k & 3)), ak = dk + (uint64_t)((k >> 2) * 1024 + 2 * (k & 3));
            umma_bf16(tmem_base + AT_COL_S, aq, ak, idesc_n64, k > 0 ? 1u : 0u);
            umma_bf16(tmem_base + AT_COL_S, aq + 1024, ak, idesc_n64, 1u);
            umma_bf16(tmem_base + AT_COL_S, aq, ak + 512, idesc_n64, 1u);
            umma_bf16(tmem_base + AT_COL_S, aq + 1024, ak + 512, idesc_n64, 1u);
          }
        }
        umma_commit(bar);
      }
      __syncwarp();
    }
    // the next step's rows start to arrive while the MMAs run (issued after them: the MMAs are the critical path)
    if (blk + 1 < nblk) {
      prefetch(kb, p.k_ld, j0 + AT_K, AT_OFF_SK, IntC<NQ>(), Dp, true);
      prefetch(vb, p.v_ld, j0 + AT_K, AT_OFF_SV, IntC<NE>(), Ep, false);
      cp_async_commit();
    }
    wait_mma();
    tc_fence_after();
    {
      // this thread's 32 keys in one round trip to tensor memory
      uint32_t a[32];
      tmem_ld16(tlane + AT_COL_S + 32 * hf, a);
      tmem_ld16(tlane + AT_COL_S + 32 * hf + 16, a + 16);
      tmem_ld_wait();
      // maximum of the visible scores of this step: over this thread's 32 keys, then over the row's two threads
      const int lim = jmax - j0 - 32 * hf, low = jmin - j0 - 32 * hf;  // key e of this thread is visible iff low <= e <= lim
      float mloc = -INFINITY;
#pragma unroll
      for (int e = 0; e < 32; ++e)
        if (e <= lim && (PLAIN || e >= low)) mloc = fmaxf(mloc, __uint_as_float(a[e]));
      red[hf * 128 + r] = mloc;
      __syncthreads();
      const float mstep = fmaxf(red[r], red[128 + r]);
      // The reference maximum only moves when the step's maximum exceeds it by more than AT_TAU
      // (probabilities then stay below e^AT_TAU, harmless in fp32 / split bf16); when it moves, O and
      // the row sum accumulated so far are rescaled.  Softmax is invariant to the shift, so this is
      // the two-pass result up to rounding.  Without a window step 0 always sees key 0; with one, m stays
      // -inf (and every probability zero) until the row's first visible key.
      const bool move = mstep > m + AT_TAU;  // also true at the first visible key (m = -inf)
      const float m_new = move ? mstep : m;
      if (blk > 0 && __any_sync(0xffffffffu, move)) {
        const float scale = move ? exp2f((m - m_new) * kAtInvLn2) : 1.0f;
        lsum *= scale;
#pragma unroll
        for (int w = 0; w < NE; ++w) {
          uint32_t o[32];
          tmem_ld16(tlane + AT_COL_O + 64 * w + 32 * hf, o);
          tmem_ld16(tlane + AT_COL_O + 64 * w + 32 * hf + 16, o + 16);
          tmem_ld_wait();
#pragma unroll
          for (int e = 0; e < 32; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * scale);
          tmem_st16(tlane + AT_COL_O + 64 * w + 32 * hf, o);
          tmem_st16(tlane + AT_COL_O + 64 * w + 32 * hf + 16, o + 16);
        }
      }
      m = m_new;
#pragma unroll
      for (int c = 0; c < 2; ++c) {
        float pr[16];
#pragma unroll
        for (int e = 0; e < 16; ++e) {
          const float val = __uint_as_float(a[16 * c + e]);
          pr[e] = (16 * c + e <= lim && (PLAIN || 16 * c + e >= low)) ? ex2_approx((val - m) * kAtInvLn2) : 0.0f;
          lsum += pr[e];
        }
        uint32_t phi[8], plo[8];
#pragma unroll
        for (int e = 0; e < 8; ++e) {
          phi[e] = pack_bf16(pr[2 * e], pr[2 * e + 1]);
          plo[e] = pack_bf16(bf16_lo(pr[2 * e]), bf16_lo(pr[2 * e + 1]));
        }
        // 16 keys = 8 columns; key k of the step sits in column k / 2
        tmem_st8(tlane + AT_COL_P + 16 * hf + 8 * c, phi);
        tmem_st8(tlane + AT_COL_P + 32 + 16 * hf + 8 * c, plo);
      }
    }
    tmem_st_wait();
    tc_fence_before();
    cp_async_wait_all();
    ok = __syncthreads_and(ok);  // P is written; the next step's rows are staged
    if (!ok) break;
    if (warp == 0) {  // converged warp, one elected lane: the descriptors stay in uniform registers
      tc_fence_after();
      if (elect_one()) {
#pragma unroll
        for (int w = 0; w < NE; ++w) {
          const uint32_t acc = tmem_base + AT_COL_O + 64 * w;
          const uint64_t dv_hi = dv + (uint64_t)(1024 * w), dv_lo = dv_hi + 512;
#pragma unroll
          for (int k4 = 0; k4 < 4; ++k4) {
            const uint64_t adv = (uint64_t)(64 * 2 * k4);  // 16 keys = 16 rows of 128 bytes = 128 descriptor units
            const uint32_t p_hi = tmem_base + AT_COL_P + 8 * k4, p_lo = p_hi + 32;
            umma_bf16_ts(acc, p_hi, dv_hi + adv, idesc_pv, (blk > 0 || k4 > 0) ? 1u : 0u);
            umma_bf16_ts(acc, p_lo, dv_hi + adv, idesc_pv, 1u);
            umma_bf16_ts(acc, p_hi, dv_lo + adv, idesc_pv, 1u);
          }
        }
        umma_commit(bar);
      }
      __syncwarp();
    }
  }
  if (ok && nblk > 0) wait_mma();
  tc_fence_after();
  red[hf * 128 + r] = lsum;
  ok = __syncthreads_and(ok);
  if (ok) {
    float inv = 1.0f / (red[r] + red[128 + r]);
    const int64_t orow = (int64_t)b * s + q0 + r;
    if (!PLAIN && p.gate_off >= 0 && q0 + r < s) inv *= 1.0f / (1.0f + expf(-p.qkv[orow * p.ld + p.gate_off + h]));
#pragma unroll
    for (int w = 0; w < NE; ++w) {
      uint32_t a[32];
      tmem_ld16(tlane + AT_COL_O + 64 * w + 32 * hf, a);
      tmem_ld16(tlane + AT_COL_O + 64 * w + 32 * hf + 16, a + 16);
      tmem_ld_wait();
      float o[32];
#pragma unroll
      for (int e = 0; e < 32; ++e) o[e] = __uint_as_float(a[e]) * inv;
      if (q0 + r < s) {
        const int c0 = 64 * w + 32 * hf;
        const int64_t at = orow * p.out_ld + (int64_t)h * Ep + c0;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (!PLAIN && c0 + 8 * i >= Ep) continue;
          const float *v = o + 8 * i;
          if (p.bf.hi) {
            *reinterpret_cast<uint4 *>(p.bf.hi + at + 8 * i) =
                make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
            if (p.bf.lo)
              *reinterpret_cast<uint4 *>(p.bf.lo + at + 8 * i) =
                  make_uint4(pack_bf16(bf16_lo(v[0]), bf16_lo(v[1])), pack_bf16(bf16_lo(v[2]), bf16_lo(v[3])),
                             pack_bf16(bf16_lo(v[4]), bf16_lo(v[5])), pack_bf16(bf16_lo(v[6]), bf16_lo(v[7])));
          } else {
            *reinterpret_cast<float4 *>(p.out + at + 8 * i) = make_float4(v[0], v[1], v[2], v[3]);
            *reinterpret_cast<float4 *>(p.out + at + 8 * i + 4) = make_float4(v[4], v[5], v[6], v[7]);
          }
        }
      }
    }
  } else if (tid == 0) {
    atomicCAS(status, 0, DEV_WAIT_TIMEOUT);
    status[1] = 10;
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 0) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(Lay::COLS) : "memory");
  }
}

template <int NQ, int NE, bool PLAIN = false>
static int launch_at(caten_b200_ctx *ctx, const AttnArgs &a, float qscale) {
  const uint32_t base = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(AT_Q >> 4) << 24);  // fp32 accumulate, bf16 x bf16, M = 128
  const uint32_t idesc_n64 = base | ((uint32_t)(64 >> 3) << 17);
  constexpr size_t smem = AtLayout<NQ, NE>::SMEM;
  CB_CUDA(ctx, cudaFuncSetAttribute(attn_prefill_tc_kernel<NQ, NE, PLAIN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_k(ctx, attn_prefill_tc_kernel<NQ, NE, PLAIN>, dim3((unsigned)((a.s + AT_Q - 1) / AT_Q), (unsigned)a.H, (unsigned)a.B), dim3(256), smem, a, qscale,
           ctx->d_status, idesc_n64);
  CB_LAUNCH_CHECK(ctx, "attn_prefill_tc_kernel");
  return 0;
}

int launch_attention_tc_ex(caten_b200_ctx *ctx, const AttnArgs &args, float qscale) {
  AttnArgs a = args;
  a.fill_strides();
  if (a.Dp > 128 || a.Ep > 128) return fail(ctx, CATEN_B200_EUNSUPPORTED, "attention_tc: head size above 128");
  const bool wq = a.Dp > 64, we = a.Ep > 64;
  if (wq && we) return launch_at<2, 2>(ctx, a, qscale);
  if (wq) return launch_at<2, 1>(ctx, a, qscale);
  if (we) return launch_at<1, 2>(ctx, a, qscale);
  return launch_at<1, 1>(ctx, a, qscale);
}

int launch_attention_tc(caten_b200_ctx *ctx, const float *qkv, const float *kc, const float *vc, float *out, int64_t B, int64_t s,
                        int64_t n, int64_t H, int64_t T, BfOut bf) {
  AttnArgs a;
  a.qkv = const_cast<float *>(qkv);
  a.ld = 3 * H * 64;
  a.kc = const_cast<float *>(kc);
  a.vc = const_cast<float *>(vc);
  a.cap = T;
  a.out = out; a.bf = bf; a.out_ld = H * 64;
  a.B = (int)B; a.s = (int)s; a.n = (int)n; a.H = a.G = (int)H;
  a.D = a.Dp = a.E = a.Ep = 64;
  return launch_at<1, 1, true>(ctx, a, 0.125f);
}

}  // namespace cb
