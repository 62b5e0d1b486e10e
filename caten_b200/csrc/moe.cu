// Mixture of experts: per token the `top` experts with the largest router logits, weighted by sigmoid(logit)
// as it is (not renormalised), and the (token, expert) pairs brought into the order of the experts, so that an
// expert's linear is a dense product over consecutive rows (ExpertRows).  Everything is fp32 and the order is
// fixed by the tokens' order, not by timing.
#include "moe.cuh"

namespace cb {

namespace {

constexpr int MR_THREADS = 1024, MR_WARPS = MR_THREADS / 32, MR_MAX_EXPERTS = 1024, MR_FUSED_ROWS = 256, MR_U = 4;

// One warp, one row: lane holds experts lane, lane + 32, ...
template <int VPL>
__device__ __forceinline__ void choose(const RouteArgs &a, int64_t row, int lane) {
  float z[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const int e = lane + 32 * i;
    z[i] = e >= a.experts ? -INFINITY : a.pin.splits > 0 ? partin_load1(a.pin, row, e) : a.z[row * a.ld + e];
  }
  for (int k = 0; k < a.top; ++k) {
    float best = -INFINITY;
    int at = MR_MAX_EXPERTS;   // (a row whose logits are not numbers still chooses experts that exist, below)
#pragma unroll
    for (int i = 0; i < VPL; ++i)
      if (z[i] > best) { best = z[i]; at = lane + 32 * i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float v = __shfl_xor_sync(0xffffffffu, best, o);
      const int w = __shfl_xor_sync(0xffffffffu, at, o);
      if (v > best || (v == best && w < at)) { best = v; at = w; }
    }
    if (at >= a.experts) at = k;
#pragma unroll
    for (int i = 0; i < VPL; ++i)
      if (at == lane + 32 * i) z[i] = -INFINITY;
    if (lane == 0) {
      a.expert[row * a.top + k] = at;
      a.weight[row * a.top + k] = 1.0f / (1.0f + expf(-best));
    }
  }
}

__device__ __forceinline__ void choose_any(const RouteArgs &a, int64_t row, int lane) {
  if (a.experts <= 64) choose<2>(a, row, lane);
  else if (a.experts <= 256) choose<8>(a, row, lane);
  else choose<32>(a, row, lane);
}

}  // namespace

__global__ void __launch_bounds__(256) moe_choose_kernel(const RouteArgs a) {
  pdl_enter();
  const int64_t row = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (row < a.rows) choose_any(a, row, threadIdx.x & 31);
}

// One CTA.  Each warp counts a contiguous share of the pairs by expert; a prefix over experts and warps gives every warp
// its first place in every expert, and the warps then place their pairs in order.
__global__ void __launch_bounds__(MR_THREADS) moe_sort_kernel(const RouteArgs a, int fused) {
  extern __shared__ int counts[];   // [MR_WARPS][experts]
  __shared__ int warp_total[MR_WARPS];
  pdl_enter();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, E = a.experts;
  const int pairs = a.rows * a.top;
  for (int i = tid; i < MR_WARPS * E; i += MR_THREADS) counts[i] = 0;
  if (fused)
    for (int64_t row = warp; row < a.rows; row += MR_WARPS) choose_any(a, row, lane);
  __syncthreads();
  const int share = (pairs + MR_WARPS * 32 - 1) / (MR_WARPS * 32) * 32;
  const int p0 = min(warp * share, pairs), p1 = min(p0 + share, pairs);
  int *mine = counts + warp * E;
  for (int q = p0; q < p1; q += 32 * MR_U) {
    int e[MR_U];   // requested together
#pragma unroll
    for (int u = 0; u < MR_U; ++u) e[u] = q + 32 * u + lane < p1 ? a.expert[q + 32 * u + lane] : -1 - lane;
#pragma unroll
    for (int u = 0; u < MR_U; ++u) {
      const unsigned same = __match_any_sync(0xffffffffu, e[u]);
      if (e[u] >= 0 && lane == __ffs(same) - 1) mine[e[u]] += __popc(same);
      __syncwarp();
    }
  }
  __syncthreads();
  int total = 0;
  if (tid < E)
    for (int w = 0; w < MR_WARPS; ++w) {
      const int c = counts[w * E + tid];
      counts[w * E + tid] = total;
      total += c;
    }
  int inc = total;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int up = __shfl_up_sync(0xffffffffu, inc, o);
    if (lane >= o) inc += up;
  }
  if (lane == 31) warp_total[warp] = inc;
  __syncthreads();
  int before = inc - total;
  for (int w = 0; w < warp; ++w) before += warp_total[w];
  if (tid < E) {
    a.offsets[tid] = before;
    if (tid == E - 1) a.offsets[E] = pairs;
    for (int w = 0; w < MR_WARPS; ++w) counts[w * E + tid] += before;
  }
  __syncthreads();
  for (int q = p0; q < p1; q += 32 * MR_U) {
    int e[MR_U];
    float w[MR_U];
#pragma unroll
    for (int u = 0; u < MR_U; ++u) {
      const int p = q + 32 * u + lane;
      e[u] = p < p1 ? a.expert[p] : -1 - lane;
      w[u] = p < p1 ? a.weight[p] : 0.0f;
    }
#pragma unroll
    for (int u = 0; u < MR_U; ++u) {
      const int p = q + 32 * u + lane;
      const unsigned same = __match_any_sync(0xffffffffu, e[u]);
      int at = 0;
      if (e[u] >= 0) at = mine[e[u]] + __popc(same & ((1u << lane) - 1u));
      __syncwarp();
      if (e[u] >= 0) {
        a.pos[p] = at;
        a.src[at] = p / a.top;
        a.sorted_weight[at] = w[u];
        if (lane == __ffs(same) - 1) mine[e[u]] += __popc(same);
      }
      __syncwarp();
    }
  }
}

int launch_moe_route(caten_b200_ctx *ctx, const RouteArgs &a, bool sort) {
  if (a.rows <= 0) return 0;
  if (a.experts < 1 || a.experts > MR_MAX_EXPERTS || a.top < 1 || a.top > a.experts || (int64_t)a.rows * a.top > 0x3fffffff)
    return fail(ctx, CATEN_B200_EUNSUPPORTED, "moe: %d of %d experts", a.top, a.experts);
  const bool fused = sort && a.rows <= MR_FUSED_ROWS;
  if (!fused) {
    launch_k(ctx, moe_choose_kernel, dim3((unsigned)((a.rows + 7) / 8)), dim3(256), 0, a);
    CB_LAUNCH_CHECK(ctx, "moe_choose_kernel");
  }
  if (sort) {
    const size_t smem = (size_t)MR_WARPS * a.experts * sizeof(int);
    if (smem > 40 * 1024) CB_CUDA(ctx, cudaFuncSetAttribute(moe_sort_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_k(ctx, moe_sort_kernel, dim3(1), dim3(MR_THREADS), smem, a, fused ? 1 : 0);
    CB_LAUNCH_CHECK(ctx, "moe_sort_kernel");
  }
  return 0;
}

// one warp per sorted row
__global__ void __launch_bounds__(256) moe_gather_kernel(BfOut x, const int *__restrict__ src, int64_t pairs, int c8, BfOut out) {
  pdl_enter();
  const int64_t i = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= pairs) return;
  const int64_t from = (int64_t)src[i] * c8, to = i * c8;
  for (int c = threadIdx.x & 31; c < c8; c += 32) {
    reinterpret_cast<uint4 *>(out.hi)[to + c] = reinterpret_cast<const uint4 *>(x.hi)[from + c];
    if (x.lo) reinterpret_cast<uint4 *>(out.lo)[to + c] = reinterpret_cast<const uint4 *>(x.lo)[from + c];
  }
}

int launch_moe_gather(caten_b200_ctx *ctx, BfOut x, const int *src, int64_t pairs, int64_t cols, BfOut out) {
  if (pairs <= 0) return 0;
  if (cols % 8 || (pairs + 7) / 8 > 0x7fffffff) return fail(ctx, CATEN_B200_EUNSUPPORTED, "moe: rows of %lld", (long long)cols);
  launch_k(ctx, moe_gather_kernel, dim3((unsigned)((pairs + 7) / 8)), dim3(256), 0, x, src, pairs, (int)(cols / 8), out);
  CB_LAUNCH_CHECK(ctx, "moe_gather_kernel");
  return 0;
}

}  // namespace cb
