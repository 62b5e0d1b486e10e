// Mixture of experts (moe.cu): routing of tokens to experts, and their rows sorted by expert.
#pragma once
#include "common.cuh"

namespace cb {

struct RouteArgs {
  const float *z = nullptr;     // router logits [rows, ld], or
  PartIn pin;                   // the router linear's split-K partial tiles
  int64_t ld = 0;
  int rows = 0, experts = 0, top = 0;
  int *expert = nullptr;        // [rows * top] chosen experts, largest score first
  float *weight = nullptr;      // [rows * top] their scores
  // the pairs (token, choice) sorted by expert, in the order of the tokens within one
  int *offsets = nullptr;       // [experts + 1]
  int *src = nullptr;           // [rows * top] token of a sorted row
  float *sorted_weight = nullptr;
  int *pos = nullptr;           // [rows * top] sorted row of a pair
};

// Scores sigmoid(z), the `top` largest of a row; with `sort` also the sorted order.
int launch_moe_route(caten_b200_ctx *ctx, const RouteArgs &a, bool sort);
// Sorted rows of x (bf16): out[i] = x[src[i]], cols a multiple of 8.
int launch_moe_gather(caten_b200_ctx *ctx, BfOut x, const int *src, int64_t pairs, int64_t cols, BfOut out);

}  // namespace cb
