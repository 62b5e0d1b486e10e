// Device-resident decoding shared by the models: input ids, position and produced ids live on the
// device, and the launch sequence of a single-token step is captured into a CUDA graph and replayed.
#pragma once
#include "common.cuh"

namespace cb {

struct StepLoop {
  int64_t *ids_io = nullptr;    // [B] input ids of the next step
  int64_t *out_ids = nullptr;   // [B] ids the last step produced
  int64_t *hist = nullptr;      // [T, B] row n = ids produced by the step that started at position n
  int *d_pos = nullptr;         // position of the next step
  cudaGraphExec_t graph = nullptr;
  void *graph_xbf = nullptr, *graph_wtmp = nullptr, *graph_side = nullptr;  // scratch pointers baked into the graph
  int64_t launches_per_step = 0;
};

inline int step_loop_alloc(caten_b200_ctx *ctx, StepLoop *l, int64_t B, int64_t T) {
  int rc = caten_b200_malloc(ctx, (size_t)B * sizeof(int64_t), (void **)&l->out_ids);
  if (!rc) rc = caten_b200_malloc(ctx, (size_t)B * sizeof(int64_t), (void **)&l->ids_io);
  if (!rc) rc = caten_b200_malloc(ctx, (size_t)B * T * sizeof(int64_t), (void **)&l->hist);
  if (!rc) rc = caten_b200_malloc(ctx, sizeof(int), (void **)&l->d_pos);
  return rc;
}

inline void step_loop_free(StepLoop *l) {
  if (l->graph) cudaGraphExecDestroy(l->graph);
  for (void *p : {(void *)l->ids_io, (void *)l->out_ids, (void *)l->hist, (void *)l->d_pos})
    if (p) cudaFree(p);
  *l = StepLoop();
}

// Runs `steps` single-token steps from the device-side state (ids_io and d_pos already loaded).  `step(n)` queues one
// step's kernels, which read ids and position from device memory; the host-side n only feeds argument checks.  With
// use_graph its launch sequence is captured the first time and replayed.
template <class Step>
int step_loop_run(caten_b200_ctx *ctx, StepLoop *l, int64_t n, int64_t steps, int64_t T, bool use_graph, Step step) {
  int64_t done = 0;
  if (use_graph && l->graph && (l->graph_xbf != ctx->xbf.ptr || l->graph_wtmp != ctx->wtmp.ptr || l->graph_side != ctx->wtmp_side.ptr)) {
    cudaGraphExecDestroy(l->graph);  // scratch was re-allocated since the capture: its pointers are stale
    l->graph = nullptr;
  }
  if (use_graph && !l->graph) {
    // the first step runs eagerly: it sizes the scratch buffers and sets kernel attributes, which
    // must not happen during capture
    if (int rc = step(n)) return rc;
    done = 1;
    cudaGraph_t g = nullptr;
    CB_CUDA(ctx, cudaStreamBeginCapture(ctx->stream, cudaStreamCaptureModeThreadLocal));
    const int64_t before = ctx->launches;
    const int rc = step(n + 1 < T ? n + 1 : T - 1);
    const cudaError_t e = cudaStreamEndCapture(ctx->stream, &g);
    l->launches_per_step = ctx->launches - before;
    ctx->launches = before;  // captured, not launched
    if (rc) { if (g) cudaGraphDestroy(g); return rc; }
    if (e != cudaSuccess) return cuda_fail(ctx, e, "cudaStreamEndCapture");
    const cudaError_t e2 = cudaGraphInstantiate(&l->graph, g, 0);
    cudaGraphDestroy(g);
    if (e2 != cudaSuccess) { l->graph = nullptr; return cuda_fail(ctx, e2, "cudaGraphInstantiate"); }
    l->graph_xbf = ctx->xbf.ptr;
    l->graph_wtmp = ctx->wtmp.ptr;
    l->graph_side = ctx->wtmp_side.ptr;
  }
  for (; done < steps; ++done) {
    if (use_graph && l->graph) {
      CB_CUDA(ctx, cudaGraphLaunch(l->graph, ctx->stream));
      ctx->launches += l->launches_per_step;
    } else if (int rc = step(n + done)) {
      return rc;
    }
  }
  return 0;
}

}  // namespace cb
