// Decoders described layer by layer (caten_b200_decoder_desc): the layer loop, caches and states, and
// the step entry points.  The kernels are those of the other models where they exist (linears,
// arg-max, device-resident step loop) plus stream_norm.cu, attn_window.cu / attention_tc.cu and wkv.cu.
#include <stdlib.h>
#include <string.h>

#include <new>
#include <vector>

#include "attn_window.cuh"
#include "step_loop.cuh"
#include "stream_norm.cuh"
#include "wkv.cuh"

using namespace cb;

namespace {

int64_t p16(int64_t n) { return (n + 15) / 16 * 16; }
int64_t p64(int64_t n) { return (n + 63) / 64 * 64; }

struct Run {            // one execution of a layer in a step
  int layer = 0;
  bool pass_start = false;   // loop_in comes right before it
  float *kc = nullptr, *vc = nullptr;        // attention: ring caches [B, G, cap, Dp / Ep]
  int64_t cap = 0;
  float *state = nullptr, *shift = nullptr;  // time mixing: [B, H, Dp, Dp] and [B, wp]
};

}  // namespace

struct caten_b200_decoder {
  caten_b200_ctx *ctx = nullptr;
  caten_b200_decoder_desc desc;
  std::vector<caten_b200_layer_desc> layers;
  std::vector<Run> runs;
  int64_t wp = 0, max_rows = 0, portion = 0, cap_rows = 0, cache_bytes = 0;
  int64_t planes = 1, act_cols = 0;
  bool any_wkv = false, any_loop = false;
  // activations, [max_rows, ...] each
  float *x = nullptr, *x0 = nullptr, *y = nullptr, *y2 = nullptr, *hrow = nullptr, *d = nullptr, *o = nullptr;
  float *hp = nullptr;    // fp32 operand of the next linear: `planes` planes of hp_rows rows
  float *act = nullptr;   // fp32 operand of out_w / ff_out
  float *tl = nullptr;    // fp32 operand of w2
  int64_t hp_rows = 0;    // fp32 operands feed the GEMV (up to 4 rows) and the exact GEMM
  BfOut hp_bf, act_bf, tl_bf, last_bf;
  float *last = nullptr, *logits = nullptr;
  int *d_rows = nullptr;
  int64_t *ids = nullptr, *h_ids = nullptr, *h_out = nullptr;
  StepLoop loop;
  int64_t pos = 0;        // where the next step continues
  float *capture = nullptr;
  std::vector<void *> owned;
  int64_t launches0 = 0;
};

typedef caten_b200_decoder Dec;

static int dec_alloc(Dec *m, void **p, size_t bytes) {
  const int rc = caten_b200_malloc(m->ctx, bytes, p);
  if (!rc) m->owned.push_back(*p);
  return rc;
}
static int dec_floats(Dec *m, float **p, int64_t n) { return dec_alloc(m, (void **)p, (size_t)n * sizeof(float)); }
static int dec_bf(Dec *m, BfOut *b, int64_t n) {
  if (m->desc.precision == CATEN_B200_PREC_FP32) return 0;
  int rc = dec_alloc(m, (void **)&b->hi, (size_t)n * 2);
  if (!rc && m->desc.precision == CATEN_B200_PREC_BF16X3) rc = dec_alloc(m, (void **)&b->lo, (size_t)n * 2);
  return rc;
}

static bool shape_is(const caten_b200_weight *w, int64_t rows, int64_t cols) { return w && w->rows == rows && w->cols == cols; }

static int check_layer(caten_b200_ctx *ctx, int l, const caten_b200_layer_desc &c, int64_t wp) {
  const int64_t Dp = p16(c.dim);
  if (c.heads <= 0 || c.dim <= 0 || c.dim > 256) return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: %d heads of %d (sizes 1..256)", l, c.heads, c.dim);
  int64_t out_cols = 0;
  if (c.mixer == CATEN_B200_MIX_ATTENTION) {
    if (c.kv_heads <= 0 || c.heads % c.kv_heads || c.vdim <= 0 || c.vdim > 256 || c.window < 0 || c.rot_dims < 0 || c.rot_dims % 2 || c.rot_dims > c.dim || (c.rot_dims && !c.rot_freq))
      return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: bad attention shape", l);
    const int64_t rows = p64(c.heads * Dp + c.kv_heads * (Dp + p16(c.vdim)) + (c.gated ? c.heads : 0));
    if (!shape_is(c.in_w, rows, wp)) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: in_w must be %lldx%lld", l, (long long)rows, (long long)wp);
    out_cols = p64(c.heads * p16(c.vdim));
  } else if (c.mixer == CATEN_B200_MIX_WKV) {
    if (c.group_rows % 128 || c.group_rows < c.heads * Dp || c.low_rank <= 0 || c.low_rank % 64 || c.low_rank > c.group_rows || !c.mu || !c.w0 || !c.u || !c.norm)
      return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: bad time-mixing shape", l);
    if (!shape_is(c.in_w, 4ll * c.group_rows + c.low_rank, wp) || !shape_is(c.w2, p64(c.heads * Dp), c.low_rank) || c.w2->type != CATEN_B200_BF16)
      return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: in_w or w2 has the wrong shape or type", l);
    out_cols = p64(c.heads * Dp);
  } else {
    return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: unknown mixer %d", l, c.mixer);
  }
  if (!shape_is(c.out_w, wp, out_cols)) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: out_w must be %lldx%lld", l, (long long)wp, (long long)out_cols);
  if (c.ff_in && (c.ff_in->cols != wp || c.ff_in->rows % 128 || !shape_is(c.ff_out, wp, c.ff_in->rows / 2)))
    return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: the feed-forward weights do not fit each other", l);
  return 0;
}

extern "C" {

int caten_b200_decoder_create(caten_b200_ctx *ctx, const caten_b200_decoder_desc *dsc, caten_b200_decoder **out) {
  if (!ctx) return fail(nullptr, CATEN_B200_EINVAL, "decoder_create: ctx is NULL");
  cudaSetDevice(ctx->device);
  if (!dsc || !out || !dsc->layers) return fail(ctx, CATEN_B200_EINVAL, "decoder_create: NULL argument");
  *out = nullptr;
  const int64_t L = dsc->n_layers, B = dsc->batch, V = dsc->vocab, T = dsc->max_seq_len, wp = p64(dsc->width);
  if (L <= 0 || dsc->width <= 0 || V <= 0 || T <= 0 || B <= 0) return fail(ctx, CATEN_B200_EINVAL, "decoder_create: non-positive size");
  if (wp > 8192) return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder_create: width %d (at most 8192)", dsc->width);
  if (dsc->precision < CATEN_B200_PREC_FP32 || dsc->precision > CATEN_B200_PREC_BF16X3) return fail(ctx, CATEN_B200_EINVAL, "decoder_create: unknown precision %d", dsc->precision);
  if (!shape_is(dsc->embed, V, wp) || dsc->embed->type != CATEN_B200_BF16 || !shape_is(dsc->head, V, wp))
    return fail(ctx, CATEN_B200_EINVAL, "decoder_create: embed (BF16) and head must be %lldx%lld", (long long)V, (long long)wp);
  const bool loops = dsc->loop_stop > dsc->loop_start;
  if (loops && (dsc->loop_start < 0 || dsc->loop_stop > L || dsc->loop_times < 1 || !shape_is(dsc->loop_in, wp, 2 * wp)))
    return fail(ctx, CATEN_B200_EINVAL, "decoder_create: bad loop");
  for (int l = 0; l < L; ++l)
    if (int rc = check_layer(ctx, l, dsc->layers[l], wp)) return rc;
  Dec *m = new (std::nothrow) Dec();
  if (!m) return fail(ctx, CATEN_B200_ECUDA, "out of host memory");
  m->ctx = ctx;
  m->desc = *dsc;
  m->layers.assign(dsc->layers, dsc->layers + L);
  m->desc.layers = nullptr;
  m->wp = wp;
  m->any_loop = loops;
  auto add_run = [&](int l, bool start) { Run r; r.layer = l; r.pass_start = start; m->runs.push_back(r); };
  if (loops) {
    for (int l = 0; l < dsc->loop_start; ++l) add_run(l, false);
    for (int t = 0; t < dsc->loop_times; ++t)
      for (int l = dsc->loop_start; l < dsc->loop_stop; ++l) add_run(l, l == dsc->loop_start);
    for (int l = dsc->loop_stop; l < L; ++l) add_run(l, false);
  } else {
    for (int l = 0; l < L; ++l) add_run(l, false);
  }
  // rows processed at once, and tokens of one sequence among them (which a windowed layer's ring must hold besides
  // the window): all sequences of the batch together where that leaves useful portions
  int64_t max_rows = dsc->max_rows > 0 ? dsc->max_rows : 8192;
  if (dsc->max_rows <= 0)
    if (const char *e = getenv("CATEN_B200_MAX_ROWS")) { const long v = atol(e); if (v >= 1 && v <= (1 << 20)) max_rows = v; }
  int64_t portion = dsc->max_portion > 0 ? dsc->max_portion : max_rows / B;
  if (dsc->max_portion <= 0) portion = portion < 128 ? 128 : portion > 2048 ? 2048 : portion;
  if (portion > T) portion = T;
  if (portion > max_rows) portion = max_rows;
  if (max_rows < B) max_rows = B;  // a decode step processes the whole batch at once
  if (max_rows > B * portion) max_rows = B * portion;
  m->max_rows = max_rows;
  m->portion = portion;
  const int64_t R = max_rows;
  int64_t ny = 64, nd = 0, n_act = 64, low = 64;
  for (const auto &c : m->layers) {
    if (c.in_w->rows > ny) ny = c.in_w->rows;
    if (c.out_w->cols > n_act) n_act = c.out_w->cols;
    if (c.ff_out && c.ff_out->cols > n_act) n_act = c.ff_out->cols;
    if (c.mixer == CATEN_B200_MIX_WKV) {
      m->any_wkv = true;
      if (c.w2->rows > nd) nd = c.w2->rows;
      if (c.low_rank > low) low = c.low_rank;
    }
  }
  m->planes = m->any_wkv ? 5 : loops ? 2 : 1;
  const bool exact = dsc->precision == CATEN_B200_PREC_FP32;
  m->hp_rows = exact ? R : 4;
  m->cap_rows = B > 64 ? B : 64;
  int rc = 0;
  for (auto &r : m->runs) {
    if (rc) break;
    const auto &c = m->layers[r.layer];
    const int64_t Dp = p16(c.dim);
    int64_t bytes;
    if (c.mixer == CATEN_B200_MIX_ATTENTION) {
      const int64_t Ep = p16(c.vdim);
      // a whole number of 64-key blocks, so that no block of the tensor-core kernel wraps inside
      r.cap = p64(c.window > 0 && c.window - 1 + portion < T ? c.window - 1 + portion : T);
      rc = dec_floats(m, &r.kc, B * c.kv_heads * r.cap * Dp);
      if (!rc) rc = dec_floats(m, &r.vc, B * c.kv_heads * r.cap * Ep);
      bytes = B * c.kv_heads * r.cap * (Dp + Ep) * 4;
    } else {
      rc = dec_floats(m, &r.state, B * c.heads * Dp * Dp);
      if (!rc) rc = dec_floats(m, &r.shift, B * wp);
      bytes = B * (c.heads * Dp * Dp + wp) * 4;
    }
    m->cache_bytes += bytes;
  }
  if (!rc) rc = dec_floats(m, &m->x, R * wp);
  if (!rc && loops) rc = dec_floats(m, &m->x0, R * wp);
  if (!rc) rc = dec_floats(m, &m->y, R * ny);
  if (!rc) rc = dec_floats(m, &m->y2, R * wp);
  if (!rc) rc = dec_floats(m, &m->hp, m->planes * m->hp_rows * wp);
  if (!rc) rc = dec_floats(m, &m->act, m->hp_rows * n_act);
  if (!rc) rc = dec_bf(m, &m->hp_bf, m->planes * R * wp);
  if (!rc) rc = dec_bf(m, &m->act_bf, R * n_act);
  if (!rc && m->any_wkv) {
    rc = dec_floats(m, &m->hrow, R * wp);
    if (!rc) rc = dec_floats(m, &m->d, R * nd);
    if (!rc) rc = dec_floats(m, &m->o, R * nd);
    if (!rc) rc = dec_floats(m, &m->tl, m->hp_rows * low);
    if (!rc) rc = dec_bf(m, &m->tl_bf, R * low);
  }
  if (!rc) rc = dec_floats(m, &m->last, m->cap_rows * wp);
  if (!rc) rc = dec_bf(m, &m->last_bf, m->cap_rows * wp);
  if (!rc) rc = dec_floats(m, &m->logits, m->cap_rows * V);
  if (!rc) rc = dec_alloc(m, (void **)&m->d_rows, (size_t)m->cap_rows * sizeof(int));
  if (!rc) rc = dec_alloc(m, (void **)&m->ids, (size_t)B * T * sizeof(int64_t));
  if (!rc) rc = step_loop_alloc(ctx, &m->loop, B, T);
  if (!rc && cudaMallocHost(&m->h_ids, (size_t)B * T * sizeof(int64_t)) != cudaSuccess) rc = fail(ctx, CATEN_B200_ECUDA, "cudaMallocHost(ids)");
  if (!rc && cudaMallocHost(&m->h_out, (size_t)B * sizeof(int64_t)) != cudaSuccess) rc = fail(ctx, CATEN_B200_ECUDA, "cudaMallocHost(out ids)");
  if (rc) { caten_b200_decoder_destroy(m); return rc; }
  m->launches0 = ctx->launches;
  *out = m;
  return 0;
}

int caten_b200_decoder_destroy(caten_b200_decoder *m) {
  if (!m) return 0;
  cudaSetDevice(m->ctx->device);
  cudaStreamSynchronize(m->ctx->stream);
  step_loop_free(&m->loop);
  for (void *p : m->owned) cudaFree(p);
  if (m->h_ids) cudaFreeHost(m->h_ids);
  if (m->h_out) cudaFreeHost(m->h_out);
  delete m;
  return 0;
}

}  // extern "C"

namespace {

// One portion of a step: sequences [b0, b0 + nb), s tokens each at positions n .. (or *d_n).
struct Portion {
  const int64_t *ids = nullptr;   // token i of sequence b0 + b: ids[b * ids_ld + i]
  int64_t ids_ld = 1, b0 = 0, nb = 0, s = 0, n = 0;
  const int *d_n = nullptr;
};

// What is pending on the residual stream: how the next stream_norm launch forms the row.
struct Pending {
  int in = SN_EMBED;
  PartIn pin;
  float post = 1.0f;
};

class StepRunner {
 public:
  StepRunner(Dec *m, const Portion &p) : m_(m), ctx_(m->ctx), p_(p), R_(p.nb * p.s), prec_(m->desc.precision) {
    fused_ = prec_ != CATEN_B200_PREC_FP32 && R_ > 4;
    defer_ = fused_ && R_ <= 256;
    plane_ = fused_ ? m->max_rows : m->hp_rows;
  }

  // All layer runs; the stream of the last one stays pending.
  int layers() {
    for (size_t i = 0; i < m_->runs.size(); ++i) {
      const Run &r = m_->runs[i];
      if (r.pass_start) {
        if (int rc = boundary(SN_CONCAT, 0.0f, i)) return rc;
        if (int rc = linear(m_->desc.loop_in, m_->hp, m_->hp_bf, nullptr, m_->y2, none_, defer_ ? &pend_.pin : nullptr)) return rc;
        pend_.in = SN_COPY;
      }
      if (int rc = layer(r, r.pass_start ? 0 : i)) return rc;
    }
    if (m_->capture) {
      if (int rc = boundary(SN_NONE, 0.0f, m_->runs.size())) return rc;
      pend_ = Pending();
      pend_.in = SN_KEEP;
    }
    return 0;
  }

  // Final norm of selected stream rows into `last` rows [at, at + count): every `stride`-th row, or the listed ones.
  int final_norm(int64_t at, int64_t count, int64_t stride, const int *rows) {
    StreamArgs a = stream();
    a.pre = m_->desc.final_gain;
    a.x_out = nullptr;  // other rows may still be wanted: the pending stage stays
    a.rows = rows;
    a.src_stride = stride;
    a.h = m_->last + at * m_->wp;
    if (prec_ != CATEN_B200_PREC_FP32) a.hb = offset(m_->last_bf, at * m_->wp);
    if (head_rows_small_) a.hb = BfOut();
    ProfScope prof(ctx_, CATEN_B200_K_LAYERNORM);
    return launch_stream_norm(ctx_, pend_.in, SN_NORM, a, count);
  }
  // Forms the pending stream rows now: the split-K tiles they are made of live in scratch that the next linear reuses.
  int materialise() { return pend_.in == SN_KEEP ? 0 : boundary(SN_NONE, 0.0f, 0); }
  void set_head_rows(int64_t rows) { head_rows_small_ = rows <= 4; }

 private:
  static BfOut offset(BfOut b, int64_t n) { if (b.hi) b.hi += n; if (b.lo) b.lo += n; return b; }
  BfOut bf(BfOut b) const { return fused_ ? b : BfOut(); }

  int linear(const caten_b200_weight *w, const float *x, BfOut xb, const float *bias, float *y, BfOut yb, PartIn *defer, int act = CATEN_B200_ACT_NONE,
             LinGroups grp = LinGroups()) {
    return model_linear(ctx_, prec_, w, x, bf(xb), bias, nullptr, act, y, yb, R_, defer, grp);
  }

  StreamArgs stream() const {
    StreamArgs a;
    a.y = m_->y2; a.pin = pend_.pin; a.post = pend_.post;
    a.x = m_->x; a.x_out = m_->x; a.x0 = m_->x0;
    a.table = (const __nv_bfloat16 *)m_->desc.embed->qs;
    a.ids = p_.ids; a.ids_ld = p_.ids_ld; a.vocab = m_->desc.vocab; a.s = (int)p_.s;
    a.eps = m_->desc.eps; a.invd = 1.0f / (float)m_->desc.width; a.d4 = (int)(m_->wp / 4);
    a.h = m_->hp; a.hb = bf(m_->hp_bf);
    a.plane = plane_;
    a.n = (int)p_.n; a.d_n = p_.d_n;
    return a;
  }

  // Ends the previous sublayer and prepares the next operation's input; afterwards the stream is x.
  int boundary(int out, float pre, size_t finished_runs, const caten_b200_layer_desc *shift_layer = nullptr, const Run *shift_run = nullptr, float *to_fp32 = nullptr) {
    StreamArgs a = stream();
    a.pre = pre;
    if (to_fp32) { a.h = to_fp32; a.hb = BfOut(); }
    if (out == SN_SHIFT) { a.mu = shift_layer->mu; a.shift = shift_run->shift + p_.b0 * m_->wp; }
    {
      ProfScope prof(ctx_, pend_.in == SN_EMBED ? CATEN_B200_K_EMBED : CATEN_B200_K_LAYERNORM);
      if (int rc = launch_stream_norm(ctx_, pend_.in, out, a, R_)) return rc;
    }
    pend_ = Pending();
    pend_.in = SN_KEEP;
    if (m_->capture && finished_runs > 0) {
      float *dst = m_->capture + ((int64_t)(finished_runs - 1) * m_->desc.batch * p_.s + p_.b0 * p_.s) * m_->desc.width;
      CB_CUDA(ctx_, cudaMemcpy2DAsync(dst, (size_t)m_->desc.width * 4, m_->x, (size_t)m_->wp * 4, (size_t)m_->desc.width * 4, (size_t)R_,
                                      cudaMemcpyDeviceToHost, ctx_->stream));
    }
    return 0;
  }

  int layer(const Run &r, size_t finished_runs) {
    const caten_b200_layer_desc &c = m_->layers[r.layer];
    if (int rc = c.mixer == CATEN_B200_MIX_ATTENTION ? attention(r, c, finished_runs) : wkv(r, c, finished_runs)) return rc;
    if (int rc = linear(c.out_w, m_->act, m_->act_bf, nullptr, m_->y2, none_, defer_ ? &pend_.pin : nullptr)) return rc;
    pend_.in = SN_ADD;
    pend_.post = c.norm1b;
    if (!c.ff_in) return 0;
    if (int rc = boundary(SN_NORM, c.norm2, 0)) return rc;
    if (int rc = linear(c.ff_in, m_->hp, m_->hp_bf, nullptr, m_->act, bf(m_->act_bf), nullptr, CATEN_B200_ACT_RELU_GLU)) return rc;
    if (int rc = linear(c.ff_out, m_->act, m_->act_bf, nullptr, m_->y2, none_, defer_ ? &pend_.pin : nullptr)) return rc;
    pend_.in = SN_ADD;
    pend_.post = c.norm2b;
    return 0;
  }

  int attention(const Run &r, const caten_b200_layer_desc &c, size_t finished_runs) {
    if (int rc = boundary(SN_NORM, c.norm1, finished_runs)) return rc;
    AttnArgs a;
    if (int rc = linear(c.in_w, m_->hp, m_->hp_bf, nullptr, m_->y, none_, defer_ && p_.s == 1 ? &a.pin : nullptr)) return rc;
    a.H = c.heads; a.G = c.kv_heads;
    a.D = c.dim; a.Dp = (int)p16(c.dim); a.E = c.vdim; a.Ep = (int)p16(c.vdim);
    a.qkv = m_->y; a.ld = c.in_w->rows;
    a.k_off = (int64_t)a.H * a.Dp; a.v_off = a.k_off + (int64_t)a.G * a.Dp;
    a.gate_off = c.gated ? a.v_off + (int64_t)a.G * a.Ep : -1;
    a.cap = r.cap;
    a.kc = r.kc + p_.b0 * a.G * r.cap * a.Dp; a.vc = r.vc + p_.b0 * a.G * r.cap * a.Ep;
    a.out = m_->act; a.bf = bf(m_->act_bf); a.out_ld = c.out_w->cols;
    a.B = (int)p_.nb; a.s = (int)p_.s; a.n = (int)p_.n; a.d_n = p_.d_n;
    a.window = c.window; a.rot_pairs = c.rot_dims / 2; a.freq = c.rot_freq; a.qk_norm = c.qk_norm; a.eps = m_->desc.eps; a.scale = c.scale;
    if (p_.s == 1) {
      ProfScope prof(ctx_, CATEN_B200_K_ATTN_DECODE);
      return launch_attn_window_decode(ctx_, a);
    }
    { ProfScope prof(ctx_, CATEN_B200_K_PREP); if (int rc = launch_attn_prep(ctx_, a)) return rc; }
    ProfScope prof(ctx_, CATEN_B200_K_ATTN_PREFILL);
    return launch_attn_window_prefill(ctx_, a, prec_ != CATEN_B200_PREC_FP32 && ctx_->attn_tc);
  }

  int wkv(const Run &r, const caten_b200_layer_desc &c, size_t finished_runs) {
    WkvArgs a;
    LinGroups grp;
    grp.group_rows = c.group_rows;
    grp.xplane = plane_;
    a.H = c.heads; a.D = c.dim; a.Dp = (int)p16(c.dim);
    a.y = m_->y; a.ld = c.in_w->rows; a.gr = c.group_rows; a.w1 = c.low_rank;
    a.w2 = (const __nv_bfloat16 *)c.w2->qs; a.w0 = c.w0; a.u = c.u; a.norm = c.norm; a.eps = m_->desc.eps;
    a.state = r.state + p_.b0 * a.H * a.Dp * a.Dp;
    a.out = m_->act; a.bf = bf(m_->act_bf); a.out_ld = c.out_w->cols;
    a.B = (int)p_.nb; a.s = (int)p_.s; a.n = (int)p_.n; a.d_n = p_.d_n;
    if (p_.s == 1) {
      if (int rc = boundary(SN_SHIFT, c.norm1, finished_runs, &c, &r)) return rc;
      if (int rc = linear(c.in_w, m_->hp, m_->hp_bf, nullptr, m_->y, none_, defer_ ? &a.pin : nullptr, CATEN_B200_ACT_NONE, grp)) return rc;
      ProfScope prof(ctx_, CATEN_B200_K_WKV);
      return launch_wkv_decode(ctx_, a);
    }
    float *shift = r.shift + p_.b0 * m_->wp;
    if (int rc = boundary(SN_NORM, c.norm1, finished_runs, nullptr, nullptr, m_->hrow)) return rc;
    {
      ProfScope prof(ctx_, CATEN_B200_K_PREP);
      if (int rc = launch_token_shift(ctx_, m_->hrow, shift, c.mu, p_.nb, p_.s, p_.n, (int)(m_->wp / 4), plane_, m_->hp, bf(m_->hp_bf))) return rc;
    }
    if (int rc = linear(c.in_w, m_->hp, m_->hp_bf, nullptr, m_->y, none_, nullptr, CATEN_B200_ACT_NONE, grp)) return rc;
    {
      ProfScope prof(ctx_, CATEN_B200_K_PREP);
      if (int rc = launch_wkv_lowrank(ctx_, a, m_->tl, bf(m_->tl_bf), m_->hrow, shift, (int)m_->wp)) return rc;
    }
    if (int rc = linear(c.w2, m_->tl, m_->tl_bf, c.w0, m_->d, none_, nullptr)) return rc;
    a.d = m_->d; a.d_ld = c.w2->rows;
    a.o = m_->o; a.o_ld = c.w2->rows;
    ProfScope prof(ctx_, CATEN_B200_K_WKV);
    return launch_wkv_scan(ctx_, a);
  }

  Dec *m_;
  caten_b200_ctx *ctx_;
  Portion p_;
  int64_t R_;
  int prec_;
  bool fused_ = false, defer_ = false, head_rows_small_ = false;
  int64_t plane_ = 0;
  Pending pend_;
  const BfOut none_;
};

int head(Dec *m, int64_t rows) {
  return model_linear(m->ctx, m->desc.precision, m->desc.head, m->last, rows > 4 ? m->last_bf : BfOut(), nullptr, nullptr, CATEN_B200_ACT_NONE, m->logits, BfOut(), rows);
}

// A step of s tokens per sequence.  want / h_logits as in caten_b200_decoder_step; `last`: also leave the last position's
// logits of every sequence in m->logits.
int run_step(Dec *m, const int64_t *d_ids, int64_t s, int64_t n, const int64_t *want, int64_t n_want, float *h_logits, bool last) {
  caten_b200_ctx *ctx = m->ctx;
  const int64_t B = m->desc.batch, V = m->desc.vocab;
  int64_t per = m->max_rows / (s < m->portion ? s : m->portion);
  if (per < 1) per = 1;
  if (per > B) per = B;
  std::vector<int> rows;
  for (int64_t b0 = 0; b0 < B; b0 += per) {
    const int64_t nb = B - b0 < per ? B - b0 : per;
    int64_t w0 = 0;
    for (int64_t t0 = 0; t0 < s; t0 += m->portion) {
      Portion p;
      p.s = s - t0 < m->portion ? s - t0 : m->portion;
      p.ids = d_ids + b0 * s + t0; p.ids_ld = s; p.b0 = b0; p.nb = nb; p.n = n + t0;
      StepRunner run(m, p);
      if (int rc = run.layers()) return rc;
      int64_t w1 = w0;
      while (w1 < n_want && want[w1] < t0 + p.s) ++w1;
      if (w1 > w0)
        if (int rc = run.materialise()) return rc;
      // wanted rows of this portion, at most cap_rows at a time (whole sequences where they fit)
      for (int64_t b = 0; b < nb; ++b)
        for (int64_t w = w0; w < w1;) {
          const int64_t c = w1 - w < m->cap_rows ? w1 - w : m->cap_rows;
          rows.resize((size_t)c);
          for (int64_t i = 0; i < c; ++i) rows[(size_t)i] = (int)(b * p.s + want[w + i] - t0);
          CB_CUDA(ctx, cudaMemcpyAsync(m->d_rows, rows.data(), (size_t)c * sizeof(int), cudaMemcpyHostToDevice, ctx->stream));
          CB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
          run.set_head_rows(c);
          if (int rc = run.final_norm(0, c, 1, m->d_rows)) return rc;
          if (int rc = head(m, c)) return rc;
          CB_CUDA(ctx, cudaMemcpyAsync(h_logits + ((b0 + b) * n_want + w) * V, m->logits, (size_t)(c * V) * sizeof(float), cudaMemcpyDeviceToHost, ctx->stream));
          CB_CUDA(ctx, cudaStreamSynchronize(ctx->stream));
          w += c;
        }
      w0 = w1;
      if (last && t0 + p.s == s) {
        run.set_head_rows(B);
        if (int rc = run.final_norm(b0, nb, p.s, nullptr)) return rc;
      }
    }
  }
  return last ? head(m, B) : 0;
}

// One single-token step whose ids and position are read from device memory.
int decode_step_device_pos(Dec *m, int64_t n_host) {
  Portion p;
  p.ids = m->loop.ids_io; p.ids_ld = 1; p.nb = m->desc.batch; p.s = 1; p.n = n_host; p.d_n = m->loop.d_pos;
  StepRunner run(m, p);
  if (int rc = run.layers()) return rc;
  run.set_head_rows(p.nb);
  if (int rc = run.final_norm(0, p.nb, 1, nullptr)) return rc;
  if (int rc = head(m, p.nb)) return rc;
  {
    ProfScope prof(m->ctx, CATEN_B200_K_ARGMAX);
    if (int rc = launch_argmax(m->ctx, m->logits, p.nb, m->desc.vocab, m->loop.out_ids)) return rc;
  }
  return launch_finish_step(m->ctx, m->loop.out_ids, m->loop.ids_io, m->loop.hist, m->loop.d_pos, p.nb);
}

int decode_run(Dec *m, int64_t n, int64_t steps) {
  const bool use_graph = m->ctx->prof_mask == 0 && !m->capture;
  return step_loop_run(m->ctx, &m->loop, n, steps, m->desc.max_seq_len, use_graph, [m](int64_t pos) { return decode_step_device_pos(m, pos); });
}

int check_step(Dec *m, const char *who, int64_t s, int64_t n) {
  if (s < 1 || n < 0 || n + s > m->desc.max_seq_len)
    return fail(m->ctx, CATEN_B200_EINVAL, "%s: s=%lld n=%lld outside max_seq_len=%d", who, (long long)s, (long long)n, m->desc.max_seq_len);
  // a recurrent state cannot be rewound
  if (n != 0 && n != m->pos)
    return fail(m->ctx, CATEN_B200_EINVAL, "%s: position %lld: the sequences are at %lld (0 starts new ones)", who, (long long)n, (long long)m->pos);
  if (m->capture && s > m->portion) return fail(m->ctx, CATEN_B200_EINVAL, "%s: capture needs steps of at most %lld tokens", who, (long long)m->portion);
  return 0;
}

}  // namespace

extern "C" {

int caten_b200_decoder_step_device(caten_b200_decoder *m, const int64_t *d_ids, int64_t s, int64_t n, int64_t *d_out_ids) {
  if (!m) return fail(nullptr, CATEN_B200_EINVAL, "decoder_step: model is NULL");
  caten_b200_ctx *ctx = m->ctx;
  cudaSetDevice(ctx->device);
  if (!d_ids) return fail(ctx, CATEN_B200_EINVAL, "decoder_step: ids is NULL");
  if (int rc = check_step(m, "decoder_step", s, n)) return rc;
  if (int rc = run_step(m, d_ids, s, n, nullptr, 0, nullptr, d_out_ids != nullptr)) return rc;
  m->pos = n + s;
  if (!d_out_ids) return 0;
  ProfScope prof(ctx, CATEN_B200_K_ARGMAX);
  return launch_argmax(ctx, m->logits, m->desc.batch, m->desc.vocab, d_out_ids);
}

int caten_b200_decoder_step(caten_b200_decoder *m, const int64_t *h_ids, int64_t s, int64_t n, const int64_t *h_want, int64_t n_want,
                            float *h_logits, int64_t *h_out_ids) {
  if (!m) return fail(nullptr, CATEN_B200_EINVAL, "decoder_step: model is NULL");
  caten_b200_ctx *ctx = m->ctx;
  cudaSetDevice(ctx->device);
  const int64_t B = m->desc.batch, V = m->desc.vocab;
  if (!h_ids || n_want < 0 || (n_want > 0 && (!h_want || !h_logits))) return fail(ctx, CATEN_B200_EINVAL, "decoder_step: NULL host buffer");
  if (int rc = check_step(m, "decoder_step", s, n)) return rc;
  for (int64_t i = 0; i < n_want; ++i)
    if (h_want[i] < 0 || h_want[i] >= s || (i > 0 && h_want[i] <= h_want[i - 1])) return fail(ctx, CATEN_B200_EINVAL, "decoder_step: wanted places must be ascending and inside the step");
  memcpy(m->h_ids, h_ids, (size_t)(B * s) * sizeof(int64_t));
  CB_CUDA(ctx, cudaMemcpyAsync(m->ids, m->h_ids, (size_t)(B * s) * sizeof(int64_t), cudaMemcpyHostToDevice, ctx->stream));
  if (s == 1) {
    // the captured graph of a single-token step; it always forms the logits
    if (int rc = launch_begin_steps(ctx, nullptr, m->ids, m->loop.ids_io, m->loop.d_pos, n, B)) return rc;
    if (int rc = decode_run(m, n, 1)) return rc;
    if (n_want) CB_CUDA(ctx, cudaMemcpyAsync(h_logits, m->logits, (size_t)(B * V) * sizeof(float), cudaMemcpyDeviceToHost, ctx->stream));
  } else {
    if (int rc = run_step(m, m->ids, s, n, h_want, n_want, h_logits, h_out_ids != nullptr)) return rc;
    if (h_out_ids) {
      ProfScope prof(ctx, CATEN_B200_K_ARGMAX);
      if (int rc = launch_argmax(ctx, m->logits, B, V, m->loop.out_ids)) return rc;
    }
  }
  m->pos = n + s;
  if (h_out_ids) CB_CUDA(ctx, cudaMemcpyAsync(m->h_out, m->loop.out_ids, (size_t)B * sizeof(int64_t), cudaMemcpyDeviceToHost, ctx->stream));
  if (int rc = caten_b200_sync(ctx)) return rc;
  if (h_out_ids) memcpy(h_out_ids, m->h_out, (size_t)B * sizeof(int64_t));
  return 0;
}

int caten_b200_decoder_decode(caten_b200_decoder *m, const int64_t *d_first_ids, int64_t n, int64_t steps, int64_t *d_out_ids) {
  if (!m) return fail(nullptr, CATEN_B200_EINVAL, "decoder_decode: model is NULL");
  caten_b200_ctx *ctx = m->ctx;
  cudaSetDevice(ctx->device);
  const int64_t B = m->desc.batch;
  if (!d_first_ids || steps < 0) return fail(ctx, CATEN_B200_EINVAL, "decoder_decode: bad argument");
  if (steps == 0) return 0;
  if (int rc = check_step(m, "decoder_decode", steps, n)) return rc;
  if (int rc = launch_begin_steps(ctx, nullptr, d_first_ids, m->loop.ids_io, m->loop.d_pos, n, B)) return rc;
  if (int rc = decode_run(m, n, steps)) return rc;
  m->pos = n + steps;
  if (d_out_ids)
    CB_CUDA(ctx, cudaMemcpyAsync(d_out_ids, m->loop.hist + n * B, (size_t)(steps * B) * sizeof(int64_t), cudaMemcpyDeviceToDevice, ctx->stream));
  return 0;
}

const float *caten_b200_decoder_logits(caten_b200_decoder *m) { return m ? m->logits : nullptr; }
int64_t caten_b200_decoder_runs(caten_b200_decoder *m) { return m ? (int64_t)m->runs.size() : -1; }
int64_t caten_b200_decoder_cache_nbytes(caten_b200_decoder *m) { return m ? m->cache_bytes : -1; }
int caten_b200_decoder_capture(caten_b200_decoder *m, float *h_buf) {
  if (!m) return fail(nullptr, CATEN_B200_EINVAL, "decoder_capture: model is NULL");
  m->capture = h_buf;
  return 0;
}
int64_t caten_b200_decoder_launch_count(caten_b200_decoder *m) { return m ? m->ctx->launches - m->launches0 : 0; }

}  // extern "C"
