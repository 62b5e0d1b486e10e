// Decoders described layer by layer (caten_b200_decoder_desc): the layer loop, caches and states, and
// the step entry points.  The kernels are those of the other models where they exist (linears,
// arg-max, device-resident step loop) plus stream_norm.cu, attn_window.cu / attention_tc.cu, latent.cu, wkv.cu,
// retention.cu and moe.cu.
#include <math.h>
#include <stdlib.h>
#include <string.h>

#include <new>
#include <utility>
#include <vector>

#include "attn_window.cuh"
#include "latent.cuh"
#include "moe.cuh"
#include "retention.cuh"
#include "step_loop.cuh"
#include "stream_norm.cuh"
#include "wkv.cuh"

using namespace cb;

namespace {

int64_t p16(int64_t n) { return (n + 15) / 16 * 16; }
int64_t p64(int64_t n) { return (n + 63) / 64 * 64; }

// A latent layer takes portions of up to this many tokens per sequence in the absorbed form (latent.cu)
constexpr int LATENT_ABSORB = 4;

struct Run {            // one execution of a layer in a step
  int layer = 0;
  bool pass_start = false;   // a pass of the loop starts right before it
  int pass = 0;              // which one
  float *kc = nullptr, *vc = nullptr;        // attention: ring caches [B, G, cap, Dp / Ep]
  int64_t cap = 0;
  float *state = nullptr, *shift = nullptr;  // time mixing: [B, H, Dp, Dp] and [B, wp]; retention: [B, H, Dp, Ep]
  uint8_t *latents = nullptr;                // latent attention: see LatentArgs::cache
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
  // latent attention
  std::vector<caten_b200_weight> uv;   // per layer: the value rows of kv_w
  int64_t abs_rows = 0, kv_rows = 0, part_floats = 0;
  float *cq = nullptr, *q = nullptr;                        // query latent, queries
  float *qn = nullptr, *qcat = nullptr, *olat = nullptr;    // absorbed form: [H][abs_rows][p64(dim)], [abs_rows, H, KC], [H][abs_rows][Kr]
  float *part = nullptr, *ml = nullptr;                     // its key splits
  float *lat = nullptr, *kr = nullptr, *kvx = nullptr;      // expanded form: latents, key parts, keys and values of kv_rows cached rows
  BfOut cq_bf, qn_bf, qcat_bf, olat_bf, lat_bf;
  float *ret_o = nullptr;                                   // retention: raw outputs of heads with values wider than 256
  // mixture of experts
  float *ex_z = nullptr;                                    // router logits
  int *ex_id = nullptr, *ex_off = nullptr, *ex_src = nullptr, *ex_pos = nullptr;
  float *ex_w = nullptr, *ex_ws = nullptr, *ea = nullptr, *ye = nullptr;   // ea: experts' activations; ye: their outputs [pairs, wp]
  BfOut xs_bf, ea_bf;                                       // rows sorted by expert
  float *last = nullptr, *logits = nullptr;
  int *d_rows = nullptr;
  int64_t *ids = nullptr, *h_ids = nullptr, *h_out = nullptr;
  // parallel layers with few rows: the feed-forward runs beside the mixer on a stream of its own
  cudaStream_t side = nullptr;
  cudaEvent_t fork = nullptr, join = nullptr;
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

static bool bf16_is(const caten_b200_weight *w, int64_t rows, int64_t cols) { return shape_is(w, rows, cols) && w->type == CATEN_B200_BF16; }
// columns of a layer's out_w that the mixer fills
static int64_t mixer_cols(const caten_b200_layer_desc &c) { return p64(c.heads * p16(c.mixer == CATEN_B200_MIX_WKV ? c.dim : c.vdim)); }

static int check_layer(caten_b200_ctx *ctx, int l, const caten_b200_layer_desc &c, int64_t wp) {
  const int64_t Dp = p16(c.dim);
  if (c.heads <= 0 || c.dim <= 0 || c.dim > (c.mixer == CATEN_B200_MIX_RETENTION ? 512 : 256)) return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: %d heads of %d (sizes 1..256)", l, c.heads, c.dim);
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
  } else if (c.mixer == CATEN_B200_MIX_LATENT) {
    const int64_t Pp = p16(c.rot_dims), Ep = p16(c.vdim), H = c.heads;
    if (c.vdim <= 0 || c.vdim > 256 || Dp + Pp > 256 || c.rot_dims < 0 || c.rot_dims % 2 || (c.rot_dims && !c.rot_freq) || c.kv_rank <= 0 || c.kv_rank > 1024 || c.q_rank <= 0 || c.q_rank > 8192 || !c.q_norm || !c.kv_norm)
      return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: latent attention with heads of %d + %d / %d, latents of %d and %d", l, c.dim, c.rot_dims, c.vdim, c.q_rank, c.kv_rank);
    if (!shape_is(c.in_w, p64(p64(c.q_rank) + p16(c.kv_rank) + Pp), wp) || !shape_is(c.uq_w, H * (Dp + Pp), p64(c.q_rank)) || !bf16_is(c.uk_w, H * p16(c.kv_rank), p64(c.dim)) ||
        !bf16_is(c.kv_w, H * (Dp + Ep), p64(c.kv_rank)))
      return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: a latent attention weight has the wrong shape or type", l);
    out_cols = p64(H * Ep);
  } else if (c.mixer == CATEN_B200_MIX_RETENTION) {
    if (c.vdim <= 0 || c.vdim > 1024 || c.rot_dims < 0 || c.rot_dims % 2 || c.rot_dims > c.dim || (c.rot_dims && !c.rot_freq) || !c.powers)
      return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: retention with heads of %d x %d", l, c.dim, c.vdim);
    if (!shape_is(c.in_w, p64(2ll * c.heads * (Dp + p16(c.vdim))), wp)) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: in_w has the wrong shape", l);
    out_cols = p64(c.heads * p16(c.vdim));
  } else {
    return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: unknown mixer %d", l, c.mixer);
  }
  if (c.parallel) {
    if (c.mixer == CATEN_B200_MIX_WKV || !c.norm1_w || (c.ff_in && !c.norm2_w)) return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: no parallel form", l);
    if (c.ff_in && !act_is_glu(c.ff_act)) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: unknown activation %d", l, c.ff_act);
    const int64_t E = c.experts;
    if (E > 0) {
      if (E > 1024 || c.top < 1 || c.top > E || !bf16_is(c.router, p64(E), wp) || !c.ff_in || c.ff_in->rows % (128 * E) || !bf16_is(c.ff_in, c.ff_in->rows, wp) ||
          !bf16_is(c.ff_out, E * wp, c.ff_in->rows / E / 2))
        return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: the experts' weights do not fit each other", l);
    } else if (c.ff_in) {
      if (c.ff_in->cols != wp || c.ff_in->rows % 128 || c.ff_out) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: the feed-forward weights do not fit each other", l);
      out_cols += c.ff_in->rows / 2;
    }
    if (!shape_is(c.out_w, wp, out_cols)) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: out_w must be %lldx%lld", l, (long long)wp, (long long)out_cols);
    return 0;
  }
  if (c.experts) return fail(ctx, CATEN_B200_EUNSUPPORTED, "decoder: layer %d: experts need a parallel layer", l);
  if (!shape_is(c.out_w, wp, out_cols)) return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: out_w must be %lldx%lld", l, (long long)wp, (long long)out_cols);
  if (c.ff_in && (c.ff_in->cols != wp || c.ff_in->rows % 128 || !shape_is(c.ff_out, wp, c.ff_in->rows / 2)))
    return fail(ctx, CATEN_B200_EINVAL, "decoder: layer %d: the feed-forward weights do not fit each other", l);
  return 0;
}

static LatentArgs latent_args(const Dec *m, const caten_b200_layer_desc &c) {
  LatentArgs a;
  a.H = c.heads; a.D = c.dim; a.Dp = (int)p16(c.dim); a.P = c.rot_dims; a.Pp = (int)p16(c.rot_dims); a.E = c.vdim; a.Ep = (int)p16(c.vdim);
  a.K = c.kv_rank; a.Kp = (int)p16(c.kv_rank); a.Kr = (int)p64(c.kv_rank); a.Q = c.q_rank; a.Qr = (int)p64(c.q_rank);
  a.freq = c.rot_freq; a.q_norm = c.q_norm; a.kv_norm = c.kv_norm; a.eps = m->desc.eps; a.scale = c.scale;
  a.cache_bf16 = m->desc.precision == CATEN_B200_PREC_BF16;
  a.tiled = a.cache_bf16 && a.KC() <= 576;
  a.cap = (m->desc.max_seq_len + 127) / 128 * 128;
  return a;
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
  if (loops && (dsc->loop_start < 0 || dsc->loop_stop > L || dsc->loop_times < 1 || (!dsc->loop_in && !dsc->loop_step) || (dsc->loop_in && !shape_is(dsc->loop_in, wp, 2 * wp)) ||
                (!dsc->loop_in && !dsc->layers[dsc->loop_start].parallel)))
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
  auto add_run = [&](int l, bool start, int pass = 0) { Run r; r.layer = l; r.pass_start = start; r.pass = pass; m->runs.push_back(r); };
  if (loops) {
    for (int l = 0; l < dsc->loop_start; ++l) add_run(l, false);
    for (int t = 0; t < dsc->loop_times; ++t)
      for (int l = dsc->loop_start; l < dsc->loop_stop; ++l) add_run(l, l == dsc->loop_start, t);
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
  int64_t l_cq = 0, l_q = 0, l_qn = 0, l_cat = 0, l_o = 0, l_c = 0, l_kr = 0, l_kv = 0, l_part = 0, ret_o = 0, experts = 0, top = 0, ex_ff = 0;   // floats per row
  bool any_par = false;
  m->kv_rows = T > max_rows ? T : max_rows;
  m->abs_rows = max_rows < LATENT_ABSORB * B ? max_rows : LATENT_ABSORB * B;
  auto most = [](int64_t *a, int64_t b) { if (b > *a) *a = b; };
  m->uv.resize(L);
  for (const auto &c : m->layers) {
    if (c.in_w->rows > ny) ny = c.in_w->rows;
    if (c.out_w->cols > n_act) n_act = c.out_w->cols;
    if (c.ff_out && c.ff_out->cols > n_act) n_act = c.ff_out->cols;
    if (c.mixer == CATEN_B200_MIX_WKV) {
      m->any_wkv = true;
      if (c.w2->rows > nd) nd = c.w2->rows;
      if (c.low_rank > low) low = c.low_rank;
    }
    if (c.parallel) any_par = true;
    if (c.mixer == CATEN_B200_MIX_LATENT) {
      const int64_t H = c.heads, Dp = p16(c.dim), Pp = p16(c.rot_dims), Kp = p16(c.kv_rank), Kr = p64(c.kv_rank);
      most(&l_cq, p64(c.q_rank)); most(&l_q, H * (Dp + Pp)); most(&l_qn, H * p64(c.dim)); most(&l_cat, H * (Kp + Pp)); most(&l_o, H * Kr);
      most(&l_c, Kr); most(&l_kr, Pp > 0 ? Pp : 16); most(&l_kv, c.kv_w->rows);
      LatentArgs a = latent_args(m, c);
      a.B = (int)B;
      most(&l_part, latent_splits(ctx, a, B, a.cap) * B * H * Kr);
      most(&l_part, 4 * B * H * Kr);
      caten_b200_weight &uv = m->uv[(size_t)(&c - m->layers.data())];
      uv = *c.kv_w;
      uv.rows = H * p16(c.vdim);
      uv.qs = (uint16_t *)uv.qs + H * Dp * uv.cols;
    }
    if (c.mixer == CATEN_B200_MIX_RETENTION && p16(c.vdim) > 256) most(&ret_o, c.heads * p16(c.vdim));
    if (c.experts) { most(&experts, c.experts); most(&top, c.top); most(&ex_ff, c.ff_out->cols); }
  }
  m->planes = m->any_wkv ? 5 : loops || any_par ? 2 : 1;
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
    } else if (c.mixer == CATEN_B200_MIX_LATENT) {
      const LatentArgs a = latent_args(m, c);
      bytes = B * a.seq_elems() * (a.cache_bf16 ? 2 : 4);
      rc = dec_alloc(m, (void **)&r.latents, (size_t)bytes);
    } else if (c.mixer == CATEN_B200_MIX_RETENTION) {
      bytes = B * c.heads * Dp * p16(c.vdim) * 4;
      rc = dec_floats(m, &r.state, bytes / 4);
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
  if (!rc && l_q) {
    const int64_t A = m->abs_rows, small = A < m->hp_rows ? A : m->hp_rows;   // rows of fp32 operands
    rc = dec_floats(m, &m->cq, m->hp_rows * l_cq);
    if (!rc) rc = dec_bf(m, &m->cq_bf, R * l_cq);
    if (!rc) rc = dec_floats(m, &m->q, R * l_q);
    if (!rc) rc = dec_floats(m, &m->qn, A * l_qn);
    if (!rc) rc = dec_bf(m, &m->qn_bf, A * l_qn);
    if (!rc) rc = dec_floats(m, &m->qcat, small * l_cat);
    if (!rc) rc = dec_bf(m, &m->qcat_bf, A * l_cat);
    if (!rc) rc = dec_floats(m, &m->olat, A * l_o);
    if (!rc) rc = dec_bf(m, &m->olat_bf, A * l_o);
    m->part_floats = l_part;
    if (!rc) rc = dec_floats(m, &m->part, l_part);
    if (!rc) rc = dec_floats(m, &m->ml, l_part / 16);
    if (!rc) rc = dec_floats(m, &m->lat, (exact ? m->kv_rows : 4) * l_c);
    if (!rc) rc = dec_bf(m, &m->lat_bf, m->kv_rows * l_c);
    if (!rc) rc = dec_floats(m, &m->kr, m->kv_rows * l_kr);
    if (!rc) rc = dec_floats(m, &m->kvx, m->kv_rows * l_kv);
  }
  if (!rc && ret_o) rc = dec_floats(m, &m->ret_o, R * ret_o);
  if (!rc && experts) {
    const int64_t P = R * top;
    rc = dec_floats(m, &m->ex_z, R * p64(experts));
    if (!rc) rc = dec_alloc(m, (void **)&m->ex_id, (size_t)P * sizeof(int));
    if (!rc) rc = dec_alloc(m, (void **)&m->ex_off, (size_t)(experts + 1) * sizeof(int));
    if (!rc) rc = dec_alloc(m, (void **)&m->ex_src, (size_t)P * sizeof(int));
    if (!rc) rc = dec_alloc(m, (void **)&m->ex_pos, (size_t)P * sizeof(int));
    if (!rc) rc = dec_floats(m, &m->ex_w, P);
    if (!rc) rc = dec_floats(m, &m->ex_ws, P);
    if (!rc) rc = dec_floats(m, &m->ea, m->hp_rows * top * ex_ff);
    if (!rc) rc = dec_bf(m, &m->ea_bf, P * ex_ff);
    if (!rc) rc = dec_bf(m, &m->xs_bf, P * wp);
    if (!rc) rc = dec_floats(m, &m->ye, P * wp);
  }
  if (!rc) rc = dec_floats(m, &m->last, m->cap_rows * wp);
  if (!rc) rc = dec_bf(m, &m->last_bf, m->cap_rows * wp);
  if (!rc) rc = dec_floats(m, &m->logits, m->cap_rows * V);
  if (!rc) rc = dec_alloc(m, (void **)&m->d_rows, (size_t)m->cap_rows * sizeof(int));
  if (!rc) rc = dec_alloc(m, (void **)&m->ids, (size_t)B * T * sizeof(int64_t));
  if (!rc) rc = step_loop_alloc(ctx, &m->loop, B, T);
  if (!rc && cudaMallocHost(&m->h_ids, (size_t)B * T * sizeof(int64_t)) != cudaSuccess) rc = fail(ctx, CATEN_B200_ECUDA, "cudaMallocHost(ids)");
  if (!rc && cudaMallocHost(&m->h_out, (size_t)B * sizeof(int64_t)) != cudaSuccess) rc = fail(ctx, CATEN_B200_ECUDA, "cudaMallocHost(out ids)");
  if (!rc && any_par) {
    const char *e = getenv("CATEN_B200_SIDE_STREAM");   // 0: one kernel after the other
    if (!e || atoi(e) != 0)
      if (cudaStreamCreateWithFlags(&m->side, cudaStreamNonBlocking) != cudaSuccess || cudaEventCreateWithFlags(&m->fork, cudaEventDisableTiming) != cudaSuccess ||
          cudaEventCreateWithFlags(&m->join, cudaEventDisableTiming) != cudaSuccess)
        rc = fail(ctx, CATEN_B200_ECUDA, "decoder_create: side stream");
  }
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
  if (m->side) { cudaStreamSynchronize(m->side); cudaStreamDestroy(m->side); }
  if (m->fork) cudaEventDestroy(m->fork);
  if (m->join) cudaEventDestroy(m->join);
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
  const float *ye = nullptr;   // SN_SUM: outputs of experts
  const int *pos = nullptr;
  int top = 0;
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
      size_t finished = i;
      if (r.pass_start && m_->desc.loop_in) {
        if (int rc = boundary(SN_CONCAT, 0.0f, i)) return rc;
        if (int rc = linear(m_->desc.loop_in, m_->hp, m_->hp_bf, nullptr, m_->y2, none_, defer_ ? &pend_.pin : nullptr)) return rc;
        pend_.in = SN_COPY;
        finished = 0;
      } else if (r.pass_start && m_->capture && i > 0) {   // the stream as the layer before left it
        if (int rc = boundary(SN_NONE, 0.0f, i)) return rc;
        finished = 0;
      }
      if (int rc = layer(r, finished)) return rc;
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
    a.w1 = m_->desc.final_norm;
    a.x_out = nullptr;  // other rows may still be wanted: the pending stage stays
    a.rows = rows;
    a.src_stride = stride;
    a.h = m_->last + at * m_->wp;
    if (prec_ != CATEN_B200_PREC_FP32) a.hb = offset(m_->last_bf, at * m_->wp);
    if (head_rows_small_) a.hb = BfOut();
    ProfScope prof(ctx_, CATEN_B200_K_LAYERNORM);
    return launch_stream_norm(ctx_, pend_.in, a.w1 ? SN_NORM2 : SN_NORM, a, count);
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
    a.ye = pend_.ye; a.pos = pend_.pos; a.top = pend_.top;
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
  int boundary(int out, float pre, size_t finished_runs, const caten_b200_layer_desc *shift_layer = nullptr, const Run *shift_run = nullptr, float *to_fp32 = nullptr,
               const caten_b200_layer_desc *parallel = nullptr, const Run *pass = nullptr) {
    StreamArgs a = stream();
    a.pre = pre;
    if (parallel) { a.w1 = parallel->norm1_w; a.w2 = parallel->ff_in ? parallel->norm2_w : nullptr; }
    if (pass) { a.step = m_->desc.loop_step + (int64_t)pass->pass * m_->wp; a.add_x0 = pass->pass > 0; }
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
    if (c.parallel) return parallel_layer(r, c, finished_runs);
    if (c.mixer != CATEN_B200_MIX_WKV)
      if (int rc = boundary(SN_NORM, c.norm1, finished_runs)) return rc;
    if (int rc = mixer(r, c, finished_runs)) return rc;
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

  int mixer(const Run &r, const caten_b200_layer_desc &c, size_t finished_runs) {
    switch (c.mixer) {
      case CATEN_B200_MIX_ATTENTION: return attention(r, c);
      case CATEN_B200_MIX_LATENT: return latent(r, c);
      case CATEN_B200_MIX_RETENTION: return retention(r, c);
      default: return wkv(r, c, finished_runs);   // (its norm is part of the token shift)
    }
  }

  // Mixer and feed-forward of the same stream, and one linear over both outputs.  With few rows both are chains of short kernels,
  // and run side by side on two streams.
  int parallel_layer(const Run &r, const caten_b200_layer_desc &c, size_t finished_runs) {
    if (int rc = boundary(SN_NORM2, 0.0f, finished_runs, nullptr, nullptr, nullptr, &c, r.pass_start && !m_->desc.loop_in ? &r : nullptr)) return rc;
    Pending next;
    next.in = SN_SUM;
    const bool beside = m_->side && c.ff_in && R_ <= 256 && ctx_->prof_mask == 0;
    if (beside) {
      CB_CUDA(ctx_, cudaEventRecord(m_->fork, ctx_->stream));
      CB_CUDA(ctx_, cudaStreamWaitEvent(m_->side, m_->fork, 0));
      if (int rc = on_side([&] { return feed_forward(c, &next); })) return rc;
      CB_CUDA(ctx_, cudaEventRecord(m_->join, m_->side));
    }
    if (int rc = mixer(r, c, finished_runs)) return rc;
    if (beside) {
      CB_CUDA(ctx_, cudaStreamWaitEvent(ctx_->stream, m_->join, 0));
      full_edge();
    } else if (c.ff_in) {
      if (int rc = feed_forward(c, &next)) return rc;
    }
    if (int rc = linear(c.out_w, m_->act, m_->act_bf, nullptr, m_->y2, none_, defer_ ? &next.pin : nullptr)) return rc;
    pend_ = next;
    return 0;
  }

  size_t c_index(const caten_b200_layer_desc &c) const { return (size_t)(&c - m_->layers.data()); }

  // The next launch waits for everything before it to complete (a programmatic dependent launch has one predecessor only).
  void full_edge() { ctx_->weights_pending = true; }

  // Launches of f go to the side stream, with scratch of their own.
  template <class F>
  int on_side(F f) {
    cudaStream_t main = ctx_->stream;
    std::swap(ctx_->wtmp, ctx_->wtmp_side);
    ctx_->stream = m_->side;
    full_edge();
    const int rc = f();
    ctx_->stream = main;
    std::swap(ctx_->wtmp, ctx_->wtmp_side);
    return rc;
  }

  // Feed-forward of the second norm's rows: dense, its activations beside the mixer's output; experts, their outputs into ye.
  int feed_forward(const caten_b200_layer_desc &c, Pending *next) {
    const float *h2 = m_->hp + plane_ * m_->wp;
    const BfOut h2_bf = offset(m_->hp_bf, plane_ * m_->wp);
    if (c.experts) return experts(c, h2, h2_bf, next);
    LinGroups to;
    to.ldy = c.out_w->cols;
    const int64_t col = mixer_cols(c);
    return linear(c.ff_in, h2, h2_bf, nullptr, m_->act + col, offset(bf(m_->act_bf), col), nullptr, c.ff_act, to);
  }

  int experts(const caten_b200_layer_desc &c, const float *h2, BfOut h2_bf, Pending *next) {
    RouteArgs a;
    if (int rc = linear(c.router, h2, h2_bf, nullptr, m_->ex_z, none_, defer_ ? &a.pin : nullptr)) return rc;
    const bool sorted = R_ > 4;
    const int64_t rows_in = c.ff_in->rows / c.experts, pairs = R_ * c.top;
    a.z = m_->ex_z; a.ld = c.router->rows; a.rows = (int)R_; a.experts = c.experts; a.top = c.top;
    a.expert = m_->ex_id; a.weight = m_->ex_w; a.offsets = m_->ex_off; a.src = m_->ex_src; a.sorted_weight = m_->ex_ws; a.pos = m_->ex_pos;
    {
      ProfScope prof(ctx_, CATEN_B200_K_PREP);
      if (int rc = launch_moe_route(ctx_, a, sorted)) return rc;
      if (fused_)
        if (int rc = launch_moe_gather(ctx_, h2_bf, m_->ex_src, pairs, m_->wp, m_->xs_bf)) return rc;
    }
    next->ye = m_->ye;
    next->top = c.top;
    next->pos = sorted ? m_->ex_pos : nullptr;
    ProfScope prof(ctx_, CATEN_B200_K_EXPERTS);
    if (!sorted) {
      if (int rc = launch_gemv_experts(ctx_, c.ff_in, rows_in, h2, m_->ex_id, m_->ex_w, pairs, c.top, c.ff_act, m_->ea)) return rc;
      return launch_gemv_experts(ctx_, c.ff_out, m_->wp, m_->ea, m_->ex_id, nullptr, pairs, 1, CATEN_B200_ACT_NONE, m_->ye);
    }
    ExpertRows er;
    er.experts = c.experts; er.top = c.top; er.pairs = pairs; er.offsets = m_->ex_off; er.src = m_->ex_src;
    ExpertRows in = er;
    in.weight = m_->ex_ws;
    if (!fused_) {
      if (int rc = launch_gemm_simt_experts(ctx_, c.ff_in, in, h2, m_->ex_src, c.ff_act, m_->ea)) return rc;
      return launch_gemm_simt_experts(ctx_, c.ff_out, er, m_->ea, nullptr, CATEN_B200_ACT_NONE, m_->ye);
    }
    const int nsplit = prec_ == CATEN_B200_PREC_BF16X3 ? 3 : 1;
    if (int rc = launch_gemm_experts(ctx_, c.ff_in, in, m_->xs_bf, c.ff_act, nullptr, m_->ea_bf, nsplit)) return rc;
    return launch_gemm_experts(ctx_, c.ff_out, er, m_->ea_bf, CATEN_B200_ACT_NONE, m_->ye, none_, nsplit);
  }

  int latent(const Run &r, const caten_b200_layer_desc &c) {
    LatentArgs a = latent_args(m_, c);
    PartIn pin;
    if (int rc = linear(c.in_w, m_->hp, m_->hp_bf, nullptr, m_->y, none_, defer_ ? &pin : nullptr)) return rc;
    a.cache = r.latents + p_.b0 * a.seq_elems() * (a.cache_bf16 ? 2 : 4);
    a.B = (int)p_.nb; a.s = (int)p_.s; a.n = (int)p_.n; a.d_n = p_.d_n;
    { ProfScope prof(ctx_, CATEN_B200_K_PREP); if (int rc = launch_latent_prep(ctx_, a, m_->y, pin, c.in_w->rows, m_->cq, bf(m_->cq_bf))) return rc; }
    const bool absorbed = p_.s <= LATENT_ABSORB;
    pin = PartIn();
    if (int rc = linear(c.uq_w, m_->cq, m_->cq_bf, nullptr, m_->q, none_, defer_ && absorbed ? &pin : nullptr)) return rc;
    const int64_t ldq = c.uq_w->rows;
    if (absorbed) {
      LatentAbsorbed x;
      x.qcat = m_->qcat; x.qcat_bf = bf(m_->qcat_bf); x.o = m_->olat; x.plane = m_->abs_rows; x.part = m_->part; x.ml = m_->ml;
      x.splits = latent_splits(ctx_, a, R_, p_.d_n ? a.cap : p_.n + p_.s);
      while (x.splits > 1 && x.splits * R_ * a.H * a.Kr > m_->part_floats) --x.splits;
      // (the queries' kernel starts nothing before the kernels in front of it, the cache's append among them, are complete)
      x.early = true;
      if (latent_fused(a, R_)) {
        { ProfScope prof(ctx_, CATEN_B200_K_PREP); if (int rc = launch_latent_up(ctx_, a, c.uk_w, m_->q, pin, ldq, m_->qcat, bf(m_->qcat_bf))) return rc; }
        x.combine = false;
        { ProfScope prof(ctx_, CATEN_B200_K_ATTN_DECODE); if (int rc = launch_latent_absorbed(ctx_, a, x)) return rc; }
        ProfScope prof(ctx_, CATEN_B200_K_PREP);
        return launch_latent_down(ctx_, a, x, &m_->uv[c_index(c)], m_->act, bf(m_->act_bf), c.out_w->cols);
      }
      { ProfScope prof(ctx_, CATEN_B200_K_PREP);
        if (int rc = launch_latent_q_absorbed(ctx_, a, m_->q, pin, ldq, m_->abs_rows, m_->qn, bf(m_->qn_bf), m_->qcat, bf(m_->qcat_bf))) return rc; }
      LinGroups up;
      up.group_rows = a.Kp; up.xplane = m_->abs_rows; up.ygroup = a.KC(); up.ldy = (int64_t)a.H * a.KC();
      if (int rc = linear(c.uk_w, m_->qn, m_->qn_bf, nullptr, m_->qcat, bf(m_->qcat_bf), nullptr, CATEN_B200_ACT_NONE, up)) return rc;
      x.o_bf = bf(m_->olat_bf);
      { ProfScope prof(ctx_, CATEN_B200_K_ATTN_DECODE); if (int rc = launch_latent_absorbed(ctx_, a, x)) return rc; }
      LinGroups down;
      down.group_rows = a.Ep; down.xplane = m_->abs_rows; down.ygroup = a.Ep; down.ldy = c.out_w->cols;
      return linear(&m_->uv[c_index(c)], m_->olat, m_->olat_bf, nullptr, m_->act, bf(m_->act_bf), nullptr, CATEN_B200_ACT_NONE, down);
    }
    { ProfScope prof(ctx_, CATEN_B200_K_PREP); if (int rc = launch_latent_q_expanded(ctx_, a, m_->q, ldq)) return rc; }
    // keys and values of every cached token, for as many sequences at a time as the buffer takes
    const int64_t t = p_.n + p_.s, per = m_->kv_rows / t < 1 ? 1 : m_->kv_rows / t;
    for (int64_t b = 0; b < p_.nb; b += per) {
      const int64_t nb = p_.nb - b < per ? p_.nb - b : per, rows = nb * t;
      const bool small = prec_ == CATEN_B200_PREC_FP32 || rows <= 4;
      { ProfScope prof(ctx_, CATEN_B200_K_PREP); if (int rc = launch_latent_gather(ctx_, a, (int)b, (int)nb, (int)t, m_->lat, small ? BfOut() : m_->lat_bf, m_->kr)) return rc; }
      if (int rc = model_linear(ctx_, prec_, c.kv_w, m_->lat, small ? BfOut() : m_->lat_bf, nullptr, nullptr, CATEN_B200_ACT_NONE, m_->kvx, none_, rows)) return rc;
      AttnArgs x;
      x.H = x.G = a.H;
      x.D = a.D + a.P; x.Dp = a.Dq(); x.E = a.E; x.Ep = a.Ep;
      x.qkv = m_->q + b * p_.s * ldq; x.ld = ldq;
      x.kc = m_->kvx; x.vc = m_->kvx + (int64_t)a.H * a.Dp;
      x.cap = t;
      x.k_ld = x.v_ld = c.kv_w->rows; x.k_head = a.Dp; x.v_head = a.Ep; x.k_seq = x.v_seq = t * x.k_ld;
      x.kx = a.Pp ? m_->kr : nullptr; x.kx_ld = a.Pp; x.kx_from = a.Dp;
      x.out_ld = c.out_w->cols;
      x.out = m_->act + b * p_.s * x.out_ld;
      x.bf = offset(bf(m_->act_bf), b * p_.s * x.out_ld);
      x.B = (int)nb; x.s = (int)p_.s; x.n = (int)p_.n;
      ProfScope prof(ctx_, CATEN_B200_K_ATTN_PREFILL);
      if (int rc = launch_attn_window_prefill(ctx_, x, prec_ != CATEN_B200_PREC_FP32 && ctx_->attn_tc)) return rc;
    }
    return 0;
  }

  int retention(const Run &r, const caten_b200_layer_desc &c) {
    RetentionArgs a;
    if (int rc = linear(c.in_w, m_->hp, m_->hp_bf, nullptr, m_->y, none_, defer_ && p_.s == 1 ? &a.pin : nullptr)) return rc;
    a.H = c.heads; a.D = c.dim; a.Dp = (int)p16(c.dim); a.E = c.vdim; a.Ep = (int)p16(c.vdim);
    a.y = m_->y; a.ld = c.in_w->rows;
    a.k_off = a.H * a.Dp; a.v_off = 2 * a.k_off; a.g_off = a.v_off + a.H * a.Ep;
    a.freq = c.rot_freq; a.rot_pairs = c.rot_dims / 2; a.kscale = (float)(1.0 / sqrt((double)c.dim)); a.powers = c.powers; a.eps = m_->desc.eps;
    a.state = r.state + p_.b0 * a.H * a.Dp * a.Ep;
    a.out = m_->act; a.bf = bf(m_->act_bf); a.out_ld = c.out_w->cols;
    a.o = m_->ret_o;
    a.B = (int)p_.nb; a.s = (int)p_.s; a.n = (int)p_.n; a.d_n = p_.d_n;
    if (p_.s == 1) {
      ProfScope prof(ctx_, CATEN_B200_K_WKV);
      return launch_retention_decode(ctx_, a);
    }
    { ProfScope prof(ctx_, CATEN_B200_K_PREP); if (int rc = launch_retention_prep(ctx_, a)) return rc; }
    ProfScope prof(ctx_, CATEN_B200_K_WKV);
    return launch_retention_chunks(ctx_, a);
  }

  int attention(const Run &r, const caten_b200_layer_desc &c) {
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
