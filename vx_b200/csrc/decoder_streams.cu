/* decoder_streams.cu -- decoders of layers around a residual of several streams:
 * mixers of two kinds (latent attention over a sliding window, gated linear attention)
 * and feed-forwards, each reading a weighted sum of the streams and mixing them with
 * its output.  The step function, its graph, the positions, the tokens and the entry
 * points are decoder.cu's; this file says what a step and a portion of a prompt launch.
 *
 * A step of latent attention is four kernels: one projection to both latents (streams
 * and norm in front), the queries out of theirs (norm in front), attention with the
 * two products through the latents and the new row of the ring, the output projection
 * with the streams' mixing behind. One of gated linear attention is three: one
 * projection for every matrix that reads h, the recurrence with norm and gate, the
 * output projection. A feed-forward is two. A portion of a prompt has the same
 * products as GEMMs over its positions.
 *
 * The cache holds a ring of latents or a state for every run of a layer.
 */
#include "decoder_rows.h"
#include "decoder_state.h"
#include "kernels.h"
#include "vx_b200.h"

#include <algorithm>
#include <cstdio>

namespace {

using vxb::NormGain;

int fmt_of(const vx_decoder *d) {
  return d->c.weights_bf16 ? vxb::kFmtBf16 : vxb::kFmtF32;
}

/* Whether the projection kernel can apply a norm to `cols` values of every sequence,
   which it holds in shared memory. */
bool norm_fits(const vx_decoder *d, int cols) {
  return (size_t)d->c.batch * ((cols + 255) / 256 * 256) * sizeof(float) <= 96 * 1024;
}

vxb::LatentArgs latent_args(const vx_decoder *d, const StreamLayer &r) {
  const vx_stream_layer &l = r.l;
  vxb::LatentArgs a{};
  a.heads = l.heads;
  a.dim = l.dim;
  a.rot = l.rot_dim;
  a.vdim = l.vdim;
  a.kv_rank = l.kv_rank;
  a.window = r.window;
  a.cache_rows = r.cache_rows;
  a.scale = l.scale;
  a.ring = d->k_cache + r.at;
  a.ring_batch_stride = r.batch_stride;
  a.gain = l.kv_norm;
  a.kv_mean = l.kv_mean;
  a.eps = d->c.eps;
  a.turns = l.turns;
  a.positions = d->positions;
  a.w_ukv = l.w_ukv;
  a.w_uk_t = l.w_uk_t;
  a.fmt = fmt_of(d);
  return a;
}

vxb::GatedLinearArgs gated_args(const vx_decoder *d, const StreamLayer &r) {
  const vx_stream_layer &l = r.l;
  vxb::GatedLinearArgs a{};
  a.heads = l.heads;
  a.dim = l.dim;
  a.vdim = l.vdim;
  a.rank = l.a_rank;
  a.q_scale = l.scale;
  a.inv_tau = l.inv_tau;
  a.eps = d->c.eps;
  a.v_mean = l.v_mean;
  a.a2 = l.a2;
  a.a2_bias = l.a2_bias;
  a.gain = l.o_norm;
  a.state = d->k_cache + r.at;
  a.state_batch_stride = r.batch_stride;
  a.positions = d->positions;
  return a;
}

vxb::StreamMix mix_of(const vx_decoder *d, const vx_stream_mix &m) {
  return vxb::StreamMix{d->streams->streams, m.in, m.mix, m.out};
}

void embed(vx_decoder *d, float *x, const int32_t *tokens, int count, bool per_sequence) {
  vxb::PositionEmbedArgs e{};
  e.x = x;
  e.table = d->embed;
  e.table_bf16 = d->c.weights_bf16 != 0;
  e.tokens = tokens;
  e.count = count;
  e.vocab = d->c.vocab;
  e.width = d->streams->width;
  e.dim = d->c.dim;
  e.scale = d->streams->embed_scale;
  e.positions = d->positions;
  e.per_sequence = per_sequence;
  e.copies = d->streams->streams;
  need(vxb::position_embed(e, d->stream), "embed");
}

/* ---- a step ---------------------------------------------------------------------- */

/* y = f(w norm(sum_s in[s] x_s)) */
void project_streams(vx_decoder *d, int mode, const void *w, int rows, const float *in,
                     const float *gain, float *y, int y_stride, int &launches,
                     const char *what) {
  const StreamPlan &p = *d->streams;
  const vx_decoder_config &c = d->c;
  vxb::StreamProj a{};
  a.mode = mode;
  a.w = w;
  a.fmt = fmt_of(d);
  a.rows = rows;
  a.cols = c.dim;
  a.batch = c.batch;
  a.streams = p.streams;
  a.stream_stride = c.dim;
  a.x_stride = (int64_t)p.streams * c.dim;
  a.x = d->x;
  a.in = in;
  a.norm_w = gain;
  a.norm_n = p.width;
  a.eps = c.eps;
  a.y = y;
  a.y_stride = y_stride;
  a.logit_scale = p.logit_scale;
  a.logit_cap = p.logit_cap;
  if (!norm_fits(d, c.dim)) {
    need(vxb::streams_norm(d->xn, d->x, a.x_stride,
                           vxb::StreamMix{p.streams, in, nullptr, nullptr},
                           NormGain(gain, p.width), c.batch, c.dim, c.eps, d->stream),
         what);
    ++launches;
    a.x = d->xn;
    a.x_stride = c.dim;
    a.streams = 1;
    a.norm_w = nullptr;
  }
  need(vxb::stream_proj(a, d->stream), what);
  ++launches;
}

/* The streams mixed with w x */
void mix_streams(vx_decoder *d, const void *w, int cols, const float *x,
                 const vx_stream_mix &m, int &launches, const char *what) {
  vxb::StreamProj a{};
  a.mode = vxb::kStreamsMix;
  a.w = w;
  a.fmt = fmt_of(d);
  a.rows = d->c.dim;
  a.cols = cols;
  a.batch = d->c.batch;
  a.streams = d->streams->streams;
  a.stream_stride = d->c.dim;
  a.x = x;
  a.x_stride = cols;
  a.mix = m.mix;
  a.out = m.out;
  a.y = d->x;
  a.y_stride = (int64_t)a.streams * d->c.dim;
  need(vxb::stream_proj(a, d->stream), what);
  ++launches;
}

/* The queries out of the normalised query latent, the first q_rank values of p.in. */
void project_queries(vx_decoder *d, const StreamLayer &r, int &launches) {
  const StreamPlan &p = *d->streams;
  const vx_stream_layer &l = r.l;
  vxb::StreamProj a{};
  a.mode = vxb::kStreamsStore;
  a.w = l.w_uq;
  a.fmt = fmt_of(d);
  a.rows = l.heads * (l.dim + l.rot_dim);
  a.cols = l.q_rank;
  a.batch = d->c.batch;
  a.streams = 1;
  a.x = p.in;
  a.x_stride = r.in_rows;
  a.norm_w = l.q_norm;
  a.norm_n = l.q_mean;
  a.eps = d->c.eps;
  a.y = p.q;
  a.y_stride = a.rows;
  if (!norm_fits(d, l.q_rank)) {
    need(vxb::streams_norm(p.q_latent, p.in, r.in_rows,
                           vxb::StreamMix{1, nullptr, nullptr, nullptr},
                           NormGain(l.q_norm, l.q_mean), d->c.batch, l.q_rank, d->c.eps,
                           d->stream),
         "the query latent");
    ++launches;
    a.x = p.q_latent;
    a.x_stride = l.q_rank;
    a.norm_w = nullptr;
  }
  need(vxb::stream_proj(a, d->stream), "the queries");
  ++launches;
}

/* ---- a portion of a prompt -------------------------------------------------------- */

/* The positions whose latents a portion of t positions from `base` on reads. */
int first_seen(const StreamLayer &r, int base) {
  return std::max(0, base - r.window + 1);
}

void make_room(vx_decoder *d, int t, int n_want) {
  StreamPlan &p = *d->streams;
  const vx_decoder_config &c = d->c;
  if (t > d->rows_cap) {
    grow(d->rows_x, (size_t)t * p.streams * c.dim);
    grow_terms(d->rows_terms, (size_t)t * c.dim);
    grow(d->rows_tokens, t);
    d->rows_cap = t;
  }
  SumsRoom sums{d, 0};
  size_t q = 0, alpha = 0, o = 0, kv = 0, terms = 0;
  for (const StreamLayer &r : p.layers) {
    const vx_stream_layer &l = r.l;
    sums.add(t, r.in_rows, c.dim);
    sums.add(t, c.dim, r.out_cols);
    terms = std::max(terms, (size_t)t * r.out_cols);
    if (l.kind == VX_MIXER_LATENT) {
      const size_t n = d->host_pos + t - first_seen(r, d->host_pos);
      const int q_rows = l.heads * (l.dim + l.rot_dim);
      sums.add(t, q_rows, l.q_rank);
      q = std::max(q, (size_t)t * q_rows);
      kv = std::max(kv, n * l.heads * (l.dim + l.vdim));
      terms = std::max({terms, (size_t)t * l.q_rank, n * l.kv_rank});
    } else {
      alpha = std::max(alpha, (size_t)t * l.heads * l.dim);
      o = std::max(o, (size_t)t * l.heads * l.vdim);
    }
    if (l.hidden) {
      sums.add(t, l.hidden, c.dim);
      sums.add(t, c.dim, l.hidden);
      terms = std::max(terms, (size_t)t * l.hidden);
    }
  }
  grow_to(p.rows_q, p.q_floats, q);
  grow_to(p.rows_alpha, p.alpha_floats, alpha);
  grow_to(p.rows_o, p.o_floats, o);
  grow_to(p.rows_kv, p.kv_floats, kv);
  grow_terms_to(p.rows_terms, p.term_values, terms);
  sums.add_logits(n_want, p.vocab_rows, c.dim);
  make_rows_room(d, p.rows, sums, n_want, p.vocab_rows);
}

/* Latent attention of t positions, from the terms of h in d->rows_terms to terms of
   [t][out_cols] in p.rows_terms; only_cache: no further than the ring. */
void latent_rows(vx_decoder *d, const StreamLayer &r, int t, bool only_cache) {
  StreamPlan &p = *d->streams;
  const vx_stream_layer &l = r.l;
  const vxb::LatentArgs a = latent_args(d, r);
  cudaStream_t s = d->stream;
  int runs = 1;
  rows_product(d, d->rows_terms, l.w_in, t, r.in_rows, d->c.dim, &runs, "the latents");
  need(vxb::latent_rows_down(a, d->rows_partials, runs, t, l.q_rank, l.q_norm, l.q_mean,
                             p.rows_terms, s),
       "the latents");
  if (only_cache)
    return;
  const int q_rows = l.heads * (l.dim + l.rot_dim);
  rows_product(d, p.rows_terms, l.w_uq, t, q_rows, l.q_rank, &runs, "the queries");
  need(vxb::latent_rows_q(a, d->rows_partials, runs, t, p.rows_q, s), "the queries");
  /* keys and values of the positions that anyone here sees */
  const int first = first_seen(r, d->host_pos), n = d->host_pos + t - first;
  const int kv_rows = l.heads * (l.dim + l.vdim);
  need(vxb::latent_rows_gather(a, first, n, p.rows_terms, s), "the window's latents");
  need(d->c.weights_bf16
           ? vxb::rows_gemm_of(p.rows_terms, 3 * (int64_t)l.kv_rank, l.w_ukv, l.kv_rank,
                               n, kv_rows, p.rows_kv, &runs, s, 1)
           : vxb::rows_gemm_f32(p.rows_terms, (const float *)l.w_ukv, n, kv_rows,
                                l.kv_rank, p.rows_kv, s),
       "keys and values");
  need(vxb::latent_attention_rows(a, p.rows_q, p.rows_kv, first, t, p.rows_terms,
                                  r.out_cols, s),
       "attention");
}

/* The same for gated linear attention; only_cache: no further than the state. */
void gated_rows(vx_decoder *d, const StreamLayer &r, int t, bool only_cache) {
  StreamPlan &p = *d->streams;
  const vxb::GatedLinearArgs a = gated_args(d, r);
  cudaStream_t s = d->stream;
  int runs = 1;
  rows_product(d, d->rows_terms, r.l.w_in, t, r.in_rows, d->c.dim, &runs,
               "the input projection");
  if (runs > 1)
    need(vxb::rows_sum(d->rows_partials, d->rows_partials, runs, t, r.in_rows, s),
         "the input projection");
  need(vxb::gated_linear_decays(a, d->rows_partials, r.in_rows, t, p.rows_alpha, s),
       "the decays");
  need(vxb::gated_linear_scan(a, d->rows_partials, r.in_rows, p.rows_alpha, t, p.rows_o, s),
       "the recurrence");
  if (!only_cache)
    need(vxb::gated_linear_finish(a, d->rows_partials, r.in_rows, p.rows_o, t,
                                  p.rows_terms, r.out_cols, s),
         "norm and gate");
}

/* A sentence saying why not, or NULL. */
const char *refuse_layer(const vx_stream_layer &l) {
  if (l.kind != VX_MIXER_LATENT && l.kind != VX_MIXER_GATED_LINEAR)
    return "an unknown kind of mixer";
  if (l.heads < 1 || l.dim < 8 || l.dim % 8 || l.vdim < 8 || l.vdim % 8 ||
      (int64_t)l.heads * l.vdim % 64)
    return "head sizes must be multiples of 8 and heads * vdim of 64";
  if (l.hidden < 0 || l.hidden % 64)
    return "the feed-forward's size must be a multiple of 64";
  if (!l.norm1 || !l.w_in || !l.w_o || !l.hc1.in || !l.hc1.mix || !l.hc1.out ||
      (l.hidden && (!l.norm2 || !l.w_up || !l.w_down || !l.hc2.in || !l.hc2.mix ||
                    !l.hc2.out)))
    return "a null pointer";
  if (l.kind == VX_MIXER_LATENT) {
    if (l.rot_dim < 0 || l.rot_dim % 8 || l.q_rank < 64 || l.q_rank % 64 ||
        l.kv_rank < 64 || l.kv_rank % 64 || l.dim + l.rot_dim > 512 || l.vdim > 512 ||
        l.kv_rank + l.rot_dim > 1024 || l.q_rank + l.kv_rank > 51200)
      return "latent attention takes latents in multiples of 64, a rotated part in "
             "multiples of 8, keys and values of at most 512 values and a row of the "
             "cache of at most 1024";
    if (l.q_mean < 1 || l.q_mean > l.q_rank || l.kv_mean < 1 || l.kv_mean > l.kv_rank ||
        l.window < 1)
      return "a latent and a window have at least one value";
    if (!l.q_norm || !l.kv_norm || !l.w_uq || !l.w_ukv || !l.w_uk_t ||
        (l.rot_dim && !l.turns))
      return "a null pointer of latent attention";
    return nullptr;
  }
  if (l.dim > 512 || l.vdim > 16384 || l.a_rank < 8 || l.a_rank % 8 || l.a_rank > 512 ||
      l.v_mean < 1 || l.v_mean > l.vdim)
    return "gated linear attention takes keys and a rank of at most 512 in multiples of 8";
  if (!l.a2 || !l.a2_bias || !l.o_norm)
    return "a null pointer of gated linear attention";
  return nullptr;
}

const char *refuse(const vx_stream_config &c) {
  static thread_local char msg[256];
  if (!c.layers || !c.embed || !c.classifier || !c.final_norm)
    return "a null pointer in the configuration";
  if (c.width < 1 || c.dim < c.width || c.dim % 64 != 0 || c.dim > 51200 ||
      c.n_layers < 1 || c.vocab < 1 || c.vocab_rows < c.vocab || c.vocab_rows % 8 != 0 ||
      c.max_seq < 1 || c.prefill_rows < 0)
    return "dim must be width filled up to a multiple of 64 (51200 at most), vocab_rows "
           "vocab filled up to a multiple of 8, and there must be layers and positions";
  if (c.streams < 1 || c.streams > vxb::kMaxStreams)
    return "a residual has 1 to 32 streams";
  if (c.batch != 1 && c.batch != 2 && c.batch != 4 && c.batch != 8 && c.batch != 16)
    return "batch must be 1, 2, 4, 8 or 16";
  for (int i = 0; i < c.n_layers; ++i)
    if (const char *why = refuse_layer(c.layers[i])) {
      snprintf(msg, sizeof msg, "layer %d: %s", i, why);
      return msg;
    }
  return nullptr;
}

} // namespace

void decoder_record_stream_step(vx_decoder *d) {
  StreamPlan &p = *d->streams;
  const int B = d->c.batch;
  cudaStream_t s = d->stream;
  int launches = 1;
  embed(d, d->x, d->tokens, B, true);
  for (const StreamLayer &r : p.layers) {
    const vx_stream_layer &l = r.l;
    project_streams(d, vxb::kStreamsStore, l.w_in, r.in_rows, l.hc1.in, l.norm1, p.in,
                    r.in_rows, launches, "the input projection");
    if (l.kind == VX_MIXER_LATENT) {
      project_queries(d, r, launches);
      need(vxb::latent_attention_decode(latent_args(d, r), p.q,
                                        l.heads * (l.dim + l.rot_dim), p.in + l.q_rank,
                                        r.in_rows, B, p.mixed, r.out_cols, s),
           "attention");
    } else {
      need(vxb::gated_linear_decode(gated_args(d, r), p.in, r.in_rows, B, p.mixed,
                                    r.out_cols, s),
           "the recurrence");
    }
    ++launches;
    mix_streams(d, l.w_o, r.out_cols, p.mixed, l.hc1, launches, "the output projection");
    if (!l.hidden)
      continue;
    project_streams(d, vxb::kStreamsGelu, l.w_up, l.hidden, l.hc2.in, l.norm2, p.hidden,
                    l.hidden, launches, "the up projection");
    mix_streams(d, l.w_down, l.hidden, p.hidden, l.hc2, launches, "the down projection");
  }
  project_streams(d, vxb::kStreamsLogits, d->lm_head, p.vocab_rows, nullptr, p.final_norm,
                  d->logits, p.vocab_rows, launches, "the logits");
  decoder_record_tail(d, launches);
}

void decoder_stream_rows(vx_decoder *d, const int32_t *tokens, int t, const int32_t *want,
                         int n_want, float *logits) {
  StreamPlan &p = *d->streams;
  const vx_decoder_config &c = d->c;
  cudaStream_t s = d->stream;
  make_room(d, t, n_want);
  CUDA_OK(cudaMemcpyAsync(d->rows_tokens, tokens, (size_t)t * sizeof(int32_t),
                          cudaMemcpyHostToDevice, s));
  embed(d, d->rows_x, d->rows_tokens, t, false);
  const vx_stream_layer &l0 = p.layers[0].l;
  need(vxb::rows_streams_norm(d->rows_terms, d->rows_x, mix_of(d, l0.hc1),
                              NormGain(l0.norm1, p.width), t, c.dim, c.eps, s),
       "RMSNorm");
  int runs = 1;
  /* The product in d->rows_partials goes into the streams; the terms of the next
     sublayer's norm follow. */
  auto mix = [&](const vx_stream_mix &m, const float *next_gain,
                 const vx_stream_mix *next) {
    need(vxb::rows_streams_mix(next ? d->rows_terms : nullptr, d->rows_x, d->rows_partials,
                               runs, t, mix_of(d, m), next ? next->in : nullptr,
                               NormGain(next_gain, p.width), c.dim, c.eps, s),
         "the mixing of the streams");
  };
  for (int i = 0; i < c.n_layers; ++i) {
    const StreamLayer &r = p.layers[i];
    const vx_stream_layer &l = r.l;
    const vx_stream_layer *after = i + 1 < c.n_layers ? &p.layers[i + 1].l : nullptr;
    /* no logits: nothing past the last ring or state is read by anyone later */
    const bool only_cache = !after && n_want == 0;
    if (l.kind == VX_MIXER_LATENT)
      latent_rows(d, r, t, only_cache);
    else
      gated_rows(d, r, t, only_cache);
    if (only_cache)
      break;
    rows_product(d, p.rows_terms, l.w_o, t, c.dim, r.out_cols, &runs,
                 "the output projection");
    if (l.hidden) {
      mix(l.hc1, l.norm2, &l.hc2);
      rows_product(d, d->rows_terms, l.w_up, t, l.hidden, c.dim, &runs,
                   "the up projection");
      need(vxb::rows_gelu_finish(p.rows_terms, d->rows_partials, runs, t, l.hidden, s),
           "gelu");
      rows_product(d, p.rows_terms, l.w_down, t, c.dim, l.hidden, &runs,
                   "the down projection");
    }
    mix(l.hidden ? l.hc2 : l.hc1, after ? after->norm1 : nullptr,
        after ? &after->hc1 : nullptr);
  }
  rows_logits(d, p.rows, want, n_want, logits, p.vocab_rows, p.logit_scale, p.logit_cap,
              [&](int n) {
                return vxb::rows_streams_norm(
                    p.rows.want_terms, d->rows_x,
                    vxb::StreamMix{p.streams, nullptr, nullptr, nullptr},
                    NormGain(p.final_norm, p.width), n, c.dim, c.eps, s, p.rows.want);
              });
  decoder_advance(d, t);
}

void decoder_free_streams(vx_decoder *d) {
  if (!d->streams)
    return;
  StreamPlan &p = *d->streams;
  for (void *m : {(void *)p.in, (void *)p.q, (void *)p.mixed, (void *)p.hidden,
                  (void *)p.q_latent, (void *)p.rows_q, (void *)p.rows_alpha,
                  (void *)p.rows_o, (void *)p.rows_kv, p.rows_terms})
    cudaFree(m);
  free_rows(p.rows);
  delete d->streams;
}

extern "C" {

vx_decoder *vx_decoder_create_streams(const vx_stream_config *config) {
  const char *why = config ? refuse(*config) : "a null argument";
  if (why) {
    vxb::set_last_error(why);
    return nullptr;
  }
  const vx_stream_config &sc = *config;
  vx_decoder *d = new vx_decoder();
  StreamPlan *p = d->streams = new StreamPlan();
  vx_decoder_config &c = d->c;
  c.dim = sc.dim;
  c.n_layers = sc.n_layers;
  c.vocab = sc.vocab;
  c.max_seq = sc.max_seq;
  c.eps = sc.eps;
  c.weights_bf16 = sc.weights_bf16 ? 1 : 0;
  c.batch = sc.batch;
  c.tp_ranks = 1;
  d->ranks = 1;
  d->vocab_local = sc.vocab;
  d->logit_stride = sc.vocab_rows;
  d->embed = sc.embed;
  d->lm_head = sc.classifier;
  p->width = sc.width;
  p->vocab_rows = sc.vocab_rows;
  p->streams = sc.streams;
  p->rows.prefill_rows = std::min(sc.prefill_rows ? sc.prefill_rows : 2048, sc.max_seq);
  p->embed_scale = sc.embed_scale;
  p->logit_scale = sc.logit_scale;
  p->logit_cap = sc.logit_cap;
  p->final_norm = sc.final_norm;
  for (int i = 0; i < sc.n_layers; ++i) {
    StreamLayer r{};
    r.l = sc.layers[i];
    const vx_stream_layer &l = r.l;
    r.out_cols = l.heads * l.vdim;
    if (l.kind == VX_MIXER_LATENT) {
      r.in_rows = l.q_rank + l.kv_rank + l.rot_dim;
      r.window = std::min(l.window, sc.max_seq);
      r.cache_rows = std::min(sc.max_seq, r.window - 1 + p->rows.prefill_rows);
      r.batch_stride = (int64_t)r.cache_rows * (l.kv_rank + l.rot_dim);
      p->q_max = std::max(p->q_max, l.heads * (l.dim + l.rot_dim));
      p->q_rank_max = std::max(p->q_rank_max, l.q_rank);
    } else {
      r.in_rows = 2 * l.heads * (l.dim + l.vdim) + l.a_rank;
      r.cache_rows = 1;
      r.batch_stride = (int64_t)l.heads * l.dim * l.vdim;
    }
    r.at = p->cache_floats;
    p->cache_floats += r.batch_stride * sc.batch;
    p->in_max = std::max(p->in_max, r.in_rows);
    p->mixed_max = std::max(p->mixed_max, r.out_cols);
    p->hidden_max = std::max(p->hidden_max, l.hidden);
    p->layers.push_back(r);
  }
  const size_t B = sc.batch;
  d->x = dev_alloc<float>(B * p->streams * c.dim);
  d->xn = dev_alloc<float>(B * c.dim);
  p->in = dev_alloc<float>(B * p->in_max);
  p->q = dev_alloc<float>(B * p->q_max + 4);
  p->mixed = dev_alloc<float>(B * p->mixed_max);
  p->hidden = dev_alloc<float>(B * p->hidden_max + 4);
  p->q_latent = dev_alloc<float>(B * p->q_rank_max + 4);
  d->logits = dev_alloc<float>(B * p->vocab_rows);
  d->k_cache = dev_alloc<float>(p->cache_floats);
  d->tokens = dev_alloc<int32_t>(32);
  d->positions = dev_alloc<int32_t>(32);
  CUDA_OK(cudaStreamCreateWithFlags(&d->stream, cudaStreamNonBlocking));
  CUDA_OK(cudaDeviceSynchronize());
  return d;
}

} /* extern "C" */
