/* decoder_parallel.cu -- decoders of parallel blocks: x += mixer(h) + ff(h) with h
 * one RMSNorm of x, attention over a sliding window of keys that are the values
 * too, and an output gate.  The step function, its graph, the positions, the
 * tokens and the entry points are decoder.cu's; this file says what a step and a
 * portion of a prompt launch.
 *
 * A step is three kernels a layer, since both sublayers read one h and are added
 * together: one projection for every matrix that reads h (norm in front; q, the
 * ring's new row, the gate's sigmoid and the squared relu behind), attention with
 * the gate behind, one projection of the two outputs side by side, added to x.  A
 * portion of a prompt is the same two products as GEMMs over its positions.
 *
 * The cache is a ring per layer and sequence: a window never needs more than its
 * own size and the portion being read, whatever the length of the sequence.
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

vxb::WindowAttnArgs attention_args(const vx_decoder *d, const ParallelLayer &l,
                                   const float *q, const float *gate) {
  vxb::WindowAttnArgs a{};
  a.q = q;
  a.q_stride = d->par->q_max;
  a.cache = d->k_cache + l.cache_at;
  a.cache_batch_stride = l.cache_batch_stride;
  a.cache_rows = l.cache_rows;
  a.window = l.window;
  a.scale = l.scale;
  a.gate = gate;
  a.gate_stride = d->par->q_max;
  a.q_heads = l.q_heads;
  a.kv_heads = l.kv_heads;
  a.head_dim = l.head_dim;
  a.positions = d->positions;
  return a;
}

vxb::PositionEmbedArgs embed_args(const vx_decoder *d, float *x, const int32_t *tokens,
                                  int count, bool per_sequence) {
  vxb::PositionEmbedArgs e{};
  e.x = x;
  e.table = d->embed;
  e.table_bf16 = d->c.weights_bf16 != 0;
  e.tokens = tokens;
  e.count = count;
  e.vocab = d->c.vocab;
  e.width = d->par->width;
  e.dim = d->c.dim;
  e.scale = d->par->embed_scale;
  e.turns = d->par->turns;
  e.gain = d->par->embed_norm;
  e.eps = d->c.eps;
  e.positions = d->positions;
  e.per_sequence = per_sequence;
  return e;
}

/* The input of a projection behind an RMSNorm: x itself when the projection can
   apply the norm, else x normalised into d->xn by a kernel of its own. */
const float *normed(vx_decoder *d, const float *gain, int &launches) {
  if (d->fused_norm)
    return d->x;
  need(vxb::rms_norm(d->xn, d->x, gain, false, d->par->width, d->c.eps, d->c.batch,
                     d->c.dim, d->stream),
       "RMSNorm");
  ++launches;
  return d->xn;
}

/* Room for t positions and for the logits of n_want of them. */
void make_room(vx_decoder *d, int t, int n_want) {
  ParallelPlan &p = *d->par;
  const vx_decoder_config &c = d->c;
  if (t > d->rows_cap) {
    grow(d->rows_x, (size_t)t * c.dim);
    grow(d->rows_q, (size_t)t * p.q_max);
    grow(p.rows_gate, (size_t)t * p.q_max);
    grow_terms(d->rows_terms, (size_t)t * c.dim);
    grow_terms(p.rows_mixed_terms, (size_t)t * p.out_cols_max);
    grow(d->rows_tokens, t);
    d->rows_cap = t;
  }
  SumsRoom sums{d, 0};
  for (const ParallelLayer &l : p.layers) {
    sums.add(t, l.in_rows, c.dim);
    sums.add(t, l.gate_row - l.k_row, c.dim);
    sums.add(t, c.dim, l.out_cols);
  }
  sums.add_logits(n_want, p.vocab_rows, c.dim);
  make_rows_room(d, p.rows, sums, n_want, p.vocab_rows);
}

/* A sentence saying why not, or NULL. */
const char *refuse(const vx_parallel_config &c) {
  static thread_local char msg[256];
  if (!c.layers || !c.embed || !c.classifier || !c.embed_norm || !c.final_norm ||
      !c.turns)
    return "a null pointer in the configuration";
  if (c.width < 1 || c.dim < c.width || c.dim % 64 != 0 || c.n_layers < 1 ||
      c.vocab < 1 || c.vocab_rows < c.vocab || c.vocab_rows % 8 != 0 || c.max_seq < 1 ||
      c.prefill_rows < 0)
    return "dim must be width filled up to a multiple of 64, vocab_rows vocab filled "
           "up to a multiple of 8, and there must be layers and positions";
  if (c.batch != 1 && c.batch != 2 && c.batch != 4 && c.batch != 8 && c.batch != 16)
    return "batch must be 1, 2, 4, 8 or 16";
  for (int i = 0; i < c.n_layers; ++i) {
    const vx_parallel_layer &l = c.layers[i];
    if (l.q_heads < 1 || l.kv_heads < 1 || l.q_heads % l.kv_heads != 0 ||
        l.head_dim < 8 || l.head_dim % 8 != 0 || l.head_dim > 512 || l.hidden < 0 ||
        l.hidden % 8 != 0 || (l.q_heads * l.head_dim + l.hidden) % 64 != 0 ||
        l.window < 1 || !l.norm || !l.w_in || !l.w_out) {
      snprintf(msg, sizeof msg,
               "layer %d: head_dim must be a multiple of 8 of at most 512, q_heads a "
               "multiple of kv_heads, q_heads * head_dim + hidden a multiple of 64, "
               "the window at least 1, and no pointer null",
               i);
      return msg;
    }
  }
  return nullptr;
}

} // namespace

void decoder_record_parallel_step(vx_decoder *d) {
  ParallelPlan &p = *d->par;
  const vx_decoder_config &c = d->c;
  const int B = c.batch;
  cudaStream_t s = d->stream;
  need(vxb::position_embed(embed_args(d, d->x, d->tokens, B, true), s), "embed");
  int launches = 1;
  for (const ParallelLayer &l : p.layers) {
    const int att_cols = l.q_heads * l.head_dim;
    vxb::FanArgs f{};
    f.w = l.w_in;
    f.fmt = fmt_of(d);
    f.rows = l.in_rows;
    f.cols = c.dim;
    f.x = normed(d, l.norm, launches);
    f.x_stride = c.dim;
    f.batch = B;
    f.norm_w = d->fused_norm ? l.norm : nullptr;
    f.norm_n = p.width;
    f.eps = c.eps;
    f.q_out = d->q;
    f.q_stride = p.q_max;
    f.k_cache = d->k_cache + l.cache_at;
    f.cache_batch_stride = l.cache_batch_stride;
    f.positions = d->positions;
    f.out.k_row = l.k_row;
    f.out.gate_row = l.gate_row;
    f.out.up_row = l.up_row;
    f.out.cache_rows = l.cache_rows;
    f.out.gate = p.gate;
    f.out.gate_stride = p.q_max;
    f.out.up = p.mixed + att_cols;
    f.out.up_stride = l.out_cols;
    need(vxb::fan_proj(f, s), "the input projection");
    need(vxb::window_attention_decode(attention_args(d, l, d->q, p.gate), B, p.mixed,
                                      l.out_cols, s),
         "attention");
    vxb::MatvecArgs o{};
    o.w = l.w_out;
    o.wfmt = fmt_of(d);
    o.rows = c.dim;
    o.cols = l.out_cols;
    o.x = p.mixed;
    o.x_stride = l.out_cols;
    o.batch = B;
    o.y = d->x;
    o.y_stride = c.dim;
    o.mode = 1;
    need(vxb::matvec(o, s), "the output projection");
    launches += 3;
  }
  vxb::MatvecArgs h{};
  h.w = d->lm_head;
  h.wfmt = fmt_of(d);
  h.rows = p.vocab_rows;
  h.cols = c.dim;
  h.x = normed(d, p.final_norm, launches);
  h.x_stride = c.dim;
  h.batch = B;
  h.norm_w = d->fused_norm ? p.final_norm : nullptr;
  h.norm_n = p.width;
  h.eps = c.eps;
  h.y = d->logits;
  h.y_stride = p.vocab_rows;
  h.mode = 0;
  need(vxb::matvec(h, s), "the logits");
  decoder_record_tail(d, launches + 1);
}

void decoder_parallel_rows(vx_decoder *d, const int32_t *tokens, int t,
                           const int32_t *want, int n_want, float *logits) {
  ParallelPlan &p = *d->par;
  const vx_decoder_config &c = d->c;
  cudaStream_t s = d->stream;
  const int w_bytes = c.weights_bf16 ? 2 : 4;
  make_room(d, t, n_want);
  CUDA_OK(cudaMemcpyAsync(d->rows_tokens, tokens, (size_t)t * sizeof(int32_t),
                          cudaMemcpyHostToDevice, s));
  need(vxb::position_embed(embed_args(d, d->rows_x, d->rows_tokens, t, false), s),
       "embed");
  const bool fuse_norm = c.dim <= 8192;
  need(vxb::rows_norm_terms(d->rows_terms, d->rows_x, NormGain(p.layers[0].norm, p.width),
                            t, c.dim, c.eps, s),
       "RMSNorm");
  int runs = 1;
  for (int i = 0; i < c.n_layers; ++i) {
    /* rows_terms hold the terms of this layer's h */
    const ParallelLayer &l = p.layers[i];
    const bool last = i == c.n_layers - 1;
    vxb::FanOut fan{};
    fan.k_row = l.k_row;
    fan.gate_row = l.gate_row;
    fan.up_row = l.up_row;
    fan.cache_rows = l.cache_rows;
    fan.gate = p.rows_gate;
    fan.gate_stride = p.q_max;
    float *ring = d->k_cache + l.cache_at;
    const int att_cols = l.q_heads * l.head_dim;
    if (last && n_want == 0) {
      /* nothing but the keys of the last layer is read by anyone later */
      const int k_rows = l.gate_row - l.k_row;
      fan.k_row = 0;
      fan.gate_row = fan.up_row = k_rows;
      rows_product(d, d->rows_terms,
                   (const char *)l.w_in + (int64_t)l.k_row * c.dim * w_bytes, t, k_rows,
                   c.dim, &runs, "the keys");
      need(vxb::rows_fan_finish(d->rows_partials, runs, t, k_rows, fan, d->positions,
                                d->rows_q, p.q_max, ring, p.rows_mixed_terms, l.out_cols,
                                att_cols, s),
           "the ring's new rows");
      break;
    }
    rows_product(d, d->rows_terms, l.w_in, t, l.in_rows, c.dim, &runs,
                 "the input projection");
    need(vxb::rows_fan_finish(d->rows_partials, runs, t, l.in_rows, fan, d->positions,
                              d->rows_q, p.q_max, ring, p.rows_mixed_terms, l.out_cols,
                              att_cols, s),
         "the parts of the input projection");
    need(vxb::window_attention_rows(attention_args(d, l, d->rows_q, p.rows_gate), t,
                                    p.rows_mixed_terms, l.out_cols, s),
         "attention");
    rows_product(d, p.rows_mixed_terms, l.w_out, t, c.dim, l.out_cols, &runs,
                 "the output projection");
    if (!last && fuse_norm) {
      need(vxb::rows_residual_norm(d->rows_terms, d->rows_x, d->rows_partials, runs, t,
                                   NormGain(p.layers[i + 1].norm, p.width), c.dim, c.eps,
                                   s),
           "the residual add and RMSNorm");
      continue;
    }
    need(vxb::rows_residual_finish(d->rows_x, d->rows_partials, runs, t, c.dim, s),
         "the residual add");
    if (!last)
      need(vxb::rows_norm_terms(d->rows_terms, d->rows_x,
                                NormGain(p.layers[i + 1].norm, p.width), t, c.dim, c.eps,
                                s),
           "RMSNorm");
  }
  rows_logits(d, p.rows, want, n_want, logits, p.vocab_rows, 1.0f, 0.0f, [&](int n) {
    return vxb::rows_norm_terms(p.rows.want_terms, d->rows_x,
                                NormGain(p.final_norm, p.width), n, c.dim, c.eps, s,
                                p.rows.want);
  });
  decoder_advance(d, t);
}

void decoder_free_parallel(vx_decoder *d) {
  if (!d->par)
    return;
  ParallelPlan &p = *d->par;
  for (void *m : {(void *)p.gate, (void *)p.mixed, (void *)p.rows_gate,
                  p.rows_mixed_terms})
    cudaFree(m);
  free_rows(p.rows);
  delete d->par;
}

extern "C" {

vx_decoder *vx_decoder_create_parallel(const vx_parallel_config *config) {
  const char *why = config ? refuse(*config) : "a null argument";
  if (why) {
    vxb::set_last_error(why);
    return nullptr;
  }
  const vx_parallel_config &pc = *config;
  vx_decoder *d = new vx_decoder();
  ParallelPlan *p = d->par = new ParallelPlan();
  vx_decoder_config &c = d->c;
  c.dim = pc.dim;
  c.n_layers = pc.n_layers;
  c.vocab = pc.vocab;
  c.max_seq = pc.max_seq;
  c.eps = pc.eps;
  c.weights_bf16 = pc.weights_bf16 ? 1 : 0;
  c.batch = pc.batch;
  c.tp_ranks = 1;
  d->ranks = 1;
  d->vocab_local = pc.vocab;
  d->logit_stride = pc.vocab_rows;
  d->embed = pc.embed;
  d->lm_head = pc.classifier;
  p->width = pc.width;
  p->vocab_rows = pc.vocab_rows;
  p->rows.prefill_rows = std::min(pc.prefill_rows ? pc.prefill_rows : 2048, pc.max_seq);
  p->embed_scale = pc.embed_scale;
  p->embed_norm = pc.embed_norm;
  p->final_norm = pc.final_norm;
  p->turns = pc.turns;
  for (int i = 0; i < pc.n_layers; ++i) {
    const vx_parallel_layer &from = pc.layers[i];
    ParallelLayer l{};
    l.q_heads = from.q_heads;
    l.kv_heads = from.kv_heads;
    l.head_dim = from.head_dim;
    l.window = std::min(from.window, pc.max_seq);
    l.cache_rows = std::min(pc.max_seq, l.window - 1 + p->rows.prefill_rows);
    l.scale = from.score_scale;
    const int att = l.q_heads * l.head_dim;
    l.k_row = att;
    l.gate_row = l.k_row + l.kv_heads * l.head_dim;
    l.up_row = l.gate_row + att;
    l.in_rows = l.up_row + from.hidden;
    l.out_cols = att + from.hidden;
    l.w_in = from.w_in;
    l.w_out = from.w_out;
    l.norm = from.norm;
    l.cache_batch_stride = (int64_t)l.cache_rows * l.kv_heads * l.head_dim;
    l.cache_at = p->cache_floats;
    p->cache_floats += l.cache_batch_stride * pc.batch;
    p->out_cols_max = std::max(p->out_cols_max, l.out_cols);
    p->q_max = std::max(p->q_max, att);
    p->layers.push_back(l);
  }
  const size_t B = pc.batch;
  /* the projection kernel can apply a norm to rows it holds in shared memory */
  d->fused_norm = B * ((c.dim + 255) / 256 * 256) * sizeof(float) <= 96 * 1024;
  d->x = dev_alloc<float>(B * c.dim);
  d->xn = dev_alloc<float>(B * c.dim);
  d->q = dev_alloc<float>(B * p->q_max);
  p->gate = dev_alloc<float>(B * p->q_max);
  p->mixed = dev_alloc<float>(B * p->out_cols_max);
  d->logits = dev_alloc<float>(B * p->vocab_rows);
  d->k_cache = dev_alloc<float>(p->cache_floats);
  d->tokens = dev_alloc<int32_t>(32);
  d->positions = dev_alloc<int32_t>(32);
  CUDA_OK(cudaStreamCreateWithFlags(&d->stream, cudaStreamNonBlocking));
  CUDA_OK(cudaDeviceSynchronize());
  return d;
}

} /* extern "C" */
