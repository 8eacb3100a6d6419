/* decoder_state.h -- what the source files of the decoder share: its state and
 * how it stops.  decoder.cu holds the Llama-2 decoders and the entry points,
 * decoder_parallel.cu the decoders of parallel blocks, decoder_streams.cu those of
 * layers around a residual of several streams. */
#ifndef VXB_DECODER_STATE_H
#define VXB_DECODER_STATE_H

#include "kernels.h"
#include "vx_b200.h"

#include <cstdarg>
#include <cstdio>
#include <cstdlib>
#include <map>
#include <vector>

namespace vxb {
void set_last_error(const char *why);
} // namespace vxb

struct vx_decoder;

namespace {

[[noreturn, maybe_unused]] void stop(const char *fmt, ...) {
  va_list ap;
  va_start(ap, fmt);
  fputs("[Vx CUDA] FATAL: ", stderr);
  vfprintf(stderr, fmt, ap);
  fputc('\n', stderr);
  va_end(ap);
  abort();
}
#define CUDA_OK(expr)                                                          \
  do {                                                                         \
    const cudaError_t e_ = (expr);                                             \
    if (e_ != cudaSuccess)                                                     \
      stop("%s failed: %s", #expr, cudaGetErrorString(e_));                    \
  } while (0)

[[maybe_unused]] void need(const char *why, const char *what) {
  if (why)
    stop("vx_decoder: %s: %s", what, why);
}

/* Zeros. The decoder's stream does not wait for the one that the memset is queued on,
   so it has to be over before anyone uses the memory. */
template <typename T> T *dev_alloc(size_t count) {
  void *p = nullptr;
  if (cudaMalloc(&p, count * sizeof(T)) != cudaSuccess)
    stop("vx_decoder: out of device memory for %zu bytes", count * sizeof(T));
  CUDA_OK(cudaMemsetAsync(p, 0, count * sizeof(T), cudaStreamLegacy));
  CUDA_OK(cudaStreamSynchronize(cudaStreamLegacy));
  return (T *)p;
}

} // namespace

struct PickSlot {
  float value;
  int32_t index, call, call_again;
};
struct PickPeers {
  PickSlot *slots[vxb::kMaxTpRanks];
};

/* What decoders that give logits of any position keep for the positions of a prompt
   (decoder_rows.h). */
struct RowsPlan {
  int prefill_rows; /* positions that go through the layers together at most */
  /* of the positions whose logits are asked for: want_cap of them */
  int32_t *want;
  void *want_terms;
  float *want_logits;
  int want_cap;
};

/* One parallel block: where its matrices are cut and where its keys are. */
struct ParallelLayer {
  int q_heads, kv_heads, head_dim;
  int window, cache_rows;
  float scale;
  int in_rows, k_row, gate_row, up_row; /* the input matrix: q | k | gate | up */
  int out_cols;                         /* the output matrix: attention | up */
  const void *w_in, *w_out;
  const float *norm;
  int64_t cache_at;           /* floats from k_cache to this layer's ring */
  int64_t cache_batch_stride; /* floats from a sequence's ring to the next one's */
};
struct ParallelPlan {
  std::vector<ParallelLayer> layers;
  RowsPlan rows;
  int width, vocab_rows, out_cols_max, q_max;
  float embed_scale;
  const float *embed_norm, *final_norm;
  const double *turns;
  int64_t cache_floats;
  float *gate, *mixed; /* of a step: [batch][q_max], [batch][out_cols] */
  /* of a portion of a prompt: rows_cap positions */
  float *rows_gate;
  void *rows_mixed_terms;
};

/* One run of a layer around a residual of several streams: its weights (a layer that
   runs several times has them several times here) and where this run's ring or state
   lies. */
struct StreamLayer {
  vx_stream_layer l;
  int in_rows, out_cols, window, cache_rows;
  int64_t at;           /* floats from k_cache to this run's ring or state */
  int64_t batch_stride; /* floats from a sequence's ring or state to the next one's */
};
struct StreamPlan {
  std::vector<StreamLayer> layers;
  RowsPlan rows;
  int width, vocab_rows, streams;
  float embed_scale, logit_scale, logit_cap;
  const float *final_norm;
  int64_t cache_floats;
  int in_max, q_max, q_rank_max, mixed_max, hidden_max;
  /* of a step: [batch][in_max], [batch][q_max], [batch][mixed_max],
     [batch][hidden_max], [batch][q_rank_max] */
  float *in, *q, *mixed, *hidden, *q_latent;
  /* of a portion of a prompt */
  float *rows_q, *rows_alpha, *rows_o, *rows_kv;
  void *rows_terms;
  size_t q_floats, alpha_floats, o_floats, kv_floats, term_values;
};

struct vx_decoder {
  vx_decoder_config c;
  int ranks, q_local, kv_local, hidden_local, vocab_local, vocab_offset;
  std::vector<const void *> attn_norm, wq, wk, wv, bqkv, wo, ffn_norm, w_gate,
      w_up, w_down, s_qkv, s_o, s_gate_up, s_down;
  int wfmt; /* 0, or kFmtFp8 / kFmtQ4 for the layers' projections */
  const void *embed, *final_norm, *lm_head;
  const float *cos_t, *sin_t;
  /* device state */
  float *x, *xn, *q, *att, *h, *tmp, *logits, *k_cache, *v_cache, *scratch;
  bool fused_norm; /* the activations of all sequences fit the projections' shared memory */
  int32_t *tokens, *positions, *counters, *local_best;
  float2 *pair, *pairs_all;
  /* tp_reduce == 1: partial sums exchanged through peer memory */
  bool push;
  vxb::TpPush tp;
  void *recv;                       /* this rank's slots + flags (IPC-shared) */
  void *peer_recv[vxb::kMaxTpRanks];
  int32_t *tp_epoch, *tp_done, *pick_epoch, *pick_gave_up;
  PickPeers pick;
  /* 8 or 16 sequences: the projections run on the tensor cores */
  bool mma;
  void *mma_xs;
  float *mma_scratch;
  /* a one-sequence decoder reading a whole prompt at once (prefill.cu):
     activations of rows_cap positions, their bf16 terms, the GEMMs' partial
     sums */
  float *rows_x, *rows_q, *rows_partials;
  void *rows_terms;
  /* quantised weights: the matrix in hand as two (Q4_0) or three (fp8) bf16
     terms, and the activations' terms spread over six or seven segments */
  void *rows_w_terms, *rows_terms6;
  size_t rows_partial_floats;
  int32_t *rows_tokens;
  int rows_cap;
  int64_t cache_layer_stride, cache_batch_stride;
  int split;
  int host_pos;
  cudaStream_t stream;
  std::map<int, cudaGraphExec_t> graphs;
  int kernels_per_step;
  void *owned_weights; /* a checkpoint this decoder loaded itself, or NULL */
  /* one sequence, bf16 weights, heads of 128 values: all layers and the logits
     of a step are one cooperative launch (step_kernel.cu) */
  bool one_kernel;
  vxb::StepOp *step_ops;
  int n_step_ops;
  float *step_scratch;
  int32_t *arrivals;
  unsigned long long *step_trace; /* VXB_STEP_TRACE=1: clock readings of the last step */
  /* values from one sequence's logits to the next one's */
  int logit_stride;
  /* a decoder of parallel blocks (decoder_parallel.cu), or NULL */
  ParallelPlan *par;
  /* a decoder of layers around several streams (decoder_streams.cu), or NULL */
  StreamPlan *streams;
};

/* decoder.cu: the tokens of a step (agreed between the ranks of a vocabulary-split
   model) and the move of the positions; the move after a portion of a prompt. */
void decoder_record_tail(vx_decoder *d, int launches);
void decoder_advance(vx_decoder *d, int count);
/* decoder_parallel.cu */
void decoder_record_parallel_step(vx_decoder *d);
void decoder_free_parallel(vx_decoder *d);
/* The next t positions of the sequence through all layers, and the logits [n_want,
   vocab] of the places `want` lists. */
void decoder_parallel_rows(vx_decoder *d, const int32_t *tokens, int t,
                           const int32_t *want, int n_want, float *logits);
/* decoder_streams.cu: the same for its decoders */
void decoder_record_stream_step(vx_decoder *d);
void decoder_free_streams(vx_decoder *d);
void decoder_stream_rows(vx_decoder *d, const int32_t *tokens, int t, const int32_t *want,
                         int n_want, float *logits);

#endif /* VXB_DECODER_STATE_H */
