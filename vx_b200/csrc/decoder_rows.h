/* decoder_rows.h -- a portion of a prompt through a decoder that gives logits of any
 * position: buffers that grow, one product of many positions, the logits of the
 * positions that are asked for. */
#ifndef VXB_DECODER_ROWS_H
#define VXB_DECODER_ROWS_H

#include "decoder_state.h"

#include <algorithm>

namespace {

constexpr int WANT_GROUP = 256; /* positions whose logits are computed together */

template <typename T> void grow(T *&p, size_t count) {
  cudaFree(p);
  p = dev_alloc<T>(count);
}
/* ... to `count` values when there are fewer */
[[maybe_unused]] void grow_to(float *&p, size_t &has, size_t count) {
  if (count <= has)
    return;
  grow(p, count);
  has = count;
}
void grow_terms(void *&p, size_t values) {
  cudaFree(p);
  p = dev_alloc<uint16_t>(values * 3);
}
[[maybe_unused]] void grow_terms_to(void *&p, size_t &has, size_t values) {
  if (values <= has)
    return;
  grow_terms(p, values);
  has = values;
}

/* One product of t positions: partials[run][t][n]. */
void rows_product(vx_decoder *d, const void *terms, const void *w, int t, int n, int cols,
                  int *runs, const char *what) {
  *runs = 1;
  need(d->c.weights_bf16
           ? vxb::rows_gemm(terms, w, t, n, cols, d->rows_partials, runs, d->stream)
           : vxb::rows_gemm_f32(terms, (const float *)w, t, n, cols, d->rows_partials,
                                d->stream),
       what);
}

/* How much room products need: the runs of one depend on how many positions it has,
   so the sums of few positions can take more than those of many. */
struct SumsRoom {
  const vx_decoder *d;
  size_t most;
  void add(int positions, int n, int cols) {
    const size_t runs =
        d->c.weights_bf16 ? vxb::rows_gemm_splits(positions, n, cols) : 1;
    most = std::max(most, runs * positions * n);
  }
  void add_logits(int n_want, int vocab_rows, int cols) {
    if (n_want >= WANT_GROUP)
      add(WANT_GROUP, vocab_rows, cols);
    if (n_want % WANT_GROUP)
      add(n_want % WANT_GROUP, vocab_rows, cols);
  }
};

/* Room for those sums and for the logits of n_want positions. */
void make_rows_room(vx_decoder *d, RowsPlan &p, const SumsRoom &sums, int n_want,
                    int vocab_rows) {
  const int group = std::min(n_want, WANT_GROUP);
  if (group > p.want_cap) {
    grow(p.want, group);
    grow_terms(p.want_terms, (size_t)group * d->c.dim);
    grow(p.want_logits, (size_t)group * vocab_rows);
    p.want_cap = group;
  }
  if (sums.most > d->rows_partial_floats) {
    grow(d->rows_partials, sums.most);
    d->rows_partial_floats = sums.most;
  }
}

/* The logits of n_want positions of the portion in d->rows_x. norm(n) leaves the terms
   of the positions p.want lists in p.want_terms; scale and cap as rows_sum's. */
template <typename Norm>
void rows_logits(vx_decoder *d, RowsPlan &p, const int32_t *want, int n_want,
                 float *logits, int vocab_rows, float scale, float cap, Norm norm) {
  const vx_decoder_config &c = d->c;
  cudaStream_t s = d->stream;
  for (int at = 0; at < n_want; at += WANT_GROUP) {
    const int n = std::min(WANT_GROUP, n_want - at);
    int runs = 1;
    CUDA_OK(cudaMemcpyAsync(p.want, want + at, n * sizeof(int32_t),
                            cudaMemcpyHostToDevice, s));
    need(norm(n), "RMSNorm");
    rows_product(d, p.want_terms, d->lm_head, n, vocab_rows, c.dim, &runs, "the logits");
    need(vxb::rows_sum(p.want_logits, d->rows_partials, runs, n, vocab_rows, s, scale,
                       cap),
         "the logits");
    CUDA_OK(cudaMemcpy2DAsync(logits + (int64_t)at * c.vocab, c.vocab * sizeof(float),
                              p.want_logits, vocab_rows * sizeof(float),
                              c.vocab * sizeof(float), n, cudaMemcpyDeviceToHost, s));
    const cudaError_t e = cudaStreamSynchronize(s);
    if (e != cudaSuccess)
      stop("a kernel of the decoder faulted: %s", cudaGetErrorString(e));
  }
}

[[maybe_unused]] void free_rows(RowsPlan &p) {
  for (void *m : {(void *)p.want, p.want_terms, (void *)p.want_logits})
    cudaFree(m);
}

} // namespace

#endif /* VXB_DECODER_ROWS_H */
