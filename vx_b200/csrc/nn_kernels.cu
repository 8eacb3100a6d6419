/* nn_kernels.cu -- the decode operators of one transformer token: bandwidth
 * bound, so every kernel is organised around streaming its weights (or its KV
 * cache) once, with 16-byte loads that a warp issues over consecutive
 * addresses, several in flight per lane, and warp-shuffle reductions.
 *
 * The arithmetic is the one the reference states in stdlib/std/nn.vx (bf16
 * weights, f32 activations, f32 sums; half-split RoPE with tables) and in
 * tests/backend/pass/llama2.vx:218-429 (f32 weights, interleaved RoPE computed
 * from pos, eps added after the mean); each kernel names the functions it
 * covers.  Where the reference launches one kernel per operator, these fuse
 * what follows a projection into it: RMSNorm in front of the q/k/v and the
 * gate/up projections, bias + RoPE + KV-cache store behind q/k/v, SwiGLU
 * behind gate/up, the residual add behind the output and down projections, and
 * the merge of the attention parts into the attention kernel itself (inside a
 * thread-block cluster, through distributed shared memory).
 *
 * No float atomics and a fixed order in every reduction: the same inputs give
 * the same bits on every run.
 */
#include "kernels.h"
#include "launch.cuh"
#include "launch_util.h"
#include "nn_device.cuh"
#include "ptx.cuh"

#include <cooperative_groups.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>

#include <algorithm>
#include <cstdio>
#include <cstdlib>
#include <mutex>

namespace vxb {
namespace {

/* Sum over the block; every thread gets the result. `red` holds 32 floats. */
__device__ float block_sum(float v, float *red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int nwarps = (blockDim.x + 31) >> 5;
  v = warp_sum(v);
  __syncthreads();
  if (lane == 0)
    red[warp] = v;
  __syncthreads();
  float t = 0.0f;
  for (int w = 0; w < nwarps; ++w) /* fixed order */
    t += red[w];
  return t;
}

/* fmt: a kFmt* code of kernels.h. */
const char *launch_rowdot(int epi, RowDotParams &p, int fmt, cudaStream_t stream) {
  const int per_word = fmt == kFmtF32 ? 4 : fmt == kFmtBf16 ? 8 : fmt == kFmtFp8 ? 16 : 32;
  if (p.cols % 8 != 0 || p.cols % per_word != 0)
    return "the number of columns must be a multiple of 8 (f32, bf16), of 128 "
           "(fp8) or of 32 (Q4_0)";
  if (((uintptr_t)p.w0 | (uintptr_t)p.w1 | (uintptr_t)p.w2 | (uintptr_t)p.x) & 15)
    return "weights and activations must be 16-byte aligned";
  if (p.x_stride % 4 != 0 && p.batch > 1)
    return "the stride between sequences must be a multiple of 4 values";
  if (fmt == kFmtFp8 || fmt == kFmtQ4) {
    if (fmt == kFmtFp8 && p.cols % 128 != 0)
      return "an fp8 matrix has a multiple of 128 columns";
    if (!p.s0 || (p.w1 && !p.s1) || (p.w2 && !p.s2))
      return "a quantised matrix needs its scales";
    if (p.batch != 1)
      return "the quantised projections take one sequence";
    if (epi == EPI_PUSH)
      return "the quantised projections are not sharded";
    return rowdot_quant(epi, p, fmt, stream);
  }
  if (reads_streams(epi) || epi == EPI_MIX)
    return fmt == kFmtBf16 ? rowdot_streams_bf16(epi, p, stream)
                           : rowdot_streams_f32(epi, p, stream);
  return fmt == kFmtBf16 ? rowdot_bf16(epi, p, stream) : rowdot_f32(epi, p, stream);
}

/* ------------------------------------------------------------- rms_norm
 * nn_rms_norm (nn.vx:212-239); one block per sequence. */
__global__ void __launch_bounds__(1024)
rms_norm_kernel(float *y, const float *x, const void *w, int wbf16, int n,
                float eps, int64_t stride) {
  __shared__ float red[32];
  chain_release();
  chain_wait();

  const float *xr = x + blockIdx.x * stride;
  float *yr = y + blockIdx.x * stride;
  float ss = 0.0f;
  for (int i = threadIdx.x; i < n; i += blockDim.x)
    ss = fmaf(xr[i], xr[i], ss);
  ss = block_sum(ss, red);
  const float inv = 1.0f / sqrtf(ss / (float)n + eps);
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float wn = wbf16 ? bf16_at(w, i) : ((const float *)w)[i];
    yr[i] = xr[i] * inv * wn;
  }
}

/* ------------------------------------------------------- rope_and_store
 * nn_rope_and_store (nn.vx:245-280), unfused. */
__global__ void rope_store_kernel(float *q_out, float *k_cache, float *v_cache,
                                  const float *q, const float *k,
                                  const float *v, const float *cos_t,
                                  const float *sin_t, int cs_cols, int pos,
                                  int q_heads, int kv_heads, int hd) {
  chain_release();
  chain_wait();
  const int h = blockIdx.x, i = threadIdx.x;
  if (i >= hd)
    return;
  const int half = hd / 2;
  const int j = i < half ? i : i - half;
  const int partner = i < half ? i + half : i - half;
  const float sign = i < half ? -1.0f : 1.0f;
  const float c = cos_t[(int64_t)pos * cs_cols + j];
  const float s = sin_t[(int64_t)pos * cs_cols + j];
  if (h < q_heads) {
    const float *qh = q + h * hd;
    q_out[h * hd + i] =
        __fadd_rn(__fmul_rn(qh[i], c), __fmul_rn(__fmul_rn(sign, qh[partner]), s));
  } else {
    const int g = h - q_heads;
    const float *kh = k + g * hd;
    const int64_t at = ((int64_t)pos * kv_heads + g) * hd + i;
    k_cache[at] =
        __fadd_rn(__fmul_rn(kh[i], c), __fmul_rn(__fmul_rn(sign, kh[partner]), s));
    v_cache[at] = v[g * hd + i];
  }
}

/* The same arithmetic with the parts of a head merged inside a cluster of
   ATT_CLUSTER blocks (distributed shared memory) instead of through global
   memory, a fence, an atomic and a last block: three round trips shorter.
   This is what kAttnAuto runs unless the process chose otherwise. */
constexpr int ATT_CLUSTER = 8;
template <int GH, int ATT_WARPS>
__global__ void __launch_bounds__(ATT_WARPS * 32)
attention_cluster_kernel(const AttnArgs a) {
  __shared__ AttnShared<GH, ATT_WARPS> sh;
  chain_release();
  attention_unit<GH, true, ATT_CLUSTER, ATT_WARPS>(
      a, blockIdx.x, blockIdx.y, blockIdx.z, threadIdx.x >> 5, threadIdx.x & 31,
      sh, 0);
}

template <int GH>
__global__ void __launch_bounds__(4 * 32)
attention_decode_kernel(const AttnArgs a) {
  __shared__ AttnShared<GH, 4> sh;
  chain_release();
  attention_unit<GH, true, 0, 4>(a, blockIdx.x, blockIdx.y, blockIdx.z,
                                 threadIdx.x >> 5, threadIdx.x & 31, sh, 0);
}

/* ----------------------------------------------------------------- top_k
 * nn_top_k (nn.vx:904-938): the router of a mixture-of-experts layer. The
 * reference sorts 64-bit keys -- the value's bits in an order that keeps the
 * order of the values, then 255 - index, so that of equal values the lower
 * index comes first -- and takes the first k; here each of the n <= 256
 * values counts the keys above its own, which is its place. Then the softmax
 * over the k values, summed in the order of their places. One block. */
__global__ void __launch_bounds__(256)
top_k_kernel(int32_t *ids, float *weights, const float *logits, int n, int k,
             int64_t ids_pitch, int64_t weights_pitch, int64_t logits_pitch) {
  __shared__ long long keys[256];
  __shared__ int order[256];
  chain_release();
  chain_wait();
  /* nn_top_k_rows (nn.vx:2897-2929): a block per position, the same arithmetic */
  ids += blockIdx.x * ids_pitch;
  weights += blockIdx.x * weights_pitch;
  logits += blockIdx.x * logits_pitch;
  const int i = threadIdx.x;
  if (i < n) {
    const int bits = __float_as_int(logits[i]);
    const int ordered = bits < 0 ? bits ^ 0x7fffffff : bits;
    keys[i] = (long long)ordered * 4294967296ll + (255 - i);
  }
  __syncthreads();
  if (i < n) {
    const long long mine = keys[i];
    int place = 0;
    for (int j = 0; j < n; ++j)
      place += keys[j] > mine;
    order[place] = i; /* keys are distinct: every place is taken once */
  }
  __syncthreads();
  if (i < k) {
    const float top = logits[order[0]];
    float total = 0.0f;
    for (int t = 0; t < k; ++t)
      total = total + expf(logits[order[t]] - top);
    const int id = order[i];
    ids[i] = id;
    weights[i] = expf(logits[id] - top) / total;
  }
}

/* ---------------------------------------------------------------- argmax
 * nn_argmax (nn.vx:870-897) and sample_argmax (llama2.vx:460-474): the lowest
 * index of the largest value. One block per sequence. */
__global__ void __launch_bounds__(1024)
argmax_kernel(int32_t *out, const float *logits, int n, int64_t stride) {
  chain_release();
  chain_wait();
  __shared__ float best_v[32];
  __shared__ int best_i[32];
  const float *row = logits + blockIdx.x * stride;
  float bv = -INFINITY;
  int bi = 0x7fffffff;
  for (int i = threadIdx.x; i < n; i += blockDim.x) {
    const float v = row[i];
    if (v > bv || (v == bv && i < bi) || bi == 0x7fffffff) {
      bv = v;
      bi = i;
    }
  }
  auto better = [](float v, int i, float ov, int oi) {
    return oi != 0x7fffffff && (i == 0x7fffffff || ov > v || (ov == v && oi < i));
  };
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
    const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
    if (better(bv, bi, ov, oi)) {
      bv = ov;
      bi = oi;
    }
  }
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (lane == 0) {
    best_v[warp] = bv;
    best_i[warp] = bi;
  }
  __syncthreads();
  if (warp == 0) {
    const int nw = (blockDim.x + 31) >> 5;
    bv = lane < nw ? best_v[lane] : -INFINITY;
    bi = lane < nw ? best_i[lane] : 0x7fffffff;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (better(bv, bi, ov, oi)) {
        bv = ov;
        bi = oi;
      }
    }
    if (lane == 0)
      out[blockIdx.x] = bi;
  }
}

/* ----------------------------------------------------------------- embed
 * nn_embed (nn.vx:942-958); a token outside the table gives a row of NaN
 * instead of a read outside it. */
__global__ void embed_kernel(float *x, const void *table, int tbf16,
                             const int32_t *token, int dim, int rows,
                             int64_t x_stride) {
  chain_release();
  chain_wait();
  const int b = blockIdx.y;
  const int t = token[b];
  for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < dim;
       i += gridDim.x * blockDim.x) {
    float v = __int_as_float(0x7fc00000);
    if (t >= 0 && t < rows)
      v = tbf16 ? bf16_at(table, (int64_t)t * dim + i)
                : ((const float *)table)[(int64_t)t * dim + i];
    x[b * x_stride + i] = v;
  }
}

} // namespace


const char *matvec(const MatvecArgs &a, cudaStream_t stream) {
  if (a.rows <= 0 || a.batch <= 0)
    return nullptr;
  RowDotParams p{};
  p.w0 = a.w;
  p.rows = a.rows;
  p.cols = a.cols;
  p.items = (a.rows + 1) / 2;
  p.x = a.x;
  p.x_stride = a.x_stride;
  p.batch = a.batch;
  p.norm_w = a.norm_w;
  p.norm_bf16 = a.norm_bf16;
  p.eps = a.eps;
  p.norm_n = a.norm_n;
  p.y = a.y;
  p.y_stride = a.y_stride;
  p.bias = a.bias;
  p.s0 = a.scales;
  p.row_base = a.row_base;
  const int fmt = a.wfmt ? a.wfmt : (a.wbf16 ? kFmtBf16 : kFmtF32);
  const int per_word = fmt == kFmtF32 ? 4 : fmt == kFmtBf16 ? 8 : fmt == kFmtFp8 ? 16 : 32;
  if (a.expert_ids) {
    if (fmt == kFmtFp8)
      return "the expert projections take bf16 or Q4_0 weights";
    p.expert_ids = a.expert_ids;
    p.expert_slot = a.expert_slot;
    p.experts = a.experts;
    p.expert_bytes = (int64_t)a.rows * (a.cols / per_word * 16);
    p.scale_bytes = fmt == kFmtQ4 ? (int64_t)a.rows * (a.cols / 32) * 2 : 0;
  }
  p.add_scale = a.add_scale;
  switch (a.mode) {
  case 0: return launch_rowdot(EPI_STORE, p, fmt, stream);
  case 1: return launch_rowdot(EPI_ADD, p, fmt, stream);
  case 2: return launch_rowdot(EPI_BIAS, p, fmt, stream);
  case 3:
    if (!a.push || a.push->ranks < 1 || a.push->ranks > kMaxTpRanks)
      return "a pushed projection needs the receive buffers of 1 to 8 ranks";
    if (a.push->count % 2 != 0 || a.y_stride % 2 != 0)
      return "a pushed projection needs an even number of rows";
    p.tp = *a.push;
    return launch_rowdot(EPI_PUSH, p, fmt, stream);
  default: return "unknown matvec mode";
  }
}

const char *matvec_f32(float *y, const float *x, const float *w, int n, int d,
                       cudaStream_t stream) {
  if (n % 8 != 0 || (((uintptr_t)w | (uintptr_t)x) & 15)) {
    /* Any n: the f32 GEMM with a one-column B. */
    return gemm_f32(w, n, x, 1, y, 1, d, 1, n, stream);
  }
  MatvecArgs a{};
  a.w = w;
  a.wbf16 = false;
  a.rows = d;
  a.cols = n;
  a.x = x;
  a.x_stride = n;
  a.y = y;
  a.y_stride = d;
  a.batch = 1;
  return matvec(a, stream);
}

const char *fan_proj(const FanArgs &a, cudaStream_t stream) {
  if ((a.rows | a.out.k_row | a.out.gate_row | a.out.up_row) % 8 != 0)
    return "the parts of an input projection are multiples of 8 rows";
  if (a.out.cache_rows < 1)
    return "the ring of keys needs a row";
  RowDotParams p{};
  p.w0 = a.w;
  p.rows = a.rows;
  p.cols = a.cols;
  p.items = a.rows / 2;
  p.x = a.x;
  p.x_stride = a.x_stride;
  p.batch = a.batch;
  p.norm_w = a.norm_w;
  p.norm_n = a.norm_n;
  p.eps = a.eps;
  p.y = a.q_out;
  p.y_stride = a.q_stride;
  p.k_cache = a.k_cache;
  p.cache_batch_stride = a.cache_batch_stride;
  p.positions = a.positions;
  p.fan = a.out;
  return launch_rowdot(EPI_FAN, p, a.fmt, stream);
}

const char *stream_proj(const StreamProj &a, cudaStream_t stream) {
  if (a.streams < 1 || a.streams > kMaxStreams)
    return "a residual has 1 to 32 streams";
  if (a.rows % 2 != 0 || a.y_stride % 2 != 0 || a.stream_stride % 4 != 0)
    return "the projections around streams take an even number of rows, and streams "
           "a multiple of 4 values apart";
  RowDotParams p{};
  p.w0 = a.w;
  p.rows = a.rows;
  p.cols = a.cols;
  p.items = a.rows / 2;
  p.x = a.x;
  p.x_stride = a.x_stride;
  p.batch = a.batch;
  p.norm_w = a.norm_w;
  p.norm_n = a.norm_n;
  p.eps = a.eps;
  p.y = a.y;
  p.y_stride = a.y_stride;
  p.streams = a.streams;
  p.stream_stride = a.stream_stride;
  p.stream_in = a.in;
  p.stream_mix = a.mix;
  p.stream_out = a.out;
  p.logit_scale = a.logit_scale;
  p.logit_cap = a.logit_cap;
  switch (a.mode) {
  case kStreamsStore: return launch_rowdot(EPI_IN_STORE, p, a.fmt, stream);
  case kStreamsGelu: return launch_rowdot(EPI_IN_GELU, p, a.fmt, stream);
  case kStreamsLogits: return launch_rowdot(EPI_IN_LOGITS, p, a.fmt, stream);
  case kStreamsMix:
    if (!a.mix || !a.out)
      return "mixing streams takes their matrix and the weights of the product";
    return launch_rowdot(EPI_MIX, p, a.fmt, stream);
  default: return "unknown mode of a projection around streams";
  }
}

const char *swiglu(const SwigluArgs &a, cudaStream_t stream) {
  if (a.rows <= 0 || a.batch <= 0)
    return nullptr;
  RowDotParams p{};
  p.w0 = a.w;
  p.w1 = a.w_up;
  p.rows = a.rows;
  p.cols = a.cols;
  p.items = a.rows;
  p.x = a.x;
  p.x_stride = a.x_stride;
  p.batch = a.batch;
  p.norm_w = a.norm_w;
  p.norm_bf16 = a.norm_bf16;
  p.eps = a.eps;
  p.y = a.out;
  p.y_stride = a.out_stride;
  p.s0 = a.scales;
  p.s1 = a.scales_up;
  p.row_base = a.row_base;
  if (a.expert_ids) {
    const int fmt = a.wfmt ? a.wfmt : (a.wbf16 ? kFmtBf16 : kFmtF32);
    const int per_word = fmt == kFmtF32 ? 4 : fmt == kFmtBf16 ? 8 : fmt == kFmtFp8 ? 16 : 32;
    if (fmt == kFmtFp8 || a.w_up)
      return "the expert projections take bf16 or Q4_0 weights, gate and up rows "
             "in one matrix";
    p.expert_ids = a.expert_ids;
    p.expert_slot = a.expert_slot;
    p.experts = a.experts;
    p.expert_bytes = (int64_t)2 * a.rows * (a.cols / per_word * 16);
    p.scale_bytes = fmt == kFmtQ4 ? (int64_t)2 * a.rows * (a.cols / 32) * 2 : 0;
  }
  return launch_rowdot(EPI_SWIGLU, p, a.wfmt ? a.wfmt : (a.wbf16 ? kFmtBf16 : kFmtF32),
                                   stream);
}

const char *qkv_rope_store(const QkvArgs &a, cudaStream_t stream) {
  if (a.head_dim % 2 != 0)
    return "head_dim must be even";
  RowDotParams p{};
  p.w0 = a.wq;
  p.w1 = a.wk;
  p.w2 = a.wv;
  p.rows = (a.q_heads + 2 * a.kv_heads) * a.head_dim;
  p.cols = a.cols;
  p.items = p.rows / 2;
  p.x = a.x;
  p.x_stride = a.x_stride;
  p.batch = a.batch;
  p.norm_w = a.norm_w;
  p.norm_bf16 = a.norm_bf16;
  p.eps = a.eps;
  p.y = a.q_out;
  p.y_stride = (int64_t)a.q_heads * a.head_dim;
  p.bias = a.bias;
  p.q_heads = a.q_heads;
  p.kv_heads = a.kv_heads;
  p.head_dim = a.head_dim;
  p.rope_mode = a.rope_mode;
  p.cos_t = a.cos_t;
  p.sin_t = a.sin_t;
  p.cs_cols = a.cs_cols;
  p.theta = a.theta;
  p.positions = a.positions;
  p.k_cache = a.k_cache;
  p.v_cache = a.v_cache;
  p.cache_batch_stride = a.cache_batch_stride;
  p.max_seq = a.max_seq;
  p.s0 = a.sq;
  p.s1 = a.sk;
  p.s2 = a.sv;
  return launch_rowdot(EPI_QKV, p, a.wfmt ? a.wfmt : (a.wbf16 ? kFmtBf16 : kFmtF32),
                                stream);
}

int tp_status(cudaStream_t stream) {
  if (cudaStreamSynchronize(stream) != cudaSuccess)
    return -1;
  const int b = rowdot_bf16_status(), f = rowdot_f32_status(), q = rowdot_quant_status();
  const int sb = rowdot_streams_bf16_status(), sf = rowdot_streams_f32_status();
  return b ? b : f ? f : q ? q : sb ? sb : sf;
}

const char *rms_norm(float *y, const float *x, const void *w, bool wbf16, int n,
                     float eps, int batch, int64_t stride, cudaStream_t stream) {
  if (n <= 0 || batch <= 0)
    return nullptr;
  launch_chained(rms_norm_kernel, dim3(batch), dim3(1024), 0, stream, y, x, w,
                 (int)wbf16, n, eps, stride);
  return check_launch("the RMSNorm launch");
}

const char *rope_and_store(float *q_out, float *k_cache, float *v_cache,
                           const float *q, const float *k, const float *v,
                           const float *cos_t, const float *sin_t, int cs_cols,
                           int pos, int q_heads, int kv_heads, int head_dim,
                           cudaStream_t stream) {
  if (head_dim > 1024)
    return "head_dim is larger than a block";
  launch_chained(rope_store_kernel, dim3(q_heads + kv_heads),
                 dim3(((head_dim + 31) / 32) * 32), 0, stream, q_out, k_cache,
                 v_cache, q, k, v, cos_t, sin_t, cs_cols, pos, q_heads,
                 kv_heads, head_dim);
  return check_launch("the RoPE launch");
}

size_t attn_scratch_floats(int batch, int q_heads, int head_dim, int max_seq,
                           int split) {
  return (size_t)batch * q_heads * ((size_t)max_seq / split + 1) *
         (head_dim + 2);
}

const char *attention_decode(const AttnArgs &a, cudaStream_t stream) {
  if (a.head_dim % 4 != 0 || a.head_dim > 128)
    return "head_dim must be a multiple of 4, and at most 128";
  if (a.q_heads % a.kv_heads != 0)
    return "q_heads must be a multiple of kv_heads";
  if (a.split < 1)
    return "the split must be at least one position";
  if (((uintptr_t)a.scratch & 7) || ((uintptr_t)a.q & 15) ||
      ((uintptr_t)a.k_cache & 15) || ((uintptr_t)a.v_cache & 15) ||
      ((uintptr_t)a.out & 15))
    return "q, the caches and out must be 16-byte aligned, the scratch 8-byte";
  const int group = a.q_heads / a.kv_heads;
  const int gh = group >= 4 ? 4 : (group >= 2 ? 2 : 1);
  const int tiles = (group + gh - 1) / gh;
  int which = a.kernel == kAttnAuto ? attention_kernel_choice(-1) : a.kernel;
  if (which == kAttnAuto)
    which = kAttnCluster;
  if (which == kAttnSplit && (!a.scratch || !a.counters))
    return "the split attention kernel needs scratch memory and counters";
  if (which != kAttnCluster && which != kAttnSplit)
    return "unknown attention kernel";
  if (which == kAttnCluster) {
    const dim3 cgrid(ATT_CLUSTER, a.kv_heads * tiles, a.batch);
    /* Warps per block by how many blocks there are: with few heads (a rank of
       a tensor-parallel job holds 4 or 8 of 32) sixteen warps per block put
       the positions of a head on 128 warps, one round trip to memory each;
       with every SM already holding several blocks, four. Measured at
       position 520 on one rank's share of the 7B shape, microseconds per
       layer for 4 / 8 / 16 warps: 1/2 of the heads 53.4 / 51.8 / 54.3, 1/4
       37.7 / 37.3 / 36.0, 1/8 28.6 / 27.3 / 26.5; all heads 387 / 389 / 361
       tokens/s. */
    const int64_t blocks = (int64_t)cgrid.x * cgrid.y * cgrid.z;
    int warps = 2 * blocks <= sm_count() ? 16 : (blocks <= 2 * sm_count() ? 8 : 4);
    /* VXB_ATTN_WARPS=4, 8 or 16 pins it (for measurements) */
    if (const char *pin = getenv("VXB_ATTN_WARPS")) {
      const int v = atoi(pin);
      if (v == 4 || v == 8 || v == 16)
        warps = v;
    }
    auto go = [&](auto kernel) {
      launch_chained_cluster(kernel, cgrid, dim3(warps * 32), ATT_CLUSTER, stream, a);
    };
    if (gh == 4) {
      if (warps == 16) go(attention_cluster_kernel<4, 16>);
      else if (warps == 8) go(attention_cluster_kernel<4, 8>);
      else go(attention_cluster_kernel<4, 4>);
    } else if (gh == 2) {
      if (warps == 16) go(attention_cluster_kernel<2, 16>);
      else if (warps == 8) go(attention_cluster_kernel<2, 8>);
      else go(attention_cluster_kernel<2, 4>);
    } else {
      if (warps == 16) go(attention_cluster_kernel<1, 16>);
      else if (warps == 8) go(attention_cluster_kernel<1, 8>);
      else go(attention_cluster_kernel<1, 4>);
    }
    return check_launch("the attention launch");
  }
  const dim3 grid(a.max_pos / a.split + 1, a.kv_heads * tiles, a.batch);
  if (gh == 4)
    launch_chained(attention_decode_kernel<4>, grid, dim3(4 * 32), 0, stream, a);
  else if (gh == 2)
    launch_chained(attention_decode_kernel<2>, grid, dim3(4 * 32), 0, stream, a);
  else
    launch_chained(attention_decode_kernel<1>, grid, dim3(4 * 32), 0, stream, a);
  return check_launch("the attention launch");
}

int attention_kernel_choice(int which) {
  static std::mutex mu;
  static int choice = kAttnAuto;
  std::lock_guard<std::mutex> lock(mu);
  const int before = choice;
  if (which == kAttnAuto || which == kAttnCluster || which == kAttnSplit)
    choice = which;
  return before;
}

const char *attention_decode_clustered(const AttnArgs &a, cudaStream_t stream) {
  AttnArgs b = a;
  b.scratch = nullptr;
  b.counters = nullptr;
  b.kernel = kAttnCluster;
  return attention_decode(b, stream);
}

const char *top_k(int32_t *ids, float *weights, const float *logits, int n, int k,
                  cudaStream_t stream) {
  return top_k_rows(ids, weights, logits, 1, n, k, 0, 0, 0, stream);
}

const char *top_k_rows(int32_t *ids, float *weights, const float *logits,
                       int positions, int n, int k, int64_t ids_pitch,
                       int64_t weights_pitch, int64_t logits_pitch,
                       cudaStream_t stream) {
  if (n < 1 || n > 256 || k < 1 || k > n)
    return "n must be 1 to 256, and k must be 1 to n";
  if (positions < 1)
    return nullptr;
  launch_chained(top_k_kernel, dim3(positions), dim3(256), 0, stream, ids, weights,
                 logits, n, k, ids_pitch, weights_pitch, logits_pitch);
  return check_launch("the router launch");
}

const char *argmax(int32_t *out, const float *logits, int n, int batch,
                   int64_t stride, cudaStream_t stream) {
  if (n <= 0 || batch <= 0)
    return nullptr;
  launch_chained(argmax_kernel, dim3(batch), dim3(1024), 0, stream, out, logits,
                 n, stride);
  return check_launch("the argmax launch");
}

const char *embed(float *x, const void *table, bool tbf16, const int32_t *token,
                  int dim, int rows, int batch, int64_t x_stride,
                  cudaStream_t stream) {
  const dim3 grid((dim + 255) / 256, batch);
  launch_chained(embed_kernel, grid, dim3(256), 0, stream, x, table, (int)tbf16,
                 token, dim, rows, x_stride);
  return check_launch("the embed launch");
}

} // namespace vxb
