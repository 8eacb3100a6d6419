/* parallel_block.cu -- the small kernels around the two products of a parallel
 * block, and the f32 product of a prompt's positions.
 *
 * A parallel block reads one norm of the residual in all its input matrices, so
 * they are one matrix with rows q | k | gate | up, and adds the sum of its two
 * outputs, so they are one matrix whose columns are the attention output's and
 * then `up`'s.  A decode step is three launches a layer (fan_proj, window
 * attention, matvec with a residual add), a prompt five (GEMM, rows_fan_finish,
 * window attention, GEMM, residual add and norm).
 */
#include "kernels.h"
#include "launch.cuh"
#include "launch_util.h"
#include "nn_device.cuh"
#include "terms.cuh"

#include <cstdio>

namespace vxb {
namespace {

/* ---- token rows with their position, normalised: a block per row, a thread per
   pair of values that share an angle ---------------------------------------------- */
__global__ void __launch_bounds__(1024) position_embed_kernel(const PositionEmbedArgs a) {
  extern __shared__ __align__(8) float embed_row[]; /* [dim] */
  __shared__ float red[32];
  chain_release();
  chain_wait();
  const int64_t t = blockIdx.x;
  const int token = a.tokens[t];
  const int pos = a.per_sequence ? a.positions[t] : a.positions[0] + (int)t;
  const int copies = a.copies > 1 ? a.copies : 1;
  float *row = a.x + t * copies * a.dim;
  if (token < 0 || token >= a.vocab) {
    for (int i = threadIdx.x; i < a.dim; i += blockDim.x)
      for (int c = 0; c < copies; ++c)
        row[c * a.dim + i] = i < a.width ? __int_as_float(0x7fc00000) : 0.0f;
    return;
  }
  float ss = 0.0f;
#pragma unroll 2
  for (int k = threadIdx.x; 2 * k < a.width; k += blockDim.x) {
    /* dim is even, so a pair of the table is one aligned load; the second value
       of an odd width's last pair is filling */
    float2 e;
    if (a.table_bf16) {
      const uint32_t two =
          ((const uint32_t *)a.table)[((int64_t)token * a.dim >> 1) + k];
      e = make_float2(bf_lo(two), bf_hi(two));
    } else {
      e = ((const float2 *)a.table)[((int64_t)token * a.dim >> 1) + k];
    }
    float sine = 0.0f, cosine = 0.0f;
    if (a.turns)
      turned(pos, a.turns[k], sine, cosine);
    const float v0 = fmaf(e.x, a.scale, sine);
    const float v1 = 2 * k + 1 < a.width ? fmaf(e.y, a.scale, cosine) : 0.0f;
    *reinterpret_cast<float2 *>(&embed_row[2 * k]) = make_float2(v0, v1);
    ss = fmaf(v0, v0, ss);
    ss = fmaf(v1, v1, ss);
  }
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0)
    red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = 0.0f;
  for (int k = 0; k < (int)blockDim.x / 32; ++k) /* fixed order */
    total += red[k];
  const float inv = 1.0f / sqrtf(total / (float)a.width + a.eps);
  for (int i = threadIdx.x; i < a.dim; i += blockDim.x) {
    const float v = i >= a.width ? 0.0f
                    : a.gain     ? embed_row[i] * inv * a.gain[i]
                                 : embed_row[i];
    for (int c = 0; c < copies; ++c)
      row[c * a.dim + i] = v;
  }
}

/* ---- after the input GEMM: a thread per (position, eight rows) ---------------- */
__global__ void __launch_bounds__(256)
fan_finish_kernel(const float *partials, int splits, int t_count, int n,
                  const FanOut f, const int32_t *positions, float *q_out,
                  int64_t q_stride, float *k_cache, __nv_bfloat16 *terms, int out_cols,
                  int out_col) {
  chain_release();
  chain_wait();
  const int per_row = n / 8;
  const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (int64_t)t_count * per_row)
    return;
  const int64_t t = idx / per_row;
  const int r = (int)(idx - t * per_row) * 8;
  const float4 lo = sum_runs4(partials, splits, t_count, n, t, r);
  const float4 hi = sum_runs4(partials, splits, t_count, n, t, r + 4);
  float v[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
  float *dst;
  if (r < f.k_row) {
    dst = q_out + t * q_stride + r;
  } else if (r < f.gate_row) {
    const int row = (positions[0] + (int)t) % f.cache_rows;
    dst = k_cache + (int64_t)row * (f.gate_row - f.k_row) + r - f.k_row;
  } else if (r < f.up_row) {
#pragma unroll
    for (int e = 0; e < 8; ++e)
      v[e] = sigmoid(v[e]);
    dst = f.gate + t * f.gate_stride + r - f.gate_row;
  } else {
#pragma unroll
    for (int e = 0; e < 8; ++e)
      v[e] = squared_relu(v[e]);
    store_terms8(terms, out_cols, t, out_col + r - f.up_row, v);
    return;
  }
  *reinterpret_cast<float4 *>(dst) = make_float4(v[0], v[1], v[2], v[3]);
  *reinterpret_cast<float4 *>(dst + 4) = make_float4(v[4], v[5], v[6], v[7]);
}

__global__ void __launch_bounds__(256)
sum_kernel(float *out, const float *partials, int splits, int t_count, int n, float scale,
           float cap) {
  chain_release();
  chain_wait();
  const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (int64_t)t_count * n)
    return;
  const int64_t t = idx / n;
  out[idx] = capped_logit(sum_runs(partials, splits, t_count, n, t, idx - t * n), scale,
                          cap);
}

/* The same for n a multiple of 4, four values a thread. */
__global__ void __launch_bounds__(256)
sum4_kernel(float *out, const float *partials, int splits, int t_count, int n, float scale,
            float cap) {
  chain_release();
  chain_wait();
  const int64_t idx = ((int64_t)blockIdx.x * blockDim.x + threadIdx.x) * 4;
  if (idx >= (int64_t)t_count * n)
    return;
  const float4 s = sum_runs4(partials, splits, 1, (int64_t)t_count * n, 0, idx);
  *reinterpret_cast<float4 *>(out + idx) =
      make_float4(capped_logit(s.x, scale, cap), capped_logit(s.y, scale, cap),
                  capped_logit(s.z, scale, cap), capped_logit(s.w, scale, cap));
}

/* ---- the f32 product on the FP32 pipe: 64 positions x 64 rows a block, 4 x 4 a
   thread, the terms added up again (exactly) on their way into shared memory --- */
constexpr int GT = 64, GC = 16;
__global__ void __launch_bounds__(256)
rows_gemm_f32_kernel(const __nv_bfloat16 *terms, const float *w, int t_count, int n,
                     int cols, float *out) {
  __shared__ __align__(16) float sx[GC][GT + 4], sw[GC][GT + 4];
  chain_release();
  chain_wait();
  const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16;
  const int t0 = blockIdx.y * GT, n0 = blockIdx.x * GT;
  /* a thread stages four columns of one position and of one matrix row */
  const int lr = tid / 4, lc = tid % 4 * 4;
  float acc[4][4] = {};
  for (int c0 = 0; c0 < cols; c0 += GC) {
    float xv[4] = {0, 0, 0, 0}, wv[4] = {0, 0, 0, 0};
    if (t0 + lr < t_count) {
      const __nv_bfloat16 *row = terms + (int64_t)(t0 + lr) * 3 * cols + c0 + lc;
#pragma unroll
      for (int e = 0; e < 4; ++e)
        xv[e] = (bf16_val(row, e) + bf16_val(row, cols + e)) +
                bf16_val(row, 2 * (int64_t)cols + e);
    }
    if (n0 + lr < n) {
      const float4 v =
          *reinterpret_cast<const float4 *>(w + (int64_t)(n0 + lr) * cols + c0 + lc);
      wv[0] = v.x; wv[1] = v.y; wv[2] = v.z; wv[3] = v.w;
    }
    __syncthreads();
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      sx[lc + e][lr] = xv[e];
      sw[lc + e][lr] = wv[e];
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < GC; ++c) {
      const float4 xa = *reinterpret_cast<const float4 *>(&sx[c][ty * 4]);
      const float4 wa = *reinterpret_cast<const float4 *>(&sw[c][tx * 4]);
      const float xs[4] = {xa.x, xa.y, xa.z, xa.w}, ws[4] = {wa.x, wa.y, wa.z, wa.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
          acc[i][j] = fmaf(xs[i], ws[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (t0 + ty * 4 + i < t_count && n0 + tx * 4 + j < n)
        out[(int64_t)(t0 + ty * 4 + i) * n + n0 + tx * 4 + j] = acc[i][j];
}

} // namespace

const char *position_embed(const PositionEmbedArgs &a, cudaStream_t stream) {
  if (a.count <= 0)
    return nullptr;
  const int smem = a.dim * (int)sizeof(float);
  if (a.dim % 2 != 0 || ((uintptr_t)a.table & 7))
    return "a row of the embedding is an even number of values, 8-byte aligned";
  if (smem > 200 * 1024 ||
      allow_dynamic_smem((const void *)position_embed_kernel, 200 * 1024) != cudaSuccess)
    return "a row of the embedding must fit in shared memory (51200 values)";
  /* few rows: a thread per pair; many: enough blocks are in flight anyway */
  int threads = a.count > 64 ? 256 : 1024;
  while (threads > 32 && threads >= a.width)
    threads /= 2;
  launch_chained(position_embed_kernel, dim3(a.count), dim3(threads), smem, stream, a);
  return check_launch("the embedding launch");
}

const char *rows_fan_finish(const float *partials, int splits, int t, int n,
                            const FanOut &out, const int32_t *positions, float *q_out,
                            int64_t q_stride, float *k_cache, void *terms, int out_cols,
                            int out_col, cudaStream_t stream) {
  if ((n | out.k_row | out.gate_row | out.up_row | out_cols | out_col) % 8 != 0)
    return "the parts of an input projection are multiples of 8 rows";
  const int64_t count = (int64_t)t * (n / 8);
  launch_chained(fan_finish_kernel, dim3((unsigned)((count + 255) / 256)), dim3(256), 0,
                 stream, partials, splits, t, n, out, positions, q_out, q_stride,
                 k_cache, (__nv_bfloat16 *)terms, out_cols, out_col);
  return check_launch("the parts of an input projection");
}

const char *rows_sum(float *out, const float *partials, int splits, int t, int n,
                     cudaStream_t stream, float scale, float cap) {
  const int64_t count = (int64_t)t * n;
  if (n % 4 == 0)
    launch_chained(sum4_kernel, dim3((unsigned)((count / 4 + 255) / 256)), dim3(256), 0,
                   stream, out, partials, splits, t, n, scale, cap);
  else
    launch_chained(sum_kernel, dim3((unsigned)((count + 255) / 256)), dim3(256), 0,
                   stream, out, partials, splits, t, n, scale, cap);
  return check_launch("the sum of a product's runs");
}

const char *rows_gemm_f32(const void *terms, const float *w, int t, int n, int cols,
                          float *partials, cudaStream_t stream) {
  if (cols % GC != 0 || ((uintptr_t)w & 15))
    return "the f32 product of many positions takes columns in multiples of 16";
  launch_chained(rows_gemm_f32_kernel, dim3((n + GT - 1) / GT, (t + GT - 1) / GT),
                 dim3(256), 0, stream, (const __nv_bfloat16 *)terms, w, t, n, cols,
                 partials);
  return check_launch("the f32 product of many positions");
}

} // namespace vxb
