/* residual_streams.cu -- a residual of several streams over the positions of a
 * prompt: their weighted sum through a norm, and their mixing with a sublayer's
 * output, which the norm of the next sublayer follows in the same pass.  (A step has
 * both inside its projections: stream_proj.)
 *
 * A block is a position; a thread keeps its values of every stream to itself, so the
 * streams of a position are read once, mixed in registers and written once.
 */
#include "kernels.h"
#include "launch.cuh"
#include "launch_util.h"
#include "nn_device.cuh"
#include "terms.cuh"

namespace vxb {
namespace {

constexpr int THREADS = 256;

/* A NormGain and a StreamMix of at most kMaxStreams streams, in shared memory. */
struct MixShared {
  float in[kMaxStreams], out[kMaxStreams], mix[kMaxStreams * kMaxStreams];
  float red[THREADS / 32];
};

__device__ __forceinline__ float gain_of(const NormGain &w, int i) {
  return w.f32 ? ((const float *)w.gain)[i] : bf16_val(w.gain, i);
}

/* 1 / sqrt(mean of ss over n + eps), ss summed over the block in a fixed order */
__device__ __forceinline__ float block_rms(float ss, int n, float eps, float *red) {
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0)
    red[threadIdx.x >> 5] = ss;
  __syncthreads();
  float total = 0.0f;
  for (int k = 0; k < THREADS / 32; ++k)
    total += red[k];
  return 1.0f / sqrtf(total / (float)n + eps);
}

/* TERMS: out is bf16 terms [t][3 dim], else f32 rows [t][dim]. */
template <bool TERMS>
__global__ void __launch_bounds__(THREADS)
streams_norm_kernel(void *out, const float *x, int64_t x_stride, const float *in,
                    int streams,
                    const NormGain w, int dim, float eps, const int32_t *pick) {
  extern __shared__ __align__(16) float u[]; /* [dim] */
  __shared__ float red[THREADS / 32];
  const int64_t t = blockIdx.x;
  const float *xr = x + (pick ? pick[t] : t) * x_stride;
  float ss = 0.0f;
  for (int i = threadIdx.x * 4; i < dim; i += THREADS * 4) {
    float4 v = make_float4(0, 0, 0, 0);
#pragma unroll 4
    for (int s = 0; s < streams; ++s)
      axpy(v, in ? in[s] : 1.0f,
           *reinterpret_cast<const float4 *>(xr + (int64_t)s * dim + i));
    *reinterpret_cast<float4 *>(u + i) = v;
    ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
  }
  const float inv = block_rms(ss, w.n ? w.n : dim, eps, red);
  for (int i = threadIdx.x * 4; i < dim; i += THREADS * 4) {
    const float4 v = *reinterpret_cast<const float4 *>(u + i);
    const float n[4] = {v.x * gain_of(w, i) * inv, v.y * gain_of(w, i + 1) * inv,
                        v.z * gain_of(w, i + 2) * inv, v.w * gain_of(w, i + 3) * inv};
    if (TERMS)
      store_terms4((__nv_bfloat16 *)out, dim, t, i, n);
    else
      *reinterpret_cast<float4 *>((float *)out + t * dim + i) =
          make_float4(n[0], n[1], n[2], n[3]);
  }
}

/* S streams, a thread four neighbouring values of all of them at a time; S 0: any
   number, a value at a time. */
template <int S>
__global__ void __launch_bounds__(THREADS)
streams_mix_kernel(__nv_bfloat16 *terms, float *x, const float *partials, int splits,
                   int t_count, const StreamMix m, const float *next_in,
                   const NormGain w, int dim, float eps) {
  extern __shared__ __align__(16) float u[]; /* [dim], S 0: then [streams][THREADS] */
  __shared__ MixShared sh;
  const int streams = S ? S : m.streams, tid = threadIdx.x;
  for (int i = tid; i < streams * streams; i += THREADS)
    sh.mix[i] = m.mix[i];
  if (tid < streams) {
    sh.out[tid] = m.out[tid];
    sh.in[tid] = next_in ? next_in[tid] : 1.0f;
  }
  __syncthreads();
  const int64_t t = blockIdx.x;
  float *xr = x + t * streams * (int64_t)dim;
  float ss = 0.0f;
  if constexpr (S > 0) {
    for (int i = tid * 4; i < dim; i += THREADS * 4) {
      float4 old[S], v = make_float4(0, 0, 0, 0);
#pragma unroll
      for (int s = 0; s < S; ++s)
        old[s] = *reinterpret_cast<const float4 *>(xr + (int64_t)s * dim + i);
      const float4 y = sum_runs4(partials, splits, t_count, dim, t, i);
#pragma unroll
      for (int to = 0; to < S; ++to) {
        float4 now = make_float4(0, 0, 0, 0);
        axpy(now, sh.out[to], y);
#pragma unroll
        for (int s = 0; s < S; ++s)
          axpy(now, sh.mix[s * S + to], old[s]);
        *reinterpret_cast<float4 *>(xr + (int64_t)to * dim + i) = now;
        axpy(v, sh.in[to], now);
      }
      *reinterpret_cast<float4 *>(u + i) = v;
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
  } else {
    float *old = u + dim;
    for (int i = tid; i < dim; i += THREADS) {
      const float y = sum_runs(partials, splits, t_count, dim, t, i);
      float v = 0.0f;
      for (int s = 0; s < streams; ++s)
        old[s * THREADS + tid] = xr[(int64_t)s * dim + i];
      for (int to = 0; to < streams; ++to) {
        float now = sh.out[to] * y;
        for (int s = 0; s < streams; ++s)
          now = fmaf(sh.mix[s * streams + to], old[s * THREADS + tid], now);
        xr[(int64_t)to * dim + i] = now;
        v = fmaf(sh.in[to], now, v);
      }
      u[i] = v;
      ss = fmaf(v, v, ss);
    }
  }
  if (!terms)
    return;
  const float inv = block_rms(ss, w.n ? w.n : dim, eps, sh.red); /* u is complete */
  for (int i = tid * 4; i < dim; i += THREADS * 4) {
    const float4 v = *reinterpret_cast<const float4 *>(u + i);
    const float n[4] = {v.x * gain_of(w, i) * inv, v.y * gain_of(w, i + 1) * inv,
                        v.z * gain_of(w, i + 2) * inv, v.w * gain_of(w, i + 3) * inv};
    store_terms4(terms, dim, t, i, n);
  }
}

/* a thread per (position, eight rows) */
__global__ void __launch_bounds__(256)
gelu_finish_kernel(__nv_bfloat16 *terms, const float *partials, int splits, int t_count,
                   int hidden) {
  const int per_row = hidden / 8;
  const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (int64_t)t_count * per_row)
    return;
  const int64_t t = idx / per_row;
  const int r = (int)(idx - t * per_row) * 8;
  const float4 lo = sum_runs4(partials, splits, t_count, hidden, t, r);
  const float4 hi = sum_runs4(partials, splits, t_count, hidden, t, r + 4);
  const float v[8] = {gelu(lo.x), gelu(lo.y), gelu(lo.z), gelu(lo.w),
                      gelu(hi.x), gelu(hi.y), gelu(hi.z), gelu(hi.w)};
  store_terms8(terms, hidden, t, r, v);
}

const char *refuse(const StreamMix &m, int dim) {
  if (m.streams < 1 || m.streams > kMaxStreams)
    return "a residual has 1 to 32 streams";
  if (dim * (int)sizeof(float) > 200 * 1024)
    return "a stream of the residual must fit in shared memory (51200 values)";
  return nullptr;
}

template <bool TERMS>
const char *launch_norm(void *out, const float *x, int64_t x_stride, const StreamMix &m,
                        NormGain w, int t, int dim, float eps, cudaStream_t stream,
                        const int32_t *pick) {
  if (const char *why = refuse(m, dim))
    return why;
  if (t <= 0)
    return nullptr;
  if (allow_dynamic_smem((const void *)streams_norm_kernel<TERMS>, 200 * 1024) !=
      cudaSuccess)
    return "the norm of the streams could not get its shared memory";
  launch_in_order(streams_norm_kernel<TERMS>, dim3(t), dim3(THREADS), dim * sizeof(float),
                 stream, out, x, x_stride, m.in, m.streams, w, dim, eps, pick);
  return check_launch("the norm of the streams");
}

template <int S>
const char *launch_mix(void *terms, float *x, const float *partials, int splits, int t,
                       const StreamMix &m, const float *next_in, NormGain w, int dim,
                       float eps, cudaStream_t stream) {
  const size_t smem = (dim + (S ? 0 : m.streams * THREADS)) * sizeof(float);
  if (smem > 216 * 1024 || dim % 4 != 0)
    return "the streams of a position must fit in shared memory";
  if (allow_dynamic_smem((const void *)streams_mix_kernel<S>, 216 * 1024) != cudaSuccess)
    return "the mixing of the streams could not get its shared memory";
  launch_in_order(streams_mix_kernel<S>, dim3(t), dim3(THREADS), smem, stream, (__nv_bfloat16 *)terms, x, partials, splits, t, m, next_in, w,
                 dim, eps);
  return check_launch("the mixing of the streams");
}

} // namespace

const char *rows_streams_norm(void *terms, const float *x, const StreamMix &m, NormGain w,
                              int t, int dim, float eps, cudaStream_t stream,
                              const int32_t *pick) {
  return launch_norm<true>(terms, x, (int64_t)m.streams * dim, m, w, t, dim, eps, stream,
                           pick);
}

const char *streams_norm(float *y, const float *x, int64_t x_stride, const StreamMix &m,
                         NormGain w, int batch, int dim, float eps, cudaStream_t stream) {
  return launch_norm<false>(y, x, x_stride, m, w, batch, dim, eps, stream, nullptr);
}

const char *rows_streams_mix(void *terms, float *x, const float *partials, int splits,
                             int t, const StreamMix &m, const float *next_in, NormGain w,
                             int dim, float eps, cudaStream_t stream) {
  if (const char *why = refuse(m, dim))
    return why;
  if (t <= 0)
    return nullptr;
  switch (m.streams) {
#define CASE(S)                                                                          \
  case S:                                                                                \
    return launch_mix<S>(terms, x, partials, splits, t, m, next_in, w, dim, eps, stream)
    CASE(1);
    CASE(2);
    CASE(3);
    CASE(4);
    CASE(8);
#undef CASE
  default:
    return launch_mix<0>(terms, x, partials, splits, t, m, next_in, w, dim, eps, stream);
  }
}

const char *rows_gelu_finish(void *terms, const float *partials, int splits, int t,
                             int hidden, cudaStream_t stream) {
  if (hidden % 8 != 0)
    return "the multi-position gelu takes a hidden size in multiples of 8";
  const int64_t count = (int64_t)t * (hidden / 8);
  launch_in_order(gelu_finish_kernel, dim3((unsigned)((count + 255) / 256)), dim3(256), 0,
                 stream, (__nv_bfloat16 *)terms, partials, splits, t, hidden);
  return check_launch("the multi-position gelu");
}

} // namespace vxb
