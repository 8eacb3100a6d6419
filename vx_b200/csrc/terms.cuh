/* terms.cuh -- f32 activations between the GEMMs of a prompt: a value as three
 * bf16 terms whose sum it is exactly, and the sum of the GEMM's runs. */
#ifndef VXB_TERMS_CUH
#define VXB_TERMS_CUH

#include <cuda_bf16.h>

#include <cstdint>

namespace vxb {
namespace {

[[maybe_unused]] __device__ __forceinline__ float bf16_val(const void *p, int64_t i) {
  return __uint_as_float((uint32_t)((const uint16_t *)p)[i] << 16);
}
/* v as three bf16 terms at column i of row t of a [T, 3 cols] matrix. */
[[maybe_unused]] __device__ __forceinline__ void store_terms(__nv_bfloat16 *terms, int cols,
                                            int64_t t, int i, float v) {
  const __nv_bfloat16 t1 = __float2bfloat16(v);
  const float r1 = v - __bfloat162float(t1);
  const __nv_bfloat16 t2 = __float2bfloat16(r1);
  const float r2 = r1 - __bfloat162float(t2);
  __nv_bfloat16 *row = terms + t * 3 * cols;
  row[i] = t1;
  row[cols + i] = t2;
  row[2 * cols + i] = __float2bfloat16(r2);
}
/* The sum of the runs' partials of (t, r), in run order. */
[[maybe_unused]] __device__ __forceinline__ float sum_runs(const float *partials, int splits,
                                          int64_t t_count, int64_t n, int64_t t,
                                          int64_t r) {
  float s = partials[t * n + r];
  for (int k = 1; k < splits; ++k)
    s += partials[((int64_t)k * t_count + t) * n + r];
  return s;
}

/* The same for four consecutive values (r a multiple of 4). */
[[maybe_unused]] __device__ __forceinline__ float4 sum_runs4(const float *partials, int splits,
                                            int64_t t_count, int64_t n, int64_t t,
                                            int64_t r) {
  float4 s = *reinterpret_cast<const float4 *>(partials + t * n + r);
  for (int k = 1; k < splits; ++k) {
    const float4 v = *reinterpret_cast<const float4 *>(
        partials + ((int64_t)k * t_count + t) * n + r);
    s.x += v.x; s.y += v.y; s.z += v.z; s.w += v.w;
  }
  return s;
}
/* Eight consecutive values (i a multiple of 8) as their three terms: one
   16-byte store per term. */
[[maybe_unused]] __device__ __forceinline__ void store_terms8(__nv_bfloat16 *terms, int cols,
                                             int64_t t, int i, const float (&v)[8]) {
  uint32_t w1[4], w2[4], w3[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    uint32_t parts[3] = {0, 0, 0};
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      const float x = v[2 * j + h];
      const __nv_bfloat16 t1 = __float2bfloat16(x);
      const float r1 = x - __bfloat162float(t1);
      const __nv_bfloat16 t2 = __float2bfloat16(r1);
      const float r2 = r1 - __bfloat162float(t2);
      const __nv_bfloat16 t3 = __float2bfloat16(r2);
      parts[0] |= (uint32_t)__bfloat16_as_ushort(t1) << (16 * h);
      parts[1] |= (uint32_t)__bfloat16_as_ushort(t2) << (16 * h);
      parts[2] |= (uint32_t)__bfloat16_as_ushort(t3) << (16 * h);
    }
    w1[j] = parts[0];
    w2[j] = parts[1];
    w3[j] = parts[2];
  }
  __nv_bfloat16 *row = terms + t * 3 * cols;
  *reinterpret_cast<uint4 *>(row + i) = make_uint4(w1[0], w1[1], w1[2], w1[3]);
  *reinterpret_cast<uint4 *>(row + cols + i) = make_uint4(w2[0], w2[1], w2[2], w2[3]);
  *reinterpret_cast<uint4 *>(row + 2 * cols + i) = make_uint4(w3[0], w3[1], w3[2], w3[3]);
}
/* Four consecutive values (i a multiple of 4), one 8-byte store per term. */
[[maybe_unused]] __device__ __forceinline__ void
store_terms4(__nv_bfloat16 *terms, int cols, int64_t t, int i, const float (&v)[4]) {
  uint32_t w[3][2] = {{0, 0}, {0, 0}, {0, 0}};
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const __nv_bfloat16 t1 = __float2bfloat16(v[j]);
    const float r1 = v[j] - __bfloat162float(t1);
    const __nv_bfloat16 t2 = __float2bfloat16(r1);
    const __nv_bfloat16 t3 = __float2bfloat16(r1 - __bfloat162float(t2));
    const int sh = 16 * (j & 1);
    w[0][j >> 1] |= (uint32_t)__bfloat16_as_ushort(t1) << sh;
    w[1][j >> 1] |= (uint32_t)__bfloat16_as_ushort(t2) << sh;
    w[2][j >> 1] |= (uint32_t)__bfloat16_as_ushort(t3) << sh;
  }
  __nv_bfloat16 *row = terms + t * 3 * cols + i;
#pragma unroll
  for (int k = 0; k < 3; ++k)
    *reinterpret_cast<uint2 *>(row + (int64_t)k * cols) = make_uint2(w[k][0], w[k][1]);
}

} // namespace
} // namespace vxb

#endif /* VXB_TERMS_CUH */
