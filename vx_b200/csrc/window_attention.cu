/* window_attention.cu -- attention over a sliding window of a ring of keys that
 * serve as the values too, with the gate on its output.
 *
 * A cached position is one row per key head, read once: the row a lane holds
 * for the score is the row it adds to the weighted sum, so a step moves half
 * the bytes of attention over separate keys and values.  The ring keeps the
 * last cache_rows positions (position t in row t % cache_rows); a token at
 * position p sees p - window + 1 .. p.  Scores, weights and sums are f32.
 */
#include "kernels.h"
#include "launch.cuh"
#include "launch_util.h"
#include "nn_device.cuh"
#include "terms.cuh"

#include <cooperative_groups.h>

#include <cstdio>
#include <cstdlib>

namespace vxb {
namespace {

namespace cg = cooperative_groups;

constexpr float LOWEST = -3.0e38f;

/* ---- one new token per sequence ----------------------------------------------
 * A cluster of RUNS blocks per (sequence, key head, tile of GH query heads that
 * share it); block r takes the r-th run of the window's positions, its NW warps
 * every NW-th of them, NB rows in flight per warp. A lane holds D4 float4s of a
 * row. The warps meet in shared memory, the blocks in distributed shared memory,
 * in a fixed order. */
constexpr int RUNS = 8;

template <int GH, int D4, int NW> struct WindowShared {
  float m[NW][GH], l[NW][GH];
  __align__(16) float acc[NW][GH][D4 * 128];
};

template <int GH, int D4, int NW>
__global__ void __launch_bounds__(NW * 32)
window_decode_kernel(const WindowAttnArgs a, float *out, int64_t out_stride) {
  constexpr int NB = 8 / D4;
  __shared__ WindowShared<GH, D4, NW> sh;
  chain_release();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int hd = a.head_dim, group = a.q_heads / a.kv_heads;
  const int tiles = (group + GH - 1) / GH;
  const int g = blockIdx.y / tiles, tile = blockIdx.y - g * tiles;
  const int h0 = g * group + tile * GH, nh = min(GH, group - tile * GH);
  const int b = blockIdx.z;
  const int pos = a.positions[b];
  const int low = max(0, pos - a.window + 1);
  const int run = (pos - low + RUNS) / RUNS; /* ceil of the count over RUNS */
  const int t_begin = low + (int)blockIdx.x * run;
  const int t_end = min(t_begin + run, pos + 1);
  const int row_low = low % a.cache_rows;
  const float *cache = a.cache + b * a.cache_batch_stride + (int64_t)g * hd;
  const int64_t row_floats = (int64_t)a.kv_heads * hd;
  bool active[D4];
#pragma unroll
  for (int c = 0; c < D4; ++c)
    active[c] = (c * 32 + lane) * 4 < hd;

  float4 kv[NB][D4];
  /* Rows below pos come from earlier steps: they may be fetched before the
     kernel in front has finished. Row pos is its output. */
  auto load = [&](int t0, bool before_wait, bool after_wait) {
#pragma unroll
    for (int j = 0; j < NB; ++j) {
      const int t = t0 + j * NW;
      if (t >= t_end || (t < pos ? after_wait : before_wait))
        continue;
      int row = row_low + (t - low);
      if (row >= a.cache_rows)
        row -= a.cache_rows;
#pragma unroll
      for (int c = 0; c < D4; ++c)
        if (active[c])
          kv[j][c] = *reinterpret_cast<const float4 *>(cache + row * row_floats +
                                                       (c * 32 + lane) * 4);
    }
  };
#pragma unroll
  for (int j = 0; j < NB; ++j)
#pragma unroll
    for (int c = 0; c < D4; ++c)
      kv[j][c] = make_float4(0, 0, 0, 0);
  load(t_begin + warp, true, false);
  chain_wait();
  load(t_begin + warp, false, true);

  float4 q[GH][D4], acc[GH][D4];
  float m[GH], l[GH];
#pragma unroll
  for (int h = 0; h < GH; ++h) {
    m[h] = LOWEST;
    l[h] = 0.0f;
#pragma unroll
    for (int c = 0; c < D4; ++c) {
      acc[h][c] = q[h][c] = make_float4(0, 0, 0, 0);
      if (active[c] && h < nh)
        q[h][c] = __ldcg(reinterpret_cast<const float4 *>(
            a.q + b * a.q_stride + (int64_t)(h0 + h) * hd + (c * 32 + lane) * 4));
    }
  }
  for (int t0 = t_begin + warp; t0 < t_end; t0 += NB * NW) {
    if (t0 != t_begin + warp)
      load(t0, false, false);
#pragma unroll
    for (int h = 0; h < GH; ++h) {
      float s[NB];
#pragma unroll
      for (int j = 0; j < NB; ++j) {
        s[j] = 0.0f;
#pragma unroll
        for (int c = 0; c < D4; ++c) {
          s[j] = fmaf(q[h][c].x, kv[j][c].x, s[j]);
          s[j] = fmaf(q[h][c].y, kv[j][c].y, s[j]);
          s[j] = fmaf(q[h][c].z, kv[j][c].z, s[j]);
          s[j] = fmaf(q[h][c].w, kv[j][c].w, s[j]);
        }
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1)
#pragma unroll
        for (int j = 0; j < NB; ++j)
          s[j] += __shfl_xor_sync(0xffffffffu, s[j], o);
      float big = m[h];
#pragma unroll
      for (int j = 0; j < NB; ++j) {
        s[j] = t0 + j * NW < t_end ? s[j] * a.scale : LOWEST;
        big = fmaxf(big, s[j]);
      }
      const float fix = expf(m[h] - big);
      m[h] = big;
      l[h] *= fix;
#pragma unroll
      for (int c = 0; c < D4; ++c) {
        acc[h][c].x *= fix; acc[h][c].y *= fix;
        acc[h][c].z *= fix; acc[h][c].w *= fix;
      }
#pragma unroll
      for (int j = 0; j < NB; ++j) {
        const float w = t0 + j * NW < t_end ? expf(s[j] - big) : 0.0f;
        l[h] += w;
#pragma unroll
        for (int c = 0; c < D4; ++c)
          axpy(acc[h][c], w, kv[j][c]);
      }
    }
  }

  /* ---- the block's warps, in warp order, into row 0 of its arrays ---- */
#pragma unroll
  for (int h = 0; h < GH; ++h) {
    if (lane == 0) {
      sh.m[warp][h] = m[h];
      sh.l[warp][h] = l[h];
    }
#pragma unroll
    for (int c = 0; c < D4; ++c)
      *reinterpret_cast<float4 *>(&sh.acc[warp][h][(c * 32 + lane) * 4]) = acc[h][c];
  }
  __syncthreads();
  for (int h = warp; h < nh; h += NW) {
    float big = LOWEST;
    for (int w = 0; w < NW; ++w)
      big = fmaxf(big, sh.m[w][h]);
    float total = 0.0f;
    float4 o[D4];
#pragma unroll
    for (int c = 0; c < D4; ++c)
      o[c] = make_float4(0, 0, 0, 0);
    for (int w = 0; w < NW; ++w) {
      const float f = expf(sh.m[w][h] - big);
      total = fmaf(f, sh.l[w][h], total);
#pragma unroll
      for (int c = 0; c < D4; ++c)
        axpy(o[c], f,
             *reinterpret_cast<const float4 *>(&sh.acc[w][h][(c * 32 + lane) * 4]));
    }
    __syncwarp();
#pragma unroll
    for (int c = 0; c < D4; ++c)
      *reinterpret_cast<float4 *>(&sh.acc[0][h][(c * 32 + lane) * 4]) = o[c];
    if (lane == 0) {
      sh.m[0][h] = big;
      sh.l[0][h] = total;
    }
  }

  /* ---- block 0 merges the runs, in order; then the gate ---- */
  cg::cluster_group cluster = cg::this_cluster();
  cluster.sync();
  if (cluster.block_rank() == 0) {
    for (int h = warp; h < nh; h += NW) {
      float pm[RUNS], pl[RUNS];
      float big = LOWEST;
#pragma unroll
      for (int r = 0; r < RUNS; ++r) {
        const WindowShared<GH, D4, NW> *peer = cluster.map_shared_rank(&sh, r);
        pm[r] = peer->m[0][h];
        pl[r] = peer->l[0][h];
        big = fmaxf(big, pm[r]);
      }
      float total = 0.0f;
      float4 o[D4];
#pragma unroll
      for (int c = 0; c < D4; ++c)
        o[c] = make_float4(0, 0, 0, 0);
#pragma unroll
      for (int r = 0; r < RUNS; ++r) {
        const WindowShared<GH, D4, NW> *peer = cluster.map_shared_rank(&sh, r);
        const float f = expf(pm[r] - big);
        total = fmaf(f, pl[r], total);
#pragma unroll
        for (int c = 0; c < D4; ++c)
          axpy(o[c], f, *reinterpret_cast<const float4 *>(
                            &peer->acc[0][h][(c * 32 + lane) * 4]));
      }
#pragma unroll
      for (int c = 0; c < D4; ++c) {
        if (!active[c])
          continue;
        const int64_t at = (int64_t)(h0 + h) * hd + (c * 32 + lane) * 4;
        const float4 gt = __ldcg(
            reinterpret_cast<const float4 *>(a.gate + b * a.gate_stride + at));
        *reinterpret_cast<float4 *>(out + b * out_stride + at) =
            make_float4(o[c].x / total * gt.x, o[c].y / total * gt.y,
                        o[c].z / total * gt.z, o[c].w / total * gt.w);
      }
    }
  }
  cluster.sync(); /* nobody leaves while block 0 may still read its part */
}

/* ---- the positions of a prompt -------------------------------------------------
 * A block per (AQ positions, query head): scores against AK keys at a time,
 * online softmax, weighted sum of the same rows; 16 x 16 threads, thread (ty, tx)
 * owning AQ/16 queries ty*(AQ/16).., keys tx + 16 b and values tx*4 + 64 c ...
 * DP: head_dim rounded up to what the threads cover, zeros beyond it. */
constexpr int ROW_THREADS = 256;
constexpr int rows_smem(int DP, int AQ, int AK) {
  return ((AQ + AK) * (DP + 4) + AQ * (AK + 4)) * 4;
}

template <int DP, int AQ, int AK>
__global__ void __launch_bounds__(ROW_THREADS)
window_rows_kernel(const WindowAttnArgs a, int t_count, __nv_bfloat16 *terms,
                   int cols) {
  constexpr int QN = AQ / 16, KN = AK / 16, CN = DP / 64, D4 = DP / 4;
  extern __shared__ __align__(16) float att_smem[];
  float (*sq)[DP + 4] = reinterpret_cast<float (*)[DP + 4]>(att_smem);
  float (*sk)[DP + 4] = reinterpret_cast<float (*)[DP + 4]>(att_smem + AQ * (DP + 4));
  float (*sp)[AK + 4] =
      reinterpret_cast<float (*)[AK + 4]>(att_smem + (AQ + AK) * (DP + 4));
  chain_release();
  chain_wait();
  const int hd = a.head_dim, head = blockIdx.y;
  const int g = head / (a.q_heads / a.kv_heads);
  const int t0 = blockIdx.x * AQ, base = a.positions[0];
  const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16;

  for (int i = tid; i < AQ * D4; i += ROW_THREADS) {
    const int r = i / D4, c = i % D4 * 4;
    float4 v = make_float4(0, 0, 0, 0);
    if (t0 + r < t_count && c < hd)
      v = *reinterpret_cast<const float4 *>(a.q + (t0 + r) * a.q_stride +
                                            (int64_t)head * hd + c);
    *reinterpret_cast<float4 *>(&sq[r][c]) = v;
  }
  float m[QN], l[QN];
  float4 o[QN][CN];
#pragma unroll
  for (int i = 0; i < QN; ++i) {
    m[i] = LOWEST;
    l[i] = 0.0f;
#pragma unroll
    for (int c = 0; c < CN; ++c)
      o[i][c] = make_float4(0, 0, 0, 0);
  }
  const int first_key = max(0, base + t0 - a.window + 1);
  const int last_key = base + min(t0 + AQ, t_count) - 1;
  for (int k0 = first_key; k0 <= last_key; k0 += AK) {
    const int row0 = k0 % a.cache_rows;
    __syncthreads(); /* the tiles of the round before are done with */
    for (int i = tid; i < AK * D4; i += ROW_THREADS) {
      const int r = i / D4, c = i % D4 * 4;
      float4 v = make_float4(0, 0, 0, 0);
      if (k0 + r <= last_key && c < hd) {
        int row = row0 + r;
        if (row >= a.cache_rows)
          row -= a.cache_rows;
        v = *reinterpret_cast<const float4 *>(
            a.cache + ((int64_t)row * a.kv_heads + g) * hd + c);
      }
      *reinterpret_cast<float4 *>(&sk[r][c]) = v;
    }
    __syncthreads();
    float s[QN][KN];
#pragma unroll
    for (int i = 0; i < QN; ++i)
#pragma unroll
      for (int j = 0; j < KN; ++j)
        s[i][j] = 0.0f;
    for (int d = 0; d < hd; d += 4) {
      float4 qv[QN], kv[KN];
#pragma unroll
      for (int i = 0; i < QN; ++i)
        qv[i] = *reinterpret_cast<const float4 *>(&sq[ty * QN + i][d]);
#pragma unroll
      for (int j = 0; j < KN; ++j)
        kv[j] = *reinterpret_cast<const float4 *>(&sk[tx + 16 * j][d]);
#pragma unroll
      for (int i = 0; i < QN; ++i)
#pragma unroll
        for (int j = 0; j < KN; ++j) {
          s[i][j] = fmaf(qv[i].x, kv[j].x, s[i][j]);
          s[i][j] = fmaf(qv[i].y, kv[j].y, s[i][j]);
          s[i][j] = fmaf(qv[i].z, kv[j].z, s[i][j]);
          s[i][j] = fmaf(qv[i].w, kv[j].w, s[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < QN; ++i) {
      const int at = base + t0 + ty * QN + i;
      bool seen[KN];
      float big = LOWEST;
#pragma unroll
      for (int j = 0; j < KN; ++j) {
        const int behind = at - (k0 + tx + 16 * j);
        seen[j] = behind >= 0 && behind < a.window;
        s[i][j] = seen[j] ? s[i][j] * a.scale : LOWEST;
        big = fmaxf(big, s[i][j]);
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1)
        big = fmaxf(big, __shfl_xor_sync(0xffffffffu, big, off));
      const float mn = fmaxf(m[i], big);
      const float fix = expf(m[i] - mn);
      float sum = 0.0f;
#pragma unroll
      for (int j = 0; j < KN; ++j) {
        const float w = seen[j] ? expf(s[i][j] - mn) : 0.0f;
        sp[ty * QN + i][tx + 16 * j] = w;
        sum += w;
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1)
        sum += __shfl_xor_sync(0xffffffffu, sum, off);
      l[i] = l[i] * fix + sum;
      m[i] = mn;
#pragma unroll
      for (int c = 0; c < CN; ++c) {
        o[i][c].x *= fix; o[i][c].y *= fix;
        o[i][c].z *= fix; o[i][c].w *= fix;
      }
    }
    __syncwarp(); /* a query's weights stay within the half warp that made them */
    for (int k = 0; k < AK; k += 4) {
      float4 w[QN];
#pragma unroll
      for (int i = 0; i < QN; ++i)
        w[i] = *reinterpret_cast<const float4 *>(&sp[ty * QN + i][k]);
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int c = 0; c < CN; ++c) {
          const float4 v =
              *reinterpret_cast<const float4 *>(&sk[k + j][tx * 4 + 64 * c]);
#pragma unroll
          for (int i = 0; i < QN; ++i)
            axpy(o[i][c], j == 0 ? w[i].x : j == 1 ? w[i].y : j == 2 ? w[i].z : w[i].w,
                 v);
        }
    }
  }
#pragma unroll
  for (int i = 0; i < QN; ++i) {
    const int t = t0 + ty * QN + i;
    if (t >= t_count)
      continue;
#pragma unroll
    for (int c = 0; c < CN; ++c) {
      const int d = tx * 4 + 64 * c;
      if (d >= hd)
        continue;
      const int at = head * hd + d;
      const float4 gt =
          *reinterpret_cast<const float4 *>(a.gate + t * a.gate_stride + at);
      const float v[4] = {o[i][c].x / l[i] * gt.x, o[i][c].y / l[i] * gt.y,
                          o[i][c].z / l[i] * gt.z, o[i][c].w / l[i] * gt.w};
      store_terms4(terms, cols, t, at, v);
    }
  }
}

const char *refuse(const WindowAttnArgs &a) {
  if (a.head_dim % 4 != 0 || a.head_dim < 4 || a.head_dim > 512)
    return "head_dim must be a multiple of 4, and at most 512";
  if (a.kv_heads < 1 || a.q_heads % a.kv_heads != 0)
    return "q_heads must be a multiple of kv_heads";
  if (a.window < 1 || a.cache_rows < 1)
    return "a window holds at least its own token";
  if (((uintptr_t)a.q | (uintptr_t)a.cache | (uintptr_t)a.gate) & 15 ||
      (a.q_stride | a.gate_stride | a.cache_batch_stride) % 4 != 0)
    return "q, the ring and the gate must be 16-byte aligned";
  return nullptr;
}

template <int GH, int D4>
void launch_decode(const WindowAttnArgs &a, dim3 grid, float *out, int64_t out_stride,
                   cudaStream_t stream) {
  const int64_t blocks = (int64_t)grid.x * grid.y * grid.z;
  auto go = [&](auto kernel, int warps) {
    launch_chained_cluster(kernel, grid, dim3(warps * 32), RUNS, stream, a, out,
                           out_stride);
  };
  /* few blocks: more warps each, so that a window is a trip or two to memory */
  int warps = 2 * blocks <= sm_count() ? 16 : (blocks <= 2 * sm_count() ? 8 : 4);
  /* VXB_ATTN_WARPS=4, 8 or 16 pins it (for measurements) */
  if (const char *pin = getenv("VXB_ATTN_WARPS")) {
    const int v = atoi(pin);
    if (v == 4 || v == 8 || v == 16)
      warps = v;
  }
  /* long rows take more shared memory per warp */
  constexpr int most = 16 / D4;
  if (warps == 16 && most >= 16)
    go(window_decode_kernel<GH, D4, most >= 16 ? 16 : 4>, 16);
  else if (warps >= 8 && most >= 8)
    go(window_decode_kernel<GH, D4, most >= 8 ? 8 : 4>, 8);
  else
    go(window_decode_kernel<GH, D4, 4>, 4);
}

template <int GH>
void launch_decode_dim(const WindowAttnArgs &a, dim3 grid, float *out,
                       int64_t out_stride, cudaStream_t stream) {
  if (a.head_dim <= 128)
    launch_decode<GH, 1>(a, grid, out, out_stride, stream);
  else if (a.head_dim <= 256)
    launch_decode<GH, 2>(a, grid, out, out_stride, stream);
  else
    launch_decode<GH, 4>(a, grid, out, out_stride, stream);
}

template <int DP, int AQ, int AK>
const char *launch_rows(const WindowAttnArgs &a, int t, __nv_bfloat16 *terms, int cols,
                        cudaStream_t stream) {
  constexpr int smem = rows_smem(DP, AQ, AK);
  if (allow_dynamic_smem((const void *)window_rows_kernel<DP, AQ, AK>, smem) !=
      cudaSuccess)
    return "the multi-position window attention could not get its shared memory";
  launch_chained(window_rows_kernel<DP, AQ, AK>, dim3((t + AQ - 1) / AQ, a.q_heads),
                 dim3(ROW_THREADS), smem, stream, a, t, terms, cols);
  return check_launch("the multi-position window attention");
}

} // namespace

const char *window_attention_decode(const WindowAttnArgs &a, int batch, float *out,
                                    int64_t out_stride, cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  if (a.cache_rows < a.window)
    return "the ring must hold a window";
  if (((uintptr_t)out & 15) || out_stride % 4 != 0)
    return "the output must be 16-byte aligned";
  const int group = a.q_heads / a.kv_heads;
  const int gh = group >= 4 ? 4 : (group >= 2 ? 2 : 1);
  const dim3 grid(RUNS, a.kv_heads * ((group + gh - 1) / gh), batch);
  if (gh == 4)
    launch_decode_dim<4>(a, grid, out, out_stride, stream);
  else if (gh == 2)
    launch_decode_dim<2>(a, grid, out, out_stride, stream);
  else
    launch_decode_dim<1>(a, grid, out, out_stride, stream);
  return check_launch("the window attention launch");
}

const char *window_attention_rows(const WindowAttnArgs &a, int t, void *terms,
                                  int cols, cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  if (cols % 4 != 0 || cols < a.q_heads * a.head_dim)
    return "the output has too few columns";
  __nv_bfloat16 *to = (__nv_bfloat16 *)terms;
  if (a.head_dim <= 64)
    return launch_rows<64, 64, 64>(a, t, to, cols, stream);
  if (a.head_dim <= 128)
    return launch_rows<128, 64, 64>(a, t, to, cols, stream);
  if (a.head_dim <= 256)
    return launch_rows<256, 64, 64>(a, t, to, cols, stream);
  return launch_rows<512, 32, 32>(a, t, to, cols, stream);
}

} // namespace vxb
