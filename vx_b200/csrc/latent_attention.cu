/* latent_attention.cu -- attention whose keys and values are products of one latent
 * per position, over a sliding window of a ring of latents.
 *
 * A step never makes a key or a value: a head's query goes through its key matrix
 * once (q W_uk is a query for the latents themselves), the softmax weighs latents, and
 * the sum goes through the head's value matrix; both products happen in the attention
 * kernel, split over the blocks of a cluster.  All heads read one row per position, so
 * a step moves kv_rank + rot values per position instead of heads * (dim + vdim).
 * Over the positions of a prompt the latents are worth expanding: keys and values of
 * the window are made by one GEMM, and a score costs dim + rot multiplications, not
 * kv_rank + rot.  Scores, weights and sums are f32.
 */
#include "kernels.h"
#include "launch.cuh"
#include "launch_util.h"
#include "nn_device.cuh"
#include "terms.cuh"

#include <cooperative_groups.h>

namespace vxb {
namespace {

namespace cg = cooperative_groups;

constexpr float LOWEST = -3.0e38f;

/* ---- one new token per sequence ----------------------------------------------
 * A cluster of CL blocks per (sequence, tile of GH heads); block r takes the r-th run
 * of the window's positions and the r-th part of the two products' rows, its NW warps
 * every NW-th position. A warp's rows come through SLOTS shared-memory slots of its
 * own, filled by bulk copies that it asks for ahead (all of them before the wait for
 * the kernel in front, since earlier steps wrote them), NB rows at a time into
 * registers, D4 float4s a lane. Warps and blocks meet in a fixed order. */
constexpr int CL = 8;
__host__ __device__ constexpr int row_slots(int D4) { return D4 <= 2 ? 8 : 4; }

/* floats of dynamic shared memory */
constexpr int latent_smem(int GH, int D4, int NW, int dim, int kv_rank) {
  return (NW * row_slots(D4) + GH + 1) * D4 * 128 + GH * dim + GH * kv_rank / CL;
}

__device__ int g_latent_status; /* 0x61: a row of the ring never arrived */

__device__ __forceinline__ float dot_word(const uint4 &w, const float *x,
                                          const __nv_bfloat16 *) {
  const float4 a = *reinterpret_cast<const float4 *>(x);
  const float4 b = *reinterpret_cast<const float4 *>(x + 4);
  float s = bf_lo(w.x) * a.x;
  s = fmaf(bf_hi(w.x), a.y, s);
  s = fmaf(bf_lo(w.y), a.z, s);
  s = fmaf(bf_hi(w.y), a.w, s);
  s = fmaf(bf_lo(w.z), b.x, s);
  s = fmaf(bf_hi(w.z), b.y, s);
  s = fmaf(bf_lo(w.w), b.z, s);
  return fmaf(bf_hi(w.w), b.w, s);
}
__device__ __forceinline__ float dot_word(const uint4 &w, const float *x, const float *) {
  const float4 a = *reinterpret_cast<const float4 *>(x);
  float s = __uint_as_float(w.x) * a.x;
  s = fmaf(__uint_as_float(w.y), a.y, s);
  s = fmaf(__uint_as_float(w.z), a.z, s);
  return fmaf(__uint_as_float(w.w), a.w, s);
}

/* y[r] = w[r] . x for `rows` rows of `cols` values, r taken in turn by the WARPS warps
   of which this one is the `warp`-th; x in shared memory, put(r, y) takes a result. As
   many lanes as a row has words take one, U rows of each such group are in flight. */
template <typename W, int WARPS, typename Put>
__device__ __forceinline__ void warp_dots(const W *w, int rows, int cols, const float *x,
                                          int warp, Put put) {
  constexpr int E = 16 / (int)sizeof(W), U = 4;
  const int lane = threadIdx.x & 31;
  const int words = cols / E;
  int lanes = 32;
  while (lanes > 1 && lanes / 2 >= words)
    lanes /= 2;
  const int groups = 32 / lanes, group = lane / lanes, first = lane % lanes;
  const int step = WARPS * groups;
#pragma unroll 1
  for (int r0 = warp * groups + group; r0 - group < rows; r0 += step * U) {
    const uint4 *at = reinterpret_cast<const uint4 *>(w) + (int64_t)r0 * words;
    float s[U];
#pragma unroll
    for (int u = 0; u < U; ++u)
      s[u] = 0.0f;
#pragma unroll 1
    for (int wd = first; wd < words; wd += lanes) {
      uint4 word[U];
#pragma unroll
      for (int u = 0; u < U; ++u)
        word[u] = r0 + u * step < rows ? __ldg(at + u * step * words + wd)
                                       : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int u = 0; u < U; ++u)
        s[u] += dot_word(word[u], x + wd * E, (const W *)nullptr);
    }
    for (int o = lanes / 2; o > 0; o >>= 1)
#pragma unroll
      for (int u = 0; u < U; ++u)
        s[u] += __shfl_xor_sync(0xffffffffu, s[u], o);
#pragma unroll
    for (int u = 0; u < U; ++u)
      if (first == 0 && r0 + u * step < rows)
        put(r0 + u * step, s[u]);
  }
}

template <typename W, int GH, int D4, int NW>
__global__ void __launch_bounds__(NW * 32, D4 <= 5 ? 2 : 1)
latent_decode_kernel(const LatentArgs a, const float *q_in, int64_t q_stride,
                     const float *down, int64_t down_stride, float *out,
                     int64_t out_stride) {
  constexpr int NB = D4 <= 2 ? 4 : D4 <= 5 ? 2 : 1;
  constexpr int WPH = NW / GH; /* warps a head, in the two products */
  constexpr int THREADS = NW * 32, ROW = D4 * 128, SLOTS = row_slots(D4);
  extern __shared__ __align__(128) float latent_shared[];
  float *slots_s = latent_shared; /* [NW][SLOTS][ROW]; the first GH then hold a warp's sums */
  float *heads_s = slots_s + NW * SLOTS * ROW; /* [GH][ROW]: queries, then weighted latents */
  float *fresh = heads_s + GH * ROW;    /* [ROW]: this position's row */
  float *qn = fresh + ROW;              /* [GH][dim] */
  float *slice = qn + GH * a.dim;       /* [GH][kv_rank / CL] */
  __shared__ float warp_m[NW][GH], warp_l[NW][GH], red[NW];
  __shared__ float block_m[GH], block_l[GH], share[GH][CL];
  __shared__ __align__(8) uint64_t bars[NW][SLOTS];
  cg::cluster_group cluster = cg::this_cluster();
  chain_release();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  static_assert(GH <= SLOTS && NW % GH == 0, "a warp's sums fit its slots");
  const int rank = blockIdx.x, h0 = blockIdx.y * GH, b = blockIdx.z;
  const int nh = min(GH, a.heads - h0);
  const int K = a.kv_rank, part = K / CL, row_floats = K + a.rot;
  const int v_part = (a.vdim + CL - 1) / CL, v0 = min(rank * v_part, a.vdim),
            vn = min(v_part, a.vdim - v0);
  const W *uk = (const W *)a.w_uk_t, *ukv = (const W *)a.w_ukv;
  auto uk_row = [&](int g, int r) {
    return uk + ((int64_t)(h0 + g) * K + rank * part + r) * a.dim;
  };
  auto uv_row = [&](int g, int r) {
    return ukv + ((int64_t)(h0 + g) * (a.dim + a.vdim) + a.dim + v0 + r) * K;
  };
  /* what depends on no kernel before: the matrices on their way to L2 */
  if (tid < nh) {
    ptx::bulk_prefetch_l2(uk_row(tid, 0), part * a.dim * (int)sizeof(W));
    if (vn > 0)
      ptx::bulk_prefetch_l2(uv_row(tid, 0), vn * K * (int)sizeof(W));
  }
  const int pos = a.positions[b];
  const int low = max(0, pos - a.window + 1);
  const int run = (pos - low + CL) / CL; /* ceil of the count over CL */
  const int t_begin = low + rank * run, t_end = min(t_begin + run, pos + 1);
  const int row_low = low % a.cache_rows;
  float *ring = a.ring + b * a.ring_batch_stride;
  bool active[D4];
#pragma unroll
  for (int c = 0; c < D4; ++c)
    active[c] = (c * 32 + lane) * 4 < row_floats;

  /* Rows below pos come from earlier steps; row pos is made here. This warp's rows are
     t_begin + warp + j NW, `have` of them in the ring. */
  const int mine = t_begin + warp;
  const int have = max(0, (min(t_end, pos) - mine + NW - 1) / NW);
  float *my_slots = slots_s + warp * SLOTS * ROW;
  auto ask = [&](int j) { /* lane 0 */
    int row = row_low + (mine + j * NW - low);
    if (row >= a.cache_rows)
      row -= a.cache_rows;
    uint64_t *bar = &bars[warp][j % SLOTS];
    ptx::mbar_expect_tx(bar, row_floats * (int)sizeof(float));
    ptx::bulk_load(my_slots + j % SLOTS * ROW, ring + (int64_t)row * row_floats,
                   row_floats * (int)sizeof(float), bar);
  };
  if (lane == 0) {
    for (int k = 0; k < SLOTS; ++k)
      ptx::mbar_init(&bars[warp][k], 1);
    ptx::fence_proxy_async_smem();
    ptx::fence_barrier_init();
    for (int j = 0; j < min(SLOTS, have); ++j)
      ask(j);
  }
  __syncwarp();
  chain_wait();

  /* ---- this position's row; the queries, rotated; what fills rows up ---- */
  for (int i = row_floats + tid; i < ROW; i += THREADS)
#pragma unroll
    for (int h = 0; h <= GH; ++h) /* fresh follows the heads */
      heads_s[h * ROW + i] = 0.0f;
  const float *dn = down + b * down_stride;
  const float *q = q_in + b * q_stride + (int64_t)h0 * (a.dim + a.rot);
  float ss = 0.0f;
  for (int i = tid; i < K; i += THREADS) {
    const float v = dn[i];
    fresh[i] = v;
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if (lane == 0)
    red[warp] = ss;
  for (int i = tid; i < nh * a.dim; i += THREADS) {
    const int g = i / a.dim;
    qn[i] = q[g * (a.dim + a.rot) + i - g * a.dim];
  }
  const int pairs = a.rot / 2;
  for (int i = tid; i < (nh + 1) * pairs; i += THREADS) {
    const int g = i / pairs, k = i - g * pairs; /* g == nh: the key */
    const float2 uv = *reinterpret_cast<const float2 *>(
        (g < nh ? q + g * (a.dim + a.rot) + a.dim : dn + K) + 2 * k);
    float sine, cosine;
    turned(pos, a.turns[k], sine, cosine);
    float *to = (g < nh ? heads_s + g * ROW : fresh) + K + 2 * k;
    to[0] = uv.x * cosine - uv.y * sine;
    to[1] = uv.y * cosine + uv.x * sine;
  }
  __syncthreads();
  float total = 0.0f;
  for (int w = 0; w < NW; ++w) /* fixed order */
    total += red[w];
  const float inv = 1.0f / sqrtf(total / (float)a.kv_mean + a.eps);
  for (int i = tid; i < K; i += THREADS)
    fresh[i] = fresh[i] * inv * a.gain[i];

  /* ---- the queries for latents: this block's part of each, then all parts ---- */
  const int g_mine = warp % GH; /* the head whose products this warp takes part in */
  if (g_mine < nh)
    warp_dots<W, WPH>(uk_row(g_mine, 0), part, a.dim, qn + g_mine * a.dim, warp / GH,
                      [&](int r, float y) { slice[g_mine * part + r] = y; });
  auto gather = [&] {
    for (int i = tid; i < nh * K / 4; i += THREADS) {
      const int g = i / (K / 4), c = (i - g * (K / 4)) * 4, r = c / part;
      *reinterpret_cast<float4 *>(heads_s + g * ROW + c) =
          *reinterpret_cast<const float4 *>(cluster.map_shared_rank(slice, r) +
                                            g * part + c - r * part);
    }
  };
  cluster.sync();
  gather();
  __syncthreads();
  if (blockIdx.y == 0 && rank == 0) {
    float *to = ring + (int64_t)(pos % a.cache_rows) * row_floats;
    for (int i = tid; i < row_floats; i += THREADS)
      to[i] = fresh[i];
  }
  float2 acc[GH][D4][2];
  float m[GH], l[GH];
#pragma unroll
  for (int h = 0; h < GH; ++h) {
    m[h] = LOWEST;
    l[h] = 0.0f;
#pragma unroll
    for (int c = 0; c < D4; ++c)
      acc[h][c][0] = acc[h][c][1] = make_float2(0, 0);
  }
  bool arrived = true;
  for (int j0 = 0; mine + j0 * NW < t_end; j0 += NB) {
    const int t0 = mine + j0 * NW;
    float4 kv[NB][D4];
#pragma unroll
    for (int k = 0; k < NB; ++k) {
      const int j = j0 + k, slot = j % SLOTS;
      const float *src = fresh;
      if (j < have) {
        uint64_t *bar = &bars[warp][slot];
        const uint32_t phase = (j / SLOTS) & 1;
        arrived = arrived && __all_sync(0xffffffffu, ptx::mbar_try_wait(bar, phase) ||
                                                         ptx::mbar_wait_alone(bar, phase));
        src = my_slots + slot * ROW;
      }
#pragma unroll
      for (int c = 0; c < D4; ++c)
        kv[k][c] = active[c] && t0 + k * NW < t_end
                       ? *reinterpret_cast<const float4 *>(src + (c * 32 + lane) * 4)
                       : make_float4(0, 0, 0, 0);
    }
    if (!arrived) {
      atomicCAS(&g_latent_status, 0, 0x61);
      for (int j = j0; j < min(j0 + SLOTS, have); ++j) /* what is still on its way */
        ptx::mbar_wait_alone(&bars[warp][j % SLOTS], (j / SLOTS) & 1);
      break;
    }
    __syncwarp(); /* every lane has the rows: their slots may be filled again */
    if (lane == 0)
      for (int j = j0 + SLOTS; j < min(j0 + NB + SLOTS, have); ++j)
        ask(j);
    float s[GH][NB];
#pragma unroll
    for (int h = 0; h < GH; ++h) {
      float2 d[NB];
#pragma unroll
      for (int k = 0; k < NB; ++k)
        d[k] = make_float2(0, 0);
#pragma unroll
      for (int c = 0; c < D4; ++c) {
        const float4 q4 =
            *reinterpret_cast<const float4 *>(heads_s + h * ROW + (c * 32 + lane) * 4);
#pragma unroll
        for (int k = 0; k < NB; ++k) {
          fma_pair(d[k], make_float2(q4.x, q4.y), make_float2(kv[k][c].x, kv[k][c].y));
          fma_pair(d[k], make_float2(q4.z, q4.w), make_float2(kv[k][c].z, kv[k][c].w));
        }
      }
#pragma unroll
      for (int k = 0; k < NB; ++k)
        s[h][k] = d[k].x + d[k].y;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1)
#pragma unroll
      for (int h = 0; h < GH; ++h)
#pragma unroll
        for (int k = 0; k < NB; ++k)
          s[h][k] += __shfl_xor_sync(0xffffffffu, s[h][k], o);
#pragma unroll
    for (int h = 0; h < GH; ++h) {
      float big = m[h];
#pragma unroll
      for (int k = 0; k < NB; ++k) {
        s[h][k] = t0 + k * NW < t_end ? s[h][k] * a.scale : LOWEST;
        big = fmaxf(big, s[h][k]);
      }
      const float fix = expf(m[h] - big);
      m[h] = big;
      l[h] *= fix;
      float w[NB];
#pragma unroll
      for (int k = 0; k < NB; ++k) {
        w[k] = t0 + k * NW < t_end ? expf(s[h][k] - big) : 0.0f;
        l[h] += w[k];
      }
#pragma unroll
      for (int c = 0; c < D4; ++c) {
        acc[h][c][0] = mul_pair(acc[h][c][0], make_float2(fix, fix));
        acc[h][c][1] = mul_pair(acc[h][c][1], make_float2(fix, fix));
#pragma unroll
        for (int k = 0; k < NB; ++k) {
          fma_pair(acc[h][c][0], make_float2(w[k], w[k]),
                   make_float2(kv[k][c].x, kv[k][c].y));
          fma_pair(acc[h][c][1], make_float2(w[k], w[k]),
                   make_float2(kv[k][c].z, kv[k][c].w));
        }
      }
    }
  }

  /* ---- the block's warps, in warp order, into row 0 of its arrays ---- */
#pragma unroll
  for (int h = 0; h < GH; ++h) {
    if (lane == 0) {
      warp_m[warp][h] = m[h];
      warp_l[warp][h] = l[h];
    }
#pragma unroll
    for (int c = 0; c < D4; ++c)
      *reinterpret_cast<float4 *>(my_slots + h * ROW + (c * 32 + lane) * 4) =
          make_float4(acc[h][c][0].x, acc[h][c][0].y, acc[h][c][1].x, acc[h][c][1].y);
  }
  __syncthreads();
  for (int i = warp; i < nh * D4; i += NW) {
    const int h = i / D4, c = i - h * D4;
    float big = LOWEST;
    for (int w = 0; w < NW; ++w)
      big = fmaxf(big, warp_m[w][h]);
    float sum = 0.0f;
    float4 o = make_float4(0, 0, 0, 0);
    for (int w = 0; w < NW; ++w) {
      const float f = expf(warp_m[w][h] - big);
      sum = fmaf(f, warp_l[w][h], sum);
      axpy(o, f,
           *reinterpret_cast<const float4 *>(slots_s + (w * SLOTS + h) * ROW +
                                             (c * 32 + lane) * 4));
    }
    *reinterpret_cast<float4 *>(slots_s + h * ROW + (c * 32 + lane) * 4) = o;
    if (lane == 0 && c == 0) {
      block_m[h] = big;
      block_l[h] = sum;
    }
  }

  /* ---- the runs, in order: each block its part of the latents, then all parts ---- */
  cluster.sync();
  if (tid < nh) {
    float pm[CL], big = LOWEST, sum = 0.0f;
#pragma unroll
    for (int r = 0; r < CL; ++r) {
      pm[r] = cluster.map_shared_rank(block_m, r)[tid];
      big = fmaxf(big, pm[r]);
    }
#pragma unroll
    for (int r = 0; r < CL; ++r) {
      pm[r] = expf(pm[r] - big);
      sum = fmaf(pm[r], cluster.map_shared_rank(block_l, r)[tid], sum);
    }
#pragma unroll
    for (int r = 0; r < CL; ++r)
      share[tid][r] = pm[r] / sum;
  }
  __syncthreads();
  for (int i = tid; i < nh * part / 4; i += THREADS) {
    const int g = i / (part / 4), c = (i - g * (part / 4)) * 4;
    float4 o = make_float4(0, 0, 0, 0);
#pragma unroll
    for (int r = 0; r < CL; ++r)
      axpy(o, share[g][r],
           *reinterpret_cast<const float4 *>(cluster.map_shared_rank(slots_s, r) + g * ROW +
                                             rank * part + c));
    *reinterpret_cast<float4 *>(slice + g * part + c) = o;
  }
  cluster.sync();
  gather();
  cluster.barrier_arrive(); /* nobody leaves while a peer may still read its part */
  __syncthreads();

  /* ---- through the value matrix ---- */
  if (vn > 0 && g_mine < nh)
    warp_dots<W, WPH>(uv_row(g_mine, 0), vn, K, heads_s + g_mine * ROW, warp / GH,
                      [&](int r, float y) {
                        out[b * out_stride + (int64_t)(h0 + g_mine) * a.vdim + v0 + r] = y;
                      });
  cluster.barrier_wait();
}

/* ---- the positions of a prompt: the ring's rows and the query latent -------------
 * A block is a position. */
__global__ void __launch_bounds__(256, 6)
latent_down_kernel(const LatentArgs a, const float *partials, int splits, int t_count,
                   int q_rank, const float *q_gain, int q_mean, __nv_bfloat16 *terms) {
  extern __shared__ __align__(16) float down_row[]; /* [q_rank + kv_rank] */
  __shared__ float red[2][8];
  const int64_t t = blockIdx.x;
  const int tid = threadIdx.x, K = a.kv_rank, both = q_rank + K, n = both + a.rot;
  const int pos = a.positions[0] + (int)t;
  float *ring = a.ring + (int64_t)(pos % a.cache_rows) * (K + a.rot);
  float sq = 0.0f, sk = 0.0f;
  for (int i = tid * 4; i < both; i += 1024) {
    const float4 v = sum_runs4(partials, splits, t_count, n, t, i);
    *reinterpret_cast<float4 *>(down_row + i) = v;
    float &ss = i < q_rank ? sq : sk;
    ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if ((tid & 31) == 0) {
    red[0][tid >> 5] = sq;
    red[1][tid >> 5] = sk;
  }
  __syncthreads();
  sq = sk = 0.0f;
  for (int w = 0; w < 8; ++w) { /* fixed order */
    sq += red[0][w];
    sk += red[1][w];
  }
  const float q_inv = 1.0f / sqrtf(sq / (float)q_mean + a.eps);
  const float k_inv = 1.0f / sqrtf(sk / (float)a.kv_mean + a.eps);
  for (int i = tid * 4; i < both; i += 1024) {
    const float4 v = *reinterpret_cast<const float4 *>(down_row + i);
    const bool of_q = i < q_rank;
    const float4 g = *reinterpret_cast<const float4 *>(of_q ? q_gain + i
                                                            : a.gain + i - q_rank);
    const float inv = of_q ? q_inv : k_inv;
    const float out[4] = {v.x * inv * g.x, v.y * inv * g.y, v.z * inv * g.z,
                          v.w * inv * g.w};
    if (of_q)
      store_terms4(terms, q_rank, t, i, out);
    else
      *reinterpret_cast<float4 *>(ring + i - q_rank) =
          make_float4(out[0], out[1], out[2], out[3]);
  }
  /* the rotated part, by the warps that have least of the rest */
  for (int k = 255 - tid; k < a.rot / 2; k += 256) {
    const float u = sum_runs(partials, splits, t_count, n, t, both + 2 * k);
    const float v = sum_runs(partials, splits, t_count, n, t, both + 2 * k + 1);
    float sine, cosine;
    turned(pos, a.turns[k], sine, cosine);
    ring[K + 2 * k] = u * cosine - v * sine;
    ring[K + 2 * k + 1] = v * cosine + u * sine;
  }
}

/* a thread per (position, four values of a head) */
__global__ void __launch_bounds__(256)
latent_q_kernel(const LatentArgs a, const float *partials, int splits, int t_count,
                float *q) {
  const int hd = a.dim + a.rot, n = a.heads * hd;
  const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (int64_t)t_count * (n / 4))
    return;
  const int64_t t = idx / (n / 4);
  const int r = (int)(idx - t * (n / 4)) * 4, d = r % hd;
  float4 v = sum_runs4(partials, splits, t_count, n, t, r);
  if (d >= a.dim) {
    const int pos = a.positions[0] + (int)t, k = (d - a.dim) / 2;
    float s0, c0, s1, c1;
    turned(pos, a.turns[k], s0, c0);
    turned(pos, a.turns[k + 1], s1, c1);
    v = make_float4(v.x * c0 - v.y * s0, v.y * c0 + v.x * s0, v.z * c1 - v.w * s1,
                    v.w * c1 + v.z * s1);
  }
  *reinterpret_cast<float4 *>(q + t * n + r) = v;
}

/* a thread per (position, eight values of its latent) */
__global__ void __launch_bounds__(256)
latent_gather_kernel(const LatentArgs a, int first, int n, __nv_bfloat16 *terms) {
  const int per_row = a.kv_rank / 8;
  const int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (idx >= (int64_t)n * per_row)
    return;
  const int64_t t = idx / per_row;
  const int c = (int)(idx - t * per_row) * 8;
  const float *row =
      a.ring + (first + t) % a.cache_rows * (int64_t)(a.kv_rank + a.rot) + c;
  const float4 lo = *reinterpret_cast<const float4 *>(row);
  const float4 hi = *reinterpret_cast<const float4 *>(row + 4);
  const float v[8] = {lo.x, lo.y, lo.z, lo.w, hi.x, hi.y, hi.z, hi.w};
  store_terms8(terms, a.kv_rank, t, c, v);
}

/* ---- the positions of a prompt: attention -----------------------------------------
 * A block per (AQ positions, head): scores against AK keys at a time, online softmax,
 * weighted sum; 16 x 16 threads, thread (ty, tx) owning AQ / 16 queries, keys
 * tx + 16 j and values tx * 4 + 64 c ... KP, VP: key and value sizes rounded up to
 * what the threads cover, zeros beyond them. Two neighbouring values go through a
 * multiply-add together. */
constexpr int ROW_THREADS = 256;
constexpr int rows_smem(int KP, int VP, int AQ, int AK) {
  return ((AQ + AK) * (KP + 4) + AK * (VP + 4) + AQ * (AK + 4)) * 4;
}

template <int KP, int VP, int AQ, int AK>
__global__ void __launch_bounds__(ROW_THREADS)
latent_rows_kernel(const LatentArgs a, const float *q, const float *kv, int first,
                   int t_count, __nv_bfloat16 *terms, int cols) {
  constexpr int QN = AQ / 16, KN = AK / 16, CN = VP / 64;
  extern __shared__ __align__(16) float att_smem[];
  float (*sq)[KP + 4] = reinterpret_cast<float (*)[KP + 4]>(att_smem);
  float (*sk)[KP + 4] = sq + AQ;
  float (*sv)[VP + 4] = reinterpret_cast<float (*)[VP + 4]>(sk + AK);
  float (*sp)[AK + 4] = reinterpret_cast<float (*)[AK + 4]>(sv + AK);
  const int dim = a.dim, hd = a.dim + a.rot, vdim = a.vdim, head = blockIdx.y;
  const int t0 = blockIdx.x * AQ, base = a.positions[0];
  const int tid = threadIdx.x, ty = tid / 16, tx = tid % 16;
  const int row_floats = a.kv_rank + a.rot;
  const int64_t kv_stride = (int64_t)a.heads * (dim + vdim);
  const float4 zero = make_float4(0, 0, 0, 0);

  for (int i = tid; i < AQ * (KP / 4); i += ROW_THREADS) {
    const int r = i / (KP / 4), c = i % (KP / 4) * 4;
    float4 v = zero;
    if (t0 + r < t_count && c < hd)
      v = *reinterpret_cast<const float4 *>(
          q + ((int64_t)(t0 + r) * a.heads + head) * hd + c);
    *reinterpret_cast<float4 *>(&sq[r][c]) = v;
  }
  float m[QN], l[QN];
  float2 o[QN][CN][2];
#pragma unroll
  for (int i = 0; i < QN; ++i) {
    m[i] = LOWEST;
    l[i] = 0.0f;
#pragma unroll
    for (int c = 0; c < CN; ++c)
      o[i][c][0] = o[i][c][1] = make_float2(0, 0);
  }
  const int first_key = max(0, base + t0 - a.window + 1);
  const int last_key = base + min(t0 + AQ, t_count) - 1;
  for (int k0 = first_key; k0 <= last_key; k0 += AK) {
    const int row0 = k0 % a.cache_rows;
    __syncthreads(); /* the tiles of the round before are done with */
    for (int i = tid; i < AK * (KP / 4); i += ROW_THREADS) {
      const int r = i / (KP / 4), c = i % (KP / 4) * 4;
      float4 v = zero;
      if (k0 + r <= last_key && c < hd) {
        int row = row0 + r;
        if (row >= a.cache_rows)
          row -= a.cache_rows;
        v = *reinterpret_cast<const float4 *>(
            c < dim ? kv + (k0 + r - first) * kv_stride + head * (dim + vdim) + c
                    : a.ring + (int64_t)row * row_floats + a.kv_rank + c - dim);
      }
      *reinterpret_cast<float4 *>(&sk[r][c]) = v;
    }
    for (int i = tid; i < AK * (VP / 4); i += ROW_THREADS) {
      const int r = i / (VP / 4), c = i % (VP / 4) * 4;
      float4 v = zero;
      if (k0 + r <= last_key && c < vdim)
        v = *reinterpret_cast<const float4 *>(kv + (k0 + r - first) * kv_stride +
                                              head * (dim + vdim) + dim + c);
      *reinterpret_cast<float4 *>(&sv[r][c]) = v;
    }
    __syncthreads();
    float2 s2[QN][KN];
#pragma unroll
    for (int i = 0; i < QN; ++i)
#pragma unroll
      for (int j = 0; j < KN; ++j)
        s2[i][j] = make_float2(0, 0);
#pragma unroll 2
    for (int d = 0; d < hd; d += 4) {
      float4 qv[QN], kq[KN];
#pragma unroll
      for (int i = 0; i < QN; ++i)
        qv[i] = *reinterpret_cast<const float4 *>(&sq[ty * QN + i][d]);
#pragma unroll
      for (int j = 0; j < KN; ++j)
        kq[j] = *reinterpret_cast<const float4 *>(&sk[tx + 16 * j][d]);
#pragma unroll
      for (int i = 0; i < QN; ++i)
#pragma unroll
        for (int j = 0; j < KN; ++j) {
          fma_pair(s2[i][j], make_float2(qv[i].x, qv[i].y), make_float2(kq[j].x, kq[j].y));
          fma_pair(s2[i][j], make_float2(qv[i].z, qv[i].w), make_float2(kq[j].z, kq[j].w));
        }
    }
#pragma unroll
    for (int i = 0; i < QN; ++i) {
      const int at = base + t0 + ty * QN + i;
      bool seen[KN];
      float s[KN], big = LOWEST;
#pragma unroll
      for (int j = 0; j < KN; ++j) {
        const int behind = at - (k0 + tx + 16 * j);
        seen[j] = behind >= 0 && behind < a.window;
        s[j] = seen[j] ? (s2[i][j].x + s2[i][j].y) * a.scale : LOWEST;
        big = fmaxf(big, s[j]);
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1)
        big = fmaxf(big, __shfl_xor_sync(0xffffffffu, big, off));
      const float mn = fmaxf(m[i], big);
      const float fix = expf(m[i] - mn);
      float sum = 0.0f;
#pragma unroll
      for (int j = 0; j < KN; ++j) {
        const float w = seen[j] ? expf(s[j] - mn) : 0.0f;
        sp[ty * QN + i][tx + 16 * j] = w;
        sum += w;
      }
#pragma unroll
      for (int off = 8; off > 0; off >>= 1)
        sum += __shfl_xor_sync(0xffffffffu, sum, off);
      l[i] = l[i] * fix + sum;
      m[i] = mn;
      const float2 fix2 = make_float2(fix, fix);
#pragma unroll
      for (int c = 0; c < CN; ++c) {
        o[i][c][0] = mul_pair(o[i][c][0], fix2);
        o[i][c][1] = mul_pair(o[i][c][1], fix2);
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
              *reinterpret_cast<const float4 *>(&sv[k + j][tx * 4 + 64 * c]);
#pragma unroll
          for (int i = 0; i < QN; ++i) {
            const float p = j == 0 ? w[i].x : j == 1 ? w[i].y : j == 2 ? w[i].z : w[i].w;
            fma_pair(o[i][c][0], make_float2(p, p), make_float2(v.x, v.y));
            fma_pair(o[i][c][1], make_float2(p, p), make_float2(v.z, v.w));
          }
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
      if (d >= vdim)
        continue;
      const float v[4] = {o[i][c][0].x / l[i], o[i][c][0].y / l[i], o[i][c][1].x / l[i],
                          o[i][c][1].y / l[i]};
      store_terms4(terms, cols, t, head * vdim + d, v);
    }
  }
}

const char *refuse(const LatentArgs &a) {
  if (a.heads < 1 || (a.dim | a.rot | a.vdim) % 8 != 0 || a.dim < 8 || a.rot < 0 ||
      a.vdim < 8 || a.dim + a.rot > 512 || a.vdim > 512 || a.kv_rank < 64 ||
      a.kv_rank % 64 != 0 || a.kv_rank + a.rot > 1024)
    return "latent attention takes head sizes in multiples of 8 and a latent in "
           "multiples of 64; keys and values of at most 512, latent and rotated part "
           "of at most 1024 values";
  if (a.window < 1 || a.cache_rows < 1)
    return "a window holds at least its own token";
  if (((uintptr_t)a.ring | (uintptr_t)a.w_ukv | (uintptr_t)a.w_uk_t) & 15 ||
      a.ring_batch_stride % 4 != 0)
    return "the ring and the matrices of latent attention must be 16-byte aligned";
  return nullptr;
}

struct StepCall {
  const float *q;
  int64_t q_stride;
  const float *down;
  int64_t down_stride;
  int batch;
  float *out;
  int64_t out_stride;
  cudaStream_t stream;
};

template <typename W, int GH, int D4> struct Step {
  static constexpr int NW = 8;
  static constexpr int most = latent_smem(GH, D4, NW, 512, D4 * 128) * (int)sizeof(float);
  static_assert(most <= 226 * 1024, "the arrays fit in shared memory");

  static int smem(const LatentArgs &a) {
    return latent_smem(GH, D4, NW, a.dim, a.kv_rank) * (int)sizeof(float);
  }
  static bool allowed() {
    return allow_dynamic_smem((const void *)latent_decode_kernel<W, GH, D4, NW>, most) ==
           cudaSuccess;
  }
  /* whether the clusters all run at once */
  static bool one_wave(const LatentArgs &a, int batch) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(CL, (a.heads + GH - 1) / GH, batch);
    cfg.blockDim = dim3(NW * 32);
    cfg.dynamicSmemBytes = smem(a);
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = CL;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = 1;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    int clusters = 0;
    if (!allowed() || cudaOccupancyMaxActiveClusters(
                          &clusters, latent_decode_kernel<W, GH, D4, NW>, &cfg) !=
                          cudaSuccess) {
      cudaGetLastError();
      return false;
    }
    return (int64_t)cfg.gridDim.y * batch <= clusters;
  }
  static const char *launch(const LatentArgs &a, const StepCall &c) {
    if (!allowed())
      return "latent attention could not get its shared memory";
    launch_chained_cluster_smem(latent_decode_kernel<W, GH, D4, NW>,
                                dim3(CL, (a.heads + GH - 1) / GH, c.batch), dim3(NW * 32),
                                CL, smem(a), c.stream, a, c.q, c.q_stride, c.down,
                                c.down_stride, c.out, c.out_stride);
    return check_launch("a step of latent attention");
  }
};

template <typename W, int D4>
const char *launch_step_heads(const LatentArgs &a, const StepCall &c) {
  /* few heads a cluster as long as the clusters all run at once */
  if ((int64_t)a.heads * c.batch * CL <= sm_count() && Step<W, 1, D4>::one_wave(a, c.batch))
    return Step<W, 1, D4>::launch(a, c);
  if (D4 > 2 || Step<W, 2, D4>::one_wave(a, c.batch))
    return Step<W, 2, D4>::launch(a, c);
  return Step<W, (D4 > 2 ? 2 : 4), D4>::launch(a, c);
}

template <typename W> const char *launch_step_row(const LatentArgs &a, const StepCall &c) {
  const int row = a.kv_rank + a.rot;
  if (row <= 128)
    return launch_step_heads<W, 1>(a, c);
  if (row <= 256)
    return launch_step_heads<W, 2>(a, c);
  if (row <= 640)
    return launch_step_heads<W, 5>(a, c);
  return launch_step_heads<W, 8>(a, c);
}

template <int KP, int VP, int AQ, int AK>
const char *launch_rows(const LatentArgs &a, const float *q, const float *kv, int first,
                        int t, __nv_bfloat16 *terms, int cols, cudaStream_t stream) {
  constexpr int smem = rows_smem(KP, VP, AQ, AK);
  if (allow_dynamic_smem((const void *)latent_rows_kernel<KP, VP, AQ, AK>, smem) !=
      cudaSuccess)
    return "the multi-position latent attention could not get its shared memory";
  launch_in_order(latent_rows_kernel<KP, VP, AQ, AK>, dim3((t + AQ - 1) / AQ, a.heads),
                 dim3(ROW_THREADS), smem, stream, a, q, kv, first, t, terms, cols);
  return check_launch("the multi-position latent attention");
}

} // namespace

const char *latent_attention_decode(const LatentArgs &a, const float *q, int64_t q_stride,
                                    const float *down, int64_t down_stride, int batch,
                                    float *out, int64_t out_stride, cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  if (a.cache_rows < a.window)
    return "the ring must hold a window";
  if ((((uintptr_t)q | (uintptr_t)down) & 7) || (q_stride | down_stride) % 2 != 0)
    return "queries and latents must be 8-byte aligned";
  const StepCall c{q, q_stride, down, down_stride, batch, out, out_stride, stream};
  return a.fmt == kFmtBf16 ? launch_step_row<__nv_bfloat16>(a, c)
                           : launch_step_row<float>(a, c);
}

int latent_status() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, g_latent_status, sizeof v) != cudaSuccess)
    return -1;
  if (v)
    cudaMemcpyToSymbol(g_latent_status, &zero, sizeof zero);
  return v;
}

const char *latent_rows_down(const LatentArgs &a, const float *partials, int splits, int t,
                             int q_rank, const float *q_gain, int q_mean, void *terms,
                             cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  const int smem = (q_rank + a.kv_rank) * (int)sizeof(float);
  if (smem > 200 * 1024 ||
      allow_dynamic_smem((const void *)latent_down_kernel, 200 * 1024) != cudaSuccess)
    return "the two latents of a position must fit in shared memory";
  launch_in_order(latent_down_kernel, dim3(t), dim3(256), smem, stream, a, partials, splits,
                 t, q_rank, q_gain, q_mean, (__nv_bfloat16 *)terms);
  return check_launch("the latents of a prompt");
}

const char *latent_rows_q(const LatentArgs &a, const float *partials, int splits, int t,
                          float *q, cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  const int64_t count = (int64_t)t * (a.heads * (a.dim + a.rot) / 4);
  launch_in_order(latent_q_kernel, dim3((unsigned)((count + 255) / 256)), dim3(256), 0,
                 stream, a, partials, splits, t, q);
  return check_launch("the queries of a prompt");
}

const char *latent_rows_gather(const LatentArgs &a, int first, int n, void *terms,
                               cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  const int64_t count = (int64_t)n * (a.kv_rank / 8);
  launch_in_order(latent_gather_kernel, dim3((unsigned)((count + 255) / 256)), dim3(256), 0,
                 stream, a, first, n, (__nv_bfloat16 *)terms);
  return check_launch("the latents of a window");
}

const char *latent_attention_rows(const LatentArgs &a, const float *q, const float *kv,
                                  int first, int t, void *terms, int cols,
                                  cudaStream_t stream) {
  if (const char *why = refuse(a))
    return why;
  if (cols % 4 != 0 || cols < a.heads * a.vdim)
    return "the output has too few columns";
  __nv_bfloat16 *to = (__nv_bfloat16 *)terms;
  const int hd = a.dim + a.rot;
  if (hd <= 64 && a.vdim <= 64)
    return launch_rows<64, 64, 64, 64>(a, q, kv, first, t, to, cols, stream);
  if (hd <= 128 && a.vdim <= 128)
    return launch_rows<128, 128, 64, 32>(a, q, kv, first, t, to, cols, stream);
  if (hd <= 192 && a.vdim <= 128)
    return launch_rows<192, 128, 64, 32>(a, q, kv, first, t, to, cols, stream);
  if (hd <= 256 && a.vdim <= 256)
    return launch_rows<256, 256, 64, 32>(a, q, kv, first, t, to, cols, stream);
  return launch_rows<512, 512, 32, 32>(a, q, kv, first, t, to, cols, stream);
}

} // namespace vxb
