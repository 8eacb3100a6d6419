/* gated_linear.cu -- gated linear attention: a matrix per head that fades by key
 * channel, takes in k v^T and is read by q.
 *
 * A column of the state needs no other column, so both forms cut the state by
 * columns.  A step streams it once (a cluster per head, so that the norm over the
 * head meets in distributed shared memory).  The positions of a prompt go through
 * one after another with the state in registers: 3 multiply-adds per value of the
 * state and position, which is what a chunked form costs on the FP32 pipe too, and
 * the result does not depend on how the prompt is cut.
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

/* sigmoid(z)^(1 / tau), by way of the logarithm, which no z overflows */
__device__ __forceinline__ float decay(float z, float inv_tau) {
  const float log_sigmoid = fminf(z, 0.0f) - log1pf(expf(-fabsf(z)));
  return expf(log_sigmoid * inv_tau);
}

/* where the parts of an input row begin */
struct Parts {
  int k, v, gate, a1;
  __host__ __device__ explicit Parts(const GatedLinearArgs &a)
      : k(a.heads * a.dim), v(2 * k), gate(v + a.heads * a.vdim),
        a1(gate + a.heads * a.vdim) {}
};

/* ---- one token of each sequence ------------------------------------------------
 * A cluster of CL blocks per (head, sequence), block r taking vdim / CL columns
 * (rounded up to 4). Threads: COLS4 groups of four columns by ROWS rows. */
constexpr int CL = 8, ROWS = 32;
constexpr int EARLY = 8; /* rows of a thread that are fetched ahead of the wait */

template <int COLS4>
__global__ void __launch_bounds__(COLS4 * ROWS)
gated_linear_step_kernel(const GatedLinearArgs a, const float *in, int64_t in_stride,
                         float *out, int64_t out_stride) {
  constexpr int STEP_THREADS = COLS4 * ROWS;
  extern __shared__ __align__(16) float step_smem[];
  const int slice4 = (a.vdim / 4 + CL - 1) / CL; /* float4 columns of a block */
  float *alpha = step_smem, *sk = alpha + a.dim, *sq = sk + a.dim; /* [dim] each */
  float *o = sq + a.dim;                                           /* [slice4 * 4] */
  __shared__ __align__(16) float part[ROWS][COLS4 * 4 + 4];
  __shared__ float ssq, red[STEP_THREADS / 32];
  chain_release();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, b = blockIdx.z, r = blockIdx.x;
  const int c4 = tid % COLS4, row = tid / COLS4;
  const int first4 = r * slice4, last4 = min(first4 + slice4, a.vdim / 4);
  const bool fresh = a.positions[b] == 0;
  float *state = a.state + b * a.state_batch_stride + (int64_t)h * a.dim * a.vdim;
  const Parts at(a);

  /* The state is what earlier steps left: the first columns' rows come while the
     kernel in front still runs. */
  float4 early[EARLY];
#pragma unroll
  for (int j = 0; j < EARLY; ++j) {
    const int i = row + j * ROWS;
    early[j] = make_float4(0, 0, 0, 0);
    if (!fresh && i < a.dim && first4 + c4 < last4)
      early[j] = *reinterpret_cast<const float4 *>(state + (int64_t)i * a.vdim +
                                                   (first4 + c4) * 4);
  }
  chain_wait();
  const float *x = in + b * in_stride;
  for (int i = tid; i < a.dim; i += STEP_THREADS) {
    float z = a.a2_bias[h * a.dim + i];
    const float4 *w = reinterpret_cast<const float4 *>(a.a2 +
                                                       (int64_t)(h * a.dim + i) * a.rank);
    const float4 *y = reinterpret_cast<const float4 *>(x + at.a1);
    for (int c = 0; c < a.rank / 4; ++c) {
      const float4 p = w[c], q = y[c];
      z = fmaf(p.x, q.x, z);
      z = fmaf(p.y, q.y, z);
      z = fmaf(p.z, q.z, z);
      z = fmaf(p.w, q.w, z);
    }
    alpha[i] = decay(z, a.inv_tau);
    sk[i] = x[at.k + h * a.dim + i];
    sq[i] = x[h * a.dim + i] * a.q_scale;
  }
  __syncthreads();

  float ss = 0.0f;
  for (int base4 = first4; base4 < last4; base4 += COLS4) {
    const int col4 = base4 + c4;
    const bool mine = col4 < last4;
    float4 v = make_float4(0, 0, 0, 0), sum = v;
    if (mine)
      v = *reinterpret_cast<const float4 *>(x + at.v + h * a.vdim + col4 * 4);
    auto advance = [&](int i, float4 s) {
      const float f = alpha[i], k = sk[i];
      s.x = fmaf(k, v.x, f * s.x);
      s.y = fmaf(k, v.y, f * s.y);
      s.z = fmaf(k, v.z, f * s.z);
      s.w = fmaf(k, v.w, f * s.w);
      *reinterpret_cast<float4 *>(state + (int64_t)i * a.vdim + col4 * 4) = s;
      axpy(sum, sq[i], s);
    };
    if (mine) {
      int i = row;
      if (base4 == first4) {
#pragma unroll
        for (int j = 0; j < EARLY; ++j, i += ROWS)
          if (i < a.dim)
            advance(i, early[j]);
      }
      for (; i < a.dim; i += ROWS)
        advance(i, fresh ? make_float4(0, 0, 0, 0)
                         : *reinterpret_cast<const float4 *>(
                               state + (int64_t)i * a.vdim + col4 * 4));
    }
    *reinterpret_cast<float4 *>(&part[row][c4 * 4]) = sum;
    __syncthreads();
    if (tid < COLS4 * 4 && (base4 - first4) * 4 + tid < slice4 * 4) {
      float total = 0.0f;
      for (int k = 0; k < ROWS; ++k) /* fixed order */
        total += part[k][tid];
      o[(base4 - first4) * 4 + tid] = total;
      ss = fmaf(total, total, ss);
    }
    __syncthreads();
  }
  ss = warp_sum(ss);
  if (lane == 0)
    red[warp] = ss;
  __syncthreads();
  if (tid == 0) {
    float total = 0.0f;
    for (int k = 0; k < STEP_THREADS / 32; ++k)
      total += red[k];
    ssq = total;
  }
  cg::cluster_group cluster = cg::this_cluster();
  cluster.sync();
  float total = 0.0f;
  for (int k = 0; k < CL; ++k) /* fixed order */
    total += *cluster.map_shared_rank(&ssq, k);
  const float inv = 1.0f / sqrtf(total / (float)a.v_mean + a.eps);
  for (int c = tid; c < (last4 - first4) * 4; c += STEP_THREADS) {
    const int col = first4 * 4 + c;
    const float g = x[at.gate + h * a.vdim + col];
    out[b * out_stride + h * a.vdim + col] = o[c] * inv * a.gain[col] * silu(g);
  }
  cluster.sync(); /* nobody leaves while a peer may still read its sum */
}

/* ---- the positions of a prompt: decays -----------------------------------------
 * A block takes TB positions and 256 channels. */
constexpr int TB = 16;
__global__ void __launch_bounds__(256)
gated_linear_decay_kernel(const GatedLinearArgs a, const float *in, int64_t in_stride,
                          int t_count, float *alpha) {
  extern __shared__ __align__(16) float low[]; /* [TB][rank] */
  const int t0 = blockIdx.x * TB, channels = a.heads * a.dim;
  const int a1 = Parts(a).a1;
  for (int i = threadIdx.x; i < TB * a.rank; i += 256) {
    const int t = i / a.rank, c = i - t * a.rank;
    low[i] = t0 + t < t_count ? in[(t0 + t) * in_stride + a1 + c] : 0.0f;
  }
  __syncthreads();
  const int ch = blockIdx.y * 256 + threadIdx.x;
  if (ch >= channels)
    return;
  float z[TB];
  const float bias = a.a2_bias[ch];
#pragma unroll
  for (int t = 0; t < TB; ++t)
    z[t] = bias;
  const float4 *w = reinterpret_cast<const float4 *>(a.a2 + (int64_t)ch * a.rank);
  for (int c = 0; c < a.rank / 4; ++c) {
    const float4 p = w[c];
#pragma unroll
    for (int t = 0; t < TB; ++t) {
      const float4 y = *reinterpret_cast<const float4 *>(&low[t * a.rank + c * 4]);
      z[t] = fmaf(p.x, y.x, z[t]);
      z[t] = fmaf(p.y, y.y, z[t]);
      z[t] = fmaf(p.z, y.z, z[t]);
      z[t] = fmaf(p.w, y.w, z[t]);
    }
  }
#pragma unroll
  for (int t = 0; t < TB; ++t)
    if (t0 + t < t_count)
      alpha[(int64_t)(t0 + t) * channels + ch] = decay(z[t], a.inv_tau);
}

/* ---- the positions of a prompt: the recurrence ----------------------------------
 * LG lanes side by side hold the key channels of RJ columns (lane g of them channels
 * 4 (LG c + g) .. + 3, c below NI), so a warp holds 32 / LG * RJ columns of a head
 * and a block SCAN_WARPS times as many. q, k, alpha and v of TT positions at a time
 * come by bulk copies into two shared-memory buffers (past the end: q = k = v = 0,
 * alpha = 1, which leave the state as it is), which a warp of their own asks for. Two
 * channels go through a multiply-add together, and the sums over the lanes are taken
 * for TS positions at once. */
constexpr int SCAN_WARPS = 8, SCAN_THREADS = (SCAN_WARPS + 1) * 32, TS = 8;
__host__ __device__ constexpr int scan_tile(int NI) { return NI > 2 ? 16 : 32; }
/* floats of shared memory */
__host__ __device__ constexpr int scan_smem(int NI, int COLS, int dim) {
  return 2 * scan_tile(NI) * (3 * dim + COLS) + scan_tile(NI) * COLS;
}

__device__ int g_scan_status; /* 0x62: a tile never arrived; 0x63: or was never used */

/* The sums of N values over the LG lanes of a group: half of the values change hands
   at every exchange while there are several, so that lane g is left with the sums of
   values first .. first + N / LG - 1 (N < LG: with value `first`, and the lowest of
   the lanes that are writes it). */
template <int LG, int N>
__device__ __forceinline__ void group_sums(float (&v)[N], int g, int &first,
                                           bool &owner) {
  first = 0;
  owner = true;
  int n = N;
#pragma unroll
  for (int off = LG / 2; off > 0; off /= 2) {
    const bool upper = (g & off) != 0;
    if (n > 1) {
#pragma unroll
      for (int j = 0; j < N / 2; ++j)
        if (j < n / 2) {
          const float give = upper ? v[j] : v[j + n / 2];
          const float keep = upper ? v[j + n / 2] : v[j];
          v[j] = keep + __shfl_xor_sync(0xffffffffu, give, off);
        }
      n /= 2;
      if (upper)
        first += n;
    } else {
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], off);
      owner = owner && !upper;
    }
  }
}

template <int LG, int NI, int RJ>
__global__ void __launch_bounds__(SCAN_THREADS)
gated_linear_scan_kernel(const GatedLinearArgs a, const float *in, int64_t in_stride,
                         const float *alpha, int t_count, float *o) {
  constexpr int TT = scan_tile(NI);
  static_assert(RJ % 4 == 0 && TT % TS == 0, "columns in fours, whole batches");
  constexpr int WARP_COLS = 32 / LG * RJ, COLS = SCAN_WARPS * WARP_COLS;
  extern __shared__ __align__(128) float scan_shared[];
  __shared__ __align__(8) uint64_t full[2], empty[2];
  const int dim = a.dim, vdim = a.vdim;
  const int step = 3 * dim + COLS; /* floats of a position: q | k | alpha | v */
  float *buf = scan_shared;        /* [2][TT][step] */
  float *so = buf + 2 * TT * step; /* [warp][TT][WARP_COLS] */
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.y, col0 = blockIdx.x * COLS;
  const int v_cols = min(COLS, vdim - col0);
  const int g = lane % LG, group = lane / LG;
  const int mine = warp * WARP_COLS + group * RJ; /* first column, in the block */
  const Parts at(a);
  const bool fresh = a.positions[0] == 0;
  float *state = a.state + (int64_t)h * dim * vdim;

  if (tid == 0) {
    for (int side = 0; side < 2; ++side) {
      ptx::mbar_init(&full[side], 1);
      ptx::mbar_init(&empty[side], SCAN_WARPS);
    }
    ptx::fence_proxy_async_smem();
    ptx::fence_barrier_init();
  }
  if (v_cols < COLS) /* the columns of nobody */
    for (int i = tid; i < 2 * TT * (COLS - v_cols); i += SCAN_THREADS) {
      const int t = i / (COLS - v_cols);
      buf[t * step + 3 * dim + v_cols + i - t * (COLS - v_cols)] = 0.0f;
    }
  __syncthreads();

  if (warp == SCAN_WARPS) {
    for (int t0 = 0, tile = 0; t0 < t_count; t0 += TT, ++tile) {
      const int side = tile & 1, n = min(TT, t_count - t0);
      const uint32_t phase = ((tile >> 1) & 1) ^ 1;
      if (!__all_sync(0xffffffffu, ptx::mbar_try_wait(&empty[side], phase) ||
                                       ptx::mbar_wait_alone(&empty[side], phase))) {
        atomicCAS(&g_scan_status, 0, 0x63);
        break;
      }
      float *to = buf + side * TT * step;
      const int filled = (n + TS - 1) / TS * TS;
      for (int i = n * step + lane; i < filled * step; i += 32) {
        const int c = i % step;
        to[i] = c >= 2 * dim && c < 3 * dim ? 1.0f : 0.0f;
      }
      __syncwarp();
      if (lane == 0)
        ptx::mbar_expect_tx(&full[side], n * (3 * dim + v_cols) * (int)sizeof(float));
      __syncwarp();
      for (int i = lane; i < n * 4; i += 32) {
        const int t = i >> 2, part = i & 3;
        const float *row = in + (int64_t)(t0 + t) * in_stride;
        const float *src = part == 0   ? row + h * dim
                           : part == 1 ? row + at.k + h * dim
                           : part == 2 ? alpha + ((int64_t)(t0 + t) * a.heads + h) * dim
                                       : row + at.v + h * vdim + col0;
        ptx::bulk_load(to + t * step + part * dim, src,
                       (part == 3 ? v_cols : dim) * (int)sizeof(float), &full[side]);
      }
    }
    return; /* the others use every tile up before they leave */
  }

  float2 s[2 * NI][RJ]; /* two neighbouring channels of a column */
  auto each_cell = [&](auto body) {
#pragma unroll
    for (int c = 0; c < 2 * NI; ++c)
#pragma unroll
      for (int j = 0; j < RJ; ++j)
        body(s[c][j], ((c >> 1) * LG + g) * 4 + (c & 1) * 2, col0 + mine + j);
  };
  each_cell([&](float2 &cell, int i, int col) {
    cell = make_float2(0, 0);
    if (!fresh && i < dim && col < vdim)
      cell = make_float2(state[(int64_t)i * vdim + col], state[(int64_t)(i + 1) * vdim + col]);
  });
  float *out = so + warp * TT * WARP_COLS;
  for (int t0 = 0, tile = 0; t0 < t_count; t0 += TT, ++tile) {
    const int side = tile & 1, n = min(TT, t_count - t0);
    const uint32_t phase = (tile >> 1) & 1;
    if (!__all_sync(0xffffffffu, ptx::mbar_try_wait(&full[side], phase) ||
                                     ptx::mbar_wait_alone(&full[side], phase))) {
      atomicCAS(&g_scan_status, 0, 0x62);
      break;
    }
    const float *now = buf + side * TT * step;
    for (int t = 0; t < n; t += TS) {
      float part[TS * RJ];
#pragma unroll
      for (int u = 0; u < TS; ++u, now += step) {
        float v[RJ];
        float2 sum[RJ];
#pragma unroll
        for (int j = 0; j < RJ; j += 4) {
          const float4 v4 = *reinterpret_cast<const float4 *>(now + 3 * dim + mine + j);
          v[j] = v4.x; v[j + 1] = v4.y; v[j + 2] = v4.z; v[j + 3] = v4.w;
        }
#pragma unroll
        for (int j = 0; j < RJ; ++j)
          sum[j] = make_float2(0, 0);
#pragma unroll
        for (int c = 0; c < NI; ++c) {
          const int i = (c * LG + g) * 4;
          float4 q = make_float4(0, 0, 0, 0), k = q, f = q;
          if (i < dim) {
            q = *reinterpret_cast<const float4 *>(now + i);
            k = *reinterpret_cast<const float4 *>(now + dim + i);
            f = *reinterpret_cast<const float4 *>(now + 2 * dim + i);
          }
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float2 q2 = e ? make_float2(q.z, q.w) : make_float2(q.x, q.y);
            const float2 k2 = e ? make_float2(k.z, k.w) : make_float2(k.x, k.y);
            const float2 f2 = e ? make_float2(f.z, f.w) : make_float2(f.x, f.y);
#pragma unroll
            for (int j = 0; j < RJ; ++j) {
              float2 &cell = s[c * 2 + e][j];
              cell = mul_pair(f2, cell);
              fma_pair(cell, k2, make_float2(v[j], v[j]));
              fma_pair(sum[j], q2, cell);
            }
          }
        }
#pragma unroll
        for (int j = 0; j < RJ; ++j)
          part[u * RJ + j] = sum[j].x + sum[j].y;
      }
      int one;
      bool owner;
      group_sums<LG>(part, g, one, owner);
      constexpr int LEFT = TS * RJ > LG ? TS * RJ / LG : 1;
      if (owner)
#pragma unroll
        for (int j = 0; j < LEFT; ++j)
          out[(t + (one + j) / RJ) * WARP_COLS + group * RJ + (one + j) % RJ] =
              part[j] * a.q_scale;
    }
    __syncwarp();
    if (lane == 0)
      ptx::mbar_arrive(&empty[side]);
    for (int i = lane; i < n * (WARP_COLS / 4); i += 32) {
      const int t = i / (WARP_COLS / 4), c = i % (WARP_COLS / 4) * 4;
      const int col = col0 + warp * WARP_COLS + c;
      if (col < vdim)
        *reinterpret_cast<float4 *>(o + (int64_t)(t0 + t) * a.heads * vdim + h * vdim +
                                    col) =
            *reinterpret_cast<const float4 *>(&out[t * WARP_COLS + c]);
    }
    __syncwarp();
  }
  each_cell([&](float2 &cell, int i, int col) {
    if (i < dim && col < vdim) {
      state[(int64_t)i * vdim + col] = cell.x;
      state[(int64_t)(i + 1) * vdim + col] = cell.y;
    }
  });
}

/* ---- the positions of a prompt: norm and gate -----------------------------------
 * A block is a position, a warp takes every eighth head. */
__global__ void __launch_bounds__(256)
gated_linear_finish_kernel(const GatedLinearArgs a, const float *in, int64_t in_stride,
                           const float *o, __nv_bfloat16 *terms, int cols) {
  const int64_t t = blockIdx.x;
  const int lane = threadIdx.x & 31, gate = Parts(a).gate;
  for (int h = threadIdx.x >> 5; h < a.heads; h += 8) {
    const float *row = o + (t * a.heads + h) * a.vdim;
    const float *g = in + t * in_stride + gate + h * a.vdim;
    float ss = 0.0f;
    for (int c = lane * 4; c < a.vdim; c += 128) {
      const float4 v = *reinterpret_cast<const float4 *>(row + c);
      ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
    }
    const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.v_mean + a.eps);
    for (int c = lane * 4; c < a.vdim; c += 128) {
      const float4 v = *reinterpret_cast<const float4 *>(row + c);
      const float4 w = *reinterpret_cast<const float4 *>(a.gain + c);
      const float4 z = *reinterpret_cast<const float4 *>(g + c);
      const float out[4] = {v.x * inv * w.x * silu(z.x), v.y * inv * w.y * silu(z.y),
                            v.z * inv * w.z * silu(z.z), v.w * inv * w.w * silu(z.w)};
      store_terms4(terms, cols, t, h * a.vdim + c, out);
    }
  }
}

const char *refuse(const GatedLinearArgs &a, int64_t in_stride) {
  if (a.heads < 1 || a.dim < 8 || a.dim > 512 || (a.dim | a.vdim | a.rank) % 8 != 0 ||
      a.vdim < 8 || a.vdim > 16384 || a.rank < 8 || a.rank > 512)
    return "gated linear attention takes head sizes and a rank in multiples of 8, keys "
           "and rank at most 512";
  if (in_stride % 4 != 0 || a.state_batch_stride % 4 != 0 ||
      ((uintptr_t)a.state | (uintptr_t)a.a2 | (uintptr_t)a.gain) & 15)
    return "the state and the rows of gated linear attention must be 16-byte aligned";
  return nullptr;
}

template <int LG, int NI, int RJ>
const char *launch_scan(const GatedLinearArgs &a, const float *in, int64_t in_stride,
                        const float *alpha, int t, float *o, cudaStream_t stream) {
  constexpr int COLS = SCAN_WARPS * 32 / LG * RJ;
  const int smem = scan_smem(NI, COLS, a.dim) * (int)sizeof(float);
  constexpr int most = scan_smem(NI, COLS, LG * NI * 4) * (int)sizeof(float);
  static_assert(most <= 227 * 1024, "the buffers fit in shared memory");
  const void *kernel = (const void *)gated_linear_scan_kernel<LG, NI, RJ>;
  if (allow_dynamic_smem(kernel, most) != cudaSuccess)
    return "gated linear attention could not get its shared memory";
  launch_in_order(gated_linear_scan_kernel<LG, NI, RJ>,
                 dim3((a.vdim + COLS - 1) / COLS, a.heads), dim3(SCAN_THREADS), smem,
                 stream, a, in, in_stride, alpha, t, o);
  return check_launch("the recurrence of gated linear attention");
}

} // namespace

const char *gated_linear_decode(const GatedLinearArgs &a, const float *in,
                                int64_t in_stride, int batch, float *out,
                                int64_t out_stride, cudaStream_t stream) {
  if (const char *why = refuse(a, in_stride))
    return why;
  const int slice4 = (a.vdim / 4 + CL - 1) / CL;
  const int smem = (3 * a.dim + slice4 * 4) * (int)sizeof(float);
  auto go = [&](auto kernel, int cols4) {
    launch_chained_cluster_smem(kernel, dim3(CL, a.heads, batch), dim3(cols4 * ROWS), CL,
                                smem, stream, a, in, in_stride, out, out_stride);
  };
  if (slice4 <= 8)
    go(gated_linear_step_kernel<8>, 8);
  else
    go(gated_linear_step_kernel<16>, 16);
  return check_launch("a step of gated linear attention");
}

const char *gated_linear_decays(const GatedLinearArgs &a, const float *in,
                                int64_t in_stride, int t, float *alpha,
                                cudaStream_t stream) {
  if (const char *why = refuse(a, in_stride))
    return why;
  launch_in_order(gated_linear_decay_kernel,
                 dim3((t + TB - 1) / TB, (a.heads * a.dim + 255) / 256), dim3(256),
                 TB * a.rank * sizeof(float), stream, a, in, in_stride, t, alpha);
  return check_launch("the decays of gated linear attention");
}

const char *gated_linear_scan(const GatedLinearArgs &a, const float *in, int64_t in_stride,
                              const float *alpha, int t, float *o, cudaStream_t stream) {
  if (const char *why = refuse(a, in_stride))
    return why;
  if (a.dim <= 32)
    return launch_scan<8, 1, 4>(a, in, in_stride, alpha, t, o, stream);
  if (a.dim <= 64)
    return launch_scan<16, 1, 4>(a, in, in_stride, alpha, t, o, stream);
  if (a.dim <= 128)
    return launch_scan<32, 1, 4>(a, in, in_stride, alpha, t, o, stream);
  if (a.dim <= 256)
    return launch_scan<32, 2, 4>(a, in, in_stride, alpha, t, o, stream);
  return launch_scan<32, 4, 4>(a, in, in_stride, alpha, t, o, stream);
}

int gated_linear_status() {
  int v = 0, zero = 0;
  if (cudaMemcpyFromSymbol(&v, g_scan_status, sizeof v) != cudaSuccess)
    return -1;
  if (v)
    cudaMemcpyToSymbol(g_scan_status, &zero, sizeof zero);
  return v;
}

const char *gated_linear_finish(const GatedLinearArgs &a, const float *in,
                                int64_t in_stride, const float *o, int t, void *terms,
                                int cols, cudaStream_t stream) {
  if (const char *why = refuse(a, in_stride))
    return why;
  if (cols % 4 != 0 || cols < a.heads * a.vdim)
    return "the output has too few columns";
  launch_in_order(gated_linear_finish_kernel, dim3(t), dim3(256), 0, stream, a, in,
                 in_stride, o, (__nv_bfloat16 *)terms, cols);
  return check_launch("the norm and gate of gated linear attention");
}

} // namespace vxb
