// GEMV over plain weight rows (f32 or bfloat16), up to eight activation rows per pass:
//   y[m, n] (+)= sum_k norm(x)[m, k] * w[n, k]
// with an optional RMSNorm prologue, a bias, an activation, a residual sum, and gated (gate, up) row
// pairs from a given row on, so that one launch serves every projection that reads the same
// normalised row.  For one row the prologue also settles the stream: what the sublayer before left
// (its output still to be normed, the embedding row of a new pass) is added to x by every CTA for
// itself, and written back by the first.
// HBM bound: a warp streams R rows with 16-byte loads, each weight byte is read once per pass.
// And its two forms for a mixture of experts, where the rows to stream are chosen per token on
// the device (route_row): expert_in_kernel (gate / up of the chosen experts) and
// expert_out_kernel (their weighted down projections, and the attention output projection in
// the same sum).
#include "layered.cuh"
#include "rows.cuh"

namespace b200 {

namespace {

constexpr int kThreads = 256, kWarps = 8;
constexpr int kSlabBytes = 64 * 1024;      // staged activations per CTA
constexpr int kMaxDynamic = 200 * 1024;

struct RowsP {
  const void *w;
  int64_t ldw;                 // row stride in elements
  int N, K, M;
  const float *x;
  int64_t ldx;
  const float *norm_w;
  float eps;
  float *y;
  int64_t ldy;
  int add;                     // y += instead of y =
  int pair_from;               // rows from here on are (gate, up) pairs; N: none
  float *y2;                   // their results
  int64_t ldy2;
  Gate gate;
  const float *bias;           // per weight row, or null
  RowAct act;
  Unsettled late;              // MT == 1, one slab
  float *x_out;
  int slab;                    // activations staged at a time (a multiple of a block, or all)
};

// 1 / rms of row m in s_r[m], for all rows of a tile
template <int MT>
__device__ void row_rms(const float *x, int64_t ldx, int K, int rows, float eps, float *s_r, float *s_red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (MT == 1) {
    float s = 0.f;
    for (int k = threadIdx.x; k < K; k += kThreads)
      s = fmaf(x[k], x[k], s);
    s = warp_sum(s);
    if (lane == 0)
      s_red[warp] = s;
    __syncthreads();
    if (threadIdx.x == 0) {
      float t = 0.f;
      for (int w = 0; w < kWarps; ++w)
        t += s_red[w];
      s_r[0] = 1.0f / sqrtf(t / (float)K + eps);
    }
  } else {
    for (int m = warp; m < MT; m += kWarps) {
      float s = 0.f;
      if (m < rows)
        for (int k = lane; k < K; k += 32) {
          const float v = x[(int64_t)m * ldx + k];
          s = fmaf(v, v, s);
        }
      s = warp_sum(s);
      if (lane == 0)
        s_r[m] = 1.0f / sqrtf(s / (float)K + eps);
    }
  }
  __syncthreads();
}

__device__ __forceinline__ float cta_sum(float s, float *s_red) {
  s = warp_sum(s);
  __syncthreads();
  if ((threadIdx.x & 31) == 0)
    s_red[threadIdx.x >> 5] = s;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < kWarps; ++w)
    t += s_red[w];
  return t;
}

// The same with the row in registers, four groups of four elements per thread (K % 4 == 0).
constexpr int kRowGroups = 4;
template <typename T>
__device__ void stage_settled_short(const RowsP &p, float4 *xs, float *s_red) {
  float4 x[kRowGroups], y[kRowGroups];
  const int groups = p.K >> 2;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < kRowGroups; ++i) {
    const int g = threadIdx.x + i * kThreads;
    x[i] = g < groups ? reinterpret_cast<const float4 *>(p.x)[g] : zero;
    y[i] = g < groups && p.late.y != nullptr ? reinterpret_cast<const float4 *>(p.late.y)[g] : zero;
  }
  float r = 0.f;
  if (p.late.y != nullptr) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < kRowGroups; ++i)
      s = fmaf(y[i].x, y[i].x, fmaf(y[i].y, y[i].y, fmaf(y[i].z, y[i].z, fmaf(y[i].w, y[i].w, s))));
    r = 1.0f / sqrtf(cta_sum(s, s_red) / (float)p.K + p.eps);
  }
  const T *emb = p.late.embed != nullptr ? reinterpret_cast<const T *>(p.late.embed) + (int64_t)p.late.tokens[0] * p.late.lde : nullptr;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < kRowGroups; ++i) {
    const int g = threadIdx.x + i * kThreads;
    if (g >= groups)
      continue;
    float4 &v = x[i];
    if (p.late.y != nullptr) {
      const float4 w = __ldg(reinterpret_cast<const float4 *>(p.late.w) + g);
      v.x = fmaf(y[i].x * r, w.x, v.x); v.y = fmaf(y[i].y * r, w.y, v.y);
      v.z = fmaf(y[i].z * r, w.z, v.z); v.w = fmaf(y[i].w * r, w.w, v.w);
    }
    if (emb != nullptr) {
      v.x = fmaf(to_float(emb[4 * g]), p.late.scale, v.x); v.y = fmaf(to_float(emb[4 * g + 1]), p.late.scale, v.y);
      v.z = fmaf(to_float(emb[4 * g + 2]), p.late.scale, v.z); v.w = fmaf(to_float(emb[4 * g + 3]), p.late.scale, v.w);
    }
    if (blockIdx.x == 0)
      reinterpret_cast<float4 *>(p.x_out)[g] = v;
    s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
  }
  const float rx = p.norm_w != nullptr ? 1.0f / sqrtf(cta_sum(s, s_red) / (float)p.K + p.eps) : 1.f;
#pragma unroll
  for (int i = 0; i < kRowGroups; ++i) {
    const int g = threadIdx.x + i * kThreads;
    if (g >= block_pad<T>(p.K) / 4)
      continue;
    float4 v = x[i];
    if (p.norm_w != nullptr && g < groups) {
      const float4 w = __ldg(reinterpret_cast<const float4 *>(p.norm_w) + g);
      v = make_float4(v.x * rx * w.x, v.y * rx * w.y, v.z * rx * w.z, v.w * rx * w.w);
    }
    xs[stage_slot<T>(g)] = v;                      // zero beyond K
  }
  __syncthreads();
}

// Stage the settled (and normed) row in xs; the first CTA writes the settled row to x_out.
template <typename T>
__device__ void stage_settled(const RowsP &p, float4 *xs, float *s_red) {
  if ((p.K & 3) == 0 && block_pad<T>(p.K) <= 4 * kRowGroups * kThreads) {
    stage_settled_short<T>(p, xs, s_red);
    return;
  }
  float r = 0.f;
  if (p.late.y != nullptr) {
    float s = 0.f;
    for (int k = threadIdx.x; k < p.K; k += kThreads)
      s = fmaf(p.late.y[k], p.late.y[k], s);
    r = 1.0f / sqrtf(cta_sum(s, s_red) / (float)p.K + p.eps);
  }
  const T *emb = p.late.embed != nullptr ? reinterpret_cast<const T *>(p.late.embed) + (int64_t)p.late.tokens[0] * p.late.lde : nullptr;
  const bool keep = blockIdx.x == 0;
  float s = 0.f;
  for (int g = threadIdx.x; g < block_pad<T>(p.K) / 4; g += kThreads) {
    float v[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = 4 * g + e;
      if (k < p.K) {
        v[e] = p.x[k];
        if (p.late.y != nullptr)
          v[e] = fmaf(p.late.y[k] * r, __ldg(p.late.w + k), v[e]);
        if (emb != nullptr)
          v[e] = fmaf(to_float(emb[k]), p.late.scale, v[e]);
        if (keep)
          p.x_out[k] = v[e];
        s = fmaf(v[e], v[e], s);
      }
    }
    xs[stage_slot<T>(g)] = make_float4(v[0], v[1], v[2], v[3]);
  }
  if (p.norm_w != nullptr) {
    const float rx = 1.0f / sqrtf(cta_sum(s, s_red) / (float)p.K + p.eps);
    for (int g = threadIdx.x; g < block_pad<T>(p.K) / 4; g += kThreads) {   // the groups this thread staged
      float4 &v = xs[stage_slot<T>(g)];
      const int k = 4 * g;
      v.x = k < p.K ? v.x * rx * __ldg(p.norm_w + k) : 0.f;
      v.y = k + 1 < p.K ? v.y * rx * __ldg(p.norm_w + k + 1) : 0.f;
      v.z = k + 2 < p.K ? v.z * rx * __ldg(p.norm_w + k + 2) : 0.f;
      v.w = k + 3 < p.K ? v.w * rx * __ldg(p.norm_w + k + 3) : 0.f;
    }
  }
  __syncthreads();
}

template <typename T, int MT, int R>
__global__ void __launch_bounds__(kThreads, MT == 1 ? 4 : 1)
gemv_rows_kernel(const RowsP p) {
  extern __shared__ __align__(16) float4 xs[];   // [MT][slab / 4]
  __shared__ float s_r[8], s_red[8];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int m0 = blockIdx.y * MT, rows = min(MT, p.M - m0);
  const float *x = p.x + (int64_t)m0 * p.ldx;
  if (MT == 1) {
    // while the kernel ahead ends: the norm weights and the beginnings of the CTA's first weight
    // rows, which nothing writes, on their way to L2
    for (int k = threadIdx.x * 32; k < p.K; k += kThreads * 32) {
      if (p.norm_w != nullptr)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(p.norm_w + k));
      if (p.late.y != nullptr)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(p.late.w + k));
    }
    constexpr int kLines = 32 / R;                 // of 128 bytes, per row
    const int64_t row = (int64_t)blockIdx.x * kWarps * R + warp * R + lane / kLines;
    const int k = lane % kLines * (128 / (int)sizeof(T));
    if (row < p.N && k < p.K)
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const T *>(p.w) + row * p.ldw + k));
  }
  chain_wait();
  chain_next();
  const bool settles = MT == 1 && p.x_out != nullptr;
  if (settles)
    stage_settled<T>(p, xs, s_red);
  else if (p.norm_w != nullptr)
    row_rms<MT>(x, p.ldx, p.K, rows, p.eps, s_r, s_red);
  const int Kp = unit_pad<T>(p.K);
  const int xs_ld = p.slab / 4;
  const bool one_slab = p.slab >= Kp;
  bool staged = settles;
  const T *w = reinterpret_cast<const T *>(p.w);
  for (int64_t base = (int64_t)blockIdx.x * kWarps * R; base < p.N; base += (int64_t)gridDim.x * kWarps * R) {
    const int64_t row0 = base + warp * R;
    const T *rowp[R];
    float acc[R][MT];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      rowp[r] = w + min(row0 + r, (int64_t)p.N - 1) * p.ldw;   // clamped rows are read but not stored
#pragma unroll
      for (int m = 0; m < MT; ++m)
        acc[r][m] = 0.f;
    }
    for (int k0 = 0; k0 < Kp; k0 += p.slab) {
      if (!(one_slab && staged)) {
        if (staged)
          __syncthreads();
#pragma unroll
        for (int m = 0; m < MT; ++m)
          if (m < rows)
            stage_row<T>(xs + m * xs_ld, x + (int64_t)m * p.ldx + k0, min(p.slab, p.K - k0),
                         p.norm_w != nullptr ? s_r[m] : 1.f, p.norm_w != nullptr ? p.norm_w + k0 : nullptr, threadIdx.x, kThreads);
        staged = true;
        __syncthreads();
      }
      dot_rows<T, MT, R>(rowp, min(p.slab, Kp - k0), xs, xs_ld, lane, acc);
#pragma unroll
      for (int r = 0; r < R; ++r)
        rowp[r] += p.slab;
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int m = 0; m < MT; ++m)
        acc[r][m] = warp_sum(acc[r][m]);
    if (lane != 0)
      continue;
    if (R >= 2 && row0 >= p.pair_from) {
#pragma unroll
      for (int r = 0; r + 1 < R; r += 2)
        if (row0 + r + 1 < p.N)
#pragma unroll
          for (int m = 0; m < MT; ++m)
            if (m < rows)
              p.y2[(int64_t)(m0 + m) * p.ldy2 + ((row0 + r - p.pair_from) >> 1)] = gate_pair(p.gate, acc[r][m], acc[r + 1 < R ? r + 1 : r][m]);
    } else {
#pragma unroll
      for (int r = 0; r < R; ++r)
        if (row0 + r < p.N)
#pragma unroll
          for (int m = 0; m < MT; ++m)
            if (m < rows) {
              float *y = p.y + (int64_t)(m0 + m) * p.ldy + row0 + r;
              const float v = row_act(p.act, p.bias != nullptr ? acc[r][m] + p.bias[row0 + r] : acc[r][m], m0 + m, row0 + r);
              *y = p.add ? *y + v : v;
            }
    }
  }
}

struct ExpertInP {
  const void *w;               // [experts][2 * ff rows (gate_j, up_j)][ldw]
  int64_t ldw;
  int ff, K, M;
  const float *x;
  int64_t ldx;
  const float *norm_w;
  float eps;
  const float *z;              // router logits of row m at z + m * ldz
  int64_t ldz;
  int experts, top;
  Gate gate;
  float *mid;                  // [M * top][ff]
  int32_t *ids;                // [M * top]
  float *weight;               // [M * top]
};

template <typename T, int R>
__global__ void __launch_bounds__(kThreads)
expert_in_kernel(const ExpertInP p) {
  extern __shared__ __align__(16) float4 xs[];   // the normalised row, then experts + 2 * top words of routing
  __shared__ float s_r[8], s_red[8];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int slot = blockIdx.y, m = slot / p.top, j = slot - m * p.top;
  float *s_z = reinterpret_cast<float *>(xs + block_pad<T>(p.K) / 4);
  float *s_w = s_z + p.experts;
  int *s_id = reinterpret_cast<int *>(s_w + p.top);
  const float *x = p.x + (int64_t)m * p.ldx;
  if (warp == 0)
    route_row(p.z + (int64_t)m * p.ldz, p.experts, p.top, s_z, s_id, s_w, lane);
  row_rms<1>(x, p.ldx, p.K, 1, p.eps, s_r, s_red);
  stage_row<T>(xs, x, p.K, s_r[0], p.norm_w, threadIdx.x, kThreads);
  __syncthreads();
  const int e = s_id[j];
  if (blockIdx.x == 0 && threadIdx.x == 0) {
    p.ids[slot] = e;
    p.weight[slot] = s_w[j];
  }
  const int N = 2 * p.ff, Kp = unit_pad<T>(p.K);
  const T *w = reinterpret_cast<const T *>(p.w) + (int64_t)e * N * p.ldw;
  for (int base = blockIdx.x * kWarps * R; base < N; base += gridDim.x * kWarps * R) {
    const int row0 = base + warp * R;
    const T *rowp[R];
    float acc[R][1];
#pragma unroll
    for (int r = 0; r < R; ++r) {
      rowp[r] = w + (int64_t)min(row0 + r, N - 1) * p.ldw;
      acc[r][0] = 0.f;
    }
    dot_rows<T, 1, R>(rowp, Kp, xs, 0, lane, acc);
#pragma unroll
    for (int r = 0; r < R; ++r)
      acc[r][0] = warp_sum(acc[r][0]);
    if (lane == 0)
#pragma unroll
      for (int r = 0; r < R; r += 2)
        if (row0 + r < N)
          p.mid[(int64_t)slot * p.ff + ((row0 + r) >> 1)] = gate_pair(p.gate, acc[r][0], acc[r + 1][0]);
  }
}

struct ExpertOutP {
  const void *w0;              // attention output projection [N][ld0], or null
  int64_t ld0;
  int K0;
  const float *x0;             // its input [M][ldx0]
  int64_t ldx0;
  const void *w;               // [experts][N][ldw]
  int64_t ldw;
  int ff, N, top;
  const float *mid;            // [M * top][ff]
  const int32_t *ids;
  const float *weight;
  float *y;                    // [M][ldy] +=
  int64_t ldy;
  int staged_once;             // every segment fits shared memory together
};

template <typename T, int R>
__global__ void __launch_bounds__(kThreads)
expert_out_kernel(const ExpertOutP p) {
  extern __shared__ __align__(16) float4 xs[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int m = blockIdx.y;
  const int first = p.w0 != nullptr ? -1 : 0;          // segment -1: the attention output
  const int seg0 = p.w0 != nullptr ? block_pad<T>(p.K0) / 4 : 0, seg = block_pad<T>(p.ff) / 4;
  auto stage = [&](int s, float4 *dst) {
    if (s < 0)
      stage_row<T>(dst, p.x0 + (int64_t)m * p.ldx0, p.K0, 1.f, nullptr, threadIdx.x, kThreads);
    else
      stage_row<T>(dst, p.mid + ((int64_t)m * p.top + s) * p.ff, p.ff, p.weight[m * p.top + s], nullptr, threadIdx.x, kThreads);
  };
  if (p.staged_once) {
    for (int s = first; s < p.top; ++s)
      stage(s, xs + (s < 0 ? 0 : seg0 + s * seg));
    __syncthreads();
  }
  for (int64_t base = (int64_t)blockIdx.x * kWarps * R; base < p.N; base += (int64_t)gridDim.x * kWarps * R) {
    const int64_t row0 = base + warp * R;
    float acc[R][1];
#pragma unroll
    for (int r = 0; r < R; ++r)
      acc[r][0] = 0.f;
    for (int s = first; s < p.top; ++s) {
      const T *rowp[R];
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int64_t row = min(row0 + r, (int64_t)p.N - 1);
        rowp[r] = s < 0 ? reinterpret_cast<const T *>(p.w0) + row * p.ld0
                        : reinterpret_cast<const T *>(p.w) + ((int64_t)p.ids[m * p.top + s] * p.N + row) * p.ldw;
      }
      const float4 *src = xs + (s < 0 ? 0 : seg0 + s * seg);
      if (!p.staged_once) {
        __syncthreads();
        stage(s, xs);
        __syncthreads();
        src = xs;
      }
      dot_rows<T, 1, R>(rowp, unit_pad<T>(s < 0 ? p.K0 : p.ff), src, 0, lane, acc);
    }
#pragma unroll
    for (int r = 0; r < R; ++r)
      acc[r][0] = warp_sum(acc[r][0]);
    if (lane == 0)
#pragma unroll
      for (int r = 0; r < R; ++r)
        if (row0 + r < p.N)
          p.y[(int64_t)m * p.ldy + row0 + r] += acc[r][0];
  }
}

template <typename K> int allow_dynamic(K kern, size_t bytes) {
  if (bytes > (size_t)kMaxDynamic)
    return fail(B200_ELIMIT, "row kernels: %zu bytes of staged activations exceed shared memory", bytes);
  if (bytes > 40 * 1024)
    B200_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynamic));
  return B200_OK;
}

// CTAs for N rows: one resident wave at most (a CTA loops over its row groups)
template <typename K> int wave_grid(K kern, int64_t groups, int y, size_t smem, int *grid) {
  int occ = 0, dev = 0, sms = 0;
  B200_CUDA(cudaGetDevice(&dev));
  B200_CUDA(cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev));
  B200_CUDA(cudaOccupancyMaxActiveBlocksPerMultiprocessor(&occ, kern, kThreads, smem));
  int64_t cap = (int64_t)sms * (occ < 1 ? 1 : occ) / (y < 1 ? 1 : y);
  if (cap < 1)
    cap = 1;
  *grid = (int)(groups < cap ? groups : cap);
  return B200_OK;
}

template <typename T, int MT, int R> int gemv_rows_run(RowsP &p, cudaStream_t st) {
  auto kern = gemv_rows_kernel<T, MT, R>;
  const int budget = kSlabBytes / (4 * MT);
  p.slab = block_pad<T>(p.K) <= budget ? block_pad<T>(p.K) : budget / 256 * 256;
  const size_t smem = (size_t)MT * p.slab * 4;
  if (int rc = allow_dynamic(kern, smem)) return rc;
  const int y = (p.M + MT - 1) / MT;
  int grid = 1;
  if (int rc = wave_grid(kern, (p.N + kWarps * R - 1) / (kWarps * R), y, smem, &grid)) return rc;
  B200_CUDA(launch_chained(kern, dim3(grid, y), kThreads, smem, st, p));
  B200_LAUNCH_CHECK();
  return B200_OK;
}

template <typename T> int gemv_rows_pick(RowsP &p, cudaStream_t st) {
  const bool pairs = p.pair_from < p.N;
  if (p.M == 1) {
    if (p.N >= 8 * 4 * 2 * 148)
      return gemv_rows_run<T, 1, 4>(p, st);
    if (pairs || p.N >= 8 * 2 * 148)
      return gemv_rows_run<T, 1, 2>(p, st);
    return gemv_rows_run<T, 1, 1>(p, st);
  }
  if (p.M == 2)
    return gemv_rows_run<T, 2, 2>(p, st);
  if (p.M <= 4)
    return gemv_rows_run<T, 4, 2>(p, st);
  return gemv_rows_run<T, 8, 2>(p, st);
}

} // namespace

bool gemv_rows_settles(int M, int K) { return M == 1 && block_pad<bf16>(K) <= kSlabBytes / 4; }

int gemv_rows_launch(int dtype, const GemvRows &g, cudaStream_t st) {
  RowsP p{};
  p.w = g.w.w;
  p.ldw = g.w.ld;
  p.N = g.w.N;
  p.K = g.w.K;
  p.M = g.M;
  p.x = g.x;
  p.ldx = g.ldx;
  p.norm_w = g.norm_w;
  p.eps = g.eps;
  p.y = g.y;
  p.ldy = g.ldy;
  p.add = g.add ? 1 : 0;
  p.pair_from = g.pair_from < g.w.N ? g.pair_from : g.w.N;
  p.y2 = g.y2;
  p.ldy2 = g.ldy2;
  p.gate = g.gate;
  p.bias = g.bias;
  p.act = g.act;
  p.late = g.late;
  p.x_out = g.x_out;
  if ((p.pair_from < g.w.N) && ((p.pair_from & 3) || (g.w.N & 1)))
    return fail(B200_EINVAL, "gemv_rows: pairs must start at a multiple of four rows");
  if (g.late.any() != (g.x_out != nullptr) || (g.x_out != nullptr && (!gemv_rows_settles(g.M, p.K) || g.x_out == g.x)))
    return fail(B200_EINVAL, "gemv_rows: only one row that fits shared memory is settled, into another buffer");
  return dtype == B200_F32 ? gemv_rows_pick<float>(p, st) : gemv_rows_pick<bf16>(p, st);
}

template <typename T>
static int expert_rows_run(const RowMatrix &in, const RowMatrix &out, int ff, int experts, int top, const Gate &gate,
                           float *x, int64_t ldx, int M, const float *norm_w, float eps, const float *z, int64_t ldz,
                           const RowMatrix *o, const float *att, int64_t lda, float *mid, int32_t *ids, float *weight,
                           cudaStream_t st) {
  {
    ExpertInP p{};
    p.w = in.w; p.ldw = in.ld; p.ff = ff; p.K = in.K; p.M = M;
    p.x = x; p.ldx = ldx; p.norm_w = norm_w; p.eps = eps;
    p.z = z; p.ldz = ldz; p.experts = experts; p.top = top; p.gate = gate;
    p.mid = mid; p.ids = ids; p.weight = weight;
    auto kern = expert_in_kernel<T, 2>;
    const size_t smem = (size_t)block_pad<T>(p.K) * 4 + (size_t)experts * 4 + (size_t)top * 8;
    if (int rc = allow_dynamic(kern, smem)) return rc;
    int grid = 1;
    if (int rc = wave_grid(kern, (2 * ff + kWarps * 2 - 1) / (kWarps * 2), M * top, smem, &grid)) return rc;
    for (int m0 = 0; m0 < M; m0 += 32768 / top) {   // gridDim.y limit
      const int mm = M - m0 < 32768 / top ? M - m0 : 32768 / top;
      ExpertInP q = p;
      q.x += (int64_t)m0 * ldx; q.z += (int64_t)m0 * ldz; q.M = mm;
      q.mid += (int64_t)m0 * top * ff; q.ids += (int64_t)m0 * top; q.weight += (int64_t)m0 * top;
      kern<<<dim3(grid, mm * top), kThreads, smem, st>>>(q);
      B200_LAUNCH_CHECK();
    }
  }
  ExpertOutP p{};
  if (o) {
    p.w0 = o->w; p.ld0 = o->ld; p.K0 = o->K; p.x0 = att; p.ldx0 = lda;
  }
  p.w = out.w; p.ldw = out.ld; p.ff = ff; p.N = out.N / experts; p.top = top;
  p.mid = mid; p.ids = ids; p.weight = weight; p.y = x; p.ldy = ldx;
  auto kern = expert_out_kernel<T, 2>;
  const size_t a = o ? (size_t)block_pad<T>(p.K0) * 4 : 0, b = (size_t)block_pad<T>(ff) * 4;
  p.staged_once = a + b * top <= 96 * 1024;
  const size_t smem = p.staged_once ? a + b * top : (a > b ? a : b);
  if (int rc = allow_dynamic(kern, smem)) return rc;
  int grid = 1;
  if (int rc = wave_grid(kern, (p.N + kWarps * 2 - 1) / (kWarps * 2), M, smem, &grid)) return rc;
  for (int m0 = 0; m0 < M; m0 += 32768) {
    const int mm = M - m0 < 32768 ? M - m0 : 32768;
    ExpertOutP q = p;
    q.x0 = q.x0 ? q.x0 + (int64_t)m0 * lda : nullptr;
    q.mid += (int64_t)m0 * top * ff; q.ids += (int64_t)m0 * top; q.weight += (int64_t)m0 * top;
    q.y += (int64_t)m0 * ldx;
    kern<<<dim3(grid, mm), kThreads, smem, st>>>(q);
    B200_LAUNCH_CHECK();
  }
  return B200_OK;
}

int expert_rows_launch(int dtype, const RowMatrix &in, const RowMatrix &out, int ff, int experts, int top,
                       const Gate &gate, float *x, int64_t ldx, int M, const float *norm_w, float eps, const float *z,
                       int64_t ldz, const RowMatrix *o, const float *att, int64_t lda, float *mid, int32_t *ids,
                       float *weight, cudaStream_t st) {
  return dtype == B200_F32
             ? expert_rows_run<float>(in, out, ff, experts, top, gate, x, ldx, M, norm_w, eps, z, ldz, o, att, lda, mid, ids, weight, st)
             : expert_rows_run<bf16>(in, out, ff, experts, top, gate, x, ldx, M, norm_w, eps, z, ldz, o, att, lda, mid, ids, weight, st);
}

} // namespace b200
