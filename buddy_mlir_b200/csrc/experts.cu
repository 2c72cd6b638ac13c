// Mixture of experts over many rows: route every row, sort the (row, choice) slots by expert, and
// feed the sorted rows to the grouped GEMM; afterwards every row adds up its choices in order.
#include "layered.cuh"
#include "rows.cuh"

namespace b200 {

namespace {

constexpr int BM = 128;        // rows per tile of the grouped GEMM

// a warp routes kRouteRows rows; counts[e] is the number of slots of expert e
constexpr int kRouteRows = 2;
__global__ void __launch_bounds__(256)
route_rows_kernel(const float *z, int64_t ldz, int experts, int top, int M, int32_t *ids, float *weight, int32_t *counts) {
  extern __shared__ float s_z[];   // per warp: experts logits, top weights, top ids; then the CTA's counts
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float *sz = s_z + warp * (experts + 2 * top), *sw = sz + experts;
  int *sid = reinterpret_cast<int *>(sw + top);
  int *s_count = reinterpret_cast<int *>(s_z + 8 * (experts + 2 * top));
  for (int e = threadIdx.x; e < experts; e += 256)
    s_count[e] = 0;
  __syncthreads();
  for (int r = 0; r < kRouteRows; ++r) {
    const int m = (blockIdx.x * 8 + warp) * kRouteRows + r;
    if (m >= M)
      break;
    route_row(z + (int64_t)m * ldz, experts, top, sz, sid, sw, lane);
    for (int j = lane; j < top; j += 32) {
      ids[(int64_t)m * top + j] = sid[j];
      weight[(int64_t)m * top + j] = sw[j];
      atomicAdd(s_count + sid[j], 1);
    }
    __syncwarp();
  }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += 256)
    if (s_count[e] > 0)
      atomicAdd(counts + e, s_count[e]);
}

// counts -> first sorted row of every expert (left in counts as a cursor) and the tile table
__global__ void __launch_bounds__(1024)
plan_tiles_kernel(int32_t *counts, int experts, int4 *tiles, int32_t *n_tiles) {
  __shared__ int s_row[1024], s_tile[1024];
  const int e = threadIdx.x;
  const int n = e < experts ? counts[e] : 0;
  s_row[e] = n;
  s_tile[e] = (n + BM - 1) / BM;
  __syncthreads();
  for (int o = 1; o < 1024; o <<= 1) {
    const int a = e >= o ? s_row[e - o] : 0, b = e >= o ? s_tile[e - o] : 0;
    __syncthreads();
    s_row[e] += a;
    s_tile[e] += b;
    __syncthreads();
  }
  if (e >= experts)
    return;
  const int row0 = s_row[e] - n, mine = (n + BM - 1) / BM, t0 = s_tile[e] - mine;
  for (int t = 0; t < mine; ++t)
    tiles[t0 + t] = make_int4(e, row0 + t * BM, min(BM, n - t * BM), 0);
  counts[e] = row0;
  if (e == experts - 1)
    *n_tiles = s_tile[e];
}

// one warp per slot: take a place among the expert's rows and copy the row there
__global__ void __launch_bounds__(256)
sort_rows_kernel(const bf16 *h, int64_t ldh, int top, int slots, const int32_t *ids, int32_t *cursor, int32_t *place, bf16 *out) {
  const int lane = threadIdx.x & 31, slot = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (slot >= slots)
    return;
  int pos = 0;
  if (lane == 0) {
    pos = atomicAdd(cursor + ids[slot], 1);
    place[slot] = pos;
  }
  pos = __shfl_sync(0xffffffffu, pos, 0);
  const uint4 *src = reinterpret_cast<const uint4 *>(h + (int64_t)(slot / top) * ldh);
  uint4 *dst = reinterpret_cast<uint4 *>(out + (int64_t)pos * ldh);
  for (int i = lane; i < ldh / 8; i += 32)
    dst[i] = src[i];
}

// x[m] += sum over j of weight[m, j] * y[place[m, j]]
__global__ void __launch_bounds__(256)
combine_experts_kernel(float *x, int W, int top, const float *y, const int32_t *place, const float *weight) {
  extern __shared__ float s_w[];   // top weights, top places
  int *s_p = reinterpret_cast<int *>(s_w + top);
  const int64_t m = blockIdx.x;
  for (int j = threadIdx.x; j < top; j += 256) {
    s_w[j] = weight[m * top + j];
    s_p[j] = place[m * top + j];
  }
  __syncthreads();
  if ((W & 3) == 0) {
    for (int n = threadIdx.x * 4; n < W; n += 1024) {
      float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int j = 0; j < top; ++j) {
        const float4 v = __ldg(reinterpret_cast<const float4 *>(y + (int64_t)s_p[j] * W + n));
        s.x = fmaf(s_w[j], v.x, s.x);
        s.y = fmaf(s_w[j], v.y, s.y);
        s.z = fmaf(s_w[j], v.z, s.z);
        s.w = fmaf(s_w[j], v.w, s.w);
      }
      float4 *dst = reinterpret_cast<float4 *>(x + m * W + n);
      const float4 v = *dst;
      *dst = make_float4(v.x + s.x, v.y + s.y, v.z + s.z, v.w + s.w);
    }
  } else {
    for (int n = threadIdx.x; n < W; n += 256) {
      float s = 0.f;
      for (int j = 0; j < top; ++j)
        s = fmaf(s_w[j], y[(int64_t)s_p[j] * W + n], s);
      x[m * W + n] += s;
    }
  }
}

} // namespace

int experts_max_tiles(int slots, int experts) { return slots / BM + (experts < slots ? experts : slots) + 1; }

int experts_sort_launch(const float *z, int64_t ldz, int experts, int top, int M, const bf16 *h, int64_t ldh, int32_t *ids,
                        float *weight, int32_t *counts, int4 *tiles, int32_t *n_tiles, int32_t *place, bf16 *sorted,
                        cudaStream_t st) {
  const size_t route_bytes = ((size_t)8 * (experts + 2 * top) + experts) * 4;
  if (route_bytes > 40 * 1024)
    B200_CUDA(cudaFuncSetAttribute(route_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 120 * 1024));
  B200_CUDA(cudaMemsetAsync(counts, 0, (size_t)experts * 4, st));
  route_rows_kernel<<<(M + 8 * kRouteRows - 1) / (8 * kRouteRows), 256, route_bytes, st>>>(z, ldz, experts, top, M, ids, weight, counts);
  B200_LAUNCH_CHECK();
  plan_tiles_kernel<<<1, 1024, 0, st>>>(counts, experts, tiles, n_tiles);
  B200_LAUNCH_CHECK();
  sort_rows_kernel<<<(M * top + 7) / 8, 256, 0, st>>>(h, ldh, top, M * top, ids, counts, place, sorted);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

int experts_combine_launch(float *x, int W, int top, int M, const float *y, const int32_t *place, const float *weight,
                           cudaStream_t st) {
  combine_experts_kernel<<<M, 256, (size_t)top * 8, st>>>(x, W, top, y, place, weight);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

} // namespace b200
