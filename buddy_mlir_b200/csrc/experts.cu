// Mixture of experts over many rows: route every row, sort the (row, choice) slots by expert, and
// feed the sorted rows to the grouped GEMM; afterwards every row adds up its choices in order.
#include "layered.cuh"
#include "rows.cuh"

namespace b200 {

namespace {

constexpr int BM = 128;        // rows per tile of the grouped GEMM

// one warp per row; counts[e] is the number of slots of expert e
__global__ void __launch_bounds__(256)
route_rows_kernel(const float *z, int64_t ldz, int experts, int top, int M, int32_t *ids, float *weight, int32_t *counts) {
  extern __shared__ float s_z[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int m = blockIdx.x * 8 + warp;
  if (m >= M)
    return;
  int32_t *id = ids + (int64_t)m * top;
  route_row(z + (int64_t)m * ldz, experts, top, s_z + warp * experts, id, weight + (int64_t)m * top, lane);
  for (int j = lane; j < top; j += 32)
    atomicAdd(counts + id[j], 1);
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
  const int m = blockIdx.x;
  for (int n = threadIdx.x; n < W; n += 256) {
    float s = 0.f;
    for (int j = 0; j < top; ++j)
      s = fmaf(weight[(int64_t)m * top + j], y[(int64_t)place[(int64_t)m * top + j] * W + n], s);
    x[(int64_t)m * W + n] += s;
  }
}

} // namespace

int experts_max_tiles(int slots, int experts) { return slots / BM + (experts < slots ? experts : slots) + 1; }

int experts_sort_launch(const float *z, int64_t ldz, int experts, int top, int M, const bf16 *h, int64_t ldh, int32_t *ids,
                        float *weight, int32_t *counts, int4 *tiles, int32_t *n_tiles, int32_t *place, bf16 *sorted,
                        cudaStream_t st) {
  B200_CUDA(cudaMemsetAsync(counts, 0, (size_t)experts * 4, st));
  route_rows_kernel<<<(M + 7) / 8, 256, (size_t)experts * 8 * 4, st>>>(z, ldz, experts, top, M, ids, weight, counts);
  B200_LAUNCH_CHECK();
  plan_tiles_kernel<<<1, 1024, 0, st>>>(counts, experts, tiles, n_tiles);
  B200_LAUNCH_CHECK();
  sort_rows_kernel<<<(M * top + 7) / 8, 256, 0, st>>>(h, ldh, top, M * top, ids, counts, place, sorted);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

int experts_combine_launch(float *x, int W, int top, int M, const float *y, const int32_t *place, const float *weight,
                           cudaStream_t st) {
  combine_experts_kernel<<<M, 256, 0, st>>>(x, W, top, y, place, weight);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

} // namespace b200
