// Models given as a list of described layers (b200_model_create_layered): weight matrices as
// plain rows, the launches of the layer mechanisms, and the per-layer state the engine keeps.
#pragma once
#include "common.cuh"
#include "rows.cuh"

namespace b200 {

// [N][ld] plain weight rows, K used elements per row (the rest of a row is zero).
struct RowMatrix {
  void *w = nullptr;
  int64_t ld = 0;
  int N = 0, K = 0;
};

// The `top` largest of the router logits z[0..experts) (the lowest index among equals) and the
// softmax over them, by one warp.  s_z: `experts` floats of scratch.
__device__ __forceinline__ void route_row(const float *z, int experts, int top, float *s_z, int *ids, float *weight, int lane) {
  for (int i = lane; i < experts; i += 32)
    s_z[i] = z[i];
  __syncwarp();
  for (int j = 0; j < top; ++j) {
    float best = -INFINITY;
    int bi = 0x7fffffff;
    for (int i = lane; i < experts; i += 32)
      if (s_z[i] > best) {
        best = s_z[i];
        bi = i;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
      if (ov > best || (ov == best && oi < bi)) {
        best = ov;
        bi = oi;
      }
    }
    if (bi >= experts)   // nothing comparable left (NaN logits): stay in bounds
      bi = j;
    if (lane == 0) {
      ids[j] = bi;
      weight[j] = best;
      s_z[bi] = -INFINITY;
    }
    __syncwarp();
  }
  if (lane == 0) {
    const float mx = weight[0];
    float sum = 0.f;
    for (int j = 0; j < top; ++j) {
      weight[j] = expf(weight[j] - mx);
      sum += weight[j];
    }
    for (int j = 0; j < top; ++j)
      weight[j] = weight[j] / sum;
  }
  __syncwarp();
}

// Where a sequence's cached rows are: row of position p of sequence s in pool + address * row stride.
struct CacheView {
  const int32_t *row_seq, *row_pos;   // per activation row
  const int32_t *table;               // [sequences][stride] page numbers
  int stride, page;
};
__device__ __forceinline__ int64_t cache_row(const CacheView &v, int seq, int pos) {
  return (int64_t)v.table[(int64_t)seq * v.stride + pos / v.page] * v.page + pos % v.page;
}

// One latent-attention layer's sizes and constants.
struct LatentDims {
  int heads, dim, rot, vdim, rank;
  int window;                  // <= 0: every position before
  float scale;
  int64_t row;                 // cache row stride in elements (latent, rotated key part, padding)
};

int gemv_rows_launch(int dtype, const RowMatrix &w, const float *x, int64_t ldx, int M, const float *norm_w, float eps,
                     float *y, int64_t ldy, bool add, int pair_from, float *y2, int64_t ldy2, const Gate &gate,
                     cudaStream_t st);
int expert_rows_launch(int dtype, const RowMatrix &in, const RowMatrix &out, int ff, int experts, int top,
                       const Gate &gate, float *x, int64_t ldx, int M, const float *norm_w, float eps, const float *z,
                       int64_t ldz, const RowMatrix *o, const float *att, int64_t lda, float *mid, int32_t *ids,
                       float *weight, cudaStream_t st);

// latent.cu.  proj: f32 rows [q | latent and key part | ...] of the layer's projections.
int latent_prep_launch(int dtype, const LatentDims &d, const float *proj, int64_t ldp, int M, const RowMatrix &uk,
                       const float *inv_freq, float *qabs, bool own, int off_down, const float *norm_w, float eps,
                       void *pool, const CacheView &cv, cudaStream_t st);
int64_t latent_scratch_floats(const LatentDims &d, int M, int splits);
int latent_splits(const LatentDims &d, int M, int max_ctx);
int latent_attend_launch(int dtype, const LatentDims &d, const float *qabs, int M, const void *pool, const CacheView &cv,
                         int splits, int max_ctx, float *scratch, cudaStream_t st);
// work: room for M * heads * (rank + 7) bf16 (the attended queries' own buffer will do), or null
int latent_value_launch(int dtype, const LatentDims &d, const float *scratch, int M, int splits, const RowMatrix &uv,
                        void *out, int64_t ldo, bool out_bf16, void *work, cudaStream_t st);
int latent_shift_launch(int dtype, const LatentDims &d, const void *cache, int src, int tail, const float *inv_freq, int delta,
                        void *stage, cudaStream_t st);   // rows moved by `delta` positions, into stage
int latent_limits(const LatentDims &d);   // 0, or an error for sizes the kernels do not take

// latent_prefill.cu: many consecutive queries of one sequence, bf16
int latent_store_launch(const LatentDims &d, const float *proj, int64_t ldp, int M, int off_down, const float *norm_w,
                        float eps, const float *inv_freq, void *pool, const CacheView &cv, cudaStream_t st);
int latent_query_launch(const LatentDims &d, const float *proj, int64_t ldp, int M, const float *inv_freq,
                        const int32_t *row_pos, bf16 *q, cudaStream_t st);
int latent_gather_launch(const LatentDims &d, const void *pool, const CacheView &cv, int seq, int first, int n, bf16 *rows,
                         cudaStream_t st);
bool latent_prefill_takes(const LatentDims &d);
int latent_prefill_launch(const LatentDims &d, const bf16 *q, int n, int pos0, const bf16 *rows, const bf16 *kv, int64_t ldkv,
                          int first, bf16 *out, int64_t ldo, cudaStream_t st);

// gemm_bf16.cu
struct GemmBf16 {
  const bf16 *A = nullptr;     // [M][lda], K used elements per row
  int64_t lda = 0;
  int M = 0;
  RowMatrix w;                 // bf16 rows
  float *C = nullptr;          // result as f32 or as bf16, rows of ldc
  bf16 *C16 = nullptr;
  int64_t ldc = 0;
  bool add = false;            // C += (f32 only)
  bool pairs = false;          // rows (2j, 2j + 1) of w are (gate_j, up_j): N / 2 gated columns
  Gate gate{};
  const int4 *tiles = nullptr; // grouped: row tiles (group, first row, rows), at most max_tiles of them
  const int32_t *n_tiles = nullptr;
  int max_tiles = 0, groups = 1;   // w holds `groups` matrices of N / groups rows
};
int64_t gemm_bf16_workspace_bytes();
int gemm_bf16_launch(const GemmBf16 &g, void *workspace, cudaStream_t st);

// experts.cu
int experts_max_tiles(int slots, int experts);
int experts_sort_launch(const float *z, int64_t ldz, int experts, int top, int M, const bf16 *h, int64_t ldh, int32_t *ids,
                        float *weight, int32_t *counts, int4 *tiles, int32_t *n_tiles, int32_t *place, bf16 *sorted,
                        cudaStream_t st);
int experts_combine_launch(float *x, int W, int top, int M, const float *y, const int32_t *place, const float *weight,
                           cudaStream_t st);

} // namespace b200
