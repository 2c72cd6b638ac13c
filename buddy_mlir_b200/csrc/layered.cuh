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
int latent_value_launch(int dtype, const LatentDims &d, const float *scratch, int M, int splits, const RowMatrix &uv,
                        void *out, int64_t ldo, bool out_bf16, cudaStream_t st);
int latent_limits(const LatentDims &d);   // 0, or an error for sizes the kernels do not take

// rows_ops in layered.cu
int place_rows_launch(int src_dtype, const void *src, int rows, int cols, int dst_dtype, void *dst, int64_t ld, int64_t row0,
                      int64_t row_step, int64_t col0, cudaStream_t st);

} // namespace b200
