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

// y (+)= act(norm(x) w^T + bias): M activation rows against plain weight rows.
struct GemvRows {
  RowMatrix w;
  const float *x = nullptr;    // [M][ldx]
  int64_t ldx = 0;
  int M = 0;
  const float *norm_w = nullptr;   // RMSNorm of x on the way in, or null
  float eps = 0.f;
  Unsettled late{};            // one row that fits shared memory (gemv_rows_settles): added to x first,
  float *x_out = nullptr;      // and the sum written here (not x)
  const float *bias = nullptr; // per weight row, or null
  RowAct act{};
  float *y = nullptr;
  int64_t ldy = 0;
  bool add = false;
  int pair_from = 0x7fffffff;  // weight rows from here on are (gate, up) pairs, their results go to y2
  float *y2 = nullptr;
  int64_t ldy2 = 0;
  Gate gate{};
};
bool gemv_rows_settles(int M, int K);
int gemv_rows_launch(int dtype, const GemvRows &g, cudaStream_t st);
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

// heads.cu: attention over keys and values cached per head
constexpr int kMaxSplits = 64, kHeadsQueryTile = 128;
struct HeadsDims {
  int heads, kv, dim, vdim, rot;   // query heads, key / value heads, sizes per head, rotated dimensions (the first ones)
  int halves;                  // rotation pairs: (i, i + rot/2), else (2i, 2i + 1)
  int window;                  // <= 0: every position before
  float scale, sink;           // sink: score of one more softmax entry without a value, -inf: none
  int dimp, vdimp;             // a head's share of a cache row: sizes padded to 8 elements
  int64_t row;                 // [keys of all kv heads | values of all kv heads]
};
struct HeadsIn {               // f32 rows of the layer's projections: queries at 0
  const float *proj;
  int64_t ldp;
  int off_k, off_v;
  const float *q_norm, *k_norm;    // norms over the whole projection, or null
  float eps;
  const double *freq;          // radians per position, per pair
};
int heads_limits(const HeadsDims &d);
bool heads_tensor_cores(const HeadsDims &d);   // sizes the bf16 mma kernels take
int heads_splits(const HeadsDims &d, int rows, int max_ctx);
int64_t heads_scratch_floats(const HeadsDims &d, int rows, int splits);
// q: [M][heads][dimp] in the compute type
int heads_prep_launch(int dtype, const HeadsDims &d, const HeadsIn &in, int M, void *q, void *pool, const CacheView &cv,
                      cudaStream_t st);
// n rows, each against its own visible keys (rows: which activation rows, null: 0 .. n - 1)
int heads_attend_launch(int dtype, const HeadsDims &d, const void *q, const int32_t *rows, int n, const void *pool,
                        const CacheView &cv, int splits, float *part, cudaStream_t st);
// tiles of at most kHeadsQueryTile consecutive queries of a sequence (first row, rows, sequence, first position)
int heads_prefill_launch(const HeadsDims &d, const bf16 *q, const int4 *tiles, int n_tiles, const bf16 *pool, const CacheView &cv,
                         const float *gate, int64_t ldg, float out_scale, bf16 *out, int64_t ldo, cudaStream_t st);
int heads_shift_launch(int dtype, const HeadsDims &d, const void *cache, int src, int tail, const double *freq, int delta,
                       void *stage, cudaStream_t st);

// memory.cu: matrix memory
struct MemoryDims {
  int heads, dim, vdim;
  float cap, q_scale, floor;   // soft cap of the gates, factor on q, added to the denominator
  int tiles;                   // ceil(vdim / 32)
  int64_t head_state, state;   // f32 values of a head, of a slot
};
struct MemoryIn {              // f32 rows of the layer's projections, and where its parts start
  const float *proj;
  int64_t ldp;
  int off_q, off_k, off_v, off_i, off_f;
};
int memory_limits(const MemoryDims &d);
bool memory_chunks_take(const MemoryDims &d);
// n segments (first row, rows, slot, -) of consecutive tokens; o: [row][ldo]
int memory_step_launch(const MemoryDims &d, const MemoryIn &in, const int4 *segs, int n, const int32_t *row_pos, float *states,
                       float *o, int64_t ldo, cudaStream_t st);
// n_segs segments in chunks of kMemoryChunk rows (first row, rows, slot, -); chunk0: the first chunk of a
// segment.  U [chunk][head][head_state] and meta [chunk][head][3]: scratch.
constexpr int kMemoryChunk = 64;
struct MemoryChunks {
  const int4 *segs, *chunks;
  const int32_t *chunk0;
  int n_segs, n_chunks;
  float *U;
  double *meta;
};
int memory_chunk_launch(const MemoryDims &d, const MemoryIn &in, const MemoryChunks &k, const int32_t *row_pos, float *states,
                        float *o, int64_t ldo, cudaStream_t st);

// The output projection's input rows from attention shares and / or memory outputs (heads.cu).
struct MixFinish {
  const int32_t *rows = nullptr;   // activation rows (null: 0 .. M - 1)
  const float *proj = nullptr;     // gates
  int64_t ldp = 0;
  float *cat = nullptr;            // f32 or bf16 rows of ldc
  bf16 *cat16 = nullptr;
  int64_t ldc = 0;
  int n_heads = 0;                 // attention: shares of the i-th listed row at part
  HeadsDims h{};
  const float *part = nullptr;
  int splits = 1, off_g = -1;      // no output gate: -1
  float h_scale = 1.f;
  int n_mem = 0;                   // memory: rows of mem_o, normed per head, gated
  int mem_vdim = 0, mem_col = 0, off_mg = 0;
  const float *mem_o = nullptr, *mem_norm = nullptr;
  int64_t ldo = 0;
  float m_scale = 1.f, eps = 0.f;
};
int mix_finish_launch(const MixFinish &f, int M, cudaStream_t st);

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
  const float *bias = nullptr; // per weight row, or null
  RowAct act{};
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
