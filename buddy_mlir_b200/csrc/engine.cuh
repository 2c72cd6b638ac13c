// The model session and the batch behind the C ABI's handles.
#pragma once
#include "common.cuh"
#include "layered.cuh"
#include "mega.cuh"

#include <map>
#include <string>
#include <vector>

namespace b200 {

inline int dev_alloc(void **p, size_t bytes) {
  cudaError_t e = cudaMalloc(p, bytes ? bytes : 16);
  if (e != cudaSuccess) {
    (void)cudaGetLastError();
    return fail(B200_ENOMEM, "cudaMalloc(%zu): %s", bytes, cudaGetErrorString(e));
  }
  return B200_OK;
}

struct DevLinear {
  b200_weight w{};
  void *w_buf = nullptr, *scale_buf = nullptr;
  float *bias_buf = nullptr;
  bool set = false;
  int64_t bytes() const {
    if (!set)
      return 0;
    int64_t b = packed_row_bytes(w.kind, w.K) * w.N;
    if (w.scale) {
      const int64_t ng =
          (w.kind == B200_W_U4 && w.group > 0 && w.group < w.K) ? w.K / w.group : 1;
      b += w.N * ng * (w.scale_dtype == B200_F32 ? 4 : 2);
    }
    if (w.bias)
      b += w.N * 4;
    return b;
  }
  void release() {
    cudaFree(w_buf);
    cudaFree(scale_buf);
    cudaFree(bias_buf);
    w_buf = scale_buf = nullptr;
    bias_buf = nullptr;
    set = false;
  }
};

struct Layer {
  float *in_norm = nullptr, *post_norm = nullptr, *q_norm = nullptr,
        *k_norm = nullptr;
  DevLinear q, k, v, o, gate, up, down;
  DevLinear qkv, gateup;  // fused at finalize
};


// ---- models of described layers ---------------------------------------------------------------
struct LayeredLayer {
  b200_layer_config cfg{};
  LatentDims d{};              // latent attention
  HeadsDims h{};               // attention over per-head keys
  MemoryDims mem{};            // matrix memory
  int off_down = 0, off_router = 0;                 // parts of `in` (queries first)
  int off_k = 0, off_v = 0, off_g = -1;
  int off_mq = 0, off_mk = 0, off_mv = 0, off_mg = 0, off_mi = 0, off_mf = 0;
  int plain = 0;               // rows of `in` before the (gate, up) pairs
  int att = 0;                 // heads * vdim
  int mem_col = 0;             // the memory's first column of `out`
  RowMatrix in;                // every matrix that reads the mixer's input: [q | latent and key part | router | padding |
                               // (gate_j, up_j) pairs], or [q | k | v | gate | memory's q, k, v, gate, i, f]
  RowMatrix out;               // [W_o | W_down] or [W_o | memory's W_o] side by side: one contraction
  RowMatrix ukv, uk, uv;       // [W_uk; W_uv], and its two parts
  RowMatrix expert_in, expert_out;   // [experts][(gate_j, up_j) pairs], [experts][W_down]
  RowMatrix up, down;          // plain feed-forward
  RowMatrix side_gate, side_proj;    // per-token layer input
  float *norm = nullptr, *down_norm = nullptr, *inv_freq = nullptr;
  double *freq = nullptr;
  float *in_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr, *mem_norm = nullptr;
  float *norm_b = nullptr, *norm2 = nullptr, *norm2_b = nullptr, *side_norm = nullptr;
  Gate gate{};
  bool latent() const { return cfg.mixer == B200_MIX_LATENT; }
  bool heads() const { return cfg.mixer == B200_MIX_HEADS || cfg.mixer == B200_MIX_HEADS_MEMORY; }
  bool memory() const { return cfg.mixer == B200_MIX_MEMORY || cfg.mixer == B200_MIX_HEADS_MEMORY; }
  bool own() const { return !latent() || cfg.kv_from < 0; }
  int64_t row() const { return latent() ? d.row : heads() ? h.row : 0; }   // elements per cached position
  int64_t state() const { return memory() ? mem.state : 0; }               // f32 values per slot
};
struct LayerCache {            // cached rows by position (or page), recurrent state by slot
  void *rows = nullptr;
  float *state = nullptr;
};
struct LayeredRun {            // one execution of a layer in a step; a looped layer has several
  int layer = 0;
  int source = 0;              // the run whose cache this one attends to (itself, or the kv_from layer's)
  bool again = false;          // the embedding output is added before it
  LayerCache cache;            // the single-sequence session's: [max_len][row], one slot
};
struct LayeredTensor {         // where a named tensor goes
  int rows, cols, dtype;
  void *dst;
  int64_t ld, row0, step, col0;
  bool set;                    // or optional
};
struct StepPlan {              // the rows of a step by sequence (device arrays)
  const int4 *segs = nullptr;  // (first row, rows, sequence, first position): n_long of at least kExpandRows rows, then n_short
  int n_long = 0, n_short = 0;
  const int4 *tiles = nullptr; // the long segments in tiles of kHeadsQueryTile
  int n_tiles = 0;
  const int4 *chunks = nullptr;       // and in chunks of kMemoryChunk, of which segment i has those from chunk0[i] on
  const int32_t *chunk0 = nullptr;
  int n_chunks = 0;
  const int32_t *singles = nullptr;   // rows outside long segments
  int n_singles = 0;
  int ctx = 0;                 // positions that some row may see
};
struct LayeredWs {             // activations of up to `rows` rows
  int rows = 0, ctx = 0;
  std::vector<void *> owned;
  float *proj = nullptr, *qabs = nullptr, *part = nullptr, *cat = nullptr, *mid = nullptr, *weight = nullptr;
  int32_t *ids = nullptr;
  int32_t *row_seq = nullptr, *row_pos = nullptr, *tokens = nullptr, *plan = nullptr;
  float *x = nullptr;
  float *x2 = nullptr, *y = nullptr, *h32 = nullptr, *mem_o = nullptr;   // sandwich blocks
  void *q = nullptr;           // rotated queries in the compute type
  // tensor-core path
  bf16 *h16 = nullptr, *cat16 = nullptr, *q16 = nullptr, *x16 = nullptr, *mid16 = nullptr;
  float *expert_y = nullptr;
  int32_t *place = nullptr, *tiles = nullptr, *counts = nullptr;
};
struct LayeredState {
  int dtype = B200_F32;
  b200_stack_config stack{1.f, 0, 0, 1, 0};
  std::vector<LayeredLayer> layers;
  std::vector<LayeredRun> runs;
  RowMatrix embed;             // also the output head
  RowMatrix side_embed;        // [vocab][layers * side_dim]
  float *final_norm = nullptr;
  std::map<std::string, LayeredTensor> tensors;
  std::vector<void *> owned;
  int32_t *zero = nullptr;     // sequence 0, page 0: the session's block table
  int ldp = 0, ldc = 0, ldq = 0, max_mid = 0, max_ff = 0, max_top = 0, max_experts = 0;
  int max_q = 0, max_row = 0, max_kv = 0, max_plain = 0, max_mem = 0, max_mem_heads = 0;
  int64_t max_state = 0;
  bool sandwich = false, memory = false;   // some layer is one / has one
  int window = 0;              // the widest window of all layers, 0: some layer sees everything
  int state_pos = 0;           // the position the session's recurrent state has reached, -1: unknown
  LayeredWs one, many;         // the captured decode step's rows, and everything else's
  float *x_want = nullptr;     // rows whose logits are asked for
  bf16 *h_want = nullptr;
  float *logits = nullptr;
  int32_t *want = nullptr, *next = nullptr;
  int want_cap = 0;
  void *gemm_ws = nullptr;     // error word, split-k partial tiles
  bf16 *keys16 = nullptr, *kv16 = nullptr;   // a prompt segment's cache rows, and their expanded keys and values
  int64_t key_rows = 0;
  float *mem_U = nullptr;      // the matrix memory's states between the chunks of a step
  double *mem_meta = nullptr;
  int64_t mem_chunks = 0;
};
struct RowSegment {            // consecutive rows of one sequence
  int row0, n, seq, pos0;
};

} // namespace b200

struct b200_model {
  b200_model_config cfg{};
  int tp = 1, rank = 0;
  int qh = 0, kvh = 0, ffn = 0, vocab = 0;  // local (sharded) sizes
  float *embed = nullptr, *inv_freq = nullptr, *final_norm = nullptr;
  std::vector<b200::Layer> layers;
  b200::DevLinear lm_head;
  std::vector<float *> kv;
  float **kv_dev = nullptr;
  float *x = nullptr, *qkv = nullptr, *attn = nullptr, *mid = nullptr,
        *part = nullptr, *logits = nullptr, *logits_shard = nullptr;
  float *attn_scratch = nullptr, *argmax_scratch = nullptr;
  float *kv_stage = nullptr;  // [2*layers][kv_heads*D]: the rows written this step
  int32_t *d_state = nullptr;  // token, pos, next, count, launches, -, error, -
  int32_t *d_history = nullptr;
  int history_cap = 0;
  int splits = 1;
  cudaStream_t stream = nullptr;
  cudaGraph_t graph = nullptr;
  cudaGraphExec_t exec = nullptr;
  cudaEvent_t ev0 = nullptr, ev1 = nullptr;
  float last_ms = 0.f;
  int kernels_per_step = 0;
  bool finalized = false;
  float *h_logits_pinned = nullptr;
  float *h_rows_pinned = nullptr;   // this step's K/V rows, fetched together with the logits
  bool rows_fresh = false;
  int32_t *h_state_pinned = nullptr;
  // persistent decode-step kernel (batch 1, int8): see mega.cu
  bool mega = false;
  b200::MegaParams mp{};
  int mega_grid = 0;
  size_t mega_smem = 0;
  int64_t mega_stream_bytes = 0;
  uint8_t *mega_stream = nullptr;
  int64_t *mega_offsets = nullptr;   // [(4L+1)+1][grid]: per-phase and per-CTA stream offsets
  const float **lvec_dev = nullptr;
  uint2 *ll_buf = nullptr;           // tagged activation buffers
  long long *d_trace = nullptr;
  // prefill (many rows at once): activations of all rows, grown on demand
  float *pf_x = nullptr, *pf_qkv = nullptr, *pf_att = nullptr, *pf_mid = nullptr, *pf_logits = nullptr;
  float *pf_norm = nullptr;   // W8A8 only: the normalised rows of a projection
  bool act_int8 = false;   // the w8a8 variant: int8 projections quantise their activations per call
  uint32_t *q_row = nullptr;   // decode: the quantised activation row of the current projection
  float *q_scale = nullptr;    //         and its scale
  cudaGraph_t graph_q = nullptr;      // the decode step with int8 activations, captured on first use
  cudaGraphExec_t exec_q = nullptr;
  int kernels_per_step_q = 0;
  void *pf_ws = nullptr;
  int32_t *pf_tokens = nullptr;
  int pf_rows = 0, pf_logit_rows = 0;
  int64_t pf_ws_bytes = 0;
  // tensor-parallel sums by peer stores (see TpPush): this rank's staging buffer and everybody's
  uint2 *tp_ll = nullptr;
  void *tp_opened[b200::kTpMaxRanks] = {};
  b200::TpPush tp_push{};   // ranks == 0: the NCCL all-reduce is used instead
  b200::LayeredState *lay = nullptr;   // a model of described layers (b200_model_create_layered): what it keeps
  size_t tp_argmax_at = 0;   // pair offset of the (value, index) exchange slots inside the staging buffers
};


struct b200_batch {
  b200_model *m = nullptr;
  int max_seqs = 0, page = 0, n_pages = 0, table_stride = 0;
  std::vector<float *> pool;            // [2 * layers] page pools [n_pages][kv_heads][page][D]
  std::vector<b200::LayerCache> caches;   // described layers, per run: page pools [n_pages][page][row], states [max_seqs]
  std::vector<int> first;               // per sequence: first page still held (pages behind every window go back)
  std::vector<int> free_pages;
  std::vector<int> len;                 // per sequence: -1 = unused slot
  std::vector<int32_t> table;           // [max_seqs][table_stride] host mirror
  int32_t *d_table = nullptr, *d_seq = nullptr, *d_pos = nullptr, *d_next = nullptr;
  float *d_part = nullptr;              // attention partials of the key-split scan, for up to part_rows rows
  int part_rows = 0, max_context = 0;
  int rows_cap = 0;
  float last_ms = 0.f;
};

namespace b200 {
int model_allocate(const b200_model_config &c, b200_model **out);   // engine.cu
// layered.cu
void layered_destroy(b200_model *m);
int layered_ready(b200_model *m);                       // every tensor set?
int layered_issue_step(b200_model *m, cudaStream_t st); // one decode step of the session from d_state, for capture
int layered_rows(b200_model *m, int M, const int32_t *tokens, const int32_t *row_seq, const int32_t *row_pos,
                 const int32_t *table_dev, int table_stride, int page, const LayerCache *caches, int max_ctx, int n_want,
                 const int32_t *want, float *logits_host, int32_t *next_host);
int layered_session_rows(b200_model *m, int M, const int32_t *tokens, int pos0, int n_want, const int32_t *want,
                         float *logits_host, int32_t *next_host);   // on the session's own cache
// Caches of every run for `positions` cached rows and `slots` recurrent states; and their release.
int layered_caches_create(const b200_model *m, int64_t positions, int slots, std::vector<LayerCache> *out);
void layered_caches_free(const b200_model *m, std::vector<LayerCache> *caches);
// The session is about to run from position pos: its recurrent state must have reached it.
int layered_state_enter(b200_model *m, int pos);
void layered_state_leave(b200_model *m, int pos);
int layered_status(b200_model *m);                      // after a synchronise: did a bounded wait give up?
int layered_clear_cache(b200_model *m);
int layered_kv_overflow(b200_model *m, int position, int keep, int *new_position);
int64_t layered_step_bytes(const b200_model *m, int ctx);
} // namespace b200
