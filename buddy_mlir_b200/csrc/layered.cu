// Models of described layers: creation, loading by tensor name, and the step over M rows of any
// mix of sequences.  The session's decode step (captured into a CUDA graph), its prefill and the
// batch calls of engine.cu all come through layered_rows / layered_issue_step; what differs is
// where a row's cache lines are (CacheView): the session's contiguous cache is one page.
//
// A parallel block x += mixer(h) + ff(h), h = RMSNorm(x), runs as
//   in    one contraction of the normalised row with every matrix that reads it: queries, latent
//         and key part, router logits, and the (gate, up) pairs of a dense feed-forward (gated in
//         the epilogue)
//   latent attention over the cache (latent.cu)
//   out   one contraction of [attention | gated feed-forward] with [W_o | W_down], added to x
// or, with experts, their own two contractions (gemv_rows.cu, experts.cu).
//
// A sandwich block norms what a sublayer returns before it is added, so the sum cannot be part of
// the sublayer's last contraction: that leaves its result y, and whatever next reads the stream
// settles it, x += RMSNorm(y) * w, before it norms x for its own use (the prologue of
// gemv_rows_kernel for one row, settle_rows_kernel for more).  The embedding row added before a
// new pass of a loop is settled in the same place; the per-token layer input is one more sublayer.
//   in    q, k, v, gates of every mixer of the layer: one contraction (with biases)
//   heads.cu attention over the cache, memory.cu recurrent state, side by side
//   out   one contraction of [attention | memory] with [W_o | W_o']
//   up, down; side gate, side proj
#include "engine.cuh"

#include <algorithm>
#include <cmath>
#include <cstring>

namespace b200 {

namespace {

// src rows [rows][cols] (row-major, tight) -> dst row (row0 + r * step), columns col0..
template <typename S, typename D>
__global__ void place_rows_kernel(const S *src, int cols, D *dst, int64_t ld, int64_t row0, int64_t step, int64_t col0) {
  const int64_t r = blockIdx.x;
  for (int c = threadIdx.x; c < cols; c += blockDim.x)
    dst[(row0 + r * step) * ld + col0 + c] = from_float<D>(to_float(src[r * cols + c]));
}

template <typename T>
__global__ void __launch_bounds__(256)
embed_table_kernel(const T *table, int64_t ld, const int32_t *tokens, float *x, int H, float scale) {
  constexpr int E = RowUnit<T>::E;
  const T *src = table + (int64_t)tokens[blockIdx.x] * ld;
  float *dst = x + (int64_t)blockIdx.x * H;
  for (int k = threadIdx.x * E; k < H; k += 256 * E) {   // rows are padded to whole units
    const uint4 u = *reinterpret_cast<const uint4 *>(src + k);
#pragma unroll
    for (int g = 0; g < RowUnit<T>::NG; ++g) {
      float f[4];
      RowUnit<T>::group(u, g, f);
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (k + 4 * g + e < H)
          dst[k + 4 * g + e] = f[e] * scale;
    }
  }
}

// h = RMSNorm(x) as bf16 rows of ldh (zero beyond H): a CTA per row
__global__ void __launch_bounds__(256)
norm_rows_kernel(const float *x, int H, const float *norm_w, float eps, bf16 *h, int64_t ldh) {
  __shared__ float s_red[8];
  const int m = blockIdx.x;
  const float *src = x + (int64_t)m * H;
  const bool vec = (H & 3) == 0;
  float s = 0.f;
  if (vec)
    for (int k = threadIdx.x * 4; k < H; k += 1024) {
      const float4 v = *reinterpret_cast<const float4 *>(src + k);
      s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    }
  else
    for (int k = threadIdx.x; k < H; k += 256)
      s = fmaf(src[k], src[k], s);
  s = warp_sum(s);
  if ((threadIdx.x & 31) == 0)
    s_red[threadIdx.x >> 5] = s;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < 8; ++w)
    t += s_red[w];
  const float r = 1.0f / sqrtf(t / (float)H + eps);
  bf16 *dst = h + (int64_t)m * ldh;
  if (vec) {
    for (int k = threadIdx.x * 4; k < ldh; k += 1024) {
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f), w = v;
      if (k < H) {
        v = *reinterpret_cast<const float4 *>(src + k);
        w = __ldg(reinterpret_cast<const float4 *>(norm_w + k));
      }
      const __nv_bfloat162 a = __floats2bfloat162_rn(v.x * r * w.x, v.y * r * w.y), b = __floats2bfloat162_rn(v.z * r * w.z, v.w * r * w.w);
      *reinterpret_cast<uint2 *>(dst + k) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
    }
  } else {
    for (int k = threadIdx.x; k < ldh; k += 256)
      dst[k] = __float2bfloat16_rn(k < H ? src[k] * r * norm_w[k] : 0.f);
  }
}

__device__ __forceinline__ float cta_sum(float s, float *s_red) {   // 256 threads
  s = warp_sum(s);
  __syncthreads();
  if ((threadIdx.x & 31) == 0)
    s_red[threadIdx.x >> 5] = s;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < 8; ++w)
    t += s_red[w];
  return t;
}

// grid M: x_out = x + what is unsettled (x_out may be x); h (rows of ldh, zero beyond H):
// RMSNorm(x_out) * norm_w, or x_out itself where norm_w is null.  VEC: four elements per thread and
// step (H % 4 == 0).  T: the embedding table's type.
template <typename T, typename D, bool VEC>
__global__ void __launch_bounds__(256)
settle_rows_kernel(const float *x, float *x_out, int H, const Unsettled u, float eps, const float *norm_w, D *h, int64_t ldh) {
  constexpr int E = VEC ? 4 : 1;
  __shared__ float s_red[8];
  const int m = blockIdx.x;
  const float *src = x + (int64_t)m * H;
  float *row = x_out + (int64_t)m * H;
  const float *y = u.y != nullptr ? u.y + (int64_t)m * H : nullptr;
  auto read = [](const float *p, float (&v)[E]) {
    if constexpr (VEC) {
      const float4 t = *reinterpret_cast<const float4 *>(p);
      v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    } else {
      v[0] = *p;
    }
  };
  float r = 0.f;
  if (y != nullptr) {
    float s = 0.f;
    for (int k = threadIdx.x * E; k < H; k += 256 * E) {
      float v[E];
      read(y + k, v);
#pragma unroll
      for (int e = 0; e < E; ++e)
        s = fmaf(v[e], v[e], s);
    }
    r = 1.0f / sqrtf(cta_sum(s, s_red) / (float)H + eps);
  }
  const T *emb = u.embed != nullptr ? reinterpret_cast<const T *>(u.embed) + (int64_t)u.tokens[m] * u.lde : nullptr;
  float s = 0.f;
  for (int k = threadIdx.x * E; k < H; k += 256 * E) {
    float v[E];
    read(src + k, v);
    if (y != nullptr) {
      float a[E], b[E];
      read(y + k, a);
      read(u.w + k, b);
#pragma unroll
      for (int e = 0; e < E; ++e)
        v[e] = fmaf(a[e] * r, b[e], v[e]);
    }
#pragma unroll
    for (int e = 0; e < E; ++e) {
      if (emb != nullptr)
        v[e] = fmaf(to_float(emb[k + e]), u.scale, v[e]);
      s = fmaf(v[e], v[e], s);
    }
    if constexpr (VEC)
      *reinterpret_cast<float4 *>(row + k) = make_float4(v[0], v[1], v[2], v[3]);
    else
      row[k] = v[0];
  }
  if (h == nullptr)
    return;
  const float rx = norm_w != nullptr ? 1.0f / sqrtf(cta_sum(s, s_red) / (float)H + eps) : 1.f;
  D *dst = h + (int64_t)m * ldh;
  for (int k = threadIdx.x * E; k < ldh; k += 256 * E) {
    float v[E] = {};
    if (k < H) {
      read(row + k, v);          // what this thread wrote
      if (norm_w != nullptr) {
        float b[E];
        read(norm_w + k, b);
#pragma unroll
        for (int e = 0; e < E; ++e)
          v[e] = v[e] * rx * b[e];
      }
    }
    if constexpr (VEC && sizeof(D) == 2) {
      const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
      *reinterpret_cast<uint2 *>(dst + k) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
    } else {
#pragma unroll
      for (int e = 0; e < E; ++e)
        dst[k + e] = from_float<D>(v[e]);
    }
  }
}

__global__ void __launch_bounds__(256)
gather_rows_kernel(const float *x, const int32_t *rows, float *y, int H) {
  const float *src = x + (int64_t)rows[blockIdx.x] * H;
#pragma unroll 4
  for (int i = threadIdx.x; i < H; i += 256)
    y[(int64_t)blockIdx.x * H + i] = src[i];
}

int64_t pad_to(int64_t n, int64_t a) { return (n + a - 1) / a * a; }

int own_alloc(std::vector<void *> &owned, void **p, size_t bytes) {
  if (int rc = dev_alloc(p, bytes)) return rc;
  owned.push_back(*p);
  B200_CUDA(cudaMemset(*p, 0, bytes ? bytes : 16));
  return B200_OK;
}
template <typename T> int own_array(std::vector<void *> &owned, T **p, int64_t n) {
  return own_alloc(owned, (void **)p, (size_t)(n > 0 ? n : 1) * sizeof(T));
}
size_t elem(int dtype) { return dtype == B200_F32 ? 4 : 2; }

void release(std::vector<void *> &owned) {
  for (void *p : owned)
    cudaFree(p);
  owned.clear();
}

int make_matrix(LayeredState *s, RowMatrix *w, int64_t N, int64_t K) {
  w->N = (int)N;
  w->K = (int)K;
  w->ld = pad_to(K, 8);
  return own_alloc(s->owned, &w->w, (size_t)N * w->ld * elem(s->dtype));
}

void add_rows(LayeredState *s, const std::string &name, const RowMatrix &w, int rows, int cols, int64_t row0,
              int64_t step = 1, int64_t col0 = 0) {
  s->tensors[name] = LayeredTensor{rows, cols, s->dtype, w.w, w.ld, row0, step, col0, false};
}
int add_vector(LayeredState *s, const std::string &name, float **p, int n) {
  if (int rc = own_array(s->owned, p, n)) return rc;
  s->tensors[name] = LayeredTensor{1, n, B200_F32, *p, n, 0, 1, 0, false};
  return B200_OK;
}

LatentDims latent_dims(const b200_layer_config &c) {
  LatentDims d{};
  d.heads = c.heads; d.dim = c.dim; d.rot = c.rot_dim; d.vdim = c.vdim; d.rank = c.kv_rank;
  d.window = c.window;
  d.scale = c.scale;
  d.row = pad_to(d.rank + d.rot, 8);
  return d;
}
HeadsDims heads_dims(const b200_layer_config &c) {
  HeadsDims d{};
  d.heads = c.heads; d.kv = c.kv_heads; d.dim = c.dim; d.vdim = c.vdim; d.rot = c.rot_dim;
  d.halves = c.rot_halves;
  d.window = c.window;
  d.scale = c.scale;
  d.sink = c.sink;
  d.dimp = (int)pad_to(d.dim, 8);
  d.vdimp = (int)pad_to(d.vdim, 8);
  d.row = (int64_t)d.kv * (d.dimp + d.vdimp);
  return d;
}
MemoryDims memory_dims(const b200_layer_config &c) {
  MemoryDims d{};
  d.heads = c.mem_heads; d.dim = c.mem_dim; d.vdim = c.mem_vdim;
  d.cap = c.mem_cap; d.q_scale = c.mem_q_scale; d.floor = c.mem_floor;
  d.tiles = (d.vdim + 31) / 32;
  d.head_state = pad_to((int64_t)d.dim * d.tiles * 32 + (int64_t)d.tiles * (d.dim + 2), 32);
  d.state = d.heads * d.head_state;
  return d;
}

int check_layer(const b200_layer_config &c, int i, const b200_layer_config *all) {
  if (c.mixer < B200_MIX_LATENT || c.mixer > B200_MIX_HEADS_MEMORY)
    return fail(B200_EINVAL, "create_layered: layer %d has an unknown mixer %d", i, c.mixer);
  LayeredLayer L;
  L.cfg = c;
  if (c.block != (L.latent() ? B200_BLOCK_PARALLEL : B200_BLOCK_SANDWICH))
    return fail(B200_EINVAL, "create_layered: layer %d: latent layers are parallel blocks, the others sandwiches", i);
  if (L.latent())
    if (int rc = latent_limits(latent_dims(c))) return rc;
  if (L.heads()) {
    if (int rc = heads_limits(heads_dims(c))) return rc;
    if (std::isnan(c.sink) || c.sink == INFINITY || !std::isfinite(c.mix_scale))
      return fail(B200_EINVAL, "create_layered: layer %d: bad sink or factor", i);
  }
  if (L.memory()) {
    if (int rc = memory_limits(memory_dims(c))) return rc;
    if (!std::isfinite(c.mem_q_scale) || !(c.mem_floor >= 0.f) || !std::isfinite(c.mem_mix_scale))
      return fail(B200_EINVAL, "create_layered: layer %d: bad constants of the matrix memory", i);
  }
  if ((L.latent() || L.heads()) && (c.window < 0 || !std::isfinite(c.scale) || !(c.rot_base > 0.f)))
    return fail(B200_EINVAL, "create_layered: layer %d: bad window, scale or rotation base", i);
  if (L.latent() && c.kv_from >= 0) {
    if (c.kv_from >= i || all[c.kv_from].mixer != B200_MIX_LATENT || all[c.kv_from].kv_from >= 0)
      return fail(B200_EINVAL, "create_layered: layer %d takes the cache of layer %d, which has none of its own before it", i, c.kv_from);
    const b200_layer_config &o = all[c.kv_from];
    if (o.kv_rank != c.kv_rank || o.rot_dim != c.rot_dim || o.rot_base != c.rot_base)
      return fail(B200_EINVAL, "create_layered: layer %d and the layer whose cache it takes differ in latent or rotation", i);
  }
  const bool known = L.latent() ? c.ff_kind == B200_FF_NONE || c.ff_kind == B200_FF_GATED || c.ff_kind == B200_FF_EXPERTS
                                : c.ff_kind == B200_FF_NONE || c.ff_kind == B200_FF_PLAIN;
  if (!known)
    return fail(B200_EINVAL, "create_layered: layer %d has an unknown feed-forward %d", i, c.ff_kind);
  if (c.ff_kind == B200_FF_PLAIN && (c.ff < 1 || c.ff_act < B200_ACT_NONE || c.ff_act > B200_ACT_GELU_TANH))
    return fail(B200_EINVAL, "create_layered: layer %d: bad feed-forward", i);
  if ((c.ff_kind == B200_FF_GATED || c.ff_kind == B200_FF_EXPERTS) && (c.ff < 1 || !(c.limit > 0.f)))
    return fail(B200_EINVAL, "create_layered: layer %d: bad feed-forward", i);
  if (c.ff_kind == B200_FF_EXPERTS && (c.experts < 1 || c.top < 1 || c.top > c.experts || c.experts > 1024))
    return fail(B200_EINVAL, "create_layered: layer %d: %d of %d experts", i, c.top, c.experts);
  return B200_OK;
}

template <typename F> int rotation(LayeredState *s, F **dst, int dims, float base) {
  std::vector<F> f((size_t)std::max(1, dims / 2));
  for (int k = 0; k < dims / 2; ++k)
    f[(size_t)k] = (F)std::pow((double)base, -2.0 * k / dims);
  if (int rc = own_array(s->owned, dst, (int64_t)f.size())) return rc;
  B200_CUDA(cudaMemcpy(*dst, f.data(), f.size() * sizeof(F), cudaMemcpyHostToDevice));
  return B200_OK;
}

// Attention over per-head keys and / or a matrix memory, in a sandwich block.
int build_sandwich(LayeredState *s, LayeredLayer &L, int i, int W) {
  const b200_layer_config &c = L.cfg;
  const std::string p = "l" + std::to_string(i) + ".";
  const bool both = L.heads() && L.memory();
  const std::string hp = p + (both ? "mix.left." : "mix."), mp = p + (both ? "mix.right." : "mix.");
  int n = 0;
  auto part = [&](int rows) {    // parts start at multiples of eight rows
    const int at = n;
    n += (int)pad_to(rows, 8);
    return at;
  };
  HeadsDims &d = L.h;
  MemoryDims &e = L.mem;
  int nq = 0, nk = 0, nv = 0, mq = 0, mv = 0;
  if (L.heads()) {
    d = heads_dims(c);
    L.att = d.heads * d.vdim;
    nq = d.heads * d.dim; nk = d.kv * d.dim; nv = d.kv * d.vdim;
    part(nq);
    L.off_k = part(nk);
    L.off_v = part(nv);
    if (c.out_gate) L.off_g = part(L.att);
  }
  if (L.memory()) {
    e = memory_dims(c);
    mq = e.heads * e.dim; mv = e.heads * e.vdim;
    L.off_mq = part(mq);
    L.off_mk = part(mq);
    L.off_mv = part(mv);
    L.off_mg = part(mv);
    L.off_mi = part(e.heads);
    L.off_mf = part(e.heads);
    L.mem_col = (int)pad_to(L.att, 8);
  }
  L.plain = n;
  if (int rc = make_matrix(s, &L.in, n, W)) return rc;
  if (int rc = make_matrix(s, &L.out, W, L.memory() ? L.mem_col + mv : L.att)) return rc;
  if (c.qkv_bias || L.memory())
    if (int rc = own_array(s->owned, &L.in_bias, n)) return rc;
  auto bias = [&](const std::string &name, int rows, int at) {
    s->tensors[name] = LayeredTensor{1, rows, B200_F32, L.in_bias + at, rows, 0, 1, 0, false};
  };
  if (L.heads()) {
    add_rows(s, hp + "q", L.in, nq, W, 0);
    add_rows(s, hp + "k", L.in, nk, W, L.off_k);
    add_rows(s, hp + "v", L.in, nv, W, L.off_v);
    add_rows(s, hp + "o", L.out, W, L.att, 0);
    if (c.out_gate) add_rows(s, hp + "g", L.in, L.att, W, L.off_g);
    if (c.qkv_bias) {
      bias(hp + "q.b", nq, 0);
      bias(hp + "k.b", nk, L.off_k);
      bias(hp + "v.b", nv, L.off_v);
    }
    if (c.qk_norm) {
      if (int rc = add_vector(s, hp + "q.norm", &L.q_norm, nq)) return rc;
      if (int rc = add_vector(s, hp + "k.norm", &L.k_norm, nk)) return rc;
    }
    if (int rc = rotation(s, &L.freq, d.rot, c.rot_base)) return rc;
  }
  if (L.memory()) {
    add_rows(s, mp + "q", L.in, mq, W, L.off_mq);
    add_rows(s, mp + "k", L.in, mq, W, L.off_mk);
    add_rows(s, mp + "v", L.in, mv, W, L.off_mv);
    add_rows(s, mp + "g", L.in, mv, W, L.off_mg);
    add_rows(s, mp + "i", L.in, e.heads, W, L.off_mi);
    add_rows(s, mp + "f", L.in, e.heads, W, L.off_mf);
    bias(mp + "i.b", e.heads, L.off_mi);
    bias(mp + "f.b", e.heads, L.off_mf);
    add_rows(s, mp + "o", L.out, W, mv, 0, 1, L.mem_col);
    if (int rc = add_vector(s, mp + "norm", &L.mem_norm, mv)) return rc;
    s->memory = true;
  }
  if (int rc = add_vector(s, p + "norm1", &L.norm, W)) return rc;
  if (int rc = add_vector(s, p + "norm1b", &L.norm_b, W)) return rc;
  if (int rc = add_vector(s, p + "norm2", &L.norm2, W)) return rc;
  if (int rc = add_vector(s, p + "norm2b", &L.norm2_b, W)) return rc;
  if (c.ff_kind == B200_FF_NONE) {
    s->tensors[p + "norm2"].set = s->tensors[p + "norm2b"].set = true;
  } else {
    if (int rc = make_matrix(s, &L.up, c.ff, W)) return rc;
    if (int rc = make_matrix(s, &L.down, W, c.ff)) return rc;
    add_rows(s, p + "mlp.up", L.up, c.ff, W, 0);
    add_rows(s, p + "mlp.down", L.down, W, c.ff, 0);
    s->max_plain = std::max(s->max_plain, c.ff);
  }
  if (const int side = s->stack.side_dim) {
    if (int rc = make_matrix(s, &L.side_gate, side, W)) return rc;
    if (int rc = make_matrix(s, &L.side_proj, W, side)) return rc;
    add_rows(s, p + "side.gate", L.side_gate, side, W, 0);
    add_rows(s, p + "side.proj", L.side_proj, W, side, 0);
    if (int rc = add_vector(s, p + "side.norm", &L.side_norm, W)) return rc;
    s->max_plain = std::max(s->max_plain, side);
  }
  s->sandwich = true;
  s->ldp = std::max(s->ldp, n);
  s->ldc = std::max(s->ldc, (int)L.out.ld);
  s->max_q = std::max(s->max_q, d.heads * d.dimp);
  s->max_row = std::max(s->max_row, (int)L.row());
  s->max_mem = std::max(s->max_mem, (int)pad_to(mv, 4));
  s->max_mem_heads = std::max(s->max_mem_heads, e.heads);
  s->max_state = std::max(s->max_state, e.state);
  return B200_OK;
}

int build_layer(LayeredState *s, LayeredLayer &L, int i, int W) {
  const b200_layer_config &c = L.cfg;
  if (!L.latent())
    return build_sandwich(s, L, i, W);
  LatentDims &d = L.d;
  d = latent_dims(c);
  L.att = d.heads * d.vdim;
  L.gate = Gate{c.limit, c.gate_slope, c.up_offset};
  const bool dense = c.ff_kind == B200_FF_GATED, experts = c.ff_kind == B200_FF_EXPERTS;
  const int nq = d.heads * (d.dim + d.rot);
  int n = nq;
  L.off_down = n;
  if (L.own()) n += d.rank + d.rot;
  L.off_router = n;
  if (experts) n += c.experts;
  L.plain = (int)pad_to(n, 4);
  const std::string p = "l" + std::to_string(i) + ".";
  if (int rc = make_matrix(s, &L.in, L.plain + (dense ? 2 * c.ff : 0), W)) return rc;
  add_rows(s, p + "mix.q", L.in, nq, W, 0);
  if (L.own()) add_rows(s, p + "mix.dkv", L.in, d.rank + d.rot, W, L.off_down);
  if (experts) add_rows(s, p + "mlp.router", L.in, c.experts, W, L.off_router);
  if (int rc = make_matrix(s, &L.ukv, (int64_t)d.heads * (d.dim + d.vdim), d.rank)) return rc;
  L.uk = L.uv = L.ukv;
  L.uk.N = d.heads * d.dim;
  L.uv.N = L.att;
  L.uv.w = (char *)L.ukv.w + (size_t)L.uk.N * L.ukv.ld * elem(s->dtype);
  add_rows(s, p + "mix.uk", L.uk, L.uk.N, d.rank, 0);
  add_rows(s, p + "mix.uv", L.uv, L.uv.N, d.rank, 0);
  if (int rc = make_matrix(s, &L.out, W, L.att + (dense ? c.ff : 0))) return rc;
  add_rows(s, p + "mix.o", L.out, W, L.att, 0);
  if (dense) {
    add_rows(s, p + "mlp.gate", L.in, c.ff, W, L.plain, 2);
    add_rows(s, p + "mlp.up", L.in, c.ff, W, L.plain + 1, 2);
    add_rows(s, p + "mlp.down", L.out, W, c.ff, 0, 1, L.att);
  }
  if (experts) {
    if (int rc = make_matrix(s, &L.expert_in, (int64_t)c.experts * 2 * c.ff, W)) return rc;
    if (int rc = make_matrix(s, &L.expert_out, (int64_t)c.experts * W, c.ff)) return rc;
    for (int e = 0; e < c.experts; ++e) {
      const std::string q = p + "mlp.e" + std::to_string(e) + ".";
      add_rows(s, q + "gate", L.expert_in, c.ff, W, (int64_t)e * 2 * c.ff, 2);
      add_rows(s, q + "up", L.expert_in, c.ff, W, (int64_t)e * 2 * c.ff + 1, 2);
      add_rows(s, q + "down", L.expert_out, W, c.ff, (int64_t)e * W);
    }
  }
  if (int rc = add_vector(s, p + "norm1", &L.norm, W)) return rc;
  if (L.own())
    if (int rc = add_vector(s, p + "mix.dkv.norm", &L.down_norm, d.rank)) return rc;
  if (int rc = rotation(s, &L.inv_freq, d.rot, c.rot_base)) return rc;
  s->ldp = std::max(s->ldp, (int)pad_to(L.plain, 4));
  s->ldc = std::max(s->ldc, (int)L.out.ld);
  s->ldq = std::max(s->ldq, d.heads * (d.rank + d.rot));
  s->max_q = std::max(s->max_q, nq);
  s->max_row = std::max(s->max_row, (int)d.row);
  s->max_kv = std::max(s->max_kv, (int)pad_to(L.ukv.N, 8));
  if (experts) {
    s->max_mid = std::max(s->max_mid, c.top * c.ff);
    s->max_top = std::max(s->max_top, c.top);
    s->max_ff = std::max(s->max_ff, c.ff);
    s->max_experts = std::max(s->max_experts, c.experts);
  }
  return B200_OK;
}

// From this many rows on a bfloat16 model contracts on the tensor cores; a run of consecutive
// rows of one sequence of this length expands its keys (latent_prefill.cu).
constexpr int kDenseRows = 9, kExpandRows = 17;
constexpr int kPlanInts = 10;            // of a StepPlan, per row: segments, tiles, chunks, single rows

bool dense(const LayeredState *s, int M) { return s->dtype == B200_BF16 && M >= kDenseRows; }

// Activations for up to `rows` rows, contexts up to `ctx` positions.
int reserve(b200_model *m, LayeredWs &ws, int rows, int ctx) {
  LayeredState *s = m->lay;
  if (rows <= ws.rows && ctx <= ws.ctx)
    return B200_OK;
  rows = std::max(rows, ws.rows);
  ctx = std::max(ctx, ws.ctx);
  B200_CUDA(cudaStreamSynchronize(m->stream));
  release(ws.owned);
  ws = LayeredWs();
  const int W = m->cfg.hidden;
  int64_t part = 0;
  for (const LayeredLayer &L : s->layers)
    for (int r = 1; r <= rows; r = r < 600 || r == rows ? r + 1 : rows) {   // beyond that many rows there is one share
      if (L.latent())
        part = std::max(part, latent_scratch_floats(L.d, r, latent_splits(L.d, r, ctx)));
      else if (L.heads())
        part = std::max(part, heads_scratch_floats(L.h, r, heads_splits(L.h, r, ctx)));
    }
  auto &o = ws.owned;
  int rc = own_array(o, &ws.x, (int64_t)rows * W);
  if (!rc) rc = own_array(o, &ws.proj, (int64_t)rows * s->ldp);
  if (!rc) rc = own_array(o, &ws.qabs, (int64_t)rows * s->ldq);
  if (!rc) rc = own_array(o, &ws.part, part);
  if (!rc) rc = own_array(o, &ws.cat, (int64_t)rows * s->ldc);
  if (!rc) rc = own_array(o, &ws.mid, (int64_t)rows * std::max(s->max_mid, s->max_plain));
  if (!rc) rc = own_array(o, &ws.weight, (int64_t)rows * s->max_top);
  if (!rc) rc = own_array(o, &ws.ids, (int64_t)rows * s->max_top);
  if (!rc) rc = own_array(o, &ws.row_seq, rows);
  if (!rc) rc = own_array(o, &ws.row_pos, rows);
  if (!rc) rc = own_array(o, &ws.tokens, rows);
  if (!rc) rc = own_array(o, &ws.plan, (int64_t)rows * kPlanInts);
  if (s->sandwich) {
    if (!rc) rc = own_array(o, &ws.x2, (int64_t)W);
    if (!rc) rc = own_array(o, &ws.y, (int64_t)rows * W);
    if (!rc) rc = own_array(o, &ws.h32, (int64_t)rows * W);
    if (!rc) rc = own_array(o, &ws.mem_o, (int64_t)rows * s->max_mem);
    if (!rc) rc = own_alloc(o, &ws.q, (size_t)rows * s->max_q * elem(s->dtype));
  }
  if (dense(s, rows)) {
    const int64_t slots = (int64_t)rows * s->max_top;
    if (!rc) rc = own_array(o, &ws.h16, rows * pad_to(W, 8));
    if (!rc) rc = own_array(o, &ws.cat16, (int64_t)rows * s->ldc);
    if (!rc) rc = own_array(o, &ws.q16, (int64_t)rows * s->max_q);
    if (!rc) rc = own_array(o, &ws.mid16, std::max(slots * pad_to(s->max_ff, 8), rows * pad_to(s->max_plain, 8)));
    if (s->max_top > 0) {
      if (!rc) rc = own_array(o, &ws.x16, slots * pad_to(W, 8));
      if (!rc) rc = own_array(o, &ws.expert_y, slots * W);
      if (!rc) rc = own_array(o, &ws.place, slots);
      if (!rc) rc = own_array(o, &ws.counts, s->max_experts + 4);
      if (!rc) rc = own_array(o, &ws.tiles, 4 * (int64_t)experts_max_tiles((int)slots, s->max_experts));
    }
    if (!rc && !s->gemm_ws) rc = own_alloc(s->owned, &s->gemm_ws, (size_t)gemm_bf16_workspace_bytes());
  }
  if (rc) {
    release(ws.owned);
    ws = LayeredWs();
    return rc;
  }
  ws.rows = rows;
  ws.ctx = ctx;
  return B200_OK;
}

int norm_rows_launch(const float *x, int H, int M, const float *norm_w, float eps, bf16 *h, int64_t ldh,
                     cudaStream_t st) {
  norm_rows_kernel<<<M, 256, 0, st>>>(x, H, norm_w, eps, h, ldh);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

// The stream of M rows, and what has not been added to it yet.
struct Stream {
  float *x;
  float *spare;                // room for one row: one row is settled from one buffer into the other
  int M;
  const int32_t *tokens;
  const float *y = nullptr;    // x += RMSNorm(y) * w
  const float *w = nullptr;
  bool again = false;          // x += scaled embedding row
  bool pending() const { return y != nullptr || again; }
};

Unsettled unsettled(const b200_model *m, const Stream &z) {
  const LayeredState *s = m->lay;
  return Unsettled{z.y, z.w, z.again ? s->embed.w : nullptr, s->embed.ld, s->stack.embed_scale, z.tokens};
}
void settled(Stream &z, float *x) {
  if (x != z.x) {
    z.spare = z.x;
    z.x = x;
  }
  z.y = z.w = nullptr;
  z.again = false;
}

template <typename T, typename D>
int settle_typed(b200_model *m, Stream &z, float *x_out, const float *norm_w, D *h, int64_t ldh, cudaStream_t st) {
  const int W = m->cfg.hidden;
  if (W % 4 == 0)
    settle_rows_kernel<T, D, true><<<z.M, 256, 0, st>>>(z.x, x_out, W, unsettled(m, z), m->cfg.eps, norm_w, h, ldh);
  else
    settle_rows_kernel<T, D, false><<<z.M, 256, 0, st>>>(z.x, x_out, W, unsettled(m, z), m->cfg.eps, norm_w, h, ldh);
  B200_LAUNCH_CHECK();
  settled(z, x_out);
  return B200_OK;
}
// Settle the stream into x_out; h: its norm under norm_w (or the stream itself) as rows of ldh, or null.
template <typename D>
int settle(b200_model *m, Stream &z, float *x_out, const float *norm_w, D *h, int64_t ldh, cudaStream_t st) {
  return m->lay->dtype == B200_F32 ? settle_typed<float>(m, z, x_out, norm_w, h, ldh, st)
                                   : settle_typed<bf16>(m, z, x_out, norm_w, h, ldh, st);
}

// y = act(norm(stream) w^T + bias), GEMV-shaped; norm_w null: the stream itself.
int rows_from_stream(b200_model *m, LayeredWs &ws, Stream &z, const RowMatrix &w, const float *norm_w, const float *bias,
                     const RowAct &act, float *y, int64_t ldy, cudaStream_t st) {
  const int W = m->cfg.hidden;
  GemvRows g;
  g.w = w; g.ldx = W; g.M = z.M; g.bias = bias; g.act = act; g.y = y; g.ldy = ldy; g.eps = m->cfg.eps;
  if (!z.pending()) {
    g.x = z.x;
    g.norm_w = norm_w;
  } else if (gemv_rows_settles(z.M, W)) {
    g.x = z.x;
    g.norm_w = norm_w;
    g.late = unsettled(m, z);
    g.x_out = z.spare;
    settled(z, g.x_out);
  } else {
    if (int rc = settle(m, z, z.x, norm_w, norm_w ? ws.h32 : nullptr, W, st)) return rc;
    g.x = norm_w ? ws.h32 : z.x;
  }
  return gemv_rows_launch(m->lay->dtype, g, st);
}

MixFinish finish_of(const LayeredState *s, const LayeredWs &ws, const LayeredLayer &L, float eps, bool heads, bool memory) {
  MixFinish f;
  f.proj = ws.proj; f.ldp = s->ldp; f.ldc = s->ldc;
  if (heads) {
    f.n_heads = L.h.heads; f.h = L.h; f.part = ws.part; f.off_g = L.off_g; f.h_scale = L.cfg.mix_scale;
  }
  if (memory) {
    f.n_mem = L.mem.heads; f.mem_vdim = L.mem.vdim; f.mem_col = L.mem_col; f.off_mg = L.off_mg;
    f.mem_o = ws.mem_o; f.ldo = s->max_mem; f.mem_norm = L.mem_norm; f.m_scale = L.cfg.mem_mix_scale; f.eps = eps;
  }
  return f;
}
HeadsIn heads_in(const LayeredState *s, const LayeredWs &ws, const LayeredLayer &L, float eps) {
  return HeadsIn{ws.proj, s->ldp, L.off_k, L.off_v, L.q_norm, L.k_norm, eps, L.freq};
}
MemoryIn memory_in(const LayeredState *s, const LayeredWs &ws, const LayeredLayer &L) {
  return MemoryIn{ws.proj, s->ldp, L.off_mq, L.off_mk, L.off_mv, L.off_mi, L.off_mf};
}
// The activation of the per-token input's gate: gelu times the layer's part of the token's row.
RowAct side_act(const LayeredState *s, int layer, const int32_t *tokens) {
  const size_t at = (size_t)layer * s->stack.side_dim * elem(s->dtype);
  return RowAct{B200_ACT_GELU_TANH, (const char *)s->side_embed.w + at, s->dtype == B200_F32, s->side_embed.ld, tokens};
}

// One sandwich layer over M rows, GEMV-shaped.
int row_sandwich(b200_model *m, LayeredWs &ws, Stream &z, const LayeredLayer &L, int layer, const LayerCache &cache,
                 const CacheView &cv, const StepPlan &plan, cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden, M = z.M;
  const float eps = m->cfg.eps;
  // y = x w^T, to be added to the stream under the norm norm_w
  auto to_stream = [&](const RowMatrix &w, const float *x, int64_t ldx, const float *norm_w) {
    GemvRows g;
    g.w = w; g.x = x; g.ldx = ldx; g.M = M; g.y = ws.y; g.ldy = W;
    z.y = ws.y;
    z.w = norm_w;
    return gemv_rows_launch(s->dtype, g, st);
  };
  if (int rc = rows_from_stream(m, ws, z, L.in, L.norm, L.in_bias, RowAct{}, ws.proj, s->ldp, st)) return rc;
  MixFinish f = finish_of(s, ws, L, eps, L.heads(), L.memory());
  f.cat = ws.cat;
  if (L.heads()) {
    if (int rc = heads_prep_launch(s->dtype, L.h, heads_in(s, ws, L, eps), M, ws.q, cache.rows, cv, st)) return rc;
    f.splits = heads_splits(L.h, M, plan.ctx);
    if (int rc = heads_attend_launch(s->dtype, L.h, ws.q, nullptr, M, cache.rows, cv, f.splits, ws.part, st)) return rc;
  }
  if (L.memory())
    if (int rc = memory_step_launch(L.mem, memory_in(s, ws, L), plan.segs, plan.n_long + plan.n_short, cv.row_pos, cache.state,
                                    ws.mem_o, s->max_mem, st))
      return rc;
  if (int rc = mix_finish_launch(f, M, st)) return rc;
  if (int rc = to_stream(L.out, ws.cat, s->ldc, L.norm_b)) return rc;
  if (L.cfg.ff_kind == B200_FF_PLAIN) {
    RowAct act{};
    act.kind = L.cfg.ff_act;
    if (int rc = rows_from_stream(m, ws, z, L.up, L.norm2, nullptr, act, ws.mid, s->max_plain, st)) return rc;
    if (int rc = to_stream(L.down, ws.mid, s->max_plain, L.norm2_b)) return rc;
  }
  if (s->stack.side_dim > 0) {
    if (int rc = rows_from_stream(m, ws, z, L.side_gate, nullptr, nullptr, side_act(s, layer, z.tokens), ws.mid, s->max_plain, st))
      return rc;
    if (int rc = to_stream(L.side_proj, ws.mid, s->max_plain, L.side_norm)) return rc;
  }
  return B200_OK;
}

// All layers over M rows, GEMV-shaped (few rows, or 32-bit).
int row_layers(b200_model *m, LayeredWs &ws, Stream &z, const CacheView &cv, const StepPlan &plan, const LayerCache *caches,
               int max_ctx, cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden, M = z.M;
  const float eps = m->cfg.eps;
  for (const LayeredRun &run : s->runs) {
    LayeredLayer &L = s->layers[run.layer];
    const LayerCache &cache = caches[run.source];
    z.again = run.again;
    if (!L.latent()) {
      if (int rc = row_sandwich(m, ws, z, L, run.layer, cache, cv, plan, st)) return rc;
      continue;
    }
    if (z.pending())
      if (int rc = settle<float>(m, z, z.x, nullptr, nullptr, 0, st)) return rc;
    float *x = z.x;
    const b200_layer_config &c = L.cfg;
    GemvRows in;
    in.w = L.in; in.x = x; in.ldx = W; in.M = M; in.norm_w = L.norm; in.eps = eps; in.y = ws.proj; in.ldy = s->ldp;
    in.pair_from = L.plain; in.y2 = ws.cat + L.att; in.ldy2 = s->ldc; in.gate = L.gate;
    if (int rc = gemv_rows_launch(s->dtype, in, st)) return rc;
    void *pool = cache.rows;
    if (int rc = latent_prep_launch(s->dtype, L.d, ws.proj, s->ldp, M, L.uk, L.inv_freq, ws.qabs, L.own(), L.off_down,
                                    L.down_norm, eps, pool, cv, st))
      return rc;
    const int splits = latent_splits(L.d, M, max_ctx);
    if (int rc = latent_attend_launch(s->dtype, L.d, ws.qabs, M, pool, cv, splits, max_ctx, ws.part, st)) return rc;
    if (int rc = latent_value_launch(s->dtype, L.d, ws.part, M, splits, L.uv, ws.cat, s->ldc, false, nullptr, st)) return rc;
    if (c.ff_kind == B200_FF_EXPERTS) {
      if (int rc = expert_rows_launch(s->dtype, L.expert_in, L.expert_out, c.ff, c.experts, c.top, L.gate, x, W, M,
                                      L.norm, eps, ws.proj + L.off_router, s->ldp, &L.out, ws.cat, s->ldc, ws.mid,
                                      ws.ids, ws.weight, st))
        return rc;
    } else {
      GemvRows out;
      out.w = L.out; out.x = ws.cat; out.ldx = s->ldc; out.M = M; out.y = x; out.ldy = W; out.add = true;
      if (int rc = gemv_rows_launch(s->dtype, out, st)) return rc;
    }
  }
  return B200_OK;
}

// Room for a segment's gathered cache rows and expanded keys.
int reserve_keys(b200_model *m, int64_t n) {
  LayeredState *s = m->lay;
  if (n <= s->key_rows)
    return B200_OK;
  B200_CUDA(cudaStreamSynchronize(m->stream));
  cudaFree(s->keys16);
  cudaFree(s->kv16);
  s->keys16 = s->kv16 = nullptr;
  s->key_rows = 0;
  if (int rc = dev_alloc((void **)&s->keys16, (size_t)n * s->max_row * 2)) return rc;
  if (int rc = dev_alloc((void **)&s->kv16, (size_t)n * s->max_kv * 2)) return rc;
  s->key_rows = n;
  return B200_OK;
}

// Room for the matrix memory's states between n chunks.
int reserve_chunks(b200_model *m, int64_t n) {
  LayeredState *s = m->lay;
  if (n <= s->mem_chunks)
    return B200_OK;
  B200_CUDA(cudaStreamSynchronize(m->stream));
  cudaFree(s->mem_U);
  cudaFree(s->mem_meta);
  s->mem_U = nullptr;
  s->mem_meta = nullptr;
  s->mem_chunks = 0;
  if (int rc = dev_alloc((void **)&s->mem_U, (size_t)n * s->max_state * 4)) return rc;
  if (int rc = dev_alloc((void **)&s->mem_meta, (size_t)n * s->max_mem_heads * 3 * 8)) return rc;
  s->mem_chunks = n;
  return B200_OK;
}

// The attention of one layer for all rows, bf16: long runs of a sequence over expanded keys,
// what lies between them in the single-query form.
int dense_attention(b200_model *m, LayeredWs &ws, LayeredLayer &L, int M, const CacheView &cv,
                    const std::vector<RowSegment> &segs, void *pool, int max_ctx, cudaStream_t st) {
  LayeredState *s = m->lay;
  const LatentDims &d = L.d;
  auto singles = [&](int r0, int n) {
    CacheView c = cv;
    c.row_seq += r0;
    c.row_pos += r0;
    const int splits = latent_splits(d, n, max_ctx);
    if (int rc = latent_prep_launch(s->dtype, d, ws.proj + (int64_t)r0 * s->ldp, s->ldp, n, L.uk, L.inv_freq, ws.qabs,
                                    false, 0, nullptr, 0.f, pool, c, st))
      return rc;
    if (int rc = latent_attend_launch(s->dtype, d, ws.qabs, n, pool, c, splits, max_ctx, ws.part, st)) return rc;
    return latent_value_launch(s->dtype, d, ws.part, n, splits, L.uv, ws.cat16 + (int64_t)r0 * s->ldc, s->ldc, true, ws.qabs, st);
  };
  int begin = 0;                         // first row not yet attended for
  for (const RowSegment &g : segs) {
    if (g.n < kExpandRows || !latent_prefill_takes(d))
      continue;
    if (g.row0 > begin)
      if (int rc = singles(begin, g.row0 - begin)) return rc;
    begin = g.row0 + g.n;
    const int first = d.window > 0 ? std::max(0, g.pos0 - d.window + 1) : 0;
    const int keys = g.pos0 + g.n - first;
    if (int rc = reserve_keys(m, keys)) return rc;
    if (int rc = latent_gather_launch(d, pool, cv, g.seq, first, keys, s->keys16, st)) return rc;
    GemmBf16 e;
    e.A = s->keys16; e.lda = d.row; e.M = keys; e.w = L.ukv; e.C16 = s->kv16; e.ldc = pad_to(L.ukv.N, 8);
    if (int rc = gemm_bf16_launch(e, s->gemm_ws, st)) return rc;
    if (int rc = latent_query_launch(d, ws.proj + (int64_t)g.row0 * s->ldp, s->ldp, g.n, L.inv_freq, cv.row_pos + g.row0,
                                     ws.q16, st))
      return rc;
    if (int rc = latent_prefill_launch(d, ws.q16, g.n, g.pos0, s->keys16, s->kv16, e.ldc, first,
                                       ws.cat16 + (int64_t)g.row0 * s->ldc, s->ldc, st))
      return rc;
  }
  return begin < M ? singles(begin, M - begin) : B200_OK;
}

// One sandwich layer over M rows on the tensor cores.
int dense_sandwich(b200_model *m, LayeredWs &ws, Stream &z, const LayeredLayer &L, int layer, const LayerCache &cache,
                   const CacheView &cv, const StepPlan &plan, cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden, M = z.M;
  const float eps = m->cfg.eps;
  const int64_t ldh = pad_to(W, 8), ldm = pad_to(s->max_plain, 8);
  auto from_stream = [&](const RowMatrix &w, const float *norm_w, const float *bias, const RowAct &act, float *y, bf16 *y16, int64_t ldy) {
    GemmBf16 g;
    if (int rc = settle(m, z, z.x, norm_w, ws.h16, ldh, st)) return rc;
    g.A = ws.h16; g.lda = ldh; g.M = M; g.w = w; g.bias = bias; g.act = act; g.C = y; g.C16 = y16; g.ldc = ldy;
    return gemm_bf16_launch(g, s->gemm_ws, st);
  };
  auto to_stream = [&](const RowMatrix &w, const bf16 *a, int64_t lda, const float *norm_w) {
    GemmBf16 g;
    g.A = a; g.lda = lda; g.M = M; g.w = w; g.C = ws.y; g.ldc = W;
    z.y = ws.y;
    z.w = norm_w;
    return gemm_bf16_launch(g, s->gemm_ws, st);
  };
  if (int rc = from_stream(L.in, L.norm, L.in_bias, RowAct{}, ws.proj, nullptr, s->ldp)) return rc;
  if (L.heads()) {
    const bf16 *q = (const bf16 *)ws.q, *pool = (const bf16 *)cache.rows;
    if (int rc = heads_prep_launch(s->dtype, L.h, heads_in(s, ws, L, eps), M, ws.q, cache.rows, cv, st)) return rc;
    const bool tiled = heads_tensor_cores(L.h);
    if (tiled && plan.n_tiles > 0)
      if (int rc = heads_prefill_launch(L.h, q, plan.tiles, plan.n_tiles, pool, cv, L.off_g >= 0 ? ws.proj + L.off_g : nullptr,
                                        s->ldp, L.cfg.mix_scale, ws.cat16, s->ldc, st))
        return rc;
    const int n = tiled ? plan.n_singles : M;
    if (n > 0) {
      MixFinish f = finish_of(s, ws, L, eps, true, false);
      f.rows = tiled ? plan.singles : nullptr;
      f.cat16 = ws.cat16;
      f.splits = heads_splits(L.h, n, plan.ctx);
      if (int rc = heads_attend_launch(s->dtype, L.h, ws.q, f.rows, n, pool, cv, f.splits, ws.part, st)) return rc;
      if (int rc = mix_finish_launch(f, n, st)) return rc;
    }
  }
  if (L.memory()) {
    const MemoryIn in = memory_in(s, ws, L);
    const int chunked = memory_chunks_take(L.mem) ? plan.n_long : 0, stepped = plan.n_long + plan.n_short - chunked;
    if (chunked > 0) {
      if (int rc = reserve_chunks(m, plan.n_chunks)) return rc;
      const MemoryChunks k{plan.segs, plan.chunks, plan.chunk0, chunked, plan.n_chunks, s->mem_U, s->mem_meta};
      if (int rc = memory_chunk_launch(L.mem, in, k, cv.row_pos, cache.state, ws.mem_o, s->max_mem, st)) return rc;
    }
    if (stepped > 0)
      if (int rc = memory_step_launch(L.mem, in, plan.segs + chunked, stepped, cv.row_pos, cache.state, ws.mem_o, s->max_mem, st))
        return rc;
    MixFinish f = finish_of(s, ws, L, eps, false, true);
    f.cat16 = ws.cat16;
    if (int rc = mix_finish_launch(f, M, st)) return rc;
  }
  if (int rc = to_stream(L.out, ws.cat16, s->ldc, L.norm_b)) return rc;
  if (L.cfg.ff_kind == B200_FF_PLAIN) {
    RowAct act{};
    act.kind = L.cfg.ff_act;
    if (int rc = from_stream(L.up, L.norm2, nullptr, act, nullptr, ws.mid16, ldm)) return rc;
    if (int rc = to_stream(L.down, ws.mid16, ldm, L.norm2_b)) return rc;
  }
  if (s->stack.side_dim > 0) {
    if (int rc = from_stream(L.side_gate, nullptr, nullptr, side_act(s, layer, z.tokens), nullptr, ws.mid16, ldm)) return rc;
    if (int rc = to_stream(L.side_proj, ws.mid16, ldm, L.side_norm)) return rc;
  }
  return B200_OK;
}

// All layers over M rows on the tensor cores (bfloat16 models, more than a handful of rows).
int dense_layers(b200_model *m, LayeredWs &ws, Stream &z, const CacheView &cv, const std::vector<RowSegment> &segs,
                 const StepPlan &plan, const LayerCache *caches, int max_ctx, cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden, M = z.M;
  const int64_t ldh = pad_to(W, 8);
  for (const LayeredRun &run : s->runs) {
    LayeredLayer &L = s->layers[run.layer];
    const LayerCache &cache = caches[run.source];
    z.again = run.again;
    if (!L.latent()) {
      if (int rc = dense_sandwich(m, ws, z, L, run.layer, cache, cv, plan, st)) return rc;
      continue;
    }
    if (z.pending())
      if (int rc = settle<float>(m, z, z.x, nullptr, nullptr, 0, st)) return rc;
    float *x = z.x;
    const b200_layer_config &c = L.cfg;
    void *pool = cache.rows;
    if (int rc = norm_rows_launch(x, W, M, L.norm, m->cfg.eps, ws.h16, ldh, st)) return rc;
    GemmBf16 in;
    in.A = ws.h16; in.lda = ldh; in.M = M; in.w = L.in; in.w.N = L.plain; in.C = ws.proj; in.ldc = s->ldp;
    if (int rc = gemm_bf16_launch(in, s->gemm_ws, st)) return rc;
    if (L.own())
      if (int rc = latent_store_launch(L.d, ws.proj, s->ldp, M, L.off_down, L.down_norm, m->cfg.eps, L.inv_freq, pool, cv, st))
        return rc;
    if (int rc = dense_attention(m, ws, L, M, cv, segs, pool, max_ctx, st)) return rc;
    if (c.ff_kind == B200_FF_GATED) {
      GemmBf16 g;
      g.A = ws.h16; g.lda = ldh; g.M = M; g.w = L.in;
      g.w.w = (bf16 *)L.in.w + (int64_t)L.plain * L.in.ld;
      g.w.N = 2 * c.ff;
      g.C16 = ws.cat16 + L.att; g.ldc = s->ldc; g.pairs = true; g.gate = L.gate;
      if (int rc = gemm_bf16_launch(g, s->gemm_ws, st)) return rc;
    }
    GemmBf16 o;
    o.A = ws.cat16; o.lda = s->ldc; o.M = M; o.w = L.out; o.C = x; o.ldc = W; o.add = true;
    if (c.ff_kind == B200_FF_EXPERTS) {
      const int slots = M * c.top;
      int4 *tiles = (int4 *)ws.tiles;
      int32_t *n_tiles = ws.counts + s->max_experts;
      const int64_t ldm = pad_to(c.ff, 8);
      if (int rc = experts_sort_launch(ws.proj + L.off_router, s->ldp, c.experts, c.top, M, ws.h16, ldh, ws.ids, ws.weight,
                                       ws.counts, tiles, n_tiles, ws.place, ws.x16, st))
        return rc;
      GemmBf16 g;
      g.A = ws.x16; g.lda = ldh; g.M = slots; g.w = L.expert_in; g.C16 = ws.mid16; g.ldc = ldm; g.pairs = true;
      g.gate = L.gate; g.tiles = tiles; g.n_tiles = n_tiles; g.groups = c.experts;
      g.max_tiles = experts_max_tiles(slots, c.experts);
      if (int rc = gemm_bf16_launch(g, s->gemm_ws, st)) return rc;
      GemmBf16 dn;
      dn.A = ws.mid16; dn.lda = ldm; dn.M = slots; dn.w = L.expert_out; dn.C = ws.expert_y; dn.ldc = W;
      dn.tiles = tiles; dn.n_tiles = n_tiles; dn.groups = c.experts; dn.max_tiles = g.max_tiles;
      if (int rc = gemm_bf16_launch(dn, s->gemm_ws, st)) return rc;
      if (int rc = gemm_bf16_launch(o, s->gemm_ws, st)) return rc;
      if (int rc = experts_combine_launch(x, W, c.top, M, ws.expert_y, ws.place, ws.weight, st)) return rc;
    } else if (int rc = gemm_bf16_launch(o, s->gemm_ws, st)) {
      return rc;
    }
  }
  return B200_OK;
}

int embed_tokens(b200_model *m, const int32_t *tokens, float *x, int M, cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden;
  if (s->dtype == B200_F32)
    embed_table_kernel<float><<<M, 256, 0, st>>>((const float *)s->embed.w, s->embed.ld, tokens, x, W, s->stack.embed_scale);
  else
    embed_table_kernel<bf16><<<M, 256, 0, st>>>((const bf16 *)s->embed.w, s->embed.ld, tokens, x, W, s->stack.embed_scale);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

int head(b200_model *m, const float *x, int n, float *logits, cudaStream_t st) {
  LayeredState *s = m->lay;
  if (dense(s, n) && s->gemm_ws) {
    const int64_t ldh = pad_to(m->cfg.hidden, 8);
    if (int rc = norm_rows_launch(x, m->cfg.hidden, n, s->final_norm, m->cfg.eps, s->h_want, ldh, st)) return rc;
    GemmBf16 g;
    g.A = s->h_want; g.lda = ldh; g.M = n; g.w = s->embed; g.C = logits; g.ldc = m->cfg.vocab;
    return gemm_bf16_launch(g, s->gemm_ws, st);
  }
  GemvRows g;
  g.w = s->embed; g.x = x; g.ldx = m->cfg.hidden; g.M = n; g.norm_w = s->final_norm; g.eps = m->cfg.eps;
  g.y = logits; g.ldy = m->cfg.vocab;
  return gemv_rows_launch(s->dtype, g, st);
}

} // namespace

int layered_ready(b200_model *m) {
  for (const auto &t : m->lay->tensors)
    if (!t.second.set)
      return fail(B200_ESTATE, "finalize: tensor %s is missing", t.first.c_str());
  return B200_OK;
}

void layered_destroy(b200_model *m) {
  LayeredState *s = m->lay;
  if (!s) return;
  for (size_t i = 0; i < s->runs.size(); ++i) {
    if (s->runs[i].source == (int)i) cudaFree(s->runs[i].cache.rows);
    cudaFree(s->runs[i].cache.state);
  }
  release(s->one.owned);
  release(s->many.owned);
  release(s->owned);
  cudaFree(s->x_want); cudaFree(s->h_want); cudaFree(s->logits); cudaFree(s->want); cudaFree(s->next);
  cudaFree(s->keys16); cudaFree(s->kv16); cudaFree(s->mem_U); cudaFree(s->mem_meta);
  delete s;
  m->lay = nullptr;
}

int layered_clear_cache(b200_model *m) {
  LayeredState *s = m->lay;
  for (const LayeredRun &r : s->runs)
    if (r.cache.rows)
      B200_CUDA(cudaMemsetAsync(r.cache.rows, 0, (size_t)m->cfg.max_len * s->layers[r.layer].row() * elem(s->dtype), m->stream));
  return B200_OK;
}

int layered_caches_create(const b200_model *m, int64_t positions, int slots, std::vector<LayerCache> *out) {
  const LayeredState *s = m->lay;
  out->assign(s->runs.size(), LayerCache{});
  for (size_t i = 0; i < s->runs.size(); ++i) {
    const LayeredLayer &L = s->layers[s->runs[i].layer];
    LayerCache &c = (*out)[i];
    if (s->runs[i].source != (int)i) {
      c.rows = (*out)[s->runs[i].source].rows;
    } else if (L.row() > 0) {
      const size_t bytes = (size_t)positions * L.row() * elem(s->dtype);
      if (int rc = dev_alloc(&c.rows, bytes)) return rc;
      B200_CUDA(cudaMemset(c.rows, 0, bytes));     // padding elements of a row are read and never written
    }
    if (L.state() > 0)
      if (int rc = dev_alloc((void **)&c.state, (size_t)slots * L.state() * 4)) return rc;
  }
  return B200_OK;
}

void layered_caches_free(const b200_model *m, std::vector<LayerCache> *caches) {
  for (size_t i = 0; i < caches->size(); ++i) {
    if (m->lay->runs[i].source == (int)i) cudaFree((*caches)[i].rows);
    cudaFree((*caches)[i].state);
  }
  caches->clear();
}

int layered_state_enter(b200_model *m, int pos) {
  LayeredState *s = m->lay;
  if (s->memory && pos != 0 && pos != s->state_pos)
    return fail(B200_ESTATE, "the recurrent state is at position %d, not %d: run from there or from 0", s->state_pos, pos);
  s->state_pos = -1;           // until the step has succeeded
  return B200_OK;
}
void layered_state_leave(b200_model *m, int pos) { m->lay->state_pos = pos; }

// The session's cache is full: keep the first `keep` positions, drop half of the rest, move what
// remains up to them (the same choice of rows as b200_kv_overflow).  A recurrent state has no
// positions: it keeps what the dropped tokens left in it.
int layered_kv_overflow(b200_model *m, int position, int keep, int *new_position) {
  LayeredState *s = m->lay;
  const int max_len = m->cfg.max_len;
  if (position < max_len) {
    *new_position = -1;
    return B200_OK;
  }
  const int cur = max_len;
  keep = std::max(0, std::min(keep, cur - 1));
  const int discard = std::max(1, (cur - keep) / 2), src = keep + discard, tail = cur - src;
  cudaStream_t st = m->stream;
  void *stage = nullptr;
  if (int rc = dev_alloc(&stage, (size_t)std::max(1, tail) * s->max_row * elem(s->dtype))) return rc;
  int rc = B200_OK;
  for (size_t i = 0; i < s->runs.size() && !rc; ++i) {
    const LayeredLayer &L = s->layers[s->runs[i].layer];
    char *cache = (char *)s->runs[i].cache.rows;
    if (s->runs[i].source != (int)i || !cache)
      continue;
    const size_t row = (size_t)L.row() * elem(s->dtype);
    if (tail > 0) {
      rc = L.latent() ? latent_shift_launch(s->dtype, L.d, cache, src, tail, L.inv_freq, -discard, stage, st)
                      : heads_shift_launch(s->dtype, L.h, cache, src, tail, L.freq, -discard, stage, st);
      if (!rc && cudaMemcpyAsync(cache + keep * row, stage, tail * row, cudaMemcpyDeviceToDevice, st) != cudaSuccess)
        rc = fail(B200_ECUDA, "kv_overflow: moving the cache rows failed");
    }
    if (!rc && cudaMemsetAsync(cache + (keep + tail) * row, 0, (cur - keep - tail) * row, st) != cudaSuccess)
      rc = fail(B200_ECUDA, "kv_overflow: clearing the cache rows failed");
  }
  if (cudaStreamSynchronize(st) != cudaSuccess && !rc)
    rc = fail(B200_ECUDA, "kv_overflow: %s", cudaGetErrorString(cudaGetLastError()));
  cudaFree(stage);
  *new_position = cur - discard;
  if (!rc && s->state_pos == position)
    s->state_pos = *new_position;
  return rc;
}

int layered_issue_step(b200_model *m, cudaStream_t st) {
  LayeredState *s = m->lay;
  const bool first = s->one.rows == 0;
  if (int rc = reserve(m, s->one, 1, m->cfg.max_len)) return rc;
  if (first) {                 // one segment of one row of sequence 0
    const int32_t seg[4] = {0, 1, 0, 0};
    B200_CUDA(cudaMemcpy(s->one.plan, seg, sizeof seg, cudaMemcpyHostToDevice));
  }
  std::vector<LayerCache> caches;
  for (const LayeredRun &r : s->runs)
    caches.push_back(r.cache);
  const CacheView cv{s->zero, m->d_state + 1, s->zero, 1, m->cfg.max_len};
  StepPlan plan;
  plan.segs = (const int4 *)s->one.plan;
  plan.n_short = 1;
  plan.ctx = m->cfg.max_len;
  Stream z{m->x, s->one.x2, 1, m->d_state};
  if (int rc = embed_tokens(m, m->d_state, m->x, 1, st)) return rc;
  if (int rc = row_layers(m, s->one, z, cv, plan, caches.data(), m->cfg.max_len, st)) return rc;
  return rows_from_stream(m, s->one, z, s->embed, s->final_norm, nullptr, RowAct{}, m->logits, m->cfg.vocab, st);
}

// The rows' segments, and what the kernels of a step want to know about them, on the device.
static int make_plan(LayeredWs &ws, const std::vector<RowSegment> &segs, bool dense_rows, StepPlan *plan, cudaStream_t st) {
  std::vector<int32_t> h;
  auto quad = [&](int a, int b, int c, int d) { h.insert(h.end(), {a, b, c, d}); };
  auto is_long = [&](const RowSegment &g) { return dense_rows && g.n >= kExpandRows; };
  for (const RowSegment &g : segs) {
    plan->ctx = std::max(plan->ctx, g.pos0 + g.n);
    if (is_long(g)) {
      quad(g.row0, g.n, g.seq, g.pos0);
      plan->n_long += 1;
    }
  }
  for (const RowSegment &g : segs)
    if (!is_long(g)) {
      quad(g.row0, g.n, g.seq, g.pos0);
      plan->n_short += 1;
    }
  const size_t tiles = h.size();
  for (const RowSegment &g : segs)
    if (is_long(g))
      for (int r = 0; r < g.n; r += kHeadsQueryTile) {
        quad(g.row0 + r, std::min(kHeadsQueryTile, g.n - r), g.seq, g.pos0 + r);
        plan->n_tiles += 1;
      }
  const size_t chunks = h.size();
  std::vector<int32_t> chunk0;
  for (const RowSegment &g : segs)
    if (is_long(g)) {
      chunk0.push_back(plan->n_chunks);
      for (int r = 0; r < g.n; r += kMemoryChunk) {
        quad(g.row0 + r, std::min(kMemoryChunk, g.n - r), g.seq, g.pos0 + r);
        plan->n_chunks += 1;
      }
    }
  const size_t firsts = h.size();
  h.insert(h.end(), chunk0.begin(), chunk0.end());
  const size_t singles = h.size();
  if (dense_rows)
    for (const RowSegment &g : segs)
      if (!is_long(g))
        for (int r = 0; r < g.n; ++r)
          h.push_back(g.row0 + r);
  plan->n_singles = (int)(h.size() - singles);
  B200_CUDA(cudaMemcpyAsync(ws.plan, h.data(), h.size() * 4, cudaMemcpyHostToDevice, st));   // pageable: copied before it returns
  plan->segs = (const int4 *)ws.plan;
  plan->tiles = (const int4 *)(ws.plan + tiles);
  plan->chunks = (const int4 *)(ws.plan + chunks);
  plan->chunk0 = ws.plan + firsts;
  plan->singles = ws.plan + singles;
  return B200_OK;
}

// M rows (host arrays) of any sequences, in chunks of rows; the logits of the `want` rows.
int layered_rows(b200_model *m, int M, const int32_t *tokens, const int32_t *row_seq, const int32_t *row_pos,
                 const int32_t *table_dev, int table_stride, int page, const LayerCache *caches, int max_ctx, int n_want,
                 const int32_t *want, float *logits_host, int32_t *next_host) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden;
  cudaStream_t st = m->stream;
  const int chunk = s->dtype == B200_F32 ? 512 : 4096;
  if (int rc = reserve(m, s->many, std::min(M, chunk), max_ctx)) return rc;
  if (n_want > s->want_cap) {
    B200_CUDA(cudaStreamSynchronize(st));
    cudaFree(s->x_want); cudaFree(s->h_want); cudaFree(s->logits); cudaFree(s->want); cudaFree(s->next);
    s->x_want = s->logits = nullptr;
    s->h_want = nullptr;
    s->want = s->next = nullptr;
    s->want_cap = 0;
    if (int rc = dev_alloc((void **)&s->x_want, (size_t)n_want * W * 4)) return rc;
    if (int rc = dev_alloc((void **)&s->h_want, (size_t)n_want * pad_to(W, 8) * 2)) return rc;
    if (int rc = dev_alloc((void **)&s->logits, (size_t)n_want * m->cfg.vocab * 4)) return rc;
    if (int rc = dev_alloc((void **)&s->want, (size_t)n_want * 4)) return rc;
    if (int rc = dev_alloc((void **)&s->next, (size_t)n_want * 4)) return rc;
    s->want_cap = n_want;
  }
  LayeredWs &ws = s->many;
  std::vector<int32_t> local;
  int done = 0;                          // wanted rows gathered so far
  for (int m0 = 0; m0 < M; m0 += chunk) {
    const int n = std::min(chunk, M - m0);
    B200_CUDA(cudaMemcpyAsync(ws.tokens, tokens + m0, (size_t)n * 4, cudaMemcpyHostToDevice, st));
    B200_CUDA(cudaMemcpyAsync(ws.row_seq, row_seq + m0, (size_t)n * 4, cudaMemcpyHostToDevice, st));
    B200_CUDA(cudaMemcpyAsync(ws.row_pos, row_pos + m0, (size_t)n * 4, cudaMemcpyHostToDevice, st));
    const CacheView cv{ws.row_seq, ws.row_pos, table_dev, table_stride, page};
    std::vector<RowSegment> segs;
    for (int r = 0; r < n; ++r) {
      const int32_t seq = row_seq[m0 + r], pos = row_pos[m0 + r];
      if (!segs.empty() && segs.back().seq == seq && segs.back().pos0 + segs.back().n == pos)
        segs.back().n += 1;
      else
        segs.push_back(RowSegment{r, 1, seq, pos});
    }
    StepPlan plan;
    if (int rc = make_plan(ws, segs, dense(s, n), &plan, st)) return rc;
    Stream z{ws.x, ws.x2, n, ws.tokens};
    if (int rc = embed_tokens(m, ws.tokens, ws.x, n, st)) return rc;
    if (dense(s, n)) {
      if (int rc = dense_layers(m, ws, z, cv, segs, plan, caches, max_ctx, st)) return rc;
    } else if (int rc = row_layers(m, ws, z, cv, plan, caches, max_ctx, st)) {
      return rc;
    }
    if (z.pending() || z.x != ws.x)
      if (int rc = settle<float>(m, z, ws.x, nullptr, nullptr, 0, st)) return rc;
    local.clear();
    for (int k = done; k < n_want && want[k] < m0 + n; ++k)
      local.push_back(want[k] - m0);
    if (!local.empty()) {
      B200_CUDA(cudaMemcpyAsync(s->want, local.data(), local.size() * 4, cudaMemcpyHostToDevice, st));
      gather_rows_kernel<<<(unsigned)local.size(), 256, 0, st>>>(ws.x, s->want, s->x_want + (int64_t)done * W, W);
      B200_LAUNCH_CHECK();
      done += (int)local.size();
      B200_CUDA(cudaStreamSynchronize(st));   // `local` is reused
    }
  }
  if (n_want > 0) {
    if (int rc = head(m, s->x_want, n_want, s->logits, st)) return rc;
    if (int rc = argmax_rows_launch(s->logits, m->cfg.vocab, n_want, s->next, st)) return rc;
    if (logits_host)
      B200_CUDA(cudaMemcpyAsync(logits_host, s->logits, (size_t)n_want * m->cfg.vocab * 4, cudaMemcpyDeviceToHost, st));
    if (next_host)
      B200_CUDA(cudaMemcpyAsync(next_host, s->next, (size_t)n_want * 4, cudaMemcpyDeviceToHost, st));
  }
  return B200_OK;
}

int layered_session_rows(b200_model *m, int M, const int32_t *tokens, int pos0, int n_want, const int32_t *want,
                         float *logits_host, int32_t *next_host) {
  // the session's cache is one page of max_len positions of one sequence
  std::vector<int32_t> rs((size_t)M, 0), rp((size_t)M);
  std::vector<LayerCache> caches;
  for (const LayeredRun &r : m->lay->runs)
    caches.push_back(r.cache);
  for (int i = 0; i < M; ++i)
    rp[(size_t)i] = pos0 + i;
  return layered_rows(m, M, tokens, rs.data(), rp.data(), m->lay->zero, 1, m->cfg.max_len, caches.data(), m->cfg.max_len, n_want,
                      want, logits_host, next_host);
}

int layered_status(b200_model *m) {
  LayeredState *s = m->lay;
  if (!s->gemm_ws)
    return B200_OK;
  int code = 0;
  B200_CUDA(cudaMemcpyAsync(&code, s->gemm_ws, 4, cudaMemcpyDeviceToHost, m->stream));
  B200_CUDA(cudaStreamSynchronize(m->stream));
  if (code == 0)
    return B200_OK;
  B200_CUDA(cudaMemsetAsync(s->gemm_ws, 0, 4, m->stream));
  return fail(B200_ECUDA, "gemm_bf16: a bounded wait gave up (code %d)", code);
}

int64_t layered_step_bytes(const b200_model *m, int ctx) {
  const LayeredState *s = m->lay;
  const int64_t e = (int64_t)elem(s->dtype), W = m->cfg.hidden;
  auto mat = [&](const RowMatrix &w) { return (int64_t)w.N * w.K * e; };
  int64_t b = (int64_t)m->cfg.vocab * W * e + W * e + W * 4;   // head, embedding row, final norm
  for (const LayeredRun &run : s->runs) {
    const LayeredLayer &L = s->layers[run.layer];
    b += mat(L.in) + mat(L.out) + mat(L.ukv) + mat(L.up) + mat(L.down) + mat(L.side_gate) + mat(L.side_proj);
    b += W * 4 * (1 + (L.norm_b != nullptr) + (L.cfg.ff_kind == B200_FF_PLAIN ? 2 : 0) + (L.side_norm != nullptr));
    if (L.cfg.ff_kind == B200_FF_EXPERTS)   // the chosen experts only
      b += (mat(L.expert_in) + mat(L.expert_out)) / L.cfg.experts * L.cfg.top;
    const int64_t seen = L.cfg.window > 0 ? std::min(L.cfg.window, ctx + 1) : ctx + 1;
    b += seen * (L.latent() ? L.d.rank + L.d.rot : L.heads() ? L.h.kv * (L.h.dim + L.h.vdim) : 0) * e;
    if (L.memory())                         // read and written
      b += (int64_t)L.mem.heads * (L.mem.dim * (L.mem.vdim + 1) + 1) * 4 * 2;
  }
  return b;
}

} // namespace b200

using namespace b200;

extern "C" {

int b200_model_create_layered(const b200_model_config *cfg, const b200_stack_config *stack, const b200_layer_config *layers,
                              int dtype, b200_model **out) {
  if (!cfg || !layers || !out)
    return fail(B200_EINVAL, "create_layered: null argument");
  if (dtype != B200_F32 && dtype != B200_BF16)
    return fail(B200_EINVAL, "create_layered: dtype must be B200_F32 or B200_BF16");
  if (cfg->hidden < 1 || cfg->n_layers < 1 || cfg->vocab < 1 || cfg->max_len < 1 || !(cfg->eps >= 0.f))
    return fail(B200_EINVAL, "create_layered: bad architecture");
  if (cfg->tp_size > 1)
    return fail(B200_EINVAL, "create_layered: single-GPU sessions only");
  const b200_stack_config sc = stack ? *stack : b200_stack_config{1.f, 0, 0, 1, 0};
  if (!std::isfinite(sc.embed_scale) || sc.loop_start < 0 || sc.loop_stop < sc.loop_start || sc.loop_stop > cfg->n_layers ||
      sc.loop_times < 1 || sc.side_dim < 0)
    return fail(B200_EINVAL, "create_layered: bad embedding factor, loop (%d .. %d, %d times) or per-token input", sc.loop_start,
                sc.loop_stop, sc.loop_times);
  for (int i = 0; i < cfg->n_layers; ++i) {
    if (int rc = check_layer(layers[i], i, layers)) return rc;
    if (sc.side_dim > 0 && layers[i].block != B200_BLOCK_SANDWICH)
      return fail(B200_EINVAL, "create_layered: layer %d: a per-token input needs sandwich blocks", i);
  }
  b200_model_config base{};
  base.hidden = cfg->hidden; base.n_layers = cfg->n_layers; base.vocab = cfg->vocab; base.max_len = cfg->max_len;
  base.eps = cfg->eps; base.head_dim = 64; base.tp_size = 1;
  b200_model *m = nullptr;
  if (int rc = model_allocate(base, &m)) return rc;
  LayeredState *s = new LayeredState();
  m->lay = s;
  s->dtype = dtype;
  s->stack = sc;
  s->layers.resize(cfg->n_layers);
  int rc = make_matrix(s, &s->embed, cfg->vocab, cfg->hidden);
  if (!rc) {
    add_rows(s, "embed", s->embed, cfg->vocab, cfg->hidden, 0);
    rc = add_vector(s, "final.norm", &s->final_norm, cfg->hidden);
  }
  if (!rc) rc = own_array(s->owned, &s->zero, 4);
  if (!rc && sc.side_dim > 0) {
    rc = make_matrix(s, &s->side_embed, cfg->vocab, (int64_t)cfg->n_layers * sc.side_dim);
    add_rows(s, "side.embed", s->side_embed, cfg->vocab, cfg->n_layers * sc.side_dim, 0);
  }
  bool all = false;
  for (int i = 0; i < cfg->n_layers && !rc; ++i) {
    LayeredLayer &L = s->layers[i];
    L.cfg = layers[i];
    rc = build_layer(s, L, i, cfg->hidden);
    if (L.latent() || L.heads()) {
      all = all || L.cfg.window == 0;
      s->window = std::max(s->window, L.cfg.window);
    }
  }
  if (all)
    s->window = 0;
  if (!rc) {
    std::vector<int> last((size_t)cfg->n_layers, 0);   // a layer's latest run
    auto run = [&](int i, bool again) {
      LayeredRun r;
      r.layer = i;
      r.again = again;
      r.source = s->layers[i].own() ? (int)s->runs.size() : last[(size_t)s->layers[i].cfg.kv_from];
      last[(size_t)i] = (int)s->runs.size();
      s->runs.push_back(r);
    };
    const bool loop = sc.loop_stop > sc.loop_start;
    for (int i = 0; i < (loop ? sc.loop_start : cfg->n_layers); ++i)
      run(i, false);
    for (int t = 0; loop && t < sc.loop_times; ++t)
      for (int i = sc.loop_start; i < sc.loop_stop; ++i)
        run(i, t > 0 && i == sc.loop_start);
    for (int i = sc.loop_stop; loop && i < cfg->n_layers; ++i)
      run(i, false);
    std::vector<LayerCache> caches;
    rc = layered_caches_create(m, cfg->max_len, 1, &caches);
    for (size_t i = 0; i < caches.size(); ++i)
      s->runs[i].cache = caches[i];
  }
  if (rc) {
    b200_model_destroy(m);
    return rc;
  }
  *out = m;
  return B200_OK;
}

int b200_model_set_tensor(b200_model *m, const char *name, int dtype, const void *host, int64_t rows, int64_t cols) {
  if (!m || !name || !host || !m->lay)
    return fail(B200_EINVAL, "set_tensor: a model of described layers, a name and data are required");
  if (m->finalized)
    return fail(B200_ESTATE, "set_tensor: model already finalised");
  if (dtype != B200_F32 && dtype != B200_BF16)
    return fail(B200_EINVAL, "set_tensor: %s: dtype must be B200_F32 or B200_BF16", name);
  auto it = m->lay->tensors.find(name);
  if (it == m->lay->tensors.end())
    return fail(B200_EINVAL, "set_tensor: the model has no tensor %s", name);
  LayeredTensor &t = it->second;
  if (rows != t.rows || cols != t.cols)
    return fail(B200_EINVAL, "set_tensor: %s is [%d, %d], got [%lld, %lld]", name, t.rows, t.cols, (long long)rows, (long long)cols);
  const size_t bytes = (size_t)rows * cols * elem(dtype);
  void *d = nullptr;
  if (int rc = dev_alloc(&d, bytes)) return rc;
  cudaStream_t st = m->stream;
  int rc = B200_OK;
  if (cudaMemcpyAsync(d, host, bytes, cudaMemcpyHostToDevice, st) != cudaSuccess)
    rc = fail(B200_ECUDA, "set_tensor: upload failed");
  if (!rc) {
    const unsigned g = (unsigned)rows;
    if (dtype == B200_F32 && t.dtype == B200_F32)
      place_rows_kernel<float, float><<<g, 256, 0, st>>>((const float *)d, (int)cols, (float *)t.dst, t.ld, t.row0, t.step, t.col0);
    else if (dtype == B200_F32)
      place_rows_kernel<float, bf16><<<g, 256, 0, st>>>((const float *)d, (int)cols, (bf16 *)t.dst, t.ld, t.row0, t.step, t.col0);
    else if (t.dtype == B200_F32)
      place_rows_kernel<bf16, float><<<g, 256, 0, st>>>((const bf16 *)d, (int)cols, (float *)t.dst, t.ld, t.row0, t.step, t.col0);
    else
      place_rows_kernel<bf16, bf16><<<g, 256, 0, st>>>((const bf16 *)d, (int)cols, (bf16 *)t.dst, t.ld, t.row0, t.step, t.col0);
    count_launch();
    if (cudaGetLastError() != cudaSuccess || cudaStreamSynchronize(st) != cudaSuccess)
      rc = fail(B200_ECUDA, "set_tensor: %s: placing the rows failed", name);
  }
  cudaFree(d);
  if (!rc)
    t.set = true;
  return rc;
}

int b200_model_read_residual(b200_model *m, float *host, int n) {
  if (!m || !host || !m->lay || n < 1 || n > m->lay->many.rows)
    return fail(B200_EINVAL, "read_residual: bad argument");
  B200_CUDA(cudaMemcpyAsync(host, m->lay->many.x, (size_t)n * m->cfg.hidden * 4, cudaMemcpyDeviceToHost, m->stream));
  B200_CUDA(cudaStreamSynchronize(m->stream));
  return B200_OK;
}

} // extern "C"
