// Models of described layers: creation, loading by tensor name, and the step over M rows of any
// mix of sequences.  The session's decode step (captured into a CUDA graph), its prefill and the
// batch calls of engine.cu all come through layered_rows / layered_issue_step; what differs is
// where a row's cache lines are (CacheView): the session's contiguous cache is one page.
//
// A layer x += mixer(h) + ff(h), h = RMSNorm(x), runs as
//   in    one contraction of the normalised row with every matrix that reads it: queries, latent
//         and key part, router logits, and the (gate, up) pairs of a dense feed-forward (gated in
//         the epilogue)
//   latent attention over the cache (latent.cu)
//   out   one contraction of [attention | gated feed-forward] with [W_o | W_down], added to x
// or, with experts, their own two contractions (gemv_rows.cu, experts.cu).
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
embed_table_kernel(const T *table, int64_t ld, const int32_t *tokens, float *x, int H) {
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
          dst[k + 4 * g + e] = f[e];
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

int check_layer(const b200_layer_config &c, int i, const b200_layer_config *all) {
  if (c.mixer != B200_MIX_LATENT)
    return fail(B200_EINVAL, "create_layered: layer %d has an unknown mixer %d", i, c.mixer);
  LatentDims d{};
  d.heads = c.heads; d.dim = c.dim; d.rot = c.rot_dim; d.vdim = c.vdim; d.rank = c.kv_rank;
  if (int rc = latent_limits(d)) return rc;
  if (c.window < 0 || !std::isfinite(c.scale) || !(c.rot_base > 0.f))
    return fail(B200_EINVAL, "create_layered: layer %d: bad window, scale or rotation base", i);
  if (c.kv_from >= 0) {
    if (c.kv_from >= i || all[c.kv_from].kv_from >= 0)
      return fail(B200_EINVAL, "create_layered: layer %d takes the cache of layer %d, which has none of its own before it", i, c.kv_from);
    const b200_layer_config &o = all[c.kv_from];
    if (o.kv_rank != c.kv_rank || o.rot_dim != c.rot_dim || o.rot_base != c.rot_base)
      return fail(B200_EINVAL, "create_layered: layer %d and the layer whose cache it takes differ in latent or rotation", i);
  }
  if (c.ff_kind != B200_FF_NONE && c.ff_kind != B200_FF_GATED && c.ff_kind != B200_FF_EXPERTS)
    return fail(B200_EINVAL, "create_layered: layer %d has an unknown feed-forward %d", i, c.ff_kind);
  if (c.ff_kind != B200_FF_NONE && (c.ff < 1 || !(c.limit > 0.f)))
    return fail(B200_EINVAL, "create_layered: layer %d: bad feed-forward", i);
  if (c.ff_kind == B200_FF_EXPERTS && (c.experts < 1 || c.top < 1 || c.top > c.experts || c.experts > 1024))
    return fail(B200_EINVAL, "create_layered: layer %d: %d of %d experts", i, c.top, c.experts);
  return B200_OK;
}

int build_layer(LayeredState *s, LayeredLayer &L, int i, int W) {
  const b200_layer_config &c = L.cfg;
  LatentDims &d = L.d;
  d.heads = c.heads; d.dim = c.dim; d.rot = c.rot_dim; d.vdim = c.vdim; d.rank = c.kv_rank;
  d.window = c.window;
  d.scale = c.scale;
  d.row = pad_to(d.rank + d.rot, 8);
  L.source = c.kv_from >= 0 ? c.kv_from : i;
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
  std::vector<float> f((size_t)std::max(1, d.rot / 2));
  for (int k = 0; k < d.rot / 2; ++k)
    f[(size_t)k] = (float)std::pow((double)c.rot_base, -2.0 * k / d.rot);
  if (int rc = own_array(s->owned, &L.inv_freq, (int64_t)f.size())) return rc;
  B200_CUDA(cudaMemcpy(L.inv_freq, f.data(), f.size() * 4, cudaMemcpyHostToDevice));
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
    for (int r = 1; r <= rows; r = r < 512 || r == rows ? r + 1 : rows)   // beyond 512 rows there is one share
      part = std::max(part, latent_scratch_floats(L.d, r, latent_splits(L.d, r, ctx)));
  auto &o = ws.owned;
  int rc = own_array(o, &ws.x, (int64_t)rows * W);
  if (!rc) rc = own_array(o, &ws.proj, (int64_t)rows * s->ldp);
  if (!rc) rc = own_array(o, &ws.qabs, (int64_t)rows * s->ldq);
  if (!rc) rc = own_array(o, &ws.part, part);
  if (!rc) rc = own_array(o, &ws.cat, (int64_t)rows * s->ldc);
  if (!rc) rc = own_array(o, &ws.mid, (int64_t)rows * s->max_mid);
  if (!rc) rc = own_array(o, &ws.weight, (int64_t)rows * s->max_top);
  if (!rc) rc = own_array(o, &ws.ids, (int64_t)rows * s->max_top);
  if (!rc) rc = own_array(o, &ws.row_seq, rows);
  if (!rc) rc = own_array(o, &ws.row_pos, rows);
  if (!rc) rc = own_array(o, &ws.tokens, rows);
  if (dense(s, rows)) {
    const int64_t slots = (int64_t)rows * s->max_top;
    if (!rc) rc = own_array(o, &ws.h16, rows * pad_to(W, 8));
    if (!rc) rc = own_array(o, &ws.cat16, (int64_t)rows * s->ldc);
    if (!rc) rc = own_array(o, &ws.q16, (int64_t)rows * s->max_q);
    if (s->max_top > 0) {
      if (!rc) rc = own_array(o, &ws.x16, slots * pad_to(W, 8));
      if (!rc) rc = own_array(o, &ws.mid16, slots * pad_to(s->max_ff, 8));
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

// All layers over M rows, GEMV-shaped (few rows, or 32-bit).
int row_layers(b200_model *m, LayeredWs &ws, float *x, int M, const CacheView &cv, void *const *pools, int max_ctx,
               cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden;
  const float eps = m->cfg.eps;
  for (LayeredLayer &L : s->layers) {
    const b200_layer_config &c = L.cfg;
    if (int rc = gemv_rows_launch(s->dtype, L.in, x, W, M, L.norm, eps, ws.proj, s->ldp, false, L.plain, ws.cat + L.att,
                                  s->ldc, L.gate, st))
      return rc;
    void *pool = pools[L.source];
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
    } else if (int rc = gemv_rows_launch(s->dtype, L.out, ws.cat, s->ldc, M, nullptr, 0.f, x, W, true, W, nullptr, 0,
                                         L.gate, st)) {
      return rc;
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

// All layers over M rows on the tensor cores (bfloat16 models, more than a handful of rows).
int dense_layers(b200_model *m, LayeredWs &ws, float *x, int M, const CacheView &cv, const std::vector<RowSegment> &segs,
                 void *const *pools, int max_ctx, cudaStream_t st) {
  LayeredState *s = m->lay;
  const int W = m->cfg.hidden;
  const int64_t ldh = pad_to(W, 8);
  for (LayeredLayer &L : s->layers) {
    const b200_layer_config &c = L.cfg;
    void *pool = pools[L.source];
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
    embed_table_kernel<float><<<M, 256, 0, st>>>((const float *)s->embed.w, s->embed.ld, tokens, x, W);
  else
    embed_table_kernel<bf16><<<M, 256, 0, st>>>((const bf16 *)s->embed.w, s->embed.ld, tokens, x, W);
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
  return gemv_rows_launch(s->dtype, s->embed, x, m->cfg.hidden, n, s->final_norm, m->cfg.eps, logits, m->cfg.vocab, false,
                          m->cfg.vocab, nullptr, 0, Gate{}, st);
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
  release(s->one.owned);
  release(s->many.owned);
  release(s->owned);
  cudaFree(s->x_want); cudaFree(s->h_want); cudaFree(s->logits); cudaFree(s->want); cudaFree(s->next);
  cudaFree(s->keys16); cudaFree(s->kv16);
  delete s;
  m->lay = nullptr;
}

int layered_clear_cache(b200_model *m) {
  LayeredState *s = m->lay;
  for (LayeredLayer &L : s->layers)
    if (L.cache)
      B200_CUDA(cudaMemsetAsync(L.cache, 0, (size_t)m->cfg.max_len * L.d.row * elem(s->dtype), m->stream));
  return B200_OK;
}

// The session's cache is full: keep the first `keep` positions, drop half of the rest, move what
// remains up to them (the same choice of rows as b200_kv_overflow).
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
  for (LayeredLayer &L : s->layers) {
    if (!L.own() || rc)
      continue;
    const size_t row = (size_t)L.d.row * elem(s->dtype);
    if (tail > 0) {
      rc = latent_shift_launch(s->dtype, L.d, L.cache, src, tail, L.inv_freq, -discard, stage, st);
      if (!rc && cudaMemcpyAsync((char *)L.cache + keep * row, stage, tail * row, cudaMemcpyDeviceToDevice, st) != cudaSuccess)
        rc = fail(B200_ECUDA, "kv_overflow: moving the cache rows failed");
    }
    if (!rc && cudaMemsetAsync((char *)L.cache + (keep + tail) * row, 0, (cur - keep - tail) * row, st) != cudaSuccess)
      rc = fail(B200_ECUDA, "kv_overflow: clearing the cache rows failed");
  }
  if (cudaStreamSynchronize(st) != cudaSuccess && !rc)
    rc = fail(B200_ECUDA, "kv_overflow: %s", cudaGetErrorString(cudaGetLastError()));
  cudaFree(stage);
  *new_position = cur - discard;
  return rc;
}

int layered_issue_step(b200_model *m, cudaStream_t st) {
  LayeredState *s = m->lay;
  if (int rc = reserve(m, s->one, 1, m->cfg.max_len)) return rc;
  std::vector<void *> pools;
  for (LayeredLayer &L : s->layers)
    pools.push_back(L.cache);
  const CacheView cv{s->zero, m->d_state + 1, s->zero, 1, m->cfg.max_len};
  if (int rc = embed_tokens(m, m->d_state, m->x, 1, st)) return rc;
  if (int rc = row_layers(m, s->one, m->x, 1, cv, pools.data(), m->cfg.max_len, st)) return rc;
  return head(m, m->x, 1, m->logits, st);
}

// M rows (host arrays) of any sequences, in chunks of rows; the logits of the `want` rows.
int layered_rows(b200_model *m, int M, const int32_t *tokens, const int32_t *row_seq, const int32_t *row_pos,
                 const int32_t *table_dev, int table_stride, int page, void *const *pools, int max_ctx, int n_want,
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
    if (int rc = embed_tokens(m, ws.tokens, ws.x, n, st)) return rc;
    if (dense(s, n)) {
      std::vector<RowSegment> segs;
      for (int r = 0; r < n; ++r) {
        const int32_t seq = row_seq[m0 + r], pos = row_pos[m0 + r];
        if (!segs.empty() && segs.back().seq == seq && segs.back().pos0 + segs.back().n == pos)
          segs.back().n += 1;
        else
          segs.push_back(RowSegment{r, 1, seq, pos});
      }
      if (int rc = dense_layers(m, ws, ws.x, n, cv, segs, pools, max_ctx, st)) return rc;
    } else if (int rc = row_layers(m, ws, ws.x, n, cv, pools, max_ctx, st)) {
      return rc;
    }
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
  for (const LayeredLayer &L : s->layers) {
    b += mat(L.in) + mat(L.out) + mat(L.ukv) + W * 4;
    if (L.cfg.ff_kind == B200_FF_EXPERTS)   // the chosen experts only
      b += (mat(L.expert_in) + mat(L.expert_out)) / L.cfg.experts * L.cfg.top;
    const int64_t seen = L.d.window > 0 ? std::min(L.d.window, ctx + 1) : ctx + 1;
    b += seen * (L.d.rank + L.d.rot) * e;
  }
  return b;
}

} // namespace b200

using namespace b200;

extern "C" {

int b200_model_create_layered(const b200_model_config *cfg, const b200_layer_config *layers, int dtype, b200_model **out) {
  if (!cfg || !layers || !out)
    return fail(B200_EINVAL, "create_layered: null argument");
  if (dtype != B200_F32 && dtype != B200_BF16)
    return fail(B200_EINVAL, "create_layered: dtype must be B200_F32 or B200_BF16");
  if (cfg->hidden < 1 || cfg->n_layers < 1 || cfg->vocab < 1 || cfg->max_len < 1 || !(cfg->eps >= 0.f))
    return fail(B200_EINVAL, "create_layered: bad architecture");
  if (cfg->tp_size > 1)
    return fail(B200_EINVAL, "create_layered: single-GPU sessions only");
  for (int i = 0; i < cfg->n_layers; ++i)
    if (int rc = check_layer(layers[i], i, layers)) return rc;
  b200_model_config base{};
  base.hidden = cfg->hidden; base.n_layers = cfg->n_layers; base.vocab = cfg->vocab; base.max_len = cfg->max_len;
  base.eps = cfg->eps; base.head_dim = 64; base.tp_size = 1;
  b200_model *m = nullptr;
  if (int rc = model_allocate(base, &m)) return rc;
  LayeredState *s = new LayeredState();
  m->lay = s;
  s->dtype = dtype;
  s->layers.resize(cfg->n_layers);
  int rc = make_matrix(s, &s->embed, cfg->vocab, cfg->hidden);
  if (!rc) {
    add_rows(s, "embed", s->embed, cfg->vocab, cfg->hidden, 0);
    rc = add_vector(s, "final.norm", &s->final_norm, cfg->hidden);
  }
  if (!rc) rc = own_array(s->owned, &s->zero, 4);
  bool all = false;
  for (int i = 0; i < cfg->n_layers && !rc; ++i) {
    LayeredLayer &L = s->layers[i];
    L.cfg = layers[i];
    rc = build_layer(s, L, i, cfg->hidden);
    all = all || L.cfg.window == 0;
    s->window = std::max(s->window, L.cfg.window);
    if (!rc && L.own())
      rc = own_alloc(s->owned, &L.cache, (size_t)cfg->max_len * L.d.row * elem(dtype));
  }
  if (all)
    s->window = 0;
  for (LayeredLayer &L : s->layers)
    L.cache = s->layers[L.source].cache;
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
