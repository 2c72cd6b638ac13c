// Attention over a cached low-rank latent, all heads sharing it: per token the cache holds one
// row [latent (rank) | rotated key part (rot)], and every head has its own up-projections
// W_uk [dim x rank] and W_uv [vdim x rank].
//
// Single-query form (decode, short portions, 32-bit models).  The up-projections are moved to
// the query and to the result: q . (W_uk c) = (W_uk^T q) . c and sum_j p_j (W_uv c_j) =
// W_uv (sum_j p_j c_j), so that a step reads each visible cache row once for all heads:
//   latent_prep_kernel    rotates, forms W_uk^T q, writes the new cache row
//   latent_attend_kernel  scores, online softmax and the weighted latent sum over a share of the
//                         visible keys (splits), f32 throughout
//   latent_value_kernel   adds the shares up and applies W_uv
// A sliding window limits the keys to (position - window, position].
#include "layered.cuh"
#include "rows.cuh"

namespace b200 {

namespace {

constexpr int kMaxDynamic = 200 * 1024;
constexpr int kKeys = 32;      // keys per tile of the single-query form: one per lane

__device__ __forceinline__ void rotate(float u, float v, float angle, float &a, float &b) {
  float s, c;
  sincosf(angle, &s, &c);
  a = u * c - v * s;
  b = v * c + u * s;
}

// cache row of one token: RMS-normed latent, rotated key part.  All threads of the CTA.
template <typename T>
__device__ void write_cache_row(const float *down, int rank, int rot, const float *norm_w, float eps, const float *inv_freq,
                                int pos, T *row, float *s_red) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  float s = 0.f;
  for (int k = threadIdx.x; k < rank; k += blockDim.x)
    s = fmaf(down[k], down[k], s);
  s = warp_sum(s);
  if (lane == 0)
    s_red[warp] = s;
  __syncthreads();
  float t = 0.f;
  for (int w = 0; w < nw; ++w)
    t += s_red[w];
  const float r = 1.0f / sqrtf(t / (float)rank + eps);
  for (int k = threadIdx.x; k < rank; k += blockDim.x)
    row[k] = from_float<T>(down[k] * r * norm_w[k]);
  for (int i = threadIdx.x; i < rot / 2; i += blockDim.x) {
    float a, b;
    rotate(down[rank + 2 * i], down[rank + 2 * i + 1], (float)pos * inv_freq[i], a, b);
    row[rank + 2 * i] = from_float<T>(a);
    row[rank + 2 * i + 1] = from_float<T>(b);
  }
}

struct PrepP {
  const float *proj;
  int64_t ldp;
  const void *uk;
  int64_t ldu;
  const float *inv_freq;
  float *qabs;
  const float *norm_w;
  float eps;
  void *pool;
  CacheView cv;
  LatentDims d;
  int off_down, col_blocks, q_blocks;
};

// grid (heads * col_blocks [+ 1], rows): CTA (h, cb) forms 64 columns of W_uk^T q of one head,
// the CTA behind them writes the cache row.
template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const PrepP p) {
  constexpr int E = RowUnit<T>::E, CL = 64 / E, DL = 256 / CL;
  __shared__ float s_part[DL][64 + 4];
  __shared__ float s_red[8];
  const int m = blockIdx.y;
  const LatentDims &d = p.d;
  const int pos = p.cv.row_pos[m];
  const float *proj = p.proj + (int64_t)m * p.ldp;
  if ((int)blockIdx.x >= p.q_blocks) {
    T *row = reinterpret_cast<T *>(p.pool) + cache_row(p.cv, p.cv.row_seq[m], pos) * d.row;
    write_cache_row<T>(proj + p.off_down, d.rank, d.rot, p.norm_w, p.eps, p.inv_freq, pos, row, s_red);
    return;
  }
  const int h = blockIdx.x / p.col_blocks, cb = blockIdx.x - h * p.col_blocks;
  const float *q = proj + h * (d.dim + d.rot);
  float *out = p.qabs + ((int64_t)m * d.heads + h) * (d.rank + d.rot);
  if (cb == 0)
    for (int i = threadIdx.x; i < d.rot / 2; i += 256) {
      float a, b;
      rotate(q[d.dim + 2 * i], q[d.dim + 2 * i + 1], (float)pos * p.inv_freq[i], a, b);
      out[d.rank + 2 * i] = a * d.scale;
      out[d.rank + 2 * i + 1] = b * d.scale;
    }
  const int cl = threadIdx.x % CL, dl = threadIdx.x / CL;
  const int col = cb * 64 + cl * E;
  float acc[E];
#pragma unroll
  for (int e = 0; e < E; ++e)
    acc[e] = 0.f;
  if (col < (int)p.ldu) {
    const T *w = reinterpret_cast<const T *>(p.uk) + (int64_t)h * d.dim * p.ldu + col;
#pragma unroll 4
    for (int k = dl; k < d.dim; k += DL) {
      const uint4 u = ld_stream_row(w + (int64_t)k * p.ldu);
      const float qk = q[k];
#pragma unroll
      for (int g = 0; g < RowUnit<T>::NG; ++g) {
        float f[4];
        RowUnit<T>::group(u, g, f);
#pragma unroll
        for (int e = 0; e < 4; ++e)
          acc[4 * g + e] = fmaf(qk, f[e], acc[4 * g + e]);
      }
    }
  }
#pragma unroll
  for (int e = 0; e < E; ++e)
    s_part[dl][cl * E + e] = acc[e];
  __syncthreads();
  if (threadIdx.x < 64) {
    float s = 0.f;
#pragma unroll
    for (int k = 0; k < DL; ++k)
      s += s_part[k][threadIdx.x];
    if (cb * 64 + (int)threadIdx.x < d.rank)
      out[cb * 64 + threadIdx.x] = s * d.scale;
  }
}

struct AttendP {
  const float *qabs;
  const void *pool;
  CacheView cv;
  LatentDims d;
  int chunk;                   // keys per split
  int splits, lq;              // lq: rank + rot rounded up to a 16-byte unit of the cache type
  int rank_pad;                // floats per partial sum
  float *ml;                   // [row][head][split][2]
  float *acc;                  // [row][head][split][rank_pad]
};

// grid (splits, head groups, rows), 8 warps x HPW heads.
template <typename T, int NR, int HPW>
__global__ void __launch_bounds__(256)
latent_attend_kernel(const AttendP p) {
  using U = RowUnit<T>;
  constexpr int E = U::E;
  extern __shared__ __align__(16) uint8_t smem[];
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int m = blockIdx.z, split = blockIdx.x;
  const int lds = p.lq + E;                                   // a 16-byte unit of padding: rows start on different banks
  float *s_q = reinterpret_cast<float *>(smem);               // [8 * HPW][lq]
  T *s_k = reinterpret_cast<T *>(s_q + 8 * HPW * p.lq);       // [kKeys][lds]
  const int h0 = blockIdx.y * 8 * HPW;
  const int pos = p.cv.row_pos[m], seq = p.cv.row_seq[m];
  const int lo = d.window > 0 ? max(0, pos - d.window + 1) : 0;
  const int k0 = lo + split * p.chunk, k1 = min(k0 + p.chunk, pos + 1);
  const int width = d.rank + d.rot;
  if (k0 < k1)
    for (int i = threadIdx.x; i < 8 * HPW * p.lq; i += 256) {
      const int h = i / p.lq, c = i - h * p.lq;
      s_q[i] = (h0 + h < d.heads && c < width) ? p.qabs[((int64_t)m * d.heads + h0 + h) * width + c] : 0.f;
    }
  float mx[HPW], l[HPW], acc[HPW][NR * E];
#pragma unroll
  for (int a = 0; a < HPW; ++a) {
    mx[a] = -INFINITY;
    l[a] = 0.f;
#pragma unroll
    for (int e = 0; e < NR * E; ++e)
      acc[a][e] = 0.f;
  }
  const bool active = h0 + warp * HPW < d.heads;
  const int units = p.lq / E;
  for (int kb = k0; kb < k1; kb += kKeys) {
    const int nk = min(kKeys, k1 - kb);
    __syncthreads();
    // a warp brings in the tile's rows 4 apart..: rows of one page are contiguous
    for (int r = warp; r < nk; r += 8) {
      const T *src = reinterpret_cast<const T *>(p.pool) + cache_row(p.cv, seq, kb + r) * d.row;
      for (int u = lane; u < units; u += 32)
        *reinterpret_cast<uint4 *>(s_k + r * lds + u * E) = *reinterpret_cast<const uint4 *>(src + u * E);
    }
    __syncthreads();
    if (!active)
      continue;
    float s[HPW];
#pragma unroll
    for (int a = 0; a < HPW; ++a)
      s[a] = 0.f;
    {
      const T *kr = s_k + min(lane, nk - 1) * lds;
      const float *qr = s_q + warp * HPW * p.lq;
#pragma unroll 2
      for (int u = 0; u < units; ++u) {
        const uint4 kv = *reinterpret_cast<const uint4 *>(kr + u * E);
#pragma unroll
        for (int g = 0; g < U::NG; ++g) {
          float f[4];
          U::group(kv, g, f);
#pragma unroll
          for (int a = 0; a < HPW; ++a) {
            const float4 qv = *reinterpret_cast<const float4 *>(qr + a * p.lq + u * E + g * 4);
            s[a] = fmaf(qv.x, f[0], s[a]);
            s[a] = fmaf(qv.y, f[1], s[a]);
            s[a] = fmaf(qv.z, f[2], s[a]);
            s[a] = fmaf(qv.w, f[3], s[a]);
          }
        }
      }
    }
#pragma unroll
    for (int a = 0; a < HPW; ++a) {
      const float sv = lane < nk ? s[a] : -INFINITY;
      const float nm = fmaxf(mx[a], warp_max(sv));
      const float corr = expf(mx[a] - nm);       // 0 for the first tile
      s[a] = expf(sv - nm);                      // 0 beyond the tile's keys
      l[a] = l[a] * corr + warp_sum(s[a]);
      mx[a] = nm;
#pragma unroll
      for (int e = 0; e < NR * E; ++e)
        acc[a][e] *= corr;
    }
    for (int j = 0; j < nk; ++j) {
      float pj[HPW];
#pragma unroll
      for (int a = 0; a < HPW; ++a)
        pj[a] = __shfl_sync(0xffffffffu, s[a], j);
#pragma unroll
      for (int i = 0; i < NR; ++i) {
        const int c = (i * 32 + lane) * E;
        if (c < d.rank) {
          const uint4 kv = *reinterpret_cast<const uint4 *>(s_k + j * lds + c);
#pragma unroll
          for (int g = 0; g < U::NG; ++g) {
            float f[4];
            U::group(kv, g, f);
#pragma unroll
            for (int a = 0; a < HPW; ++a)
#pragma unroll
              for (int e = 0; e < 4; ++e)
                acc[a][i * E + g * 4 + e] = fmaf(pj[a], f[e], acc[a][i * E + g * 4 + e]);
          }
        }
      }
    }
  }
  if (!active)
    return;
#pragma unroll
  for (int a = 0; a < HPW; ++a) {
    const int h = h0 + warp * HPW + a;
    if (h >= d.heads)
      break;
    const int64_t o = ((int64_t)m * d.heads + h) * p.splits + split;
    if (lane == 0) {
      p.ml[2 * o] = mx[a];
      p.ml[2 * o + 1] = l[a];
    }
    if (k0 >= k1)
      continue;                // an empty share is skipped by its l = 0
#pragma unroll
    for (int i = 0; i < NR; ++i) {
      const int c = (i * 32 + lane) * E;
      if (c < p.rank_pad)
#pragma unroll
        for (int e = 0; e < E; e += 4)
          *reinterpret_cast<float4 *>(p.acc + o * p.rank_pad + c + e) =
              make_float4(acc[a][i * E + e], acc[a][i * E + e + 1], acc[a][i * E + e + 2], acc[a][i * E + e + 3]);
    }
  }
}

struct ValueP {
  const float *ml, *acc;
  const void *uv;
  int64_t ldu;
  void *out;
  int64_t ldo;
  LatentDims d;
  int splits, rank_pad, rows_cta;
};

// grid (vdim / rows_cta, heads, rows): fold the shares, then rows of W_uv against the latent sum
template <typename T, typename O>
__global__ void __launch_bounds__(256)
latent_value_kernel(const ValueP p) {
  extern __shared__ __align__(16) float4 xs[];    // the latent sum, staged; then splits weights
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, m = blockIdx.z;
  float *s_w = reinterpret_cast<float *>(xs + block_pad<T>(d.rank) / 4);
  const int64_t o = ((int64_t)m * d.heads + h) * p.splits;
  if (warp == 0) {
    float mx = -INFINITY, l = 0.f;
    for (int s = lane; s < p.splits; s += 32)
      if (p.ml[2 * (o + s) + 1] > 0.f)
        mx = fmaxf(mx, p.ml[2 * (o + s)]);
    mx = warp_max(mx);
    for (int s = lane; s < p.splits; s += 32) {
      const float ls = p.ml[2 * (o + s) + 1];
      const float w = ls > 0.f ? expf(p.ml[2 * (o + s)] - mx) : 0.f;
      s_w[s] = w;
      l += w * ls;
    }
    l = warp_sum(l);
    __syncwarp();
    for (int s = lane; s < p.splits; s += 32)
      s_w[s] /= l;
  }
  __syncthreads();
  for (int g = threadIdx.x; g < block_pad<T>(d.rank) / 4; g += 256) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if (4 * g < d.rank)
      for (int s = 0; s < p.splits; ++s) {
        const float w = s_w[s];
        if (w > 0.f) {
          const float4 a = *reinterpret_cast<const float4 *>(p.acc + (o + s) * p.rank_pad + 4 * g);
          v.x = fmaf(w, a.x, v.x);
          v.y = fmaf(w, a.y, v.y);
          v.z = fmaf(w, a.z, v.z);
          v.w = fmaf(w, a.w, v.w);
        }
      }
    if (4 * g + 1 >= d.rank) v.y = 0.f;
    if (4 * g + 2 >= d.rank) v.z = 0.f;
    if (4 * g + 3 >= d.rank) v.w = 0.f;
    xs[stage_slot<T>(g)] = v;
  }
  __syncthreads();
  const T *w = reinterpret_cast<const T *>(p.uv) + (int64_t)h * d.vdim * p.ldu;
  const int r0 = blockIdx.x * p.rows_cta, r1 = min(r0 + p.rows_cta, d.vdim);
  O *out = reinterpret_cast<O *>(p.out) + (int64_t)m * p.ldo + h * d.vdim;
  for (int r = r0 + warp * 2; r < r1; r += 16) {
    const T *row[2] = {w + (int64_t)r * p.ldu, w + (int64_t)min(r + 1, d.vdim - 1) * p.ldu};
    float acc[2][1] = {{0.f}, {0.f}};
    dot_rows<T, 1, 2>(row, unit_pad<T>(d.rank), xs, 0, lane, acc);
    const float a = warp_sum(acc[0][0]), b = warp_sum(acc[1][0]);
    if (lane == 0) {
      out[r] = from_float<O>(a);
      if (r + 1 < r1)
        out[r + 1] = from_float<O>(b);
    }
  }
}

template <typename K> int allow_dynamic(K kern, size_t bytes) {
  if (bytes > (size_t)kMaxDynamic)
    return fail(B200_ELIMIT, "latent attention: %zu bytes of shared memory needed", bytes);
  if (bytes > 40 * 1024)
    B200_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, kMaxDynamic));
  return B200_OK;
}

template <typename T> int prep_run(PrepP &p, int M, bool own, cudaStream_t st) {
  p.col_blocks = (p.d.rank + 63) / 64;
  p.q_blocks = p.d.heads * p.col_blocks;
  for (int m0 = 0; m0 < M; m0 += 32768) {
    PrepP q = p;
    q.proj += (int64_t)m0 * p.ldp;
    q.qabs += (int64_t)m0 * p.d.heads * (p.d.rank + p.d.rot);
    q.cv.row_seq += m0;
    q.cv.row_pos += m0;
    latent_prep_kernel<T><<<dim3(p.q_blocks + (own ? 1 : 0), M - m0 < 32768 ? M - m0 : 32768), 256, 0, st>>>(q);
    B200_LAUNCH_CHECK();
  }
  return B200_OK;
}

template <typename T, int NR, int HPW> int attend_run(const AttendP &p, int M, cudaStream_t st) {
  auto kern = latent_attend_kernel<T, NR, HPW>;
  const size_t smem = (size_t)8 * HPW * p.lq * 4 + (size_t)kKeys * (p.lq + RowUnit<T>::E) * sizeof(T);
  if (int rc = allow_dynamic(kern, smem)) return rc;
  const int groups = (p.d.heads + 8 * HPW - 1) / (8 * HPW);
  for (int m0 = 0; m0 < M; m0 += 32768) {
    AttendP q = p;
    q.qabs += (int64_t)m0 * p.d.heads * (p.d.rank + p.d.rot);
    q.cv.row_seq += m0;
    q.cv.row_pos += m0;
    q.ml += (int64_t)m0 * p.d.heads * p.splits * 2;
    q.acc += (int64_t)m0 * p.d.heads * p.splits * p.rank_pad;
    kern<<<dim3(p.splits, groups, M - m0 < 32768 ? M - m0 : 32768), 256, smem, st>>>(q);
    B200_LAUNCH_CHECK();
  }
  return B200_OK;
}
template <typename T, int NR> int attend_heads(const AttendP &p, int M, cudaStream_t st) {
  return p.d.heads > 8 ? attend_run<T, NR, 2>(p, M, st) : attend_run<T, NR, 1>(p, M, st);
}

template <typename T, typename O> int value_run(ValueP &p, int M, cudaStream_t st) {
  // few rows: enough CTAs to fill the machine; many: a CTA per head and row
  p.rows_cta = M <= 16 ? 16 : p.d.vdim;
  const size_t smem = (size_t)block_pad<T>(p.d.rank) * 4 + (size_t)p.splits * 4;
  auto kern = latent_value_kernel<T, O>;
  if (int rc = allow_dynamic(kern, smem)) return rc;
  for (int m0 = 0; m0 < M; m0 += 32768) {
    ValueP q = p;
    q.ml += (int64_t)m0 * p.d.heads * p.splits * 2;
    q.acc += (int64_t)m0 * p.d.heads * p.splits * p.rank_pad;
    q.out = reinterpret_cast<O *>(p.out) + (int64_t)m0 * p.ldo;
    kern<<<dim3((p.d.vdim + p.rows_cta - 1) / p.rows_cta, p.d.heads, M - m0 < 32768 ? M - m0 : 32768), 256, smem, st>>>(q);
    B200_LAUNCH_CHECK();
  }
  return B200_OK;
}

int rank_pad(const LatentDims &d) { return (d.rank + 7) / 8 * 8; }

} // namespace

int latent_limits(const LatentDims &d) {
  if (d.heads < 1 || d.dim < 1 || d.vdim < 1 || d.rank < 1 || d.rot < 0 || (d.rot & 1))
    return fail(B200_EINVAL, "latent attention: bad head sizes (heads %d, dim %d, rot %d, vdim %d, rank %d)", d.heads,
                d.dim, d.rot, d.vdim, d.rank);
  if (d.rank > 1024 || d.rot > 256 || d.heads > 1024)
    return fail(B200_ELIMIT, "latent attention: rank %d (limit 1024), rot %d (limit 256), heads %d (limit 1024)", d.rank,
                d.rot, d.heads);
  return B200_OK;
}

int latent_prep_launch(int dtype, const LatentDims &d, const float *proj, int64_t ldp, int M, const RowMatrix &uk,
                       const float *inv_freq, float *qabs, bool own, int off_down, const float *norm_w, float eps,
                       void *pool, const CacheView &cv, cudaStream_t st) {
  PrepP p{};
  p.proj = proj; p.ldp = ldp; p.uk = uk.w; p.ldu = uk.ld; p.inv_freq = inv_freq; p.qabs = qabs;
  p.norm_w = norm_w; p.eps = eps; p.pool = pool; p.cv = cv; p.d = d; p.off_down = off_down;
  return dtype == B200_F32 ? prep_run<float>(p, M, own, st) : prep_run<bf16>(p, M, own, st);
}

// Shares of the visible keys per row: enough CTAs for the machine, at least one tile each.
int latent_splits(const LatentDims &d, int M, int max_ctx) {
  const int n = d.window > 0 && d.window < max_ctx ? d.window : max_ctx;
  const int groups = (d.heads + 15) / 16;
  int want = (2 * 148 + M * groups - 1) / (M * groups);
  const int tiles = (n + kKeys - 1) / kKeys;
  if (want > tiles) want = tiles;
  if (want > 128) want = 128;
  return want < 1 ? 1 : want;
}
int64_t latent_scratch_floats(const LatentDims &d, int M, int splits) {
  return ((int64_t)M * d.heads * splits * 2 + 3) / 4 * 4 + (int64_t)M * d.heads * splits * rank_pad(d);
}

int latent_attend_launch(int dtype, const LatentDims &d, const float *qabs, int M, const void *pool, const CacheView &cv,
                         int splits, int max_ctx, float *scratch, cudaStream_t st) {
  const int n = d.window > 0 && d.window < max_ctx ? d.window : max_ctx;
  AttendP p{};
  p.qabs = qabs; p.pool = pool; p.cv = cv; p.d = d; p.splits = splits;
  p.chunk = ((n + splits - 1) / splits + kKeys - 1) / kKeys * kKeys;
  p.rank_pad = rank_pad(d);
  p.ml = scratch;
  p.acc = scratch + ((int64_t)M * d.heads * splits * 2 + 3) / 4 * 4;
  if (dtype == B200_F32) {
    p.lq = unit_pad<float>(d.rank + d.rot);
    if (d.rank <= 128) return attend_heads<float, 1>(p, M, st);
    if (d.rank <= 256) return attend_heads<float, 2>(p, M, st);
    if (d.rank <= 512) return attend_heads<float, 4>(p, M, st);
    return attend_heads<float, 8>(p, M, st);
  }
  p.lq = unit_pad<bf16>(d.rank + d.rot);
  if (d.rank <= 256) return attend_heads<bf16, 1>(p, M, st);
  if (d.rank <= 512) return attend_heads<bf16, 2>(p, M, st);
  return attend_heads<bf16, 4>(p, M, st);
}

int latent_value_launch(int dtype, const LatentDims &d, const float *scratch, int M, int splits, const RowMatrix &uv,
                        void *out, int64_t ldo, bool out_bf16, cudaStream_t st) {
  ValueP p{};
  p.ml = scratch;
  p.acc = scratch + ((int64_t)M * d.heads * splits * 2 + 3) / 4 * 4;
  p.uv = uv.w; p.ldu = uv.ld; p.out = out; p.ldo = ldo; p.d = d; p.splits = splits; p.rank_pad = rank_pad(d);
  if (dtype == B200_F32)
    return value_run<float, float>(p, M, st);
  return out_bf16 ? value_run<bf16, bf16>(p, M, st) : value_run<bf16, float>(p, M, st);
}

} // namespace b200
