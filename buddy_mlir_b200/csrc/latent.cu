// Attention over a cached low-rank latent, all heads sharing it: per token the cache holds one
// row [latent (rank) | rotated key part (rot)], and every head has its own up-projections
// W_uk [dim x rank] and W_uv [vdim x rank].
//
// Single-query form (decode, short portions, 32-bit models).  The up-projections are moved to
// the query and to the result: q . (W_uk c) = (W_uk^T q) . c and sum_j p_j (W_uv c_j) =
// W_uv (sum_j p_j c_j), so that a step reads each visible cache row once for all heads:
//   latent_prep_kernel    rotates, forms W_uk^T q, writes the new cache row
//   latent_attend_kernel  (32-bit cache) and latent_attend_mma_kernel (bfloat16 cache, mma.sync):
//                         scores, online softmax and the weighted latent sum over a share of the
//                         visible keys (splits); scores, weights and sums are f32
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
  int off_down, col_blocks, q_blocks, M;
};

// the rotated, scaled part of one head's queries for `rows` rows, by the whole CTA
__device__ __forceinline__ void rotate_queries(const PrepP &p, int h, int m0, int rows) {
  const LatentDims &d = p.d;
  const int half = d.rot / 2;
  for (int i = threadIdx.x; i < rows * half; i += blockDim.x) {
    const int m = m0 + i / half, k = i % half;
    const float *q = p.proj + (int64_t)m * p.ldp + h * (d.dim + d.rot) + d.dim + 2 * k;
    float a, b;
    rotate(q[0], q[1], (float)p.cv.row_pos[m] * p.inv_freq[k], a, b);
    float *out = p.qabs + ((int64_t)m * d.heads + h) * (d.rank + d.rot) + d.rank + 2 * k;
    out[0] = a * d.scale;
    out[1] = b * d.scale;
  }
}

// grid (heads * col_blocks [+ 1], rows / MT): CTA (h, cb) forms 64 columns of W_uk^T q of one head
// for MT rows, the CTA behind them writes their cache rows.
template <typename T, int MT>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const PrepP p) {
  constexpr int E = RowUnit<T>::E, CL = 64 / E, DL = 256 / CL;
  extern __shared__ __align__(16) float s_q[];   // [MT][dim], then the warps' sums [8][MT][64]
  __shared__ float s_red[8];
  const LatentDims &d = p.d;
  const int m0 = blockIdx.y * MT, rows = min(MT, p.M - m0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if ((int)blockIdx.x >= p.q_blocks) {
    for (int m = 0; m < rows; ++m) {
      const int pos = p.cv.row_pos[m0 + m];
      T *row = reinterpret_cast<T *>(p.pool) + cache_row(p.cv, p.cv.row_seq[m0 + m], pos) * d.row;
      write_cache_row<T>(p.proj + (int64_t)(m0 + m) * p.ldp + p.off_down, d.rank, d.rot, p.norm_w, p.eps, p.inv_freq, pos,
                         row, s_red);
      __syncthreads();
    }
    return;
  }
  const int h = blockIdx.x / p.col_blocks, cb = blockIdx.x - h * p.col_blocks;
  const int64_t width = d.rank + d.rot;
  float *s_sum = s_q + MT * d.dim;
  const float *q = p.proj + (int64_t)m0 * p.ldp + h * (d.dim + d.rot);
  for (int i = threadIdx.x; i < MT * d.dim; i += 256) {
    const int m = i / d.dim, k = i - m * d.dim;
    s_q[i] = m < rows ? q[(int64_t)m * p.ldp + k] : 0.f;
  }
  if (cb == 0)
    rotate_queries(p, h, m0, rows);
  __syncthreads();
  const int cl = threadIdx.x % CL, dl = threadIdx.x / CL;
  const int col = cb * 64 + cl * E;
  float acc[MT][E];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < E; ++e)
      acc[m][e] = 0.f;
  if (col < (int)p.ldu) {
    const T *w = reinterpret_cast<const T *>(p.uk) + (int64_t)h * d.dim * p.ldu + col;
#pragma unroll 4
    for (int k = dl; k < d.dim; k += DL) {
      const uint4 u = ld_stream_row(w + (int64_t)k * p.ldu);
#pragma unroll
      for (int g = 0; g < RowUnit<T>::NG; ++g) {
        float f[4];
        RowUnit<T>::group(u, g, f);
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int e = 0; e < 4; ++e)
            acc[m][4 * g + e] = fmaf(s_q[m * d.dim + k], f[e], acc[m][4 * g + e]);
      }
    }
  }
  // lanes that share the columns, then the warps
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int e = 0; e < E; ++e) {
      float v = acc[m][e];
#pragma unroll
      for (int o = CL; o < 32; o <<= 1)
        v += __shfl_xor_sync(0xffffffffu, v, o);
      if (lane < CL)
        s_sum[(warp * MT + m) * 64 + cl * E + e] = v;
    }
  __syncthreads();
  for (int i = threadIdx.x; i < rows * 64; i += 256) {
    const int m = i >> 6, c = i & 63;
    float v = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w)
      v += s_sum[(w * MT + m) * 64 + c];
    if (cb * 64 + c < d.rank)
      p.qabs[((int64_t)(m0 + m) * d.heads + h) * width + cb * 64 + c] = v * d.scale;
  }
}

// The same for many rows of a bfloat16 model, on mma.sync: grid (rank / 64, heads, rows / 64), a
// warp per 16 rows and 32 columns, [rows x dim] queries against the head's [dim x 64] slice of W_uk.
__global__ void __launch_bounds__(256)
latent_prep_mma_kernel(const PrepP p) {
  extern __shared__ __align__(16) bf16 sm16[];
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, n0 = blockIdx.x * 64, m0 = blockIdx.z * 64, rows = min(64, p.M - m0);
  const int kp = (d.dim + 15) / 16 * 16, lda = kp + 8;
  constexpr int LDW = 64 + 8;
  bf16 *s_w = sm16, *s_a = s_w + kp * LDW;         // [kp][LDW], [64][lda]
  const bf16 *w = reinterpret_cast<const bf16 *>(p.uk) + (int64_t)h * d.dim * p.ldu + n0;
  for (int i = threadIdx.x; i < kp * 8; i += 256) {
    const int k = i >> 3, c = (i & 7) * 8;
    const bool live = k < d.dim && n0 + c < (int)p.ldu;
    cp16(s_w + k * LDW + c, live ? w + (int64_t)k * p.ldu + c : w, live);
  }
  asm volatile("cp.async.commit_group;" ::: "memory");
  const float *q = p.proj + (int64_t)m0 * p.ldp + h * (d.dim + d.rot);
  if (((d.dim | d.rot | (int)p.ldp) & 3) == 0) {
    const int g = kp / 4;
#pragma unroll 8
    for (int i = threadIdx.x; i < 64 * g; i += 256) {
      const int m = i / g, k = (i - m * g) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      if (m < rows && k < d.dim)
        v = *reinterpret_cast<const float4 *>(q + (int64_t)m * p.ldp + k);
      const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
      *reinterpret_cast<uint2 *>(s_a + m * lda + k) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
    }
  } else {
    for (int i = threadIdx.x; i < 64 * kp; i += 256) {
      const int m = i / kp, k = i - m * kp;
      s_a[m * lda + k] = __float2bfloat16_rn(m < rows && k < d.dim ? q[(int64_t)m * p.ldp + k] : 0.f);
    }
  }
  if (blockIdx.x == 0)
    rotate_queries(p, h, m0, rows);
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int rw = (warp & 3) * 16, cw = (warp >> 2) * 32;
  float o[4][4];
#pragma unroll
  for (int i = 0; i < 4; ++i)
    o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  for (int k = 0; k < kp; k += 16) {
    uint32_t a[4];
    ldsm4(a, s_a + (rw + (lane & 15)) * lda + k + (lane >> 4) * 8);
#pragma unroll
    for (int nt = 0; nt < 2; ++nt) {
      uint32_t b[4];
      ldsm4t(b, s_w + (k + (lane & 15)) * LDW + cw + nt * 16 + (lane >> 4) * 8);
      mma16816(o[2 * nt], a, b[0], b[1]);
      mma16816(o[2 * nt + 1], a, b[2], b[3]);
    }
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int m = rw + (lane >> 2) + 8 * r;
    if (m >= rows)
      continue;
    float *out = p.qabs + ((int64_t)(m0 + m) * d.heads + h) * (d.rank + d.rot);
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = n0 + cw + i * 8 + (lane & 3) * 2 + e;
        if (c < d.rank)
          out[c] = o[i][2 * r + e] * d.scale;
      }
  }
}

// cache rows [src, src + tail) of one sequence -> stage, their key parts turned by `delta` positions
template <typename T>
__global__ void __launch_bounds__(128)
latent_shift_kernel(const T *cache, LatentDims d, int src, const float *inv_freq, float delta, T *stage) {
  const T *from = cache + (int64_t)(src + blockIdx.x) * d.row;
  T *to = stage + (int64_t)blockIdx.x * d.row;
  for (int k = threadIdx.x; k < (int)d.row; k += 128)
    if (k < d.rank || k >= d.rank + d.rot)
      to[k] = from[k];
  for (int i = threadIdx.x; i < d.rot / 2; i += 128) {
    float a, b;
    rotate(to_float(from[d.rank + 2 * i]), to_float(from[d.rank + 2 * i + 1]), delta * inv_freq[i], a, b);
    to[d.rank + 2 * i] = from_float<T>(a);
    to[d.rank + 2 * i + 1] = from_float<T>(b);
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
    // a warp brings in every eighth row of the tile
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

// The same over a bfloat16 cache with the tensor cores: a CTA takes 16 heads (the rows of an
// m16n8k16 product) and its share of the keys in tiles of 32.  The scores' contraction over the
// KSW * 64 padded row elements is split over four warps, the keys of a tile over two groups of
// them; the weights enter the second product as two bf16 terms (hi + lo); every warp owns
// NTW * 8 elements of the latent sum.
template <int KSW, int NTW>
__global__ void __launch_bounds__(256, NTW <= 8 && KSW <= 9 ? 2 : 1)
latent_attend_mma_kernel(const AttendP p) {
  constexpr int KP = KSW * 64, NP = NTW * 64, LDK = (KP > NP ? KP : NP) + 8, LDS = 36, LDP = 40;
  extern __shared__ __align__(16) uint8_t smem[];
  bf16 *s_k = reinterpret_cast<bf16 *>(smem);                              // [2][kKeys][LDK]
  float *s_part = reinterpret_cast<float *>(s_k + 2 * kKeys * LDK);        // [4][16][LDS]
  bf16 *s_hi = reinterpret_cast<bf16 *>(s_part + 4 * 16 * LDS);            // [16][LDP]
  bf16 *s_lo = s_hi + 16 * LDP;
  __shared__ float s_corr[16];
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t4 = lane & 3;
  const int m = blockIdx.z, split = blockIdx.x, h0 = blockIdx.y * 16;
  const int pos = p.cv.row_pos[m], seq = p.cv.row_seq[m];
  const int lo = d.window > 0 ? max(0, pos - d.window + 1) : 0;
  const int k0 = lo + split * p.chunk, k1 = min(k0 + p.chunk, pos + 1);
  const int width = d.rank + d.rot;
  if (k0 >= k1) {                // an empty share is skipped by its l = 0
    if (threadIdx.x < 16 && h0 + threadIdx.x < d.heads) {
      const int64_t o = ((int64_t)m * d.heads + h0 + threadIdx.x) * p.splits + split;
      p.ml[2 * o] = -INFINITY;
      p.ml[2 * o + 1] = 0.f;
    }
    return;
  }
  const int units = (int)d.row / 8;
  auto load_tile = [&](int kb, int buf) {
    const int nk = min(kKeys, k1 - kb);
    // rows beyond the share repeat its last key: they are masked, and must hold finite values
    for (int r = warp; r < kKeys; r += 8) {
      const bf16 *src = reinterpret_cast<const bf16 *>(p.pool) + cache_row(p.cv, seq, kb + min(r, nk - 1)) * d.row;
      bf16 *dst = s_k + (buf * kKeys + r) * LDK;
      for (int u = lane; u < units; u += 32)
        cp16(dst + u * 8, src + u * 8, true);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  load_tile(k0, 0);
  for (int i = threadIdx.x; i < 2 * kKeys * (LDK / 8 - units); i += 256) {   // padding of the rows
    const int r = i / (LDK / 8 - units), u = i - r * (LDK / 8 - units) + units;
    *reinterpret_cast<uint4 *>(s_k + r * LDK + u * 8) = make_uint4(0, 0, 0, 0);
  }
  // this warp's quarter of the queries
  const int kg = warp & 3, ng = warp >> 2;
  uint32_t qa[KSW][4];
  {
    const float *q = p.qabs + ((int64_t)m * d.heads + h0) * width;
    auto pair = [&](int row, int k) {
      const float a = h0 + row < d.heads && k < width ? q[(int64_t)row * width + k] : 0.f;
      const float b = h0 + row < d.heads && k + 1 < width ? q[(int64_t)row * width + k + 1] : 0.f;
      const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
      return *reinterpret_cast<const uint32_t *>(&v);
    };
#pragma unroll
    for (int ks = 0; ks < KSW; ++ks) {
      const int k = (kg * KSW + ks) * 16 + t4 * 2;
      qa[ks][0] = pair(g, k);
      qa[ks][1] = pair(g + 8, k);
      qa[ks][2] = pair(g, k + 8);
      qa[ks][3] = pair(g + 8, k + 8);
    }
  }
  float o[NTW][4];
#pragma unroll
  for (int i = 0; i < NTW; ++i)
    o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};   // of heads 2 * warp, 2 * warp + 1
  const int c0 = warp * NTW * 8;
  int buf = 0;
  for (int kb = k0; kb < k1; kb += kKeys, buf ^= 1) {
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();
    if (kb + kKeys < k1)
      load_tile(kb + kKeys, buf ^ 1);
    const bf16 *k = s_k + buf * kKeys * LDK;
    {
      float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
      const bf16 *kr = k + (ng * 16 + (lane & 7) + ((lane >> 4) << 3)) * LDK + kg * KSW * 16 + ((lane >> 3) & 1) * 8;
#pragma unroll
      for (int ks = 0; ks < KSW; ++ks) {
        uint32_t b[4];
        ldsm4(b, kr + ks * 16);
        mma16816(s[0], qa[ks], b[0], b[1]);
        mma16816(s[1], qa[ks], b[2], b[3]);
      }
#pragma unroll
      for (int nt = 0; nt < 2; ++nt) {
        float *dst = s_part + (kg * 16 + g) * LDS + ng * 16 + nt * 8 + t4 * 2;
        *reinterpret_cast<float2 *>(dst) = make_float2(s[nt][0], s[nt][1]);
        *reinterpret_cast<float2 *>(dst + 8 * LDS) = make_float2(s[nt][2], s[nt][3]);
      }
    }
    __syncthreads();
#pragma unroll
    for (int a = 0; a < 2; ++a) {
      const int h = warp * 2 + a;
      float s = -INFINITY;
      if (kb + lane < k1)
        s = (s_part[h * LDS + lane] + s_part[(16 + h) * LDS + lane]) + (s_part[(32 + h) * LDS + lane] + s_part[(48 + h) * LDS + lane]);
      const float nm = fmaxf(mx[a], warp_max(s));
      const float corr = expf(mx[a] - nm);
      const float w = expf(s - nm);
      l[a] = l[a] * corr + warp_sum(w);
      mx[a] = nm;
      const bf16 hi = __float2bfloat16_rn(w);
      s_hi[h * LDP + lane] = hi;
      s_lo[h * LDP + lane] = __float2bfloat16_rn(w - __bfloat162float(hi));
      if (lane == 0)
        s_corr[h] = corr;
    }
    __syncthreads();
    if (c0 < d.rank) {
      const float ca = s_corr[g], cb = s_corr[g + 8];
#pragma unroll
      for (int i = 0; i < NTW; ++i) {
        o[i][0] *= ca;
        o[i][1] *= ca;
        o[i][2] *= cb;
        o[i][3] *= cb;
      }
#pragma unroll
      for (int kt = 0; kt < kKeys / 16; ++kt) {
        uint32_t ah[4], al[4];
        ldsm4(ah, s_hi + (lane & 15) * LDP + kt * 16 + (lane >> 4) * 8);
        ldsm4(al, s_lo + (lane & 15) * LDP + kt * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int nt = 0; nt < NTW / 2; ++nt) {
          uint32_t b[4];
          ldsm4t(b, k + (kt * 16 + (lane & 15)) * LDK + c0 + nt * 16 + (lane >> 4) * 8);
          mma16816(o[2 * nt], ah, b[0], b[1]);
          mma16816(o[2 * nt], al, b[0], b[1]);
          mma16816(o[2 * nt + 1], ah, b[2], b[3]);
          mma16816(o[2 * nt + 1], al, b[2], b[3]);
        }
      }
    }
  }
#pragma unroll
  for (int a = 0; a < 2; ++a)
    if (lane == 0 && h0 + warp * 2 + a < d.heads) {
      const int64_t i = ((int64_t)m * d.heads + h0 + warp * 2 + a) * p.splits + split;
      p.ml[2 * i] = mx[a];
      p.ml[2 * i + 1] = l[a];
    }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int h = h0 + g + 8 * r;
    if (h >= d.heads)
      continue;
    float *dst = p.acc + (((int64_t)m * d.heads + h) * p.splits + split) * p.rank_pad;
#pragma unroll
    for (int i = 0; i < NTW; ++i) {
      const int c = c0 + i * 8 + t4 * 2;
      if (c < p.rank_pad)
        *reinterpret_cast<float2 *>(dst + c) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
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
  int splits, rank_pad, rows_cta, M;
};

// weights of the shares of `rows` rows of one head: w_s = exp(m_s - max) / sum, a warp per row
__device__ __forceinline__ void share_weights(const ValueP &p, int h, int m0, int rows, float *s_w) {
  const int lane = threadIdx.x & 31;
  for (int m = threadIdx.x >> 5; m < rows; m += blockDim.x >> 5) {
    const int64_t o = ((int64_t)(m0 + m) * p.d.heads + h) * p.splits;
    float mx = -INFINITY, l = 0.f;
    for (int s = lane; s < p.splits; s += 32)
      if (p.ml[2 * (o + s) + 1] > 0.f)
        mx = fmaxf(mx, p.ml[2 * (o + s)]);
    mx = warp_max(mx);
    for (int s = lane; s < p.splits; s += 32) {
      const float ls = p.ml[2 * (o + s) + 1];
      const float w = ls > 0.f ? expf(p.ml[2 * (o + s)] - mx) : 0.f;
      s_w[m * p.splits + s] = w;
      l += w * ls;
    }
    l = warp_sum(l);
    __syncwarp();
    for (int s = lane; s < p.splits; s += 32)
      s_w[m * p.splits + s] /= l;
  }
}
// four elements from column c of the latent sum of row m (of the whole batch)
__device__ __forceinline__ float4 fold_shares(const ValueP &p, int h, int m, int c, const float *s_w) {
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  const float *src = p.acc + ((int64_t)m * p.d.heads + h) * p.splits * p.rank_pad + c;
#pragma unroll 4
  for (int s = 0; s < p.splits; ++s) {
    const float w = s_w[s];
    if (w > 0.f) {
      const float4 a = *reinterpret_cast<const float4 *>(src + (int64_t)s * p.rank_pad);
      v.x = fmaf(w, a.x, v.x);
      v.y = fmaf(w, a.y, v.y);
      v.z = fmaf(w, a.z, v.z);
      v.w = fmaf(w, a.w, v.w);
    }
  }
  if (c + 1 >= p.d.rank) v.y = 0.f;
  if (c + 2 >= p.d.rank) v.z = 0.f;
  if (c + 3 >= p.d.rank) v.w = 0.f;
  return v;
}

// grid (vdim / rows_cta, heads, rows / MT): fold the shares of MT rows, then rows of W_uv against
// their latent sums
template <typename T, typename O, int MT>
__global__ void __launch_bounds__(256)
latent_value_kernel(const ValueP p) {
  extern __shared__ __align__(16) float4 xs[];    // [MT] staged latent sums, then [MT][splits] weights
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, m0 = blockIdx.z * MT, rows = min(MT, p.M - m0);
  const int groups = block_pad<T>(d.rank) / 4;
  float *s_w = reinterpret_cast<float *>(xs + MT * groups);
  share_weights(p, h, m0, rows, s_w);
  __syncthreads();
  for (int i = threadIdx.x; i < MT * groups; i += 256) {
    const int m = i / groups, g = i - m * groups;
    xs[m * groups + stage_slot<T>(g)] =
        m < rows && 4 * g < d.rank ? fold_shares(p, h, m0 + m, 4 * g, s_w + m * p.splits) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  __syncthreads();
  const T *w = reinterpret_cast<const T *>(p.uv) + (int64_t)h * d.vdim * p.ldu;
  const int r0 = blockIdx.x * p.rows_cta, r1 = min(r0 + p.rows_cta, d.vdim);
  O *out = reinterpret_cast<O *>(p.out) + (int64_t)m0 * p.ldo + h * d.vdim;
  for (int r = r0 + warp * 2; r < r1; r += 16) {
    const T *row[2] = {w + (int64_t)r * p.ldu, w + (int64_t)min(r + 1, d.vdim - 1) * p.ldu};
    float acc[2][MT];
#pragma unroll
    for (int m = 0; m < MT; ++m)
      acc[0][m] = acc[1][m] = 0.f;
    dot_rows<T, MT, 2>(row, unit_pad<T>(d.rank), xs, groups, lane, acc);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float a = warp_sum(acc[0][m]), b = warp_sum(acc[1][m]);
      if (lane == 0 && m < rows) {
        out[(int64_t)m * p.ldo + r] = from_float<O>(a);
        if (r + 1 < r1)
          out[(int64_t)m * p.ldo + r + 1] = from_float<O>(b);
      }
    }
  }
}

// The same for many rows of a bfloat16 model in two steps: the latent sums as bf16 rows
// [row][head][rank_pad], then W_uv on mma.sync.
__global__ void __launch_bounds__(128)
latent_fold_kernel(const ValueP p, bf16 *lat) {
  __shared__ float s_w[128];                       // at most 128 shares
  const int h = blockIdx.x, m = blockIdx.y;
  share_weights(p, h, m, 1, s_w);
  __syncthreads();
  bf16 *dst = lat + ((int64_t)m * p.d.heads + h) * p.rank_pad;
  for (int c = threadIdx.x * 4; c < p.rank_pad; c += 512) {
    const float4 v = c < p.d.rank ? fold_shares(p, h, m, c, s_w) : make_float4(0.f, 0.f, 0.f, 0.f);
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(dst + c) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
  }
}
// grid (vdim / 32, heads, rows / 64), a warp per 16 rows and 16 columns
__global__ void __launch_bounds__(256)
latent_value_mma_kernel(const ValueP p, const bf16 *lat) {
  extern __shared__ __align__(16) bf16 sm16[];
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, n0 = blockIdx.x * 32, m0 = blockIdx.z * 64, rows = min(64, p.M - m0);
  const int kp = (d.rank + 15) / 16 * 16, ld = kp + 8, units = kp / 8;
  bf16 *s_v = sm16, *s_a = s_v + 32 * ld;          // [32][ld], [64][ld]
  const bf16 *w = reinterpret_cast<const bf16 *>(p.uv) + ((int64_t)h * d.vdim + n0) * p.ldu;
  const bf16 *a0 = lat + ((int64_t)m0 * d.heads + h) * p.rank_pad;
  for (int i = threadIdx.x; i < 96 * units; i += 256) {
    const int n = i / units, c = (i - n * units) * 8;
    if (n < 32) {
      const bool live = n0 + n < d.vdim && c < (int)p.ldu;
      cp16(s_v + n * ld + c, live ? w + (int64_t)n * p.ldu + c : w, live);
    } else {
      const bool live = n - 32 < rows && c < p.rank_pad;
      cp16(s_a + (n - 32) * ld + c, live ? a0 + (int64_t)(n - 32) * d.heads * p.rank_pad + c : a0, live);
    }
  }
  asm volatile("cp.async.commit_group;\n cp.async.wait_group 0;" ::: "memory");
  __syncthreads();
  const int rw = (warp & 3) * 16, cw = (warp >> 2) * 16;
  float o[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll 4
  for (int k = 0; k < kp; k += 16) {
    uint32_t a[4], b[4];
    ldsm4(a, s_a + (rw + (lane & 15)) * ld + k + (lane >> 4) * 8);
    ldsm4(b, s_v + (cw + (lane & 7) + ((lane >> 4) << 3)) * ld + k + ((lane >> 3) & 1) * 8);
    mma16816(o[0], a, b[0], b[1]);
    mma16816(o[1], a, b[2], b[3]);
  }
  bf16 *out = reinterpret_cast<bf16 *>(p.out) + (int64_t)m0 * p.ldo + h * d.vdim;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int m = rw + (lane >> 2) + 8 * r;
    if (m >= rows)
      continue;
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int c = n0 + cw + i * 8 + (lane & 3) * 2 + e;
        if (c < d.vdim)
          out[(int64_t)m * p.ldo + c] = __float2bfloat16_rn(o[i][2 * r + e]);
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

template <typename T, int MT> int prep_tile(const PrepP &p, bool own, cudaStream_t st) {
  const size_t smem = ((size_t)MT * p.d.dim + 8 * MT * 64) * 4;
  auto kern = latent_prep_kernel<T, MT>;
  if (int rc = allow_dynamic(kern, smem)) return rc;
  kern<<<dim3(p.q_blocks + (own ? 1 : 0), (p.M + MT - 1) / MT), 256, smem, st>>>(p);
  B200_LAUNCH_CHECK();
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
    q.M = M - m0 < 32768 ? M - m0 : 32768;
    const int kp = (p.d.dim + 15) / 16 * 16;
    const size_t smem = ((size_t)kp * 72 + (size_t)64 * (kp + 8)) * 2;
    if (std::is_same<T, bf16>::value && !own && q.M >= 16 && smem <= (size_t)kMaxDynamic) {
      if (int rc = allow_dynamic(latent_prep_mma_kernel, smem)) return rc;
      latent_prep_mma_kernel<<<dim3(p.col_blocks, p.d.heads, (q.M + 63) / 64), 256, smem, st>>>(q);
      B200_LAUNCH_CHECK();
    } else if (int rc = q.M >= 8 ? prep_tile<T, 8>(q, own, st) : prep_tile<T, 1>(q, own, st)) {
      return rc;
    }
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

template <int KSW, int NTW> int attend_mma_run(const AttendP &p, int M, cudaStream_t st) {
  constexpr int LDK = (KSW > NTW ? KSW : NTW) * 64 + 8;
  const size_t smem = (size_t)2 * kKeys * LDK * 2 + 4 * 16 * 36 * 4 + 2 * 16 * 40 * 2;
  auto kern = latent_attend_mma_kernel<KSW, NTW>;
  if (int rc = allow_dynamic(kern, smem)) return rc;
  for (int m0 = 0; m0 < M; m0 += 32768) {
    AttendP q = p;
    q.qabs += (int64_t)m0 * p.d.heads * (p.d.rank + p.d.rot);
    q.cv.row_seq += m0;
    q.cv.row_pos += m0;
    q.ml += (int64_t)m0 * p.d.heads * p.splits * 2;
    q.acc += (int64_t)m0 * p.d.heads * p.splits * p.rank_pad;
    kern<<<dim3(p.splits, (p.d.heads + 15) / 16, M - m0 < 32768 ? M - m0 : 32768), 256, smem, st>>>(q);
    B200_LAUNCH_CHECK();
  }
  return B200_OK;
}

template <typename T, typename O, int MT> int value_tile(ValueP &p, cudaStream_t st) {
  // few rows: enough CTAs to fill the machine; many: fewer folds of the same shares
  p.rows_cta = p.M <= 16 ? 16 : (p.M <= 128 ? 64 : p.d.vdim);
  const size_t smem = (size_t)MT * (block_pad<T>(p.d.rank) + p.splits) * 4;
  auto kern = latent_value_kernel<T, O, MT>;
  if (int rc = allow_dynamic(kern, smem)) return rc;
  kern<<<dim3((p.d.vdim + p.rows_cta - 1) / p.rows_cta, p.d.heads, (p.M + MT - 1) / MT), 256, smem, st>>>(p);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
template <typename T, typename O> int value_run(const ValueP &p, int M, bf16 *lat, cudaStream_t st) {
  for (int m0 = 0; m0 < M; m0 += 32768) {
    ValueP q = p;
    q.ml += (int64_t)m0 * p.d.heads * p.splits * 2;
    q.acc += (int64_t)m0 * p.d.heads * p.splits * p.rank_pad;
    q.out = reinterpret_cast<O *>(p.out) + (int64_t)m0 * p.ldo;
    q.M = M - m0 < 32768 ? M - m0 : 32768;
    const size_t smem = (size_t)96 * ((p.d.rank + 15) / 16 * 16 + 8) * 2;
    if (std::is_same<O, bf16>::value && lat != nullptr && q.M >= 16 && smem <= (size_t)kMaxDynamic) {
      bf16 *l16 = lat + (int64_t)m0 * p.d.heads * p.rank_pad;
      latent_fold_kernel<<<dim3(p.d.heads, q.M), 128, 0, st>>>(q, l16);
      B200_LAUNCH_CHECK();
      if (int rc = allow_dynamic(latent_value_mma_kernel, smem)) return rc;
      latent_value_mma_kernel<<<dim3((p.d.vdim + 31) / 32, p.d.heads, (q.M + 63) / 64), 256, smem, st>>>(q, l16);
      B200_LAUNCH_CHECK();
    } else if (int rc = q.M >= 8 ? value_tile<T, O, 8>(q, st) : value_tile<T, O, 1>(q, st)) {
      return rc;
    }
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

int latent_shift_launch(int dtype, const LatentDims &d, const void *cache, int src, int tail, const float *inv_freq, int delta,
                        void *stage, cudaStream_t st) {
  if (dtype == B200_F32)
    latent_shift_kernel<float><<<tail, 128, 0, st>>>((const float *)cache, d, src, inv_freq, (float)delta, (float *)stage);
  else
    latent_shift_kernel<bf16><<<tail, 128, 0, st>>>((const bf16 *)cache, d, src, inv_freq, (float)delta, (bf16 *)stage);
  B200_LAUNCH_CHECK();
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

// Shares of the visible keys per row: one resident wave of CTAs (two per SM), at least one tile each.
int latent_splits(const LatentDims &d, int M, int max_ctx) {
  const int n = d.window > 0 && d.window < max_ctx ? d.window : max_ctx;
  const int groups = (d.heads + 15) / 16;
  int want = 2 * 148 / (M * groups);
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
  const int w = d.rank + d.rot;
  if (d.rank <= 128)
    return w <= 128 ? attend_mma_run<2, 2>(p, M, st) : w <= 192 ? attend_mma_run<3, 2>(p, M, st) : attend_mma_run<6, 2>(p, M, st);
  if (d.rank <= 256)
    return w <= 320 ? attend_mma_run<5, 4>(p, M, st) : attend_mma_run<8, 4>(p, M, st);
  if (d.rank <= 512)
    return w <= 576 ? attend_mma_run<9, 8>(p, M, st) : attend_mma_run<12, 8>(p, M, st);
  return w <= 1088 ? attend_mma_run<17, 16>(p, M, st) : attend_mma_run<20, 16>(p, M, st);
}

int latent_value_launch(int dtype, const LatentDims &d, const float *scratch, int M, int splits, const RowMatrix &uv,
                        void *out, int64_t ldo, bool out_bf16, void *work, cudaStream_t st) {
  ValueP p{};
  p.ml = scratch;
  p.acc = scratch + ((int64_t)M * d.heads * splits * 2 + 3) / 4 * 4;
  p.uv = uv.w; p.ldu = uv.ld; p.out = out; p.ldo = ldo; p.d = d; p.splits = splits; p.rank_pad = rank_pad(d);
  if (dtype == B200_F32)
    return value_run<float, float>(p, M, nullptr, st);
  return out_bf16 ? value_run<bf16, bf16>(p, M, (bf16 *)work, st) : value_run<bf16, float>(p, M, nullptr, st);
}

} // namespace b200
