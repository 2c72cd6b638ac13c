// Latent attention for many consecutive queries of one sequence (prefill), bf16 operands with
// f32 scores, weights and sums.
//
// With many queries per key it pays to expand the keys: the visible cache rows are gathered,
// one GEMM with [W_uk; W_uv] gives every head's keys and values, and a tiled attention kernel
// takes [W_uk c | rotated key part] against the rotated queries:
//   latent_store_kernel    new cache rows (RMS-normed latent, rotated key part)
//   latent_query_kernel    rotated bf16 queries
//   latent_gather_kernel   cache rows first .. first + n of a sequence, contiguous
//   latent_prefill_kernel  128 queries of a head per CTA against 64-key tiles; S = Q K^T and
//                          O += P V on mma.sync, online softmax in f32; P enters as two bf16
//                          terms (hi + lo), so the weights keep 16 significant bits
#include "layered.cuh"
#include "rows.cuh"

namespace b200 {

namespace {

__device__ __forceinline__ void rotate(float u, float v, float angle, float &a, float &b) {
  float s, c;
  sincosf(angle, &s, &c);
  a = u * c - v * s;
  b = v * c + u * s;
}

// a CTA of 128 threads per row
__global__ void __launch_bounds__(128)
latent_store_kernel(const float *proj, int64_t ldp, int off, LatentDims d, const float *norm_w, float eps,
                    const float *inv_freq, bf16 *pool, CacheView cv) {
  __shared__ float s_red[4];
  const int m = blockIdx.x;
  const float *down = proj + (int64_t)m * ldp + off;
  const int pos = cv.row_pos[m];
  bf16 *row = pool + cache_row(cv, cv.row_seq[m], pos) * d.row;
  float v[8];                    // rank <= 1024
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int k = i * 128 + threadIdx.x;
    v[i] = k < d.rank ? down[k] : 0.f;
    s = fmaf(v[i], v[i], s);
  }
  s = warp_sum(s);
  if ((threadIdx.x & 31) == 0)
    s_red[threadIdx.x >> 5] = s;
  __syncthreads();
  const float r = 1.0f / sqrtf((s_red[0] + s_red[1] + s_red[2] + s_red[3]) / (float)d.rank + eps);
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const int k = i * 128 + threadIdx.x;
    if (k < d.rank)
      row[k] = __float2bfloat16_rn(v[i] * r * norm_w[k]);
  }
  for (int i = threadIdx.x; i < d.rot / 2; i += 128) {
    float a, b;
    rotate(down[d.rank + 2 * i], down[d.rank + 2 * i + 1], (float)pos * inv_freq[i], a, b);
    row[d.rank + 2 * i] = __float2bfloat16_rn(a);
    row[d.rank + 2 * i + 1] = __float2bfloat16_rn(b);
  }
}

// grid M: [heads][dim + rot], the rotated part turned to the row's position
__global__ void __launch_bounds__(256)
latent_query_kernel(const float *proj, int64_t ldp, LatentDims d, const float *inv_freq, const int32_t *row_pos, bf16 *q) {
  extern __shared__ float s_cs[];   // cos, sin per pair
  const int m = blockIdx.x, dq = d.dim + d.rot, half = d.rot / 2;
  const float pos = (float)row_pos[m];
  for (int i = threadIdx.x; i < half; i += 256)
    sincosf(pos * inv_freq[i], &s_cs[half + i], &s_cs[i]);
  __syncthreads();
  const float *src = proj + (int64_t)m * ldp;
  bf16 *dst = q + (int64_t)m * d.heads * dq;
  if ((d.dim & 1) == 0 && (ldp & 1) == 0) {   // pairs never straddle the two parts
    const int hp = dq / 2;
    for (int k = threadIdx.x; k < d.heads * hp; k += 256) {
      const int i = k % hp - d.dim / 2;
      float2 v = *reinterpret_cast<const float2 *>(src + 2 * k);
      if (i >= 0)
        v = make_float2(v.x * s_cs[i] - v.y * s_cs[half + i], v.y * s_cs[i] + v.x * s_cs[half + i]);
      *reinterpret_cast<__nv_bfloat162 *>(dst + 2 * k) = __floats2bfloat162_rn(v.x, v.y);
    }
    return;
  }
  for (int k = threadIdx.x; k < d.heads * dq; k += 256) {
    const int c = k % dq - d.dim;
    float v = src[k];
    if (c >= 0) {
      const int i = c >> 1;
      v = (c & 1) ? v * s_cs[i] + src[k - 1] * s_cs[half + i] : v * s_cs[i] - src[k + 1] * s_cs[half + i];
    }
    dst[k] = __float2bfloat16_rn(v);
  }
}

// grid n / 8, a warp per row
__global__ void __launch_bounds__(256)
latent_gather_kernel(const bf16 *pool, CacheView cv, int64_t row, int seq, int first, int n, bf16 *out) {
  const int lane = threadIdx.x & 31, r = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= n)
    return;
  const uint4 *src = reinterpret_cast<const uint4 *>(pool + cache_row(cv, seq, first + r) * row);
  uint4 *dst = reinterpret_cast<uint4 *>(out + (int64_t)r * row);
  for (int i = lane; i < row / 8; i += 32)
    dst[i] = src[i];
}

struct FlashP {
  const bf16 *q;               // [n][heads][dim + rot]
  int n, pos0;
  const bf16 *rows;            // [keys][row]: cache rows from position `first` on
  const bf16 *kv;              // [keys][ldkv]: heads * dim keys, then heads * vdim values
  int64_t ldkv;
  int first;
  bf16 *out;                   // [n][ldo]
  int64_t ldo;
  LatentDims d;
  int vec;                     // 16-byte copies possible
};

constexpr int QT = 128, KT = 64, kWarps = QT / 16, kThreads = kWarps * 32;

// grid (query tiles, heads, value columns / DV), a warp per 16 queries.  DK >= dim + rot and DV:
// padded widths; value rows wider than DV are taken DV columns per CTA.
template <int DK, int DV>
__global__ void __launch_bounds__(kThreads)
latent_prefill_kernel(const FlashP p) {
  constexpr int LK = DK + 8, LV = DV + 8;
  extern __shared__ __align__(16) bf16 sm[];
  bf16 *s_q = sm;                                  // [QT][LK]
  bf16 *s_k = s_q + QT * LK;                       // [2][KT][LK]
  bf16 *s_v = s_k + 2 * KT * LK;                   // [2][KT][LV]
  const LatentDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int h = blockIdx.y, q0 = (gridDim.x - 1 - blockIdx.x) * QT;   // the longest tiles first
  const int dq = d.dim + d.rot;
  const int v0 = blockIdx.z * DV, vdim = min(DV, d.vdim - v0);
  const int q_last = min(q0 + QT, p.n) - 1;
  // absolute positions
  const int i_min = p.pos0 + q0, i_max = p.pos0 + q_last;
  const int lo = d.window > 0 ? max(0, i_min - d.window + 1) : 0;
  const int tiles = (i_max - lo) / KT + 1;

  for (int i = threadIdx.x; i < (QT * LK + 2 * KT * LK + 2 * KT * LV) / 8; i += kThreads)
    reinterpret_cast<uint4 *>(sm)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  {
    const bf16 *src = p.q + (int64_t)q0 * d.heads * dq + (int64_t)h * dq;
    const int rows = q_last - q0 + 1;
    if (p.vec) {
      const int cpr = dq / 8;
      for (int i = threadIdx.x; i < rows * cpr; i += kThreads) {
        const int r = i / cpr, c = (i - r * cpr) * 8;
        *reinterpret_cast<uint4 *>(s_q + r * LK + c) = *reinterpret_cast<const uint4 *>(src + (int64_t)r * d.heads * dq + c);
      }
    } else {
      for (int i = threadIdx.x; i < rows * dq; i += kThreads) {
        const int r = i / dq, c = i - r * dq;
        s_q[r * LK + c] = src[(int64_t)r * d.heads * dq + c];
      }
    }
  }
  auto load_tile = [&](int t, int buf) {
    const int j0 = lo + t * KT;                    // absolute position of the tile's first key
    bf16 *kd = s_k + buf * KT * LK, *vd = s_v + buf * KT * LV;
    if (p.vec) {
      const int ck = d.dim / 8, cr = d.rot / 8, cv = vdim / 8, cpr = ck + cr + cv;
      for (int i = threadIdx.x; i < KT * cpr; i += kThreads) {
        const int r = i / cpr, c = i - r * cpr;
        const bool live = j0 + r <= i_max;
        const int64_t key = (live ? j0 + r : i_max) - p.first;
        if (c < ck)
          cp16(kd + r * LK + c * 8, p.kv + key * p.ldkv + h * d.dim + c * 8, live);
        else if (c < ck + cr)
          cp16(kd + r * LK + c * 8, p.rows + key * d.row + d.rank + (c - ck) * 8, live);
        else
          cp16(vd + r * LV + (c - ck - cr) * 8, p.kv + key * p.ldkv + d.heads * d.dim + h * d.vdim + v0 + (c - ck - cr) * 8, live);
      }
    } else {
      const int cpr = dq + vdim;
      for (int i = threadIdx.x; i < KT * cpr; i += kThreads) {
        const int r = i / cpr, c = i - r * cpr;
        const bool live = j0 + r <= i_max;
        const int64_t key = (live ? j0 + r : i_max) - p.first;
        bf16 v = __float2bfloat16_rn(0.f);
        if (live)
          v = c < d.dim ? p.kv[key * p.ldkv + h * d.dim + c]
            : c < dq    ? p.rows[key * d.row + d.rank + c - d.dim]
                        : p.kv[key * p.ldkv + d.heads * d.dim + h * d.vdim + v0 + c - dq];
        if (c < dq)
          kd[r * LK + c] = v;
        else
          vd[r * LV + c - dq] = v;
      }
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };

  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
    o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const int r0 = warp * 16 + (lane >> 2);          // this thread's rows: r0, r0 + 8
  const int qi[2] = {i_min + r0, i_min + r0 + 8};
  const float sc = d.scale * 1.4426950408889634f;  // softmax in powers of two

  load_tile(0, 0);
  for (int t = 0; t < tiles; ++t) {
    const int buf = t & 1;
    if (t + 1 < tiles) {
      load_tile(t + 1, buf ^ 1);
      asm volatile("cp.async.wait_group 1;" ::: "memory");
    } else {
      asm volatile("cp.async.wait_group 0;" ::: "memory");
    }
    __syncthreads();
    const bf16 *k = s_k + buf * KT * LK, *v = s_v + buf * KT * LV;
    float s[KT / 8][4];
#pragma unroll
    for (int i = 0; i < KT / 8; ++i)
      s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll 4
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t a[4];
      ldsm4(a, s_q + (warp * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8);
#pragma unroll
      for (int nt = 0; nt < KT / 16; ++nt) {
        uint32_t b[4];   // keys nt*16 .. +15: k halves of the first and the second eight keys
        ldsm4(b, k + (nt * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
        mma16816(s[2 * nt], a, b[0], b[1]);
        mma16816(s[2 * nt + 1], a, b[2], b[3]);
      }
    }
    // mask, running maximum
    const int j0 = lo + t * KT;
    const bool whole = j0 + KT - 1 <= i_min && (d.window <= 0 || i_max - j0 < d.window);
    float nm[2] = {mx[0], mx[1]};
#pragma unroll
    for (int i = 0; i < KT / 8; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int row = e >> 1;
        s[i][e] *= sc;
        if (!whole) {
          const int j = j0 + i * 8 + (lane & 3) * 2 + (e & 1);
          if (j > qi[row] || (d.window > 0 && qi[row] - j >= d.window))
            s[i][e] = -INFINITY;
        }
        nm[row] = fmaxf(nm[row], s[i][e]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 1));
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 2));
      const float base = nm[r] == -INFINITY ? 0.f : nm[r];   // no visible key yet
      const float corr = exp2f(mx[r] - base);
      mx[r] = nm[r];
      l[r] *= corr;
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        o[i][2 * r] *= corr;
        o[i][2 * r + 1] *= corr;
      }
#pragma unroll
      for (int i = 0; i < KT / 8; ++i) {
        s[i][2 * r] = exp2f(s[i][2 * r] - base);
        s[i][2 * r + 1] = exp2f(s[i][2 * r + 1] - base);
        l[r] += s[i][2 * r] + s[i][2 * r + 1];
      }
    }
    // O += P V, sixteen keys at a time
#pragma unroll
    for (int kt = 0; kt < KT / 16; ++kt) {
      uint32_t hi[4], lw[4];
      split2(s[2 * kt][0], s[2 * kt][1], hi[0], lw[0]);
      split2(s[2 * kt][2], s[2 * kt][3], hi[1], lw[1]);
      split2(s[2 * kt + 1][0], s[2 * kt + 1][1], hi[2], lw[2]);
      split2(s[2 * kt + 1][2], s[2 * kt + 1][3], hi[3], lw[3]);
#pragma unroll
      for (int nt = 0; nt < DV / 16; ++nt) {
        uint32_t b[4];   // values nt*16 .. +15 of sixteen keys
        ldsm4t(b, v + (kt * 16 + (lane & 15)) * LV + nt * 16 + (lane >> 4) * 8);
        mma16816(o[2 * nt], hi, b[0], b[1]);
        mma16816(o[2 * nt], lw, b[0], b[1]);
        mma16816(o[2 * nt + 1], hi, b[2], b[3]);
        mma16816(o[2 * nt + 1], lw, b[2], b[3]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    const int row = q0 + r0 + 8 * r;
    if (row >= p.n)
      continue;
    const float inv = 1.0f / l[r];
    bf16 *dst = p.out + (int64_t)row * p.ldo + h * d.vdim + v0;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      const int c = i * 8 + (lane & 3) * 2;
      if (c < vdim)
        dst[c] = __float2bfloat16_rn(o[i][2 * r] * inv);
      if (c + 1 < vdim)
        dst[c + 1] = __float2bfloat16_rn(o[i][2 * r + 1] * inv);
    }
  }
}

template <int DK, int DV> int flash_run(const FlashP &p, cudaStream_t st) {
  auto kern = latent_prefill_kernel<DK, DV>;
  const size_t smem = ((size_t)(QT + 2 * KT) * (DK + 8) + (size_t)2 * KT * (DV + 8)) * 2;
  static int configured[64] = {};
  int dev = 0;
  B200_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    B200_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    if (dev >= 0 && dev < 64)
      configured[dev] = 1;
  }
  kern<<<dim3((p.n + QT - 1) / QT, p.d.heads, (p.d.vdim + DV - 1) / DV), kThreads, smem, st>>>(p);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
template <int DK> int flash_values(const FlashP &p, cudaStream_t st) {
  if (p.d.vdim <= 64) return flash_run<DK, 64>(p, st);
  return flash_run<DK, 128>(p, st);
}

} // namespace

bool latent_prefill_takes(const LatentDims &d) { return d.dim + d.rot <= 256; }

int latent_store_launch(const LatentDims &d, const float *proj, int64_t ldp, int M, int off_down, const float *norm_w,
                        float eps, const float *inv_freq, void *pool, const CacheView &cv, cudaStream_t st) {
  latent_store_kernel<<<M, 128, 0, st>>>(proj, ldp, off_down, d, norm_w, eps, inv_freq, (bf16 *)pool, cv);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
int latent_query_launch(const LatentDims &d, const float *proj, int64_t ldp, int M, const float *inv_freq,
                        const int32_t *row_pos, bf16 *q, cudaStream_t st) {
  latent_query_kernel<<<M, 256, (size_t)d.rot * 4 + 16, st>>>(proj, ldp, d, inv_freq, row_pos, q);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
int latent_gather_launch(const LatentDims &d, const void *pool, const CacheView &cv, int seq, int first, int n, bf16 *rows,
                         cudaStream_t st) {
  latent_gather_kernel<<<(n + 7) / 8, 256, 0, st>>>((const bf16 *)pool, cv, d.row, seq, first, n, rows);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

// Queries at positions pos0 .. pos0 + n - 1; rows / kv from position `first` (no later than the
// first query's first visible key) to the last query.
int latent_prefill_launch(const LatentDims &d, const bf16 *q, int n, int pos0, const bf16 *rows, const bf16 *kv, int64_t ldkv,
                          int first, bf16 *out, int64_t ldo, cudaStream_t st) {
  FlashP p{};
  p.q = q; p.n = n; p.pos0 = pos0; p.rows = rows; p.kv = kv; p.ldkv = ldkv; p.first = first;
  p.out = out; p.ldo = ldo; p.d = d;
  p.vec = d.dim % 8 == 0 && d.rot % 8 == 0 && d.vdim % 8 == 0 && d.rank % 8 == 0 && ldkv % 8 == 0;
  const int dk = d.dim + d.rot;
  if (dk <= 64) return flash_values<64>(p, st);
  if (dk <= 96) return flash_values<96>(p, st);
  if (dk <= 128) return flash_values<128>(p, st);
  if (dk <= 192) return flash_values<192>(p, st);
  return flash_values<256>(p, st);
}

} // namespace b200
