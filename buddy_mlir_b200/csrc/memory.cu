// Matrix memory: a recurrent mixer whose state per head is a [dim][vdim] matrix S, a vector n and
// a running maximum m, all f32.  With a log input gate i and a log forget gate f per token,
//   m' = max(f + m, i);  S = exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone
//   o  = S^T q / (max(|n q|, exp(-m')) + floor)
// and S = n = 0, m = 0 before the first token (position 0 ignores what the slot holds).
//
//   memory_step_kernel   token by token, f32: a CTA keeps 32 columns of S in registers
//   long runs of tokens in chunks of 64, all chunks at once, on mma.sync.  With F the running sum of
//   f inside a chunk, a_s = i_s - F_s and M_t = max(m, max_{s<=t} a_s), unrolling gives
//     num_t = exp(m - M_t) S^T q_t + sum_{s<=t} exp(a_s - M_t) (q_t k_s) v_s,   m_t = F_t + M_t
//     memory_update_kernel  a chunk's own contribution U = sum_s exp(a_s - max a) k_s [v_s | 1]
//     memory_carry_kernel   S, n, m through the chunks of a segment: U becomes the state before each
//     memory_read_kernel    the outputs of a chunk from the state before it
//   q, k, v are the bfloat16 projections; S, the gated scores and the gated values enter the products
//   as two bf16 terms and are summed in f32; F, a and m are kept in double.
//
// State of a slot, per head: S [dim][tiles * 32], then for each 32-column tile its own copy of
// n [dim], then of m, so that the CTAs of a head need nothing from one another.  m is a sum of as
// many terms as there are tokens and is taken exponentials of: it is kept as two f32 (a double).
#include "layered.cuh"
#include "rows.cuh"

#include <algorithm>

namespace b200 {

namespace {

__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ double load_max(const float *p) { return (double)p[0] + (double)p[1]; }
__device__ __forceinline__ void store_max(float *p, double m) {
  p[0] = (float)m;
  p[1] = (float)(m - (double)p[0]);
}

// grid (segments * heads, tiles), 8 warps: a lane per column, a warp's rows d = warp + 8 r
template <int R>
__global__ void __launch_bounds__(256)
memory_step_kernel(const MemoryDims d, const MemoryIn in, const int4 *segs, const int32_t *row_pos, float *states, float *o,
                   int64_t ldo) {
  constexpr int DM = 8 * R;
  __shared__ float s_q[2][DM], s_k[2][DM], s_o[2][8][32], s_n[2][8];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x % d.heads, tile = blockIdx.y, col = tile * 32 + lane;
  chain_wait();
  chain_next();
  const int4 seg = segs[blockIdx.x / d.heads];     // first row, rows, slot
  float *st = states + (int64_t)seg.z * d.state + (int64_t)h * d.head_state;
  float *sS = st + col, *sN = st + (int64_t)d.dim * d.tiles * 32 + (int64_t)tile * d.dim;
  float *sM = st + (int64_t)d.dim * d.tiles * 32 + (int64_t)d.tiles * d.dim + 2 * tile;
  const int64_t ld = d.tiles * 32;
  const bool fresh = row_pos[seg.x] == 0;
  float S[R], n[(DM + 255) / 256];
#pragma unroll
  for (int r = 0; r < R; ++r)
    S[r] = !fresh && warp + 8 * r < d.dim ? sS[(warp + 8 * r) * ld] : 0.f;
#pragma unroll
  for (int i = 0; i < (DM + 255) / 256; ++i)
    n[i] = !fresh && tid + 256 * i < d.dim ? sN[tid + 256 * i] : 0.f;
  double m = fresh ? 0.0 : load_max(sM);
  for (int t = 0; t < seg.y; ++t) {
    const int b = t & 1;
    const float *p = in.proj + (int64_t)(seg.x + t) * in.ldp;
    for (int i = tid; i < DM; i += 256) {
      s_q[b][i] = i < d.dim ? p[in.off_q + h * d.dim + i] * d.q_scale : 0.f;
      s_k[b][i] = i < d.dim ? p[in.off_k + h * d.dim + i] : 0.f;
    }
    const float v = col < d.vdim ? p[in.off_v + h * d.vdim + col] : 0.f;
    const float ig = capped(p[in.off_i + h], d.cap), fg = log_sigmoid(capped(p[in.off_f + h], d.cap));
    const double fm = (double)fg + m, nm = fmax(fm, (double)ig);
    const float keep = expf((float)(fm - nm)), add = expf((float)((double)ig - nm));
    m = nm;
    __syncthreads();
    float acc = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      S[r] = fmaf(keep, S[r], add * s_k[b][warp + 8 * r] * v);
      acc = fmaf(S[r], s_q[b][warp + 8 * r], acc);
    }
    float nq = 0.f;
#pragma unroll
    for (int i = 0; i < (DM + 255) / 256; ++i)
      if (tid + 256 * i < DM) {
        n[i] = fmaf(keep, n[i], add * s_k[b][tid + 256 * i]);
        nq = fmaf(n[i], s_q[b][tid + 256 * i], nq);
      }
    nq = warp_sum(nq);
    s_o[b][warp][lane] = acc;
    if (lane == 0)
      s_n[b][warp] = nq;
    __syncthreads();
    if (warp == 0 && col < d.vdim) {
      float a = 0.f, c = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) {
        a += s_o[b][w][lane];
        c += s_n[b][w];
      }
      o[(int64_t)(seg.x + t) * ldo + h * d.vdim + col] = a / (fmaxf(fabsf(c), expf((float)-m)) + d.floor);
    }
  }
#pragma unroll
  for (int r = 0; r < R; ++r)
    if (warp + 8 * r < d.dim)
      sS[(warp + 8 * r) * ld] = S[r];
#pragma unroll
  for (int i = 0; i < (DM + 255) / 256; ++i)
    if (tid + 256 * i < d.dim)
      sN[tid + 256 * i] = n[i];
  if (tid == 0)
    store_max(sM, m);
}

constexpr int kChunk = kMemoryChunk;
static_assert(kChunk == 64, "two tokens per lane, sixteen per warp");

// The gates of a chunk by one warp, two tokens per lane: F, a, and the maximum of a up to the
// lane's second token; tokens from n on add nothing.
__device__ __forceinline__ void gate_scan(const MemoryDims &d, const MemoryIn &in, const float *p0, int n, int h, int lane,
                                          double (&F)[2], double (&a)[2], double &best) {
  double f[2];
  float ig[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int t = 2 * lane + i;
    const float *p = p0 + (int64_t)min(t, n - 1) * in.ldp;
    ig[i] = capped(p[in.off_i + h], d.cap);
    f[i] = t < n ? (double)log_sigmoid(capped(p[in.off_f + h], d.cap)) : 0.0;
  }
  double sum = f[0] + f[1];
#pragma unroll
  for (int w = 1; w < 32; w <<= 1) {
    const double u = __shfl_up_sync(0xffffffffu, sum, w);
    if (lane >= w)
      sum += u;
  }
  F[0] = sum - f[1];
  F[1] = sum;
#pragma unroll
  for (int i = 0; i < 2; ++i)
    a[i] = 2 * lane + i < n ? (double)ig[i] - F[i] : -1e300;
  best = fmax(a[0], a[1]);
#pragma unroll
  for (int w = 1; w < 32; w <<= 1) {
    const double u = __shfl_up_sync(0xffffffffu, best, w);
    if (lane >= w)
      best = fmax(best, u);
  }
}

// elements c .. c + 3 of a row part of `width` elements (zero from there on); vec: 16-byte loads.
// Read-only for the whole kernel, so that a thread's loads can all be under way at once.
__device__ __forceinline__ float4 load4(const float *p, int c, int width, bool vec) {
  if (vec && c + 3 < width)
    return __ldg(reinterpret_cast<const float4 *>(p + c));
  return make_float4(c < width ? __ldg(p + c) : 0.f, c + 1 < width ? __ldg(p + c + 1) : 0.f, c + 2 < width ? __ldg(p + c + 2) : 0.f,
                     c + 3 < width ? __ldg(p + c + 3) : 0.f);
}
__device__ __forceinline__ void put4(bf16 *dst, const float4 &v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2 *>(dst) = make_uint2(*reinterpret_cast<const uint32_t *>(&a), *reinterpret_cast<const uint32_t *>(&b));
}
__device__ __forceinline__ void put4_split(bf16 *hi, bf16 *lo, const float4 &v) {
  uint32_t h[2], l[2];
  split2(v.x, v.y, h[0], l[0]);
  split2(v.z, v.w, h[1], l[1]);
  *reinterpret_cast<uint2 *>(hi) = make_uint2(h[0], h[1]);
  *reinterpret_cast<uint2 *>(lo) = make_uint2(l[0], l[1]);
}
// use(row, column, elements column .. column + 3) for every group of four columns 0 .. COLS - 1 of
// rows 0 .. ROWS - 1 of src; zero from row n and column `width` on.  Eight loads per thread are under
// way at a time (vec: 16-byte ones; then width % 4 == 0).
template <int ROWS, int COLS, typename F>
__device__ __forceinline__ void each4(const float *src, int64_t ld, int n, int width, bool vec, F use) {
  constexpr int G = COLS / 4, N = ROWS * G, B = 8;
  static_assert(N % 128 == 0, "whole rounds of 128 threads");
  if (!vec) {
    for (int i = threadIdx.x; i < N; i += 128) {
      const int r = i / G, c = 4 * (i - r * G);
      use(r, c, r < n ? load4(src + (int64_t)r * ld, c, width, false) : make_float4(0.f, 0.f, 0.f, 0.f));
    }
    return;
  }
#pragma unroll 1
  for (int i0 = threadIdx.x; i0 < N; i0 += B * 128) {
    float4 v[B];
#pragma unroll
    for (int j = 0; j < B; ++j) {
      const int i = i0 + j * 128, r = i / G, c = 4 * (i - r * G);   // beyond the end: some row that exists
      v[j] = __ldg(reinterpret_cast<const float4 *>(src + (int64_t)min(r, n - 1) * ld + min(c, width - 4)));
    }
#pragma unroll
    for (int j = 0; j < B; ++j) {
      const int i = i0 + j * 128, r = i / G, c = 4 * (i - r * G);
      if (i < N)
        use(r, c, r < n && c < width ? v[j] : make_float4(0.f, 0.f, 0.f, 0.f));
    }
  }
}
// the column of ones behind VT value columns, and zeros to the end of the row: use(row, column, elements)
template <int VT, typename F> __device__ __forceinline__ void each_one(int n, F use) {
  for (int i = threadIdx.x; i < kChunk * 4; i += 128)
    use(i >> 2, VT + 4 * (i & 3), make_float4((i & 3) == 0 && (i >> 2) < n ? 1.f : 0.f, 0.f, 0.f, 0.f));
}

// grid (chunks * heads, columns / VT), 4 warps: a warp computes DK / 4 rows of U
template <int DK, int VT>
__global__ void __launch_bounds__(128)
memory_update_kernel(const MemoryDims d, const MemoryIn in, const int4 *chunks, float *U, double *meta) {
  constexpr int L = kChunk, LK = DK + 8, VA = VT + 8, LV = VA + 8, NT = VA / 8, MT = DK / 64;
  extern __shared__ __align__(16) bf16 smc[];
  bf16 *s_k = smc;                                 // [L][LK]
  bf16 *s_wh = s_k + L * LK, *s_wl = s_wh + L * LV;   // gated [v | 1], two terms
  __shared__ float s_w[L];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int chunk = blockIdx.x / d.heads, h = blockIdx.x - chunk * d.heads, v0 = blockIdx.y * VT;
  const int4 seg = chunks[chunk];
  const int n = seg.y;
  const float *p0 = in.proj + (int64_t)seg.x * in.ldp;
  if (warp == 0) {
    double F[2], a[2], best;
    gate_scan(d, in, p0, n, h, lane, F, a, best);
    const double A = __shfl_sync(0xffffffffu, best, 31);
    s_w[2 * lane] = expf((float)(a[0] - A));
    s_w[2 * lane + 1] = expf((float)(a[1] - A));
    if (lane == 31 && blockIdx.y == 0) {
      meta[(int64_t)blockIdx.x * 3] = A;
      meta[(int64_t)blockIdx.x * 3 + 1] = F[1];
    }
  }
  const bool vec = (d.dim & 3) == 0, vvec = (d.vdim & 3) == 0;
  each4<L, DK>(p0 + in.off_k + h * d.dim, in.ldp, n, d.dim, vec, [&](int r, int c, const float4 &v) { put4(s_k + r * LK + c, v); });
  __syncthreads();
  auto put = [&](int r, int c, const float4 &v) {  // the values as the bf16 they are elsewhere, times the gate
    const float w = s_w[r];
    auto g = [&](float x) { return __bfloat162float(__float2bfloat16_rn(x)) * w; };
    put4_split(s_wh + r * LV + c, s_wl + r * LV + c, make_float4(g(v.x), g(v.y), g(v.z), g(v.w)));
  };
  each4<L, VT>(p0 + in.off_v + h * d.vdim + v0, in.ldp, n, d.vdim - v0, vvec, put);
  each_one<VT>(n, put);
  __syncthreads();
  float S[MT][NT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
      S[mt][nt][0] = S[mt][nt][1] = S[mt][nt][2] = S[mt][nt][3] = 0.f;
#pragma unroll
  for (int kk = 0; kk < L / 16; ++kk)
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      uint32_t a[4];
      ldsm4t(a, s_k + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + warp * (DK / 4) + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {         // the odd last block reads its zero padding along
        uint32_t b[4];
        const int at = (kk * 16 + (lane & 15)) * LV + (lane >> 4) * 8 + nt * 8;
        ldsm4t(b, s_wh + at);
        mma16816(S[mt][nt], a, b[0], b[1]);
        if (nt + 1 < NT)
          mma16816(S[mt][nt + 1 < NT ? nt + 1 : nt], a, b[2], b[3]);
        ldsm4t(b, s_wl + at);
        mma16816(S[mt][nt], a, b[0], b[1]);
        if (nt + 1 < NT)
          mma16816(S[mt][nt + 1 < NT ? nt + 1 : nt], a, b[2], b[3]);
      }
    }
  const int64_t ld = d.tiles * 32;
  float *out = U + (int64_t)blockIdx.x * d.head_state;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int g = 0; g < 2; ++g) {
        const int r = warp * (DK / 4) + mt * 16 + (lane >> 2) + g * 8, c = nt * 8 + (lane & 3) * 2;
        if (r >= d.dim)
          continue;
        if (c < VT) {
          if (v0 + c < ld)
            *reinterpret_cast<float2 *>(out + r * ld + v0 + c) = make_float2(S[mt][nt][2 * g], S[mt][nt][2 * g + 1]);
        } else if (c == VT && blockIdx.y == 0) {
          out[d.dim * ld + r] = S[mt][nt][2 * g];
        }
      }
}

// grid (segments * heads, elements of [S | n] / 1024): four elements per thread, through the chunks
__global__ void __launch_bounds__(256)
memory_carry_kernel(const MemoryDims d, const int4 *segs, const int32_t *chunk0, const int32_t *row_pos, float *U, double *meta,
                    float *states) {
  const int sg = blockIdx.x / d.heads, h = blockIdx.x - sg * d.heads;
  const int4 seg = segs[sg];
  const int n = (seg.y + kChunk - 1) / kChunk, c0 = chunk0[sg];
  const bool fresh = row_pos[seg.x] == 0;
  float *st = states + (int64_t)seg.z * d.state + (int64_t)h * d.head_state;
  const int e = (blockIdx.y * 256 + threadIdx.x) * 4, nS = d.dim * d.tiles * 32;
  const bool live = e < nS + d.dim;
  float *sM = st + nS + d.tiles * d.dim;
  double m = fresh ? 0.0 : load_max(sM);
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (!fresh && live) {
    if (e < nS) {
      S = *reinterpret_cast<const float4 *>(st + e);
    } else {
      const float *p = st + e;                     // n, the first tile's copy
      const int w = d.dim - (e - nS);
      S = make_float4(p[0], w > 1 ? p[1] : 0.f, w > 2 ? p[2] : 0.f, w > 3 ? p[3] : 0.f);
    }
  }
  float *u = U + ((int64_t)c0 * d.heads + h) * d.head_state + e;
  double *mt = meta + ((int64_t)c0 * d.heads + h) * 3;
  const int64_t du = (int64_t)d.heads * d.head_state, dm = (int64_t)d.heads * 3;
  constexpr int B = 4;
  for (int c = 0; c < n; c += B) {
    float4 v[B];
    double A[B], F[B];
#pragma unroll
    for (int i = 0; i < B; ++i)
      if (c + i < n) {
        A[i] = mt[(c + i) * dm];
        F[i] = mt[(c + i) * dm + 1];
        if (live)
          v[i] = *reinterpret_cast<const float4 *>(u + (c + i) * du);
      }
#pragma unroll
    for (int i = 0; i < B; ++i)
      if (c + i < n) {
        const double M = fmax(m, A[i]);
        const float keep = expf((float)(m - M)), add = expf((float)(A[i] - M));
        if (blockIdx.y == 0 && threadIdx.x == 0)
          mt[(c + i) * dm + 2] = m;
        if (live) {
          *reinterpret_cast<float4 *>(u + (c + i) * du) = S;
          S = make_float4(fmaf(keep, S.x, add * v[i].x), fmaf(keep, S.y, add * v[i].y), fmaf(keep, S.z, add * v[i].z),
                          fmaf(keep, S.w, add * v[i].w));
        }
        m = F[i] + M;
      }
  }
  if (live && e < nS) {
    *reinterpret_cast<float4 *>(st + e) = S;
  } else if (live) {
    const float a[4] = {S.x, S.y, S.z, S.w};
    for (int t = 0; t < d.tiles; ++t)
      for (int i = 0; i < 4; ++i)
        if (e - nS + i < d.dim)
          st[nS + t * d.dim + e - nS + i] = a[i];
  }
}

// grid (chunks * heads, columns / VT), 4 warps of 16 tokens; a segment's last chunk leaves the
// running maximum in the state (the carry kernel, whose CTAs all read the old one, has ended)
template <int DK, int VT>
__global__ void __launch_bounds__(128)
memory_read_kernel(const MemoryDims d, const MemoryIn in, const int4 *chunks, int n_chunks, const float *U, const double *meta,
                   float *states, float *o, int64_t ldo) {
  constexpr int L = kChunk, LK = DK + 8, VA = VT + 8, LV = VA + 8, NT = VA / 8;
  extern __shared__ __align__(16) bf16 smc[];
  bf16 *s_q = smc, *s_k = s_q + L * LK;            // [L][LK]
  bf16 *s_v = s_k + L * LK;                        // [L][LV]: v | 1
  bf16 *s_sh = s_v + L * LV, *s_sl = s_sh + DK * LV;  // [DK][LV]: [S | n], two terms
  __shared__ double s_a[L], s_top[L];              // a, M
  __shared__ float s_inter[L], s_floor[L];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int chunk = blockIdx.x / d.heads, h = blockIdx.x - chunk * d.heads, v0 = blockIdx.y * VT;
  const int4 seg = chunks[chunk];
  const int n = seg.y;
  const float *p0 = in.proj + (int64_t)seg.x * in.ldp;
  if (warp == 0) {
    double F[2], a[2], best;
    gate_scan(d, in, p0, n, h, lane, F, a, best);
    const double m0 = meta[(int64_t)blockIdx.x * 3 + 2];
    double before = __shfl_up_sync(0xffffffffu, best, 1);
    before = lane == 0 ? m0 : fmax(before, m0);
    const double top[2] = {fmax(before, a[0]), fmax(before, fmax(a[0], a[1]))};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 2 * lane + i;
      s_a[t] = a[i];
      s_top[t] = top[i];
      s_inter[t] = expf((float)(m0 - top[i]));
      s_floor[t] = expf((float)-(F[i] + top[i]));
    }
    if (lane == 31 && blockIdx.y == 0 && (chunk + 1 == n_chunks || chunks[chunk + 1].z != seg.z)) {
      float *sM = states + (int64_t)seg.z * d.state + (int64_t)h * d.head_state + (int64_t)d.dim * d.tiles * 32 + d.tiles * d.dim;
      for (int t = 0; t < d.tiles; ++t)
        store_max(sM + 2 * t, F[1] + top[1]);
    }
  }
  const bool vec = (d.dim & 3) == 0, vvec = (d.vdim & 3) == 0;
  const float qs = d.q_scale;
  each4<L, DK>(p0 + in.off_q + h * d.dim, in.ldp, n, d.dim, vec,
               [&](int r, int c, const float4 &v) { put4(s_q + r * LK + c, make_float4(v.x * qs, v.y * qs, v.z * qs, v.w * qs)); });
  each4<L, DK>(p0 + in.off_k + h * d.dim, in.ldp, n, d.dim, vec, [&](int r, int c, const float4 &v) { put4(s_k + r * LK + c, v); });
  auto put = [&](int r, int c, const float4 &v) { put4(s_v + r * LV + c, v); };
  each4<L, VT>(p0 + in.off_v + h * d.vdim + v0, in.ldp, n, d.vdim - v0, vvec, put);
  each_one<VT>(n, put);
  const int ld = d.tiles * 32;
  const float *S = U + (int64_t)blockIdx.x * d.head_state;
  each4<DK, VT>(S + v0, ld, d.dim, ld - v0, true, [&](int r, int c, const float4 &v) { put4_split(s_sh + r * LV + c, s_sl + r * LV + c, v); });
  for (int i = tid; i < DK * 4; i += 128) {
    const int r = i >> 2, c = VT + 4 * (i & 3);
    put4_split(s_sh + r * LV + c, s_sl + r * LV + c, make_float4((i & 3) == 0 && r < d.dim ? __ldg(S + d.dim * ld + r) : 0.f, 0.f, 0.f, 0.f));
  }
  __syncthreads();
  if (warp * 16 >= n)
    return;
  const int t0 = warp * 16 + (lane >> 2);          // this thread's tokens: t0, t0 + 8
  float acc[NT][4], s[8][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
    acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i)
    s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f;
#pragma unroll 2
  for (int kk = 0; kk < DK / 16; ++kk) {
    uint32_t a[4];
    ldsm4(a, s_q + (warp * 16 + (lane & 15)) * LK + kk * 16 + (lane >> 4) * 8);
#pragma unroll
    for (int nt = 0; nt < 4; ++nt)
      if (nt <= warp) {                            // tokens after this warp's are not seen
        uint32_t b[4];
        ldsm4(b, s_k + (nt * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
        mma16816(s[2 * nt], a, b[0], b[1]);
        mma16816(s[2 * nt + 1], a, b[2], b[3]);
      }
    const int at = (kk * 16 + (lane & 15)) * LV + (lane >> 4) * 8;
#pragma unroll
    for (int nt = 0; nt < NT; nt += 2) {
      uint32_t b[4];
      ldsm4t(b, s_sh + at + nt * 8);
      mma16816(acc[nt], a, b[0], b[1]);
      if (nt + 1 < NT)
        mma16816(acc[nt + 1 < NT ? nt + 1 : nt], a, b[2], b[3]);
      ldsm4t(b, s_sl + at + nt * 8);
      mma16816(acc[nt], a, b[0], b[1]);
      if (nt + 1 < NT)
        mma16816(acc[nt + 1 < NT ? nt + 1 : nt], a, b[2], b[3]);
    }
  }
  const double top[2] = {s_top[t0], s_top[t0 + 8]};
  const float inter[2] = {s_inter[t0], s_inter[t0 + 8]};
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e)
      acc[i][e] *= inter[e >> 1];
#pragma unroll
  for (int i = 0; i < 8; ++i)
    if (i < 2 * warp + 2)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int j = i * 8 + (lane & 3) * 2 + (e & 1);
        s[i][e] = j <= t0 + (e >> 1) * 8 ? s[i][e] * expf((float)(s_a[j] - top[e >> 1])) : 0.f;
      }
#pragma unroll
  for (int kt = 0; kt < 4; ++kt)
    if (kt <= warp) {
      uint32_t hi[4], lw[4];
      split2(s[2 * kt][0], s[2 * kt][1], hi[0], lw[0]);
      split2(s[2 * kt][2], s[2 * kt][3], hi[1], lw[1]);
      split2(s[2 * kt + 1][0], s[2 * kt + 1][1], hi[2], lw[2]);
      split2(s[2 * kt + 1][2], s[2 * kt + 1][3], hi[3], lw[3]);
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t b[4];
        ldsm4t(b, s_v + (kt * 16 + (lane & 15)) * LV + (lane >> 4) * 8 + nt * 8);
        mma16816(acc[nt], hi, b[0], b[1]);
        mma16816(acc[nt], lw, b[0], b[1]);
        if (nt + 1 < NT) {
          mma16816(acc[nt + 1 < NT ? nt + 1 : nt], hi, b[2], b[3]);
          mma16816(acc[nt + 1 < NT ? nt + 1 : nt], lw, b[2], b[3]);
        }
      }
    }
#pragma unroll
  for (int g = 0; g < 2; ++g) {
    const int t = t0 + 8 * g;
    const float nq = __shfl_sync(0xffffffffu, acc[NT - 1][2 * g], lane & ~3);   // the column of ones
    if (t >= n)
      continue;
    const float inv = 1.0f / (fmaxf(fabsf(nq), s_floor[t]) + d.floor);
    float *dst = o + (int64_t)(seg.x + t) * ldo + h * d.vdim + v0;
#pragma unroll
    for (int i = 0; i < NT - 1; ++i) {
      const int c = i * 8 + (lane & 3) * 2;
      if (v0 + c < d.vdim)
        dst[c] = acc[i][2 * g] * inv;
      if (v0 + c + 1 < d.vdim)
        dst[c + 1] = acc[i][2 * g + 1] * inv;
    }
  }
}

template <int R>
int step_run(const MemoryDims &d, const MemoryIn &in, const int4 *segs, int n, const int32_t *row_pos, float *states, float *o,
             int64_t ldo, cudaStream_t st) {
  B200_CUDA(launch_chained(memory_step_kernel<R>, dim3(n * d.heads, d.tiles), 256, 0, st, d, in, segs, row_pos, states, o, ldo));
  B200_LAUNCH_CHECK();
  return B200_OK;
}
template <auto Kern> int allow(size_t bytes) {
  static int configured[64] = {};
  int dev = 0;
  B200_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    B200_CUDA(cudaFuncSetAttribute(Kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    if (dev >= 0 && dev < 64)
      configured[dev] = 1;
  }
  return B200_OK;
}

template <int DK, int VT>
int chunk_run(const MemoryDims &d, const MemoryIn &in, const MemoryChunks &k, const int32_t *row_pos, float *states, float *o,
              int64_t ldo, cudaStream_t st) {
  constexpr int L = kChunk, LK = DK + 8, LV = VT + 16;
  const size_t update = ((size_t)L * LK + (size_t)2 * L * LV) * 2;
  const size_t read = ((size_t)2 * L * LK + (size_t)L * LV + (size_t)2 * DK * LV) * 2;
  if (int rc = allow<memory_update_kernel<DK, VT>>(update)) return rc;
  if (int rc = allow<memory_read_kernel<DK, VT>>(read)) return rc;
  const dim3 grid(k.n_chunks * d.heads, (d.tiles * 32 + VT - 1) / VT);
  memory_update_kernel<DK, VT><<<grid, 128, update, st>>>(d, in, k.chunks, k.U, k.meta);
  B200_LAUNCH_CHECK();
  const int elems = d.dim * d.tiles * 32 + d.dim;
  memory_carry_kernel<<<dim3(k.n_segs * d.heads, (elems + 1023) / 1024), 256, 0, st>>>(d, k.segs, k.chunk0, row_pos, k.U, k.meta, states);
  B200_LAUNCH_CHECK();
  memory_read_kernel<DK, VT><<<grid, 128, read, st>>>(d, in, k.chunks, k.n_chunks, k.U, k.meta, states, o, ldo);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

} // namespace

int memory_limits(const MemoryDims &d) {
  if (d.heads < 1 || d.dim < 1 || d.dim > 512 || d.vdim < 1 || !(d.cap > 0.f))
    return fail(B200_EINVAL, "matrix memory: bad sizes (%d heads, %d x %d)", d.heads, d.dim, d.vdim);
  return B200_OK;
}
bool memory_chunks_take(const MemoryDims &d) { return d.dim <= 256 && d.tiles <= 128; }

int memory_step_launch(const MemoryDims &d, const MemoryIn &in, const int4 *segs, int n, const int32_t *row_pos, float *states,
                       float *o, int64_t ldo, cudaStream_t st) {
  if (d.dim <= 32) return step_run<4>(d, in, segs, n, row_pos, states, o, ldo, st);
  if (d.dim <= 64) return step_run<8>(d, in, segs, n, row_pos, states, o, ldo, st);
  if (d.dim <= 128) return step_run<16>(d, in, segs, n, row_pos, states, o, ldo, st);
  if (d.dim <= 256) return step_run<32>(d, in, segs, n, row_pos, states, o, ldo, st);
  return step_run<64>(d, in, segs, n, row_pos, states, o, ldo, st);
}

int memory_chunk_launch(const MemoryDims &d, const MemoryIn &in, const MemoryChunks &k, const int32_t *row_pos, float *states,
                        float *o, int64_t ldo, cudaStream_t st) {
  if (d.dim <= 64)
    return d.vdim <= 32 ? chunk_run<64, 32>(d, in, k, row_pos, states, o, ldo, st) : chunk_run<64, 64>(d, in, k, row_pos, states, o, ldo, st);
  if (d.dim <= 128)
    return chunk_run<128, 64>(d, in, k, row_pos, states, o, ldo, st);
  return chunk_run<256, 32>(d, in, k, row_pos, states, o, ldo, st);
}

} // namespace b200
