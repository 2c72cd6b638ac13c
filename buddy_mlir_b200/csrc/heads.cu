// Softmax attention over keys and values cached per head (grouped query heads), for layers of
// described models: optional norms over the whole query / key projection, rotation of the first
// dimensions of a head in either layout, a sliding window, a sink (one more softmax entry of a
// given score and no value), an output gate.
//
//   heads_prep_kernel     norms, rotation, cache row [keys of all kv heads | values], queries
//   heads_attend_kernel   one row's keys split over CTAs, f32 FMAs (32-bit models, very wide heads)
//   heads_decode_kernel   the same on mma.sync: the query heads of a group are the tile's rows, every
//                         warp streams its own keys through cp.async
//   heads_prefill_kernel  128 consecutive queries of a head per CTA against 64-key tiles of the
//                         paged cache, online softmax in f32, P as two bf16 terms
//   mix_finish_kernel     fold of the splits, sink, output gate; the norm and gate of a matrix
//                         memory's output (memory.cu); both into the output projection's input
//   heads_shift_kernel    rows moved by some positions, keys turned along
#include "layered.cuh"
#include "rows.cuh"

#include <algorithm>

namespace b200 {

namespace {

constexpr float kLog2e = 1.4426950408889634f;

// cos and sin of pos * freq[i] for all pairs: cs[i], cs[half + i].  The angle is reduced to one
// turn in double, so that it is as exact far from the start as near it.
__device__ __forceinline__ void turn_table(float *cs, const double *freq, int half, int pos, int t, int nt) {
  constexpr double kTurn = 6.283185307179586476925286766559;
  for (int i = t; i < half; i += nt) {
    const double a = (double)pos * freq[i];
    sincosf((float)(a - rint(a * (1.0 / kTurn)) * kTurn), &cs[half + i], &cs[i]);
  }
}

// value c of a head of x (pointing at the head) after norm and rotation; r: 1 / rms, w: norm
// weights of the head, cs: cos then sin of the pairs
__device__ __forceinline__ float turned(const HeadsDims &d, const float *x, int c, float r, const float *w, const float *cs) {
  auto at = [&](int i) { return w != nullptr ? x[i] * r * w[i] : x[i]; };
  if (c >= d.rot)
    return at(c);
  const int half = d.rot >> 1;
  if (d.halves)
    return c < half ? at(c) * cs[c] - at(c + half) * cs[half + c] : at(c) * cs[c - half] + at(c - half) * cs[c];
  const int i = c >> 1;
  return (c & 1) ? at(c) * cs[i] + at(c - 1) * cs[half + i] : at(c) * cs[i] - at(c + 1) * cs[half + i];
}

__device__ __forceinline__ void put2(float *p, float a, float b) { *reinterpret_cast<float2 *>(p) = make_float2(a, b); }
__device__ __forceinline__ void put2(bf16 *p, float a, float b) { *reinterpret_cast<__nv_bfloat162 *>(p) = __floats2bfloat162_rn(a, b); }
__device__ __forceinline__ float2 get2(const float *x, const float *w, int c, float r) {
  float2 v = *reinterpret_cast<const float2 *>(x + c);
  if (w != nullptr) {
    const float2 n = __ldg(reinterpret_cast<const float2 *>(w + c));
    v.x *= r * n.x;
    v.y *= r * n.y;
  }
  return v;
}
// A head by one warp, two elements at a time (dim even, and rot / 2 for split halves).
template <typename T>
__device__ __forceinline__ void turn_head(const HeadsDims &d, const float *x, float r, const float *w, const float *cs, T *dst, int lane) {
  const int half = d.rot >> 1;
  if (d.halves) {
#pragma unroll 2
    for (int i = 2 * lane; i < half; i += 64) {
      const float2 u = get2(x, w, i, r), v = get2(x, w, i + half, r);
      const float2 c = *reinterpret_cast<const float2 *>(cs + i), n = *reinterpret_cast<const float2 *>(cs + half + i);
      put2(dst + i, u.x * c.x - v.x * n.x, u.y * c.y - v.y * n.y);
      put2(dst + half + i, v.x * c.x + u.x * n.x, v.y * c.y + u.y * n.y);
    }
  } else {
#pragma unroll 2
    for (int i = lane; i < half; i += 32) {
      const float2 v = get2(x, w, 2 * i, r);
      put2(dst + 2 * i, v.x * cs[i] - v.y * cs[half + i], v.y * cs[i] + v.x * cs[half + i]);
    }
  }
#pragma unroll 2
  for (int c = d.rot + 2 * lane; c < d.dim; c += 64) {
    const float2 v = get2(x, w, c, r);
    put2(dst + c, v.x, v.y);
  }
}

// grid (M, y): a row's query, key and value heads are dealt to the warps of its y CTAs
template <typename T>
__global__ void __launch_bounds__(256)
heads_prep_kernel(const HeadsDims d, const HeadsIn in, T *q, T *pool, const CacheView cv) {
  extern __shared__ __align__(16) float s_cs[];
  __shared__ float s_red[16];
  const int m = blockIdx.x, tid = threadIdx.x, lane = tid & 31;
  chain_wait();
  chain_next();
  const float *src = in.proj + (int64_t)m * in.ldp, *ks = src + in.off_k, *vs = src + in.off_v;
  const int pos = cv.row_pos[m];
  turn_table(s_cs, in.freq, d.rot >> 1, pos, tid, 256);
  float rq = 1.f, rk = 1.f;
  if (in.q_norm != nullptr) {
    const int nq = d.heads * d.dim, nk = d.kv * d.dim;
    float a = 0.f, b = 0.f;
    auto squares = [tid](const float *x, int n) {
      float t = 0.f;
      if ((n & 3) == 0) {
#pragma unroll 4
        for (int i = tid; i < n / 4; i += 256) {
          const float4 v = reinterpret_cast<const float4 *>(x)[i];
          t = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, t))));
        }
      } else {
        for (int i = tid; i < n; i += 256)
          t = fmaf(x[i], x[i], t);
      }
      return t;
    };
    a = squares(src, nq);
    b = squares(ks, nk);
    a = warp_sum(a);
    b = warp_sum(b);
    if (lane == 0) {
      s_red[tid >> 5] = a;
      s_red[8 + (tid >> 5)] = b;
    }
    __syncthreads();
    a = b = 0.f;
    for (int w = 0; w < 8; ++w) {
      a += s_red[w];
      b += s_red[8 + w];
    }
    rq = 1.0f / sqrtf(a / (float)nq + in.eps);
    rk = 1.0f / sqrtf(b / (float)nk + in.eps);
  }
  __syncthreads();
  T *row = pool + cache_row(cv, cv.row_seq[m], pos) * d.row;
  const bool twos = (d.dim & 1) == 0 && (d.vdim & 1) == 0 && (!d.halves || (d.rot & 3) == 0);
  for (int u = blockIdx.y * 8 + (tid >> 5); u < d.heads + 2 * d.kv; u += gridDim.y * 8) {
    if (u < d.heads + d.kv) {                      // a query or a key head
      const bool query = u < d.heads;
      const int h = query ? u : u - d.heads;
      const float *x = (query ? src : ks) + h * d.dim, *w = query ? in.q_norm : in.k_norm;
      const float r = query ? rq : rk;
      T *dst = query ? q + ((int64_t)m * d.heads + h) * d.dimp : row + h * d.dimp;
      if (w != nullptr)
        w += h * d.dim;
      if (twos) {
        turn_head(d, x, r, w, s_cs, dst, lane);
      } else {
        for (int c = lane; c < d.dim; c += 32)
          dst[c] = from_float<T>(turned(d, x, c, r, w, s_cs));
      }
      if (query && d.dim + lane < d.dimp)          // a cache row's padding is zero already
        dst[d.dim + lane] = from_float<T>(0.f);
    } else {
      const int h = u - d.heads - d.kv;
      const float *x = vs + h * d.vdim;
      T *dst = row + d.kv * d.dimp + h * d.vdimp;
      if (twos) {
#pragma unroll 2
        for (int c = 2 * lane; c < d.vdim; c += 64) {
          const float2 v = *reinterpret_cast<const float2 *>(x + c);
          put2(dst + c, v.x, v.y);
        }
      } else {
        for (int c = lane; c < d.vdim; c += 32)
          dst[c] = from_float<T>(x[c]);
      }
    }
  }
}

// The keys of split sp of S for a query at `pos`: [k0, k1), whole multiples of `unit` but the last.
__device__ __forceinline__ void split_range(const HeadsDims &d, int pos, int sp, int S, int unit, int &k0, int &k1) {
  const int lo = d.window > 0 ? max(0, pos - d.window + 1) : 0, n = pos + 1 - lo;
  const int per = ((n + S - 1) / S + unit - 1) / unit * unit;
  k0 = lo + sp * per;
  k1 = min(k0 + per, pos + 1);
}
// A head's partial result: vdimp values, then the running maximum (in powers of two) and the sum.
__device__ __forceinline__ float *partial_of(float *part, const HeadsDims &d, int64_t n, int h, int S, int sp) {
  return part + ((n * d.heads + h) * S + sp) * (d.vdimp + 4);
}

constexpr int kGroup = 8, kTile = 64;

// grid (splits, kv * head chunks, rows), 128 threads
template <typename T>
__global__ void __launch_bounds__(128)
heads_attend_kernel(const HeadsDims d, const T *q, const int32_t *rows, const T *pool, const CacheView cv, float *part) {
  extern __shared__ float sm[];
  const int g_all = d.heads / d.kv, chunks = (g_all + kGroup - 1) / kGroup;
  const int kvh = blockIdx.y / chunks, g0 = (blockIdx.y - kvh * chunks) * kGroup, g = min(kGroup, g_all - g0);
  chain_wait();
  chain_next();
  const int m = rows ? rows[blockIdx.z] : (int)blockIdx.z, h0 = kvh * g_all + g0;
  const int pos = cv.row_pos[m], seq = cv.row_seq[m];
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  float *s_q = sm, *s_o = s_q + kGroup * d.dimp, *s_p = s_o + kGroup * d.vdimp;   // s_p [kGroup][kTile]
  __shared__ float s_m[kGroup], s_l[kGroup], s_c[kGroup];
  int k0, k1;
  split_range(d, pos, blockIdx.x, gridDim.x, kTile, k0, k1);
  const float sc = d.scale * kLog2e;
  for (int i = tid; i < g * d.dimp; i += 128)
    s_q[i] = to_float(q[((int64_t)m * d.heads + h0) * d.dimp + i]) * sc;
  for (int i = tid; i < g * d.vdimp; i += 128)
    s_o[i] = 0.f;
  if (tid < kGroup) {
    s_m[tid] = -INFINITY;
    s_l[tid] = 0.f;
  }
  __syncthreads();
  for (int t0 = k0; t0 < k1; t0 += kTile) {
    const int n = min(kTile, k1 - t0);
    for (int j = warp; j < n; j += 4) {
      const T *k = pool + cache_row(cv, seq, t0 + j) * d.row + kvh * d.dimp;
      float a[kGroup];
#pragma unroll
      for (int h = 0; h < kGroup; ++h)
        a[h] = 0.f;
      for (int c = lane; c < d.dimp; c += 32) {
        const float kv = to_float(k[c]);
#pragma unroll
        for (int h = 0; h < kGroup; ++h)
          if (h < g)
            a[h] = fmaf(kv, s_q[h * d.dimp + c], a[h]);
      }
#pragma unroll
      for (int h = 0; h < kGroup; ++h)
        if (h < g) {
          a[h] = warp_sum(a[h]);
          if (lane == 0)
            s_p[h * kTile + j] = a[h];
        }
    }
    __syncthreads();
    for (int h = warp; h < g; h += 4) {
      float mx = s_m[h];
      const float old = mx;
      for (int j = lane; j < n; j += 32)
        mx = fmaxf(mx, s_p[h * kTile + j]);
      mx = warp_max(mx);
      float l = 0.f;
      for (int j = lane; j < n; j += 32) {
        const float p = exp2f(s_p[h * kTile + j] - mx);
        s_p[h * kTile + j] = p;
        l += p;
      }
      l = warp_sum(l);
      __syncwarp();
      if (lane == 0) {
        s_c[h] = exp2f(old - mx);
        s_l[h] = s_l[h] * s_c[h] + l;
        s_m[h] = mx;
      }
    }
    __syncthreads();
    for (int c = tid; c < d.vdimp; c += 128) {
      float a[kGroup];
#pragma unroll
      for (int h = 0; h < kGroup; ++h)
        a[h] = h < g ? s_o[h * d.vdimp + c] * s_c[h] : 0.f;
      for (int j = 0; j < n; ++j) {
        const float v = to_float(pool[cache_row(cv, seq, t0 + j) * d.row + d.kv * d.dimp + kvh * d.vdimp + c]);
#pragma unroll
        for (int h = 0; h < kGroup; ++h)
          if (h < g)
            a[h] = fmaf(s_p[h * kTile + j], v, a[h]);
      }
#pragma unroll
      for (int h = 0; h < kGroup; ++h)
        if (h < g)
          s_o[h * d.vdimp + c] = a[h];
    }
    __syncthreads();
  }
  for (int h = 0; h < g; ++h) {
    float *out = partial_of(part, d, blockIdx.z, h0 + h, gridDim.x, blockIdx.x);
    if (k0 < k1)
      for (int c = tid; c < d.vdimp; c += 128)
        out[c] = s_o[h * d.vdimp + c];
    if (tid == 0) {
      out[d.vdimp] = s_m[h];
      out[d.vdimp + 1] = s_l[h];
    }
  }
}

// grid (splits, kv * head chunks of 16 * value chunks of DV, rows), 4 warps
template <int DK, int DV>
__global__ void __launch_bounds__(128)
heads_decode_kernel(const HeadsDims d, const bf16 *q, const int32_t *rows, const bf16 *pool, const CacheView cv, float *part) {
  constexpr int LK = DK + 8, LV = DV + 8, ST = 2;
  constexpr int WARP = ST * 16 * (LK + LV);        // elements of a warp's ring
  extern __shared__ __align__(16) bf16 smb[];
  bf16 *s_q = smb, *ring = s_q + 16 * LK;
  __shared__ float s_m[4][16], s_l[4][16];
  const int g_all = d.heads / d.kv, hchunks = (g_all + 15) / 16, vchunks = (d.vdimp + DV - 1) / DV;
  int y = blockIdx.y;
  const int vc = y % vchunks;
  y /= vchunks;
  const int kvh = y / hchunks, g0 = (y - kvh * hchunks) * 16, g = min(16, g_all - g0), h0 = kvh * g_all + g0;
  const int v0 = vc * DV, nv = min(DV, d.vdimp - v0);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  for (int i = tid; i < (16 * LK + 4 * WARP) / 8; i += 128)
    reinterpret_cast<uint4 *>(smb)[i] = make_uint4(0, 0, 0, 0);
  chain_wait();
  chain_next();
  const int m = rows ? rows[blockIdx.z] : (int)blockIdx.z;
  const int pos = cv.row_pos[m], seq = cv.row_seq[m];
  int k0, k1;
  split_range(d, pos, blockIdx.x, gridDim.x, 64, k0, k1);
  if (k0 >= k1) {
    if (vc == 0 && tid < g) {
      float *out = partial_of(part, d, blockIdx.z, h0 + tid, gridDim.x, blockIdx.x);
      out[d.vdimp] = -INFINITY;
      out[d.vdimp + 1] = 0.f;
    }
    return;
  }
  __syncthreads();
  for (int i = tid; i < g * d.dimp / 8; i += 128) {
    const int r = i / (d.dimp / 8), c = (i - r * (d.dimp / 8)) * 8;
    *reinterpret_cast<uint4 *>(s_q + r * LK + c) = *reinterpret_cast<const uint4 *>(q + ((int64_t)m * d.heads + h0 + r) * d.dimp + c);
  }
  __syncthreads();
  bf16 *mine = ring + warp * WARP;
  const int ck = d.dimp / 8, cn = nv / 8;
  auto load = [&](int j, int st) {                 // keys j .. j + 15
    bf16 *kd = mine + st * 16 * (LK + LV), *vd = kd + 16 * LK;
    const int64_t at = cache_row(cv, seq, min(j + (lane & 15), k1 - 1)) * d.row;
    for (int r = 0; r < 16; r += 2) {              // half a warp per row
      const int rr = r + (lane >> 4);
      const bf16 *src = pool + __shfl_sync(0xffffffffu, at, rr);
      const bool live = j + rr < k1;
      for (int c = lane & 15; c < ck; c += 16)
        cp16(kd + rr * LK + c * 8, src + kvh * d.dimp + c * 8, live);
      for (int c = lane & 15; c < cn; c += 16)
        cp16(vd + rr * LV + c * 8, src + d.kv * d.dimp + kvh * d.vdimp + v0 + c * 8, live);
    }
  };
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
    o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
  const float sc = d.scale * kLog2e;
  int st = 0;
  if (k0 + warp * 16 < k1)
    load(k0 + warp * 16, 0);
  asm volatile("cp.async.commit_group;" ::: "memory");
  for (int j = k0 + warp * 16; j < k1; j += 64, st ^= 1) {
    if (j + 64 < k1)
      load(j + 64, st ^ 1);
    asm volatile("cp.async.commit_group;" ::: "memory");
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncwarp();
    const bf16 *k = mine + st * 16 * (LK + LV), *v = k + 16 * LK;
    float s[2][4] = {};
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t a[4], b[4];
      ldsm4(a, s_q + (lane & 15) * LK + kk * 16 + (lane >> 4) * 8);
      ldsm4(b, k + ((lane & 7) + ((lane >> 4) << 3)) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
      mma16816(s[0], a, b[0], b[1]);
      mma16816(s[1], a, b[2], b[3]);
    }
    float nm[2] = {mx[0], mx[1]};
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        s[i][e] = j + i * 8 + (lane & 3) * 2 + (e & 1) < k1 ? s[i][e] * sc : -INFINITY;
        nm[e >> 1] = fmaxf(nm[e >> 1], s[i][e]);
      }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 1));
      nm[r] = fmaxf(nm[r], __shfl_xor_sync(0xffffffffu, nm[r], 2));   // key j is live: finite
      const float corr = exp2f(mx[r] - nm[r]);
      mx[r] = nm[r];
      l[r] *= corr;
#pragma unroll
      for (int i = 0; i < DV / 8; ++i) {
        o[i][2 * r] *= corr;
        o[i][2 * r + 1] *= corr;
      }
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        s[i][2 * r] = exp2f(s[i][2 * r] - nm[r]);
        s[i][2 * r + 1] = exp2f(s[i][2 * r + 1] - nm[r]);
        l[r] += s[i][2 * r] + s[i][2 * r + 1];
      }
    }
    uint32_t hi[4], lw[4];
    split2(s[0][0], s[0][1], hi[0], lw[0]);
    split2(s[0][2], s[0][3], hi[1], lw[1]);
    split2(s[1][0], s[1][1], hi[2], lw[2]);
    split2(s[1][2], s[1][3], hi[3], lw[3]);
#pragma unroll
    for (int nt = 0; nt < DV / 16; ++nt) {
      uint32_t b[4];
      ldsm4t(b, v + (lane & 15) * LV + nt * 16 + (lane >> 4) * 8);
      mma16816(o[2 * nt], hi, b[0], b[1]);
      mma16816(o[2 * nt], lw, b[0], b[1]);
      mma16816(o[2 * nt + 1], hi, b[2], b[3]);
      mma16816(o[2 * nt + 1], lw, b[2], b[3]);
    }
    __syncwarp();
  }
  asm volatile("cp.async.wait_group 0;" ::: "memory");
  // the four warps' shares, folded
  const int r0 = lane >> 2;
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 1);
    l[r] += __shfl_xor_sync(0xffffffffu, l[r], 2);
    if ((lane & 3) == 0) {
      s_m[warp][r0 + 8 * r] = mx[r];
      s_l[warp][r0 + 8 * r] = l[r];
    }
  }
  __syncthreads();                                 // every warp is done with the ring
  float *s_o = reinterpret_cast<float *>(smb);     // [4][16][DV]
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
#pragma unroll
    for (int r = 0; r < 2; ++r)
      *reinterpret_cast<float2 *>(s_o + (warp * 16 + r0 + 8 * r) * DV + i * 8 + (lane & 3) * 2) = make_float2(o[i][2 * r], o[i][2 * r + 1]);
  __syncthreads();
  for (int i = tid; i < g * nv; i += 128) {
    const int r = i / nv, c = i - r * nv;
    const float M = fmaxf(fmaxf(s_m[0][r], s_m[1][r]), fmaxf(s_m[2][r], s_m[3][r]));
    float a = 0.f, b = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float e = exp2f(s_m[w][r] - M);
      a = fmaf(e, s_o[(w * 16 + r) * DV + c], a);
      b = fmaf(e, s_l[w][r], b);
    }
    float *out = partial_of(part, d, blockIdx.z, h0 + r, gridDim.x, blockIdx.x);
    out[v0 + c] = a;
    if (vc == 0 && c == 0) {
      out[d.vdimp] = M;
      out[d.vdimp + 1] = b;
    }
  }
}

// a row of either result: f32 or bf16
struct CatRow {
  float *f;
  bf16 *b;
  __device__ __forceinline__ void set(int64_t i, float v) const {
    if (f != nullptr)
      f[i] = v;
    else
      b[i] = __float2bfloat16_rn(v);
  }
};
__device__ __forceinline__ float gated(float v, const float *g) { return g != nullptr ? v / (1.0f + expf(-*g)) : v; }

// grid (rows, attention heads + memory heads / 4), 128 threads: four warps share the splits of an
// attention head, or take a memory head each
__global__ void __launch_bounds__(128)
mix_finish_kernel(const MixFinish f) {
  __shared__ float s_w[kMaxSplits];
  __shared__ float4 s_o[4][32];
  chain_wait();
  chain_next();
  const int m = f.rows ? f.rows[blockIdx.x] : (int)blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const CatRow out{f.cat ? f.cat + (int64_t)m * f.ldc : nullptr, f.cat16 ? f.cat16 + (int64_t)m * f.ldc : nullptr};
  const float *proj = f.proj + (int64_t)m * f.ldp;
  int h = blockIdx.y;
  if (h < f.n_heads) {
    const HeadsDims &d = f.h;
    const int64_t ld = d.vdimp + 4;
    const float *part = f.part + ((int64_t)blockIdx.x * d.heads + h) * f.splits * ld;
    // maxima and sums, two splits per lane (kMaxSplits = 64), the same in every warp
    const float sink = d.sink * kLog2e;
    float ms[2], ls[2], mx = sink;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int sp = lane + 32 * i;
      ms[i] = sp < f.splits ? part[sp * ld + d.vdimp] : -INFINITY;
      ls[i] = sp < f.splits ? part[sp * ld + d.vdimp + 1] : 0.f;
      mx = fmaxf(mx, ms[i]);
    }
    mx = warp_max(mx);
    float l = 0.f;
    int live = 0;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const float w = ls[i] > 0.f ? exp2f(ms[i] - mx) : 0.f;
      if (warp == 0)
        s_w[lane + 32 * i] = w;
      l = fmaf(w, ls[i], l);
      const unsigned some = __ballot_sync(0xffffffffu, ls[i] > 0.f);
      if (some)
        live = 32 * i + 32 - __clz(some);
    }
    l = warp_sum(l) + exp2f(sink - mx);
    const float inv = f.h_scale / l;
    __syncthreads();
    for (int c0 = 0; c0 < d.vdimp; c0 += 128) {
      const int c = c0 + lane * 4;
      float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < d.vdimp)
#pragma unroll 4
        for (int sp = warp; sp < live; sp += 4) {
          const float w = s_w[sp];
          if (w > 0.f) {       // an empty split has no values
            const float4 v = *reinterpret_cast<const float4 *>(part + sp * ld + c);
            a.x = fmaf(w, v.x, a.x); a.y = fmaf(w, v.y, a.y); a.z = fmaf(w, v.z, a.z); a.w = fmaf(w, v.w, a.w);
          }
        }
      s_o[warp][lane] = a;
      __syncthreads();
      const int cc = c0 + tid;
      if (cc < d.vdim) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w)
          v += reinterpret_cast<const float *>(s_o[w])[tid];
        out.set(h * d.vdim + cc, gated(v * inv, f.off_g >= 0 ? proj + f.off_g + h * d.vdim + cc : nullptr));
      }
      __syncthreads();
    }
    return;
  }
  h = (h - f.n_heads) * 4 + warp;
  if (h >= f.n_mem)
    return;
  const int vd = f.mem_vdim;
  const float *o = f.mem_o + (int64_t)m * f.ldo + h * vd;
  float s = 0.f;
  const float *g = proj + f.off_mg + h * vd, *nw = f.mem_norm + h * vd;
  if ((vd & 3) == 0) {
#pragma unroll 2
    for (int c = 4 * lane; c < vd; c += 128) {
      const float4 v = *reinterpret_cast<const float4 *>(o + c);
      s = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, s))));
    }
    const float r = f.m_scale / sqrtf(warp_sum(s) / (float)vd + f.eps);
#pragma unroll 2
    for (int c = 4 * lane; c < vd; c += 128) {
      const float4 v = *reinterpret_cast<const float4 *>(o + c), z = *reinterpret_cast<const float4 *>(g + c);
      const float4 w = __ldg(reinterpret_cast<const float4 *>(nw + c));
      const float4 a = make_float4(gated(v.x * r * w.x, &z.x), gated(v.y * r * w.y, &z.y), gated(v.z * r * w.z, &z.z), gated(v.w * r * w.w, &z.w));
      const int64_t at = f.mem_col + h * vd + c;
      if (out.f != nullptr) {
        *reinterpret_cast<float4 *>(out.f + at) = a;
      } else {
        put2(out.b + at, a.x, a.y);
        put2(out.b + at + 2, a.z, a.w);
      }
    }
    return;
  }
  for (int c = lane; c < vd; c += 32)
    s = fmaf(o[c], o[c], s);
  const float r = f.m_scale / sqrtf(warp_sum(s) / (float)vd + f.eps);
  for (int c = lane; c < vd; c += 32)
    out.set(f.mem_col + h * vd + c, gated(o[c] * r * nw[c], g + c));
}

struct FlashP {
  const bf16 *q;               // [rows][heads][dimp]
  const bf16 *pool;
  const int4 *tiles;           // (first row, rows, sequence, first position)
  bf16 *out;                   // [rows][ldo]
  int64_t ldo;
  const float *gate;           // [rows][ldg] or null
  int64_t ldg;
  float out_scale;
  HeadsDims d;
  CacheView cv;
};

constexpr int QT = kHeadsQueryTile, KT = 64, kWarps = QT / 16, kThreads = kWarps * 32;

// grid (tiles, heads, value chunks of DV), a warp per 16 queries
template <int DK, int DV>
__global__ void __launch_bounds__(kThreads)
heads_prefill_kernel(const FlashP p) {
  constexpr int LK = DK + 8, LV = DV + 8;
  extern __shared__ __align__(16) bf16 sm16[];
  bf16 *s_q = sm16;                                // [QT][LK]
  bf16 *s_k = s_q + QT * LK;                       // [2][KT][LK]
  bf16 *s_v = s_k + 2 * KT * LK;                   // [2][KT][LV]
  __shared__ int64_t s_at[2][KT];                  // cache offsets of a tile's rows
  const HeadsDims &d = p.d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tid = threadIdx.x;
  const int4 tile = p.tiles[gridDim.x - 1 - blockIdx.x];             // later positions first
  const int h = blockIdx.y, kvh = h / (d.heads / d.kv);
  const int v0 = blockIdx.z * DV, nv = min(DV, d.vdimp - v0), vdim = min(DV, d.vdim - v0);
  const int i_min = tile.w, i_max = tile.w + tile.y - 1;             // positions of the queries
  const int lo = d.window > 0 ? max(0, i_min - d.window + 1) : 0;
  const int tiles = (i_max - lo) / KT + 1;
  for (int i = tid; i < (QT * LK + 2 * KT * LK + 2 * KT * LV) / 8; i += kThreads)
    reinterpret_cast<uint4 *>(sm16)[i] = make_uint4(0, 0, 0, 0);
  auto addresses = [&](int t) {
    if (tid < KT && t < tiles)
      s_at[t & 1][tid] = cache_row(p.cv, tile.z, min(lo + t * KT + tid, i_max)) * d.row;
  };
  addresses(0);
  addresses(1);
  __syncthreads();
  const int ck = d.dimp / 8, cn = nv / 8;
  {
    const bf16 *src = p.q + ((int64_t)tile.x * d.heads + h) * d.dimp;
    for (int i = tid; i < tile.y * ck; i += kThreads) {
      const int r = i / ck, c = (i - r * ck) * 8;
      *reinterpret_cast<uint4 *>(s_q + r * LK + c) = *reinterpret_cast<const uint4 *>(src + (int64_t)r * d.heads * d.dimp + c);
    }
  }
  auto load_tile = [&](int t, int buf) {
    const int live = i_max - (lo + t * KT);        // rows 0 .. live exist
    bf16 *kd = s_k + buf * KT * LK, *vd = s_v + buf * KT * LV;
    const int cpr = ck + cn;
    for (int i = tid; i < KT * cpr; i += kThreads) {
      const int r = i / cpr, c = i - r * cpr;
      const bf16 *src = p.pool + s_at[buf][r];
      if (c < ck)
        cp16(kd + r * LK + c * 8, src + kvh * d.dimp + c * 8, r <= live);
      else
        cp16(vd + r * LV + (c - ck) * 8, src + d.kv * d.dimp + kvh * d.vdimp + v0 + (c - ck) * 8, r <= live);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  float o[DV / 8][4];
#pragma unroll
  for (int i = 0; i < DV / 8; ++i)
    o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  // the sink is a first entry of weight 1, counted by one lane of a row
  const float sink = d.sink * kLog2e;
  const float one = sink > -INFINITY && (lane & 3) == 0 ? 1.f : 0.f;
  float mx[2] = {sink, sink}, l[2] = {one, one};
  const int r0 = warp * 16 + (lane >> 2);          // this thread's rows: r0, r0 + 8
  const int qi[2] = {i_min + r0, i_min + r0 + 8};
  const float sc = d.scale * kLog2e;

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
    addresses(t + 2);                              // this buffer's addresses have been used
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
        uint32_t b[4];
        ldsm4(b, k + (nt * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
        mma16816(s[2 * nt], a, b[0], b[1]);
        mma16816(s[2 * nt + 1], a, b[2], b[3]);
      }
    }
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
      const float base = nm[r] == -INFINITY ? 0.f : nm[r];   // nothing visible yet
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
#pragma unroll
    for (int kt = 0; kt < KT / 16; ++kt) {
      uint32_t hi[4], lw[4];
      split2(s[2 * kt][0], s[2 * kt][1], hi[0], lw[0]);
      split2(s[2 * kt][2], s[2 * kt][3], hi[1], lw[1]);
      split2(s[2 * kt + 1][0], s[2 * kt + 1][1], hi[2], lw[2]);
      split2(s[2 * kt + 1][2], s[2 * kt + 1][3], hi[3], lw[3]);
#pragma unroll
      for (int nt = 0; nt < DV / 16; ++nt) {
        uint32_t b[4];
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
    const int row = r0 + 8 * r;
    if (row >= tile.y)
      continue;
    const float inv = p.out_scale / l[r];
    const int64_t col = h * d.vdim + v0;
    bf16 *dst = p.out + (int64_t)(tile.x + row) * p.ldo + col;
    const float *g = p.gate != nullptr ? p.gate + (int64_t)(tile.x + row) * p.ldg + col : nullptr;
#pragma unroll
    for (int i = 0; i < DV / 8; ++i) {
      const int c = i * 8 + (lane & 3) * 2;
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (c + e < vdim)
          dst[c + e] = __float2bfloat16_rn(gated(o[i][2 * r + e] * inv, g != nullptr ? g + c + e : nullptr));
    }
  }
}

// rows src .. src + tail of a contiguous cache, keys turned by delta positions, into stage
template <typename T>
__global__ void __launch_bounds__(256)
heads_shift_kernel(const HeadsDims d, const T *cache, int src, const double *freq, int delta, T *stage) {
  extern __shared__ __align__(16) float s_cs[];
  const int half = d.rot >> 1;
  turn_table(s_cs, freq, half, delta, threadIdx.x, 256);
  __syncthreads();
  const T *row = cache + (int64_t)(src + blockIdx.x) * d.row;
  T *dst = stage + (int64_t)blockIdx.x * d.row;
  for (int64_t i = threadIdx.x; i < d.row; i += 256) {
    const int h = (int)(i / d.dimp), c = (int)(i - (int64_t)h * d.dimp);
    if (h >= d.kv || c >= d.rot) {
      dst[i] = row[i];
      continue;
    }
    const int a = d.halves ? (c < half ? c : c - half) : c >> 1;
    const bool second = d.halves ? c >= half : (c & 1);
    const int o = d.halves ? (second ? c - half : c + half) : (c ^ 1);
    const float x = to_float(row[i]), y = to_float(row[i - c + o]);
    dst[i] = from_float<T>(second ? x * s_cs[a] + y * s_cs[half + a] : x * s_cs[a] - y * s_cs[half + a]);
  }
}

// Allow `bytes` of dynamic shared memory for a kernel, once per device and kernel.
template <auto Kern> int allow(size_t bytes) {
  static int configured[64] = {};
  int dev = 0;
  B200_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || configured[dev] < (int)bytes) {
    B200_CUDA(cudaFuncSetAttribute(Kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes));
    if (dev >= 0 && dev < 64)
      configured[dev] = (int)bytes;
  }
  return B200_OK;
}

template <int DK, int DV>
int decode_run(const HeadsDims &d, const bf16 *q, const int32_t *rows, int n, const bf16 *pool, const CacheView &cv, int splits,
               float *part, cudaStream_t st) {
  const size_t ring = ((size_t)16 * (DK + 8) + (size_t)4 * 2 * 16 * (DK + DV + 16)) * 2, fold = (size_t)4 * 16 * DV * 4;
  const size_t smem = std::max(ring, fold);
  if (int rc = allow<heads_decode_kernel<DK, DV>>(smem)) return rc;
  const int g = d.heads / d.kv;
  const dim3 grid(splits, d.kv * ((g + 15) / 16) * ((d.vdimp + DV - 1) / DV), n);
  B200_CUDA(launch_chained(heads_decode_kernel<DK, DV>, grid, 128, smem, st, d, q, rows, pool, cv, part));
  B200_LAUNCH_CHECK();
  return B200_OK;
}
template <int DK, int DV> int flash_run(const FlashP &p, int n_tiles, cudaStream_t st) {
  const size_t smem = ((size_t)(QT + 2 * KT) * (DK + 8) + (size_t)2 * KT * (DV + 8)) * 2;
  if (int rc = allow<heads_prefill_kernel<DK, DV>>(smem)) return rc;
  heads_prefill_kernel<DK, DV><<<dim3(n_tiles, p.d.heads, (p.d.vdimp + DV - 1) / DV), kThreads, smem, st>>>(p);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

} // namespace

int heads_limits(const HeadsDims &d) {
  if (d.heads < 1 || d.kv < 1 || d.heads % d.kv || d.dim < 1 || d.dim > 1024 || d.vdim < 1 || d.vdim > 1024 || d.rot < 0 ||
      (d.rot & 1) || d.rot > d.dim)
    return fail(B200_EINVAL, "heads attention: bad sizes (%d query heads, %d key heads, %d / %d wide, %d rotated)", d.heads, d.kv,
                d.dim, d.vdim, d.rot);
  return B200_OK;
}
bool heads_tensor_cores(const HeadsDims &d) { return d.dimp <= 256; }

int heads_splits(const HeadsDims &d, int rows, int max_ctx) {
  const int per_row = d.kv * ((d.heads / d.kv + 15) / 16);
  int s = (4 * 148 + rows * per_row - 1) / (rows * per_row);
  s = std::min(s, (max_ctx + 63) / 64);
  return std::max(1, std::min(s, kMaxSplits));
}
int64_t heads_scratch_floats(const HeadsDims &d, int rows, int splits) {
  return (int64_t)rows * d.heads * splits * (d.vdimp + 4);
}

int heads_prep_launch(int dtype, const HeadsDims &d, const HeadsIn &in, int M, void *q, void *pool, const CacheView &cv,
                      cudaStream_t st) {
  const size_t smem = (size_t)d.rot * 4 + 16;
  const int units = (d.heads + 2 * d.kv + 7) / 8;
  const dim3 grid(M, std::max(1, std::min(units, 592 / M)));
  if (dtype == B200_F32)
    B200_CUDA(launch_chained(heads_prep_kernel<float>, grid, 256, smem, st, d, in, (float *)q, (float *)pool, cv));
  else
    B200_CUDA(launch_chained(heads_prep_kernel<bf16>, grid, 256, smem, st, d, in, (bf16 *)q, (bf16 *)pool, cv));
  B200_LAUNCH_CHECK();
  return B200_OK;
}

int heads_attend_launch(int dtype, const HeadsDims &d, const void *q, const int32_t *rows, int n, const void *pool,
                        const CacheView &cv, int splits, float *part, cudaStream_t st) {
  if (dtype == B200_BF16 && heads_tensor_cores(d)) {
    const bf16 *q16 = (const bf16 *)q, *p16 = (const bf16 *)pool;
    const bool wide = d.vdimp > 64;
    if (d.dimp <= 64)
      return wide ? decode_run<64, 128>(d, q16, rows, n, p16, cv, splits, part, st) : decode_run<64, 64>(d, q16, rows, n, p16, cv, splits, part, st);
    if (d.dimp <= 128)
      return wide ? decode_run<128, 128>(d, q16, rows, n, p16, cv, splits, part, st) : decode_run<128, 64>(d, q16, rows, n, p16, cv, splits, part, st);
    return wide ? decode_run<256, 128>(d, q16, rows, n, p16, cv, splits, part, st) : decode_run<256, 64>(d, q16, rows, n, p16, cv, splits, part, st);
  }
  const int g = d.heads / d.kv;
  const dim3 grid(splits, d.kv * ((g + kGroup - 1) / kGroup), n);
  const size_t smem = (size_t)kGroup * (d.dimp + d.vdimp + kTile) * 4;
  if (dtype == B200_F32) {
    if (int rc = allow<heads_attend_kernel<float>>(smem)) return rc;
    B200_CUDA(launch_chained(heads_attend_kernel<float>, grid, 128, smem, st, d, (const float *)q, rows, (const float *)pool, cv, part));
  } else {
    if (int rc = allow<heads_attend_kernel<bf16>>(smem)) return rc;
    B200_CUDA(launch_chained(heads_attend_kernel<bf16>, grid, 128, smem, st, d, (const bf16 *)q, rows, (const bf16 *)pool, cv, part));
  }
  B200_LAUNCH_CHECK();
  return B200_OK;
}

int mix_finish_launch(const MixFinish &f, int M, cudaStream_t st) {
  B200_CUDA(launch_chained(mix_finish_kernel, dim3(M, f.n_heads + (f.n_mem + 3) / 4), 128, 0, st, f));
  B200_LAUNCH_CHECK();
  return B200_OK;
}

int heads_prefill_launch(const HeadsDims &d, const bf16 *q, const int4 *tiles, int n_tiles, const bf16 *pool, const CacheView &cv,
                         const float *gate, int64_t ldg, float out_scale, bf16 *out, int64_t ldo, cudaStream_t st) {
  FlashP p{};
  p.q = q; p.pool = pool; p.tiles = tiles; p.out = out; p.ldo = ldo; p.gate = gate; p.ldg = ldg; p.out_scale = out_scale;
  p.d = d; p.cv = cv;
  const bool wide = d.vdimp > 64;
  if (d.dimp <= 64) return wide ? flash_run<64, 128>(p, n_tiles, st) : flash_run<64, 64>(p, n_tiles, st);
  if (d.dimp <= 96) return wide ? flash_run<96, 128>(p, n_tiles, st) : flash_run<96, 64>(p, n_tiles, st);
  if (d.dimp <= 128) return wide ? flash_run<128, 128>(p, n_tiles, st) : flash_run<128, 64>(p, n_tiles, st);
  return wide ? flash_run<256, 128>(p, n_tiles, st) : flash_run<256, 64>(p, n_tiles, st);
}

int heads_shift_launch(int dtype, const HeadsDims &d, const void *cache, int src, int tail, const double *freq, int delta,
                       void *stage, cudaStream_t st) {
  const size_t smem = (size_t)d.rot * 4 + 16;
  if (dtype == B200_F32)
    heads_shift_kernel<float><<<tail, 256, smem, st>>>(d, (const float *)cache, src, freq, delta, (float *)stage);
  else
    heads_shift_kernel<bf16><<<tail, 256, smem, st>>>(d, (const bf16 *)cache, src, freq, delta, (bf16 *)stage);
  B200_LAUNCH_CHECK();
  return B200_OK;
}

} // namespace b200
