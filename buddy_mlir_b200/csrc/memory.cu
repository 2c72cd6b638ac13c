// Matrix memory: a recurrent mixer whose state per head is a [dim][vdim] matrix S, a vector n and
// a running maximum m, all f32.  With a log input gate i and a log forget gate f per token,
//   m' = max(f + m, i);  S = exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone
//   o  = S^T q / (max(|n q|, exp(-m')) + floor)
// and S = n = 0, m = 0 before the first token (position 0 ignores what the slot holds).
//
//   memory_step_kernel   token by token, f32: a CTA keeps 32 columns of S in registers
//   memory_chunk_kernel  64 tokens at a time on mma.sync.  With F the running sum of f inside the
//                        chunk, a_s = i_s - F_s and M_t = max(m, max_{s<=t} a_s), unrolling gives
//                          num_t = exp(m - M_t) S^T q_t + sum_{s<=t} exp(a_s - M_t) (q_t k_s) v_s
//                        and m_t = F_t + M_t: three products per chunk.  q, k, v are the bfloat16
//                        projections; S, the gated scores and the gated values enter as two bf16
//                        terms and are summed in f32; F and a are kept in double.
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

constexpr int kChunk = 64;

// grid (segments * heads, columns / VT), 4 warps
template <int DK, int VT>
__global__ void __launch_bounds__(128)
memory_chunk_kernel(const MemoryDims d, const MemoryIn in, const int4 *segs, const int32_t *row_pos, float *states, float *o,
                    int64_t ldo) {
  constexpr int L = kChunk, LK = DK + 8, VA = VT + 8, LV = VA + 8, NT = VA / 8, MT = DK / 64;
  extern __shared__ __align__(16) bf16 smc[];
  bf16 *s_q = smc, *s_k = s_q + L * LK;            // [L][LK]
  bf16 *s_v = s_k + L * LK;                        // [L][LV]: v | 1
  bf16 *s_wh = s_v + L * LV, *s_wl = s_wh + L * LV;   // gated [v | 1], two terms
  bf16 *s_sh = s_wl + L * LV, *s_sl = s_sh + DK * LV; // [DK][LV]: [S | n], two terms
  __shared__ double s_a[L];
  __shared__ double s_top[L];                      // M_t
  __shared__ float s_inter[L], s_floor[L], s_w[L], s_keep;
  __shared__ double s_m;                           // m before the chunk
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int h = blockIdx.x % d.heads, v0 = blockIdx.y * VT;
  const int4 seg = segs[blockIdx.x / d.heads];
  float *st = states + (int64_t)seg.z * d.state + (int64_t)h * d.head_state;
  const int64_t ld = d.tiles * 32;
  float *sN = st + d.dim * ld, *sM = sN + (int64_t)d.tiles * d.dim;
  const int tile0 = v0 / 32, tile1 = min(tile0 + VT / 32, d.tiles);
  const bool fresh = row_pos[seg.x] == 0;
  // this thread's part of [S | n]: rows warp * DK/4 + 16 mt + (lane >> 2) (+ 8), columns 8 nt + 2 (lane & 3) (+ 1)
  float S[MT][NT][4];
  auto each = [&](auto f) {
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e)
          f(S[mt][nt][e], warp * (DK / 4) + mt * 16 + (lane >> 2) + (e >> 1) * 8, nt * 8 + (lane & 3) * 2 + (e & 1));
  };
  each([&](float &x, int r, int c) {
    x = 0.f;
    if (!fresh && r < d.dim) {
      if (c < VT && v0 + c < ld)
        x = st[r * ld + v0 + c];
      else if (c == VT)
        x = sN[(int64_t)tile0 * d.dim + r];
    }
  });
  if (tid == 0)
    s_m = fresh ? 0.0 : load_max(sM + 2 * tile0);
  for (int i = tid; i < (2 * L * LK + 3 * L * LV + 2 * DK * LV) / 8; i += 128)
    reinterpret_cast<uint4 *>(smc)[i] = make_uint4(0, 0, 0, 0);
  __syncthreads();
  for (int c0 = 0; c0 < seg.y; c0 += L) {
    const int n = min(L, seg.y - c0);
    const float *p0 = in.proj + (int64_t)(seg.x + c0) * in.ldp;
    // gates: a scan over the chunk by the first warp, two tokens per lane
    if (warp == 0) {
      double f[2], a[2], top[2];
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
      const double F[2] = {sum - f[1], sum};
#pragma unroll
      for (int i = 0; i < 2; ++i)
        a[i] = 2 * lane + i < n ? (double)ig[i] - F[i] : -1e300;
      const double m0 = s_m;
      double best = fmax(a[0], a[1]);
#pragma unroll
      for (int w = 1; w < 32; w <<= 1) {
        const double u = __shfl_up_sync(0xffffffffu, best, w);
        if (lane >= w)
          best = fmax(best, u);
      }
      double before = __shfl_up_sync(0xffffffffu, best, 1);
      before = lane == 0 ? m0 : fmax(before, m0);
      top[0] = fmax(before, a[0]);
      top[1] = fmax(top[0], a[1]);
      const double last = __shfl_sync(0xffffffffu, top[1], 31), Fl = __shfl_sync(0xffffffffu, F[1], 31);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        s_a[t] = a[i];
        s_top[t] = top[i];
        s_inter[t] = expf((float)(m0 - top[i]));
        s_floor[t] = expf((float)-(F[i] + top[i]));
        s_w[t] = expf((float)(a[i] - last));
      }
      __syncwarp();
      if (lane == 0) {
        s_keep = expf((float)(m0 - last));
        s_m = Fl + last;
      }
    }
    // the rows, bf16
    for (int i = tid; i < L * (DK / 2); i += 128) {
      const int r = i / (DK / 2), c = 2 * (i - r * (DK / 2));
      if (c >= d.dim)
        continue;
      float2 q = make_float2(0.f, 0.f), k = q;
      if (r < n) {
        const float *p = p0 + (int64_t)r * in.ldp + h * d.dim + c;
        q.x = p[in.off_q] * d.q_scale;
        k.x = p[in.off_k];
        if (c + 1 < d.dim) {
          q.y = p[in.off_q + 1] * d.q_scale;
          k.y = p[in.off_k + 1];
        }
      }
      *reinterpret_cast<__nv_bfloat162 *>(s_q + r * LK + c) = __floats2bfloat162_rn(q.x, q.y);
      *reinterpret_cast<__nv_bfloat162 *>(s_k + r * LK + c) = __floats2bfloat162_rn(k.x, k.y);
    }
    for (int i = tid; i < L * (VA / 2); i += 128) {
      const int r = i / (VA / 2), c = 2 * (i - r * (VA / 2));
      float2 v = make_float2(0.f, 0.f);
      if (r < n) {
        const float *p = p0 + (int64_t)r * in.ldp + in.off_v + h * d.vdim + v0 + c;
        if (c == VT)
          v.x = 1.f;
        else if (c < VT) {
          if (v0 + c < d.vdim) v.x = p[0];
          if (v0 + c + 1 < d.vdim) v.y = p[1];
        }
      }
      *reinterpret_cast<__nv_bfloat162 *>(s_v + r * LV + c) = __floats2bfloat162_rn(v.x, v.y);
    }
    // [S | n] as two terms
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          const int at = (warp * (DK / 4) + mt * 16 + (lane >> 2) + g * 8) * LV + nt * 8 + (lane & 3) * 2;
          uint32_t hi, lo;
          split2(S[mt][nt][2 * g], S[mt][nt][2 * g + 1], hi, lo);
          *reinterpret_cast<uint32_t *>(s_sh + at) = hi;
          *reinterpret_cast<uint32_t *>(s_sl + at) = lo;
        }
    __syncthreads();
    // gated values of the update
    for (int i = tid; i < L * (VA / 2); i += 128) {
      const int r = i / (VA / 2), c = 2 * (i - r * (VA / 2));
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162 *>(s_v + r * LV + c));
      uint32_t hi, lo;
      split2(v.x * s_w[r], v.y * s_w[r], hi, lo);
      *reinterpret_cast<uint32_t *>(s_wh + r * LV + c) = hi;
      *reinterpret_cast<uint32_t *>(s_wl + r * LV + c) = lo;
    }
    const int t0 = warp * 16 + (lane >> 2);        // this thread's tokens: t0, t0 + 8
    if (warp * 16 < n) {
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
          if (nt <= warp) {                        // tokens after this warp's are not seen
            uint32_t b[4];
            ldsm4(b, s_k + (nt * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + kk * 16 + ((lane >> 3) & 1) * 8);
            mma16816(s[2 * nt], a, b[0], b[1]);
            mma16816(s[2 * nt + 1], a, b[2], b[3]);
          }
        const int at = (kk * 16 + (lane & 15)) * LV + (lane >> 4) * 8;
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {       // the odd last block reads its zero padding along
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
        float *dst = o + (int64_t)(seg.x + c0 + t) * ldo + h * d.vdim + v0;
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
    __syncthreads();                               // gated values are complete
    // [S | n] = keep * [S | n] + K^T [gated v | gate]
    const float keep = s_keep;
    each([&](float &x, int, int) { x *= keep; });
#pragma unroll
    for (int kk = 0; kk < L / 16; ++kk) {
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t a[4];
        ldsm4t(a, s_k + (kk * 16 + (lane & 7) + ((lane >> 4) << 3)) * LK + warp * (DK / 4) + mt * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
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
    }
    __syncthreads();                               // the next chunk overwrites the operands
  }
  each([&](float &x, int r, int c) {
    if (r < d.dim) {
      if (c < VT && v0 + c < ld)
        st[r * ld + v0 + c] = x;
      else if (c == VT)
        for (int t = tile0; t < tile1; ++t)
          sN[(int64_t)t * d.dim + r] = x;
    }
  });
  if (tid >= tile0 && tid < tile1)
    store_max(sM + 2 * tid, s_m);
}

template <int R>
int step_run(const MemoryDims &d, const MemoryIn &in, const int4 *segs, int n, const int32_t *row_pos, float *states, float *o,
             int64_t ldo, cudaStream_t st) {
  memory_step_kernel<R><<<dim3(n * d.heads, d.tiles), 256, 0, st>>>(d, in, segs, row_pos, states, o, ldo);
  B200_LAUNCH_CHECK();
  return B200_OK;
}
template <int DK, int VT>
int chunk_run(const MemoryDims &d, const MemoryIn &in, const int4 *segs, int n, const int32_t *row_pos, float *states, float *o,
              int64_t ldo, cudaStream_t st) {
  const size_t smem = ((size_t)2 * kChunk * (DK + 8) + (size_t)3 * kChunk * (VT + 16) + (size_t)2 * DK * (VT + 16)) * 2;
  static int configured[64] = {};
  int dev = 0;
  B200_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    B200_CUDA(cudaFuncSetAttribute(memory_chunk_kernel<DK, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    if (dev >= 0 && dev < 64)
      configured[dev] = 1;
  }
  memory_chunk_kernel<DK, VT><<<dim3(n * d.heads, (d.tiles * 32 + VT - 1) / VT), 128, smem, st>>>(d, in, segs, row_pos, states, o, ldo);
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

int memory_chunk_launch(const MemoryDims &d, const MemoryIn &in, const int4 *segs, int n, const int32_t *row_pos, float *states,
                        float *o, int64_t ldo, cudaStream_t st) {
  if (d.dim <= 64)
    return d.vdim <= 32 ? chunk_run<64, 32>(d, in, segs, n, row_pos, states, o, ldo, st) : chunk_run<64, 64>(d, in, segs, n, row_pos, states, o, ldo, st);
  if (d.dim <= 128)
    return chunk_run<128, 32>(d, in, segs, n, row_pos, states, o, ldo, st);
  return chunk_run<256, 32>(d, in, segs, n, row_pos, states, o, ldo, st);
}

} // namespace b200
