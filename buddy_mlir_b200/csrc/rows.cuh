// Plain weight rows (f32 or bfloat16, k in its natural order): the streaming dot
// product that the GEMV-shaped kernels share, and the gate of a gated feed-forward pair.
#pragma once
#include "common.cuh"

#include <type_traits>

namespace b200 {

typedef __nv_bfloat16 bf16;

// E elements per 16-byte unit, in NG groups of four.
template <typename T> struct RowUnit;
template <> struct RowUnit<float> {
  static constexpr int E = 4, NG = 1;
  static __device__ __forceinline__ void group(const uint4 &u, int, float (&w)[4]) {
    w[0] = __uint_as_float(u.x);
    w[1] = __uint_as_float(u.y);
    w[2] = __uint_as_float(u.z);
    w[3] = __uint_as_float(u.w);
  }
};
template <> struct RowUnit<bf16> {
  static constexpr int E = 8, NG = 2;
  static __device__ __forceinline__ void group(const uint4 &u, int g, float (&w)[4]) {
    const uint32_t a = g == 0 ? u.x : u.z, b = g == 0 ? u.y : u.w;
    w[0] = __uint_as_float(a << 16);
    w[1] = __uint_as_float(a & 0xFFFF0000u);
    w[2] = __uint_as_float(b << 16);
    w[3] = __uint_as_float(b & 0xFFFF0000u);
  }
};
template <typename T> __device__ __forceinline__ T from_float(float v);
template <> __device__ __forceinline__ float from_float<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_float<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float to_float(float v) { return v; }
__device__ __forceinline__ float to_float(bf16 v) { return __bfloat162float(v); }

__device__ __forceinline__ uint4 ld_stream_row(const void *p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(p));
  return v;
}

// Elements of a row rounded up to whole units, and of a staged activation row to whole blocks of
// 32 units (what one warp reads per step).
template <typename T> __host__ __device__ inline int unit_pad(int n) {
  constexpr int E = std::is_same<T, float>::value ? 4 : 8;
  return (n + E - 1) / E * E;
}
template <typename T> __host__ __device__ inline int block_pad(int n) {
  constexpr int B = std::is_same<T, float>::value ? 128 : 256;
  return (n + B - 1) / B * B;
}
// Slot of the four activations 4g..4g+3 inside a staged row: a lane's groups lie 32 slots apart,
// so that neighbouring lanes read neighbouring 16-byte slots.
template <typename T> __device__ __forceinline__ int stage_slot(int g) {
  constexpr int NG = RowUnit<T>::NG;
  if (NG == 1)
    return g;
  return (g & ~63) + ((g & 1) << 5) + ((g & 63) >> 1);
}
// Stage x[0..n) (f32) as slots; elements from n to the end of the last block become zero.
// norm_w != null: x * r * norm_w; otherwise x * r.
template <typename T>
__device__ __forceinline__ void stage_row(float4 *xs, const float *x, int n, float r, const float *norm_w, int t, int nt) {
  const bool vec = (reinterpret_cast<uintptr_t>(x) & 15) == 0 && (norm_w == nullptr || (reinterpret_cast<uintptr_t>(norm_w) & 15) == 0);
  for (int g = t; g < block_pad<T>(n) / 4; g += nt) {
    const int k = 4 * g;
    float v[4] = {0.f, 0.f, 0.f, 0.f};
    if (vec && k + 3 < n) {
      const float4 a = *reinterpret_cast<const float4 *>(x + k);
      v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else {
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (k + e < n)
          v[e] = x[k + e];
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      v[e] *= r;
      if (norm_w != nullptr && k + e < n)
        v[e] *= __ldg(norm_w + k + e);
    }
    xs[stage_slot<T>(g)] = make_float4(v[0], v[1], v[2], v[3]);
  }
}
// acc[r][m] += sum over k < kc of row r * staged row m; kc a multiple of E, rows readable up to kc.
// UN blocks of every row are requested before the first is used.
template <typename T, int MT, int R>
__device__ __forceinline__ void dot_rows(const T *const (&row)[R], int kc, const float4 *xs, int xs_ld, int lane,
                                         float (&acc)[R][MT]) {
  using U = RowUnit<T>;
  constexpr int BLK = 32 * U::E;
  constexpr int UN = MT * R >= 16 ? 2 : (R >= 4 ? 2 : (R == 2 ? 4 : 6));
  for (int b0 = 0; b0 < kc; b0 += BLK * UN) {
    uint4 wv[UN][R];
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      const int k = b0 + u * BLK + lane * U::E;
#pragma unroll
      for (int r = 0; r < R; ++r)
        wv[u][r] = k < kc ? ld_stream_row(row[r] + k) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int u = 0; u < UN; ++u) {
      const int b = b0 + u * BLK;
      if (b + lane * U::E < kc) {
#pragma unroll
        for (int g = 0; g < U::NG; ++g) {
          float wf[R][4];
#pragma unroll
          for (int r = 0; r < R; ++r)
            U::group(wv[u][r], g, wf[r]);
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            const float4 xv = xs[m * xs_ld + (b >> 2) + g * 32 + lane];
#pragma unroll
            for (int r = 0; r < R; ++r) {
              acc[r][m] = fmaf(xv.x, wf[r][0], acc[r][m]);
              acc[r][m] = fmaf(xv.y, wf[r][1], acc[r][m]);
              acc[r][m] = fmaf(xv.z, wf[r][2], acc[r][m]);
              acc[r][m] = fmaf(xv.w, wf[r][3], acc[r][m]);
            }
          }
        }
      }
    }
  }
}

// A gated pair: g' = min(g, limit), u' = clamp(u, -limit, limit), g' * sigmoid(slope * g') * (u' + offset).
// limit = infinity, slope = 1, offset = 0 is the SiLU gate.
struct Gate {
  float limit, slope, offset;
};
__device__ __forceinline__ float gate_pair(const Gate &p, float g, float u) {
  g = fminf(g, p.limit);
  u = fminf(fmaxf(u, -p.limit), p.limit);
  return (g / (1.0f + expf(-p.slope * g))) * (u + p.offset);
}

// What a contraction's epilogue does to a result (row m, column n) besides the bias: an activation,
// and a factor mul[row[m]][n] (a table in the compute type).
struct RowAct {
  int kind;                    // B200_ACT_*
  const void *mul;             // null: none
  int mul_f32;
  int64_t ld;
  const int32_t *row;
};
__device__ __forceinline__ float activate(int kind, float z) {
  if (kind == B200_ACT_RELU2) {
    z = fmaxf(z, 0.f);
    return z * z;
  }
  if (kind == B200_ACT_GELU_TANH)
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
  return z;
}
__device__ __forceinline__ float row_act(const RowAct &a, float z, int64_t m, int64_t n) {
  z = activate(a.kind, z);
  if (a.mul != nullptr) {
    const int64_t i = (int64_t)a.row[m] * a.ld + n;
    z *= a.mul_f32 ? reinterpret_cast<const float *>(a.mul)[i] : __bfloat162float(reinterpret_cast<const bf16 *>(a.mul)[i]);
  }
  return z;
}

// What is still to be added to rows of the residual stream: RMSNorm(y) * w (y null: nothing), and the
// scaled embedding row of the token (embed null: nothing; a table in the compute type).
struct Unsettled {
  const float *y;              // rows as long as the stream's, tight
  const float *w;
  const void *embed;
  int64_t lde;
  float scale;
  const int32_t *tokens;
  __host__ __device__ bool any() const { return y != nullptr || embed != nullptr; }
};

// mma.sync building blocks
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], const void *p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], const void *p) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void mma16816(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp16(void *dst, const void *src, bool live) {
  const uint32_t a = (uint32_t)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(a), "l"(src), "r"(live ? 16 : 0) : "memory");
}
// two f32 as packed bf16 (first in the low half), and what the rounding left
__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __low2float(h), y - __high2float(h));
  hi = *reinterpret_cast<const uint32_t *>(&h);
  lo = *reinterpret_cast<const uint32_t *>(&l);
}

} // namespace b200
