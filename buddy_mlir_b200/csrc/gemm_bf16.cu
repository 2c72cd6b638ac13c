// bf16 x bf16 -> f32 GEMM on the 5th-generation tensor cores over plain weight rows,
// C[M, N] = A[M, K] * W[N, K]^T, for prefill and batched decode of models whose weights are
// bfloat16.
//
// Both operands arrive by TMA (cp.async.bulk.tensor, no multicast) as 128-byte-swizzled rows of
// 64 k; one thread issues tcgen05.mma (128 x 128 or 128 x 256 x 16) into a f32 accumulator in
// tensor memory; eight warps read it back (tcgen05.ld), apply the epilogue and write whole rows:
// plain or added to C, f32 or bf16, with a bias and an activation, or the gate of (gate, up) column pairs.  Two CTAs share an
// SM, so one's epilogue runs under the other's main loop.  Few output tiles: the k range is split
// over gridDim.z and a second kernel adds the partial tiles in split order.
//
// Grouped form (mixture of experts): rows of A are sorted by expert, a tile table made on the
// device says which expert's weight rows a row tile meets and how many of its rows are real.
//
// Every wait is bounded; on expiry an error word is set, all roles fall through and tensor memory
// is released.
#include "layered.cuh"
#include "rows.cuh"
#include "tc.cuh"

#include <algorithm>

namespace b200 {

namespace {

constexpr int BM = 128, BK = 64, kThreads = 320, kMaxStages = 6;
constexpr int kEpiWarps = 8, kLds = 128 + 4;
constexpr int kMaxPartialTiles = 320;

struct Bars {
  uint64_t full[kMaxStages], empty[kMaxStages], accum;
  uint32_t tmem_base;
  int abort_flag;
};

struct Params {
  int M, N, K;
  float *C;                    // f32 result, or null
  bf16 *C16;                   // bf16 result, or null
  int64_t ldc;
  int add, pairs;
  Gate gate;
  const float *bias;
  RowAct act;
  int stages, splits;
  float *partial;              // [tile][split][128][128]
  const int4 *tiles;           // grouped: (expert, first row, rows, -)
  const int *n_tiles;
  int *error;
};

template <int BNT>
__device__ __forceinline__ void mma(uint32_t tmem_d, uint64_t da, uint64_t db, uint32_t accumulate) {
  // kind::f16 descriptor: D = f32, A = B = bf16, both K-major
  constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BNT >> 3) << 17) | ((uint32_t)(BM >> 4) << 24);
  asm volatile(
      "{\n .reg .pred p;\n setp.ne.b32 p, %4, 0;\n"
      " tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n}" ::"r"(tmem_d),
      "l"(da), "l"(db), "r"(idesc), "r"(accumulate)
      : "memory");
}

// Store `cols` staged values of row m from column n on: 1 or 4 at a time.
__device__ __forceinline__ void store4(const Params &p, int64_t m, int64_t n, float4 v, int valid, bool vec) {
  if (p.bias != nullptr || p.act.kind != B200_ACT_NONE || p.act.mul != nullptr) {
    float a[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int e = 0; e < 4; ++e)
      if (e < valid)
        a[e] = row_act(p.act, p.bias != nullptr ? a[e] + p.bias[n + e] : a[e], m, n + e);
    v = make_float4(a[0], a[1], a[2], a[3]);
  }
  if (p.C != nullptr) {
    float *dst = p.C + m * p.ldc + n;
    if (vec && valid == 4) {
      if (p.add) {
        const float4 c = *reinterpret_cast<const float4 *>(dst);
        v.x += c.x; v.y += c.y; v.z += c.z; v.w += c.w;
      }
      *reinterpret_cast<float4 *>(dst) = v;
    } else {
      const float a[4] = {v.x, v.y, v.z, v.w};
      for (int e = 0; e < valid; ++e)
        dst[e] = p.add ? dst[e] + a[e] : a[e];
    }
  } else {
    bf16 *dst = p.C16 + m * p.ldc + n;
    if (vec && valid == 4) {
      const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
      *reinterpret_cast<uint2 *>(dst) = make_uint2(*reinterpret_cast<const uint32_t *>(&lo), *reinterpret_cast<const uint32_t *>(&hi));
    } else {
      const float a[4] = {v.x, v.y, v.z, v.w};
      for (int e = 0; e < valid; ++e)
        dst[e] = __float2bfloat16_rn(a[e]);
    }
  }
}
__device__ __forceinline__ bool vector_rows(const Params &p) {
  return (p.ldc & 3) == 0 && (p.C != nullptr ? ((uintptr_t)p.C & 15) == 0 : ((uintptr_t)p.C16 & 7) == 0);
}

template <int BNT>
__global__ void __launch_bounds__(kThreads)
gemm_bf16_tc_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, const Params p) {
  constexpr uint32_t A_BYTES = BM * BK * 2, W_BYTES = BNT * BK * 2, STAGE = A_BYTES + W_BYTES;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint8_t *tiles = reinterpret_cast<uint8_t *>(((uintptr_t)smem + 1023) & ~(uintptr_t)1023);
  const int stages = p.stages;
  Bars &bars = *reinterpret_cast<Bars *>(tiles + stages * STAGE);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  int m0 = blockIdx.y * BM, rows_end = p.M, wrow = 0;
  if (p.tiles != nullptr) {
    if ((int)blockIdx.y >= *p.n_tiles)
      return;
    const int4 t = p.tiles[blockIdx.y];
    m0 = t.y;
    rows_end = t.y + t.z;
    wrow = t.x * p.N;
  }
  const int n0 = blockIdx.x * BNT;
  const int nkb_all = (p.K + BK - 1) / BK;
  const int kb0 = (int)((int64_t)nkb_all * blockIdx.z / p.splits);
  const int nkb = (int)((int64_t)nkb_all * (blockIdx.z + 1) / p.splits) - kb0;
  volatile int *ab = &bars.abort_flag;

  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) {
      mbar_init(&bars.full[s], 1);
      mbar_init(&bars.empty[s], 1);
    }
    mbar_init(&bars.accum, 1);
    bars.abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&bars.tmem_base)), "n"(BNT) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const uint32_t tmem = bars.tmem_base;

  if (warp == 0) {
    if (lane == 0) {
      for (int i = 0; i < nkb; ++i) {
        const int s = i % stages, use = i / stages;
        if (use > 0 && !mbar_wait(&bars.empty[s], (use - 1) & 1, ab, p.error, 721))
          break;
        uint8_t *st = tiles + s * STAGE;
        mbar_expect_tx(&bars.full[s], STAGE);
        tma_load_2d(st, &map_a, (kb0 + i) * BK, m0, &bars.full[s]);
        tma_load_2d(st + A_BYTES, &map_w, (kb0 + i) * BK, wrow + n0, &bars.full[s]);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      for (int i = 0; i < nkb; ++i) {
        const int s = i % stages, use = i / stages;
        if (!mbar_wait(&bars.full[s], use & 1, ab, p.error, 722))
          break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const uint32_t a = smem_u32(tiles + s * STAGE), w = a + A_BYTES;
#pragma unroll
        for (int k = 0; k < BK / 16; ++k)
          mma<BNT>(tmem, smem_desc<64>(a + k * 32), smem_desc<64>(w + k * 32), (i | k) != 0);
        tc_commit(&bars.empty[s]);
      }
      tc_commit(&bars.accum);
    }
  } else {
    const bool ok = mbar_wait(&bars.accum, 0, ab, p.error, 723);
    float *ep = reinterpret_cast<float *>(tiles);     // [BM][kLds], in the idle ring
    const bool vec = vector_rows(p);
    const int quad = warp & 3, ew = warp - 2;
    const int rows = min(BM, rows_end - m0);
#pragma unroll 1
    for (int h = 0; h < BNT / 128; ++h) {
      const int n0h = n0 + h * 128;
      if (h > 0)
        asm volatile("bar.sync 1, %0;" ::"n"(kEpiWarps * 32) : "memory");
      if (ok && n0h < p.N && quad * 32 < rows) {
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        const int cb0 = (ew >> 2) * 64;
#pragma unroll 1
        for (int cb = cb0; cb < cb0 + 64; cb += 32) {
          uint32_t v[32];
          const uint32_t taddr = tmem + ((uint32_t)(quad * 32) << 16) + (uint32_t)(h * 128 + cb);
          asm volatile(
              "tcgen05.ld.sync.aligned.32x32b.x32.b32 "
              "{%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,"
              "%16,%17,%18,%19,%20,%21,%22,%23,%24,%25,%26,%27,%28,%29,%30,%31}, [%32];"
              : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
                "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15]),
                "=r"(v[16]), "=r"(v[17]), "=r"(v[18]), "=r"(v[19]), "=r"(v[20]), "=r"(v[21]), "=r"(v[22]), "=r"(v[23]),
                "=r"(v[24]), "=r"(v[25]), "=r"(v[26]), "=r"(v[27]), "=r"(v[28]), "=r"(v[29]), "=r"(v[30]), "=r"(v[31])
              : "r"(taddr)
              : "memory");
          asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
          float *erow = ep + (quad * 32 + lane) * kLds;
          if (p.pairs && p.splits == 1) {
#pragma unroll
            for (int j = 0; j < 32; j += 8)
              *reinterpret_cast<float4 *>(erow + ((cb + j) >> 1)) =
                  make_float4(gate_pair(p.gate, __uint_as_float(v[j]), __uint_as_float(v[j + 1])),
                              gate_pair(p.gate, __uint_as_float(v[j + 2]), __uint_as_float(v[j + 3])),
                              gate_pair(p.gate, __uint_as_float(v[j + 4]), __uint_as_float(v[j + 5])),
                              gate_pair(p.gate, __uint_as_float(v[j + 6]), __uint_as_float(v[j + 7])));
          } else {
#pragma unroll
            for (int j = 0; j < 32; j += 4)
              *reinterpret_cast<float4 *>(erow + cb + j) =
                  make_float4(__uint_as_float(v[j]), __uint_as_float(v[j + 1]), __uint_as_float(v[j + 2]), __uint_as_float(v[j + 3]));
          }
        }
      }
      asm volatile("bar.sync 1, %0;" ::"n"(kEpiWarps * 32) : "memory");
      if (ok && n0h < p.N) {
        if (p.splits > 1) {
          const int64_t tile = (int64_t)blockIdx.y * gridDim.x + blockIdx.x;
          float *dst = p.partial + (tile * p.splits + blockIdx.z) * BM * 128;
          for (int idx = ew * 32 + lane; idx < rows * 32; idx += kEpiWarps * 32)
            *reinterpret_cast<float4 *>(dst + (idx >> 5) * 128 + (idx & 31) * 4) =
                *reinterpret_cast<const float4 *>(ep + (idx >> 5) * kLds + (idx & 31) * 4);
        } else {
          const int per_row = p.pairs ? 16 : 32;           // groups of four columns
          const int cols = p.pairs ? min(128, p.N - n0h) >> 1 : min(128, p.N - n0h);
          const int64_t nc = p.pairs ? n0h >> 1 : n0h;
          for (int idx = ew * 32 + lane; idx < rows * per_row; idx += kEpiWarps * 32) {
            const int r = idx / per_row, c = (idx - r * per_row) * 4;
            if (c < cols)
              store4(p, m0 + r, nc + c, *reinterpret_cast<const float4 *>(ep + r * kLds + c), min(4, cols - c), vec);
          }
        }
      }
    }
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    if (*ab) {   // copies of an abandoned tile may still be in flight: let them land before the CTA ends
      const unsigned long long t0 = now_ns();
      while (now_ns() - t0 < 2000000ull) {
      }
    }
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(BNT) : "memory");
  }
}

// grid (tiles, 16): eight rows of a tile, four columns per thread; splits are added in order
__global__ void __launch_bounds__(256)
gemm_bf16_combine_kernel(const Params p, int tiles_x) {
  const int tile = blockIdx.x;
  const int r = blockIdx.y * 8 + (threadIdx.x >> 5), c = (threadIdx.x & 31) * 4;
  const int m = tile / tiles_x * BM + r, n = tile % tiles_x * 128 + c;
  if (m >= p.M || n >= p.N)
    return;
  const float *src = p.partial + (int64_t)tile * p.splits * BM * 128 + r * 128 + c;
  float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
  for (int z = 0; z < p.splits; ++z) {
    const float4 v = *reinterpret_cast<const float4 *>(src + (int64_t)z * BM * 128);
    a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
  }
  if (p.pairs) {
    const float4 g = make_float4(gate_pair(p.gate, a.x, a.y), gate_pair(p.gate, a.z, a.w), 0.f, 0.f);
    store4(p, m, n >> 1, g, n + 3 < p.N ? 2 : 1, false);
  } else {
    store4(p, m, n, a, min(4, p.N - n), vector_rows(p));
  }
}

template <int BNT> int launch(const CUtensorMap &ma, const CUtensorMap &mw, Params &p, int row_tiles, cudaStream_t st) {
  constexpr int STAGE = (BM + BNT) * BK * 2;
  p.stages = 96 * 1024 / STAGE;
  const int smem = p.stages * STAGE + 1024 + 256;
  static int configured[64] = {};
  int dev = 0;
  B200_CUDA(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || configured[dev] < smem) {
    B200_CUDA(cudaFuncSetAttribute(gemm_bf16_tc_kernel<BNT>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    if (dev >= 0 && dev < 64)
      configured[dev] = smem;
  }
  const dim3 grid((p.N + BNT - 1) / BNT, row_tiles, p.splits);
  gemm_bf16_tc_kernel<BNT><<<grid, kThreads, smem, st>>>(ma, mw, p);
  B200_LAUNCH_CHECK();
  if (p.splits > 1) {
    gemm_bf16_combine_kernel<<<dim3(grid.x * grid.y, BM / 8), 256, 0, st>>>(p, (int)grid.x);
    B200_LAUNCH_CHECK();
  }
  return B200_OK;
}

} // namespace

int64_t gemm_bf16_workspace_bytes() { return 256 + (int64_t)kMaxPartialTiles * BM * 128 * 4; }

int gemm_bf16_launch(const GemmBf16 &g, void *workspace, cudaStream_t st) {
  if (g.M < 1 || g.w.N < 1 || g.w.K < 1 || (g.pairs && (g.w.N & 1)) || (g.lda & 7) || (g.w.ld & 7) || (!g.C == !g.C16))
    return fail(B200_EINVAL, "gemm_bf16: bad argument (M %d, N %d, K %d)", g.M, g.w.N, g.w.K);
  if (((uintptr_t)g.A & 15) || ((uintptr_t)g.w.w & 15) || ((uintptr_t)workspace & 255))
    return fail(B200_EINVAL, "gemm_bf16: operands must be 16-byte aligned, the workspace 256-byte aligned");
  Params p{};
  p.M = g.M;
  p.N = g.tiles ? g.w.N / g.groups : g.w.N;
  p.K = g.w.K;
  p.C = g.C;
  p.C16 = g.C16;
  p.ldc = g.ldc;
  p.add = g.add ? 1 : 0;
  p.pairs = g.pairs ? 1 : 0;
  p.gate = g.gate;
  p.bias = g.bias;
  p.act = g.act;
  p.splits = 1;
  p.tiles = g.tiles;
  p.n_tiles = g.n_tiles;
  p.error = (int *)workspace;
  p.partial = (float *)((char *)workspace + 256);
  const int row_tiles = g.tiles ? g.max_tiles : (g.M + BM - 1) / BM;
  // 256 weight rows per CTA when that leaves enough CTAs; else 128, split over k when few
  const bool wide = p.N >= 256 && ((p.N + 255) / 256) * row_tiles >= 148;
  if (!wide && !g.tiles) {
    const int tiles = ((p.N + 127) / 128) * row_tiles, nkb = (p.K + BK - 1) / BK;
    if (tiles < 148) {
      int splits = 296 / tiles;
      splits = std::min(splits, nkb / 4);
      if (splits * tiles > kMaxPartialTiles)
        splits = kMaxPartialTiles / tiles;
      p.splits = std::max(1, splits);
    }
  }
  CUtensorMap ma, mw;
  if (int rc = make_map(&ma, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, BK, const_cast<bf16 *>(g.A), p.K, g.M, (uint64_t)g.lda * 2,
                        CU_TENSOR_MAP_SWIZZLE_128B, BM))
    return rc;
  if (int rc = make_map(&mw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, BK, g.w.w, p.K, g.w.N, (uint64_t)g.w.ld * 2,
                        CU_TENSOR_MAP_SWIZZLE_128B, wide ? 256 : 128))
    return rc;
  return wide ? launch<256>(ma, mw, p, row_tiles, st) : launch<128>(ma, mw, p, row_tiles, st);
}

} // namespace b200
