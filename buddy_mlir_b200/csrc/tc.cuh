// Building blocks of the tensor-core kernels: bounded mbarrier waits, TMA loads, shared-memory
// and tensor maps, tcgen05 commit.
#pragma once
#include "common.cuh"

#include <cuda.h>

#include <mutex>

namespace b200 {

constexpr uint32_t kSpin = 1u << 26;
constexpr unsigned long long kWaitNs = 2000000000ull;

__device__ __forceinline__ uint32_t smem_u32(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ unsigned long long now_ns() {
  unsigned long long t;
  asm volatile("mov.u64 %0, %%globaltimer;" : "=l"(t));
  return t;
}
__device__ __forceinline__ void mbar_init(uint64_t *bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t *bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t *bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_try(uint64_t *bar, uint32_t parity) {
  uint32_t ok;
  asm volatile("{\n .reg .pred p;\n mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n selp.u32 %0, 1, 0, p;\n}"
               : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
  return ok != 0;
}
// Bounded wait; false when it gave up or the CTA already failed.
__device__ __forceinline__ bool mbar_wait(uint64_t *bar, uint32_t parity, volatile int *ab, int *err, int code) {
  unsigned long long t0 = 0;
  for (uint32_t it = 0; it < kSpin; ++it) {
    if (mbar_try(bar, parity))
      return !*ab;
    if ((it & 0x3FF) == 0x3FF) {
      if (*ab)
        return false;
      const unsigned long long t = now_ns();
      if (t0 == 0)
        t0 = t;
      else if (t - t0 > kWaitNs)
        break;
    }
  }
  atomicCAS(err, 0, code);
  *ab = 1;
  return false;
}
__device__ __forceinline__ void tma_load_2d(void *dst, const CUtensorMap *map, int x, int y, uint64_t *bar) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(smem_u32(dst)), "l"(map), "r"(smem_u32(bar)), "r"(x), "r"(y)
      : "memory");
}
// K-major operand tile in shared memory, rows of 128 bytes (128-byte swizzle) or
// 64 bytes (64-byte swizzle): start address / 16, leading byte offset (unused for
// swizzled K-major: 1), stride byte offset = 8 rows, descriptor version 1,
// layout 2 (128-byte swizzle) or 4 (64-byte swizzle).
template <int BKT> __device__ __forceinline__ uint64_t smem_desc(uint32_t addr) {
  uint64_t d = 0;
  d |= (uint64_t)((addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)1 << 16;
  d |= (uint64_t)((8 * BKT * 2) >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)(BKT == 64 ? 2 : 4) << 61;
  return d;
}
__device__ __forceinline__ void tc_commit(uint64_t *bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar)) : "memory");
}

using EncodeFn = CUresult (*)(CUtensorMap *, CUtensorMapDataType, cuuint32_t, void *, const cuuint64_t *,
                              const cuuint64_t *, const cuuint32_t *, const cuuint32_t *, CUtensorMapInterleave,
                              CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);

inline EncodeFn encode_fn() {
  static EncodeFn fn = nullptr;
  static std::once_flag once;
  std::call_once(once, [] {
    void *p = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) == cudaSuccess &&
        q == cudaDriverEntryPointSuccess)
      fn = reinterpret_cast<EncodeFn>(p);
  });
  return fn;
}

inline int make_map(CUtensorMap *map, CUtensorMapDataType dt, int bk, void *base, uint64_t inner, uint64_t rows,
             uint64_t pitch_bytes, CUtensorMapSwizzle swz, int box_rows = 128) {
  EncodeFn fn = encode_fn();
  if (!fn)
    return fail(B200_ECUDA, "cuTensorMapEncodeTiled is not available from this driver");
  const cuuint64_t dims[2] = {inner, rows};
  const cuuint64_t strides[1] = {pitch_bytes};
  const cuuint32_t box[2] = {(cuuint32_t)bk, (cuuint32_t)box_rows};
  const cuuint32_t estr[2] = {1, 1};
  const CUresult rc = fn(map, dt, 2, base, dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, swz,
                         CU_TENSOR_MAP_L2_PROMOTION_L2_128B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  if (rc != CUDA_SUCCESS)
    return fail(B200_ECUDA, "cuTensorMapEncodeTiled failed (%d)", (int)rc);
  return B200_OK;
}

} // namespace b200
