// Warp-level building blocks of the attention kernels that read the paged cache directly: ldmatrix, mma.sync
// m16n8k16 (bf16 in, fp32 out), 16-byte cp.async, and the page-table guards.
#pragma once

#include "common.cuh"

__device__ __forceinline__ void ldsm_x4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
  __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<uint32_t*>(&v);
}

__device__ __forceinline__ float ex2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void cp_async16(void* smem_dst, const void* gmem_src, bool valid) {
  // src-size 0 zero-fills the 16 bytes without touching global memory
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(smem_dst)), "l"(gmem_src), "r"(valid ? 16 : 0)
               : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_async_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// Page-table guards shared by the decode and prefill kernels.  A context longer than the
// table can describe is cut to the table's reach, and a page id at or beyond the cache is
// treated as a hole; both are recorded in the status word (PRISM_ERR_BOUNDS) and the access
// is skipped, so a stale table or an over-long length costs wrong tokens that the engine
// reports, never an out-of-range read.
__device__ __forceinline__ int clamp_context(int ctx, int max_blocks, int page) {
  const long long reach = (long long)max_blocks * page;
  if ((long long)ctx > reach) {
    if (threadIdx.x == 0) prism_report(PRISM_ERR_BOUNDS, 1);
    return (int)reach;
  }
  return ctx < 0 ? 0 : ctx;
}
__device__ __forceinline__ int checked_page(int blk, int num_blocks) {
  if (num_blocks > 0 && blk >= num_blocks) {
    prism_report(PRISM_ERR_BOUNDS, 2);
    return -1;
  }
  return blk;
}
