// Shared device helpers for the sm_100a kernels: PTX wrappers for mbarrier, TMA
// (cp.async.bulk.tensor, never with a cluster qualifier on the load), tcgen05
// (alloc / mma / commit / ld), programmatic dependent launch, bounded waits and the
// device status word that every bounded wait reports into.
#pragma once

#include <cuda.h>
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_fp8.h>
#include <cuda_runtime.h>
#include <stdint.h>

#define PRISM_API extern "C" __attribute__((visibility("default")))

// ---- status word ----------------------------------------------------------------
// One int per device, written by kernels whose bounded waits ran out or whose
// debug bounds checks failed.  0 = healthy.  Host code reads it with
// prism_read_status(); nothing traps, so the CUDA context stays usable.
enum PrismStatus : int {
  PRISM_OK = 0,
  PRISM_ERR_MBAR_TIMEOUT = 1,
  PRISM_ERR_PEER_TIMEOUT = 2,
  PRISM_ERR_BOUNDS = 3,
};

// Each translation unit owns a private copy (no relocatable device code is used);
// PRISM_DEFINE_TU_STATUS(name) exports prism_status_<name>(out4, reset) to read it.
static __device__ int g_prism_status[4];  // [0]=code, [1]=detail, [2]=block, [3]=count

#define PRISM_DEFINE_TU_STATUS(name)                                                        \
  PRISM_API int prism_status_##name(int* out4, int reset) {                                 \
    cudaError_t e = cudaMemcpyFromSymbol(out4, g_prism_status, 4 * sizeof(int));            \
    if (e != cudaSuccess) return (int)e;                                                    \
    if (reset) {                                                                            \
      int z[4] = {0, 0, 0, 0};                                                              \
      e = cudaMemcpyToSymbol(g_prism_status, z, 4 * sizeof(int));                           \
    }                                                                                       \
    return (int)e;                                                                          \
  }

__device__ __forceinline__ void prism_report(int code, int detail) {
  if (atomicCAS(&g_prism_status[0], 0, code) == 0) {
    g_prism_status[1] = detail;
    g_prism_status[2] = (int)blockIdx.x;
  }
  atomicAdd(&g_prism_status[3], 1);
}

// ---- small numeric helpers --------------------------------------------------------
__device__ __forceinline__ float bf16_round(float x) {
  return __bfloat162float(__float2bfloat16_rn(x));
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}
// tanh.approx.f32 is one MUFU instruction with about 2^-11 relative error, far below the
// bf16 rounding of the result; the library tanhf costs tens of instructions per element,
// which made the GELU epilogue of the vision MLP longer than its main loop.
__device__ __forceinline__ float tanh_fast(float x) {
  float y;
  asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float gelu_tanh(float x) {
  const float k0 = 0.7978845608028654f, k1 = 0.044715f;
  return 0.5f * x * (1.0f + tanh_fast(k0 * (x + k1 * x * x * x)));
}
__device__ __forceinline__ float gelu_erf(float x) {
  return 0.5f * x * (1.0f + erff(x * 0.7071067811865476f));
}
__device__ __forceinline__ float silu(float x) { return x / (1.0f + __expf(-x)); }
// Gated linear units of the two-matrix GEMM epilogues.  SILU_ROUNDED keeps the rounding points of an eager bf16 graph;
// the others stay in 32-bit until the product is stored.
// BOUNDED: with g at most `limit` and u within it, g sigmoid(1.702 g) (u + 1).
enum PrismGlu : int { PRISM_GLU_SILU_ROUNDED = 0, PRISM_GLU_SILU = 1, PRISM_GLU_GELU_TANH = 2, PRISM_GLU_BOUNDED = 3 };
constexpr float PRISM_GLU_SLOPE = 1.702f;
__device__ __forceinline__ float glu(float g, float u, int act, float limit = 0.0f) {
  if (act == PRISM_GLU_BOUNDED) {
    g = fminf(g, limit);
    return g / (1.0f + __expf(-PRISM_GLU_SLOPE * g)) * (fminf(fmaxf(u, -limit), limit) + 1.0f);
  }
  if (act == PRISM_GLU_SILU_ROUNDED) return bf16_round(silu(bf16_round(g))) * bf16_round(u);
  return (act == PRISM_GLU_GELU_TANH ? gelu_tanh(g) : silu(g)) * u;
}

// Decay of a recurrence from the logarithm of its rate, in 32-bit.
__device__ __forceinline__ float decay_of(float x) { return expf(-expf(x)); }
__device__ __forceinline__ float sigmoid_fast(float x) { return 1.0f / (1.0f + __expf(-x)); }

// ---- packed pairs of floats: two fused multiply-adds per instruction -----------------
__device__ __forceinline__ unsigned long long pair_of(float lo, float hi) {
  unsigned long long d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float2 unpair(unsigned long long v) {
  float2 f;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(f.x), "=f"(f.y) : "l"(v));
  return f;
}
__device__ __forceinline__ unsigned long long fma2(unsigned long long a, unsigned long long b, unsigned long long c) {
  unsigned long long d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ unsigned long long mul2(unsigned long long a, unsigned long long b) {
  unsigned long long d;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

// ---- row sections of a stacked projection -------------------------------------------
// One GEMM over several weight matrices stacked by rows: rows [row_end[i - 1], row_end[i]) are
// scaled by alpha[i] (then the bias is added) and pass through activation act[i].
enum PrismAct : int { PRISM_ACT_NONE = 0, PRISM_ACT_GELU_TANH = 1, PRISM_ACT_GELU_ERF = 2, PRISM_ACT_SIGMOID = 3, PRISM_ACT_SOFTCAP = 4,
                      PRISM_ACT_DECAY = 5 };
constexpr int PRISM_MAX_SECTIONS = 8;
struct PrismSections {
  int n;      // 0: no sections
  float cap;  // bound of the PRISM_ACT_SOFTCAP sections: cap * tanh(v / cap)
  int row_end[PRISM_MAX_SECTIONS];
  int act[PRISM_MAX_SECTIONS];
  float alpha[PRISM_MAX_SECTIONS];
};
// Section of row m (rows past the last end belong to the last section).
__device__ __forceinline__ void prism_section_of(const PrismSections& s, int m, float& alpha, int& act) {
  alpha = s.alpha[0];
  act = s.act[0];
#pragma unroll
  for (int i = 1; i < PRISM_MAX_SECTIONS; ++i)
    if (i < s.n && m >= s.row_end[i - 1]) {
      alpha = s.alpha[i];
      act = s.act[i];
    }
}
// Copies host arrays into the kernel argument; false when they are not a valid partition of M rows.
static inline bool prism_fill_sections(PrismSections& s, int n, const int* row_end, const float* alpha, const int* act, float cap,
                                       int M) {
  if (n < 1 || n > PRISM_MAX_SECTIONS) return false;
  s.n = n;
  s.cap = cap;
  for (int i = 0; i < PRISM_MAX_SECTIONS; ++i) {
    s.row_end[i] = i < n ? row_end[i] : M;
    s.alpha[i] = i < n ? alpha[i] : 1.0f;
    s.act[i] = i < n ? act[i] : 0;
    if (i < n && ((i > 0 && row_end[i] <= row_end[i - 1]) || act[i] < 0 || act[i] > PRISM_ACT_DECAY)) return false;
    if (i < n && act[i] == PRISM_ACT_SOFTCAP && !(cap > 0.0f)) return false;
  }
  return row_end[n - 1] == M;
}

// ---- programmatic dependent launch -------------------------------------------------
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
__device__ __forceinline__ void pdl_launch_dependents() {
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
}

// ---- shared memory address / mbarrier -----------------------------------------------
__device__ __forceinline__ uint32_t smem_u32(const void* p) {
  return static_cast<uint32_t>(__cvta_generic_to_shared(p));
}
__device__ __forceinline__ void mbar_init(uint64_t* bar, uint32_t count) {
  asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(smem_u32(bar)), "r"(count));
}
__device__ __forceinline__ void mbar_expect_tx(uint64_t* bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(smem_u32(bar)), "r"(bytes)
               : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint64_t* bar) {
  asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ bool mbar_try_wait(uint64_t* bar, uint32_t parity) {
  uint32_t ok;
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(ok)
      : "r"(smem_u32(bar)), "r"(parity)
      : "memory");
  return ok != 0;
}
// Bounded wait: returns false (and records PRISM_ERR_MBAR_TIMEOUT) when the phase does
// not complete within PRISM_WAIT_CYCLES SM clock cycles (about two seconds), far beyond
// any legitimate wait.  The caller then unwinds: no trap, the context stays usable.
#ifndef PRISM_WAIT_CYCLES
#define PRISM_WAIT_CYCLES (4000000000ll)
#endif
__device__ __forceinline__ bool mbar_wait(uint64_t* bar, uint32_t parity, int tag) {
  if (mbar_try_wait(bar, parity)) return true;
  const long long t0 = clock64();
  for (;;) {
#pragma unroll 1
    for (int i = 0; i < 128; ++i) {
      if (mbar_try_wait(bar, parity)) return true;
    }
    if (clock64() - t0 > PRISM_WAIT_CYCLES) break;
  }
  prism_report(PRISM_ERR_MBAR_TIMEOUT, tag);
  return false;
}
__device__ __forceinline__ void fence_barrier_init() {
  asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
}
__device__ __forceinline__ void fence_proxy_async() {
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
}

// ---- TMA (tiled bulk tensor copies; no cluster qualifier on loads) -------------------
__device__ __forceinline__ void tma_prefetch_desc(const CUtensorMap* m) {
  asm volatile("prefetch.tensormap [%0];" ::"l"(reinterpret_cast<uint64_t>(m)) : "memory");
}
// x (innermost coordinate) times the element size must be a multiple of 16 bytes.
__device__ __forceinline__ void tma_load_2d(void* smem_dst, const CUtensorMap* m, uint64_t* bar, int x, int y) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y)
      : "memory");
}
__device__ __forceinline__ void tma_load_3d(void* smem_dst, const CUtensorMap* m, uint64_t* bar, int x, int y, int z) {
  asm volatile(
      "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z)
      : "memory");
}
__device__ __forceinline__ void tma_load_2d_hint(void* smem_dst, const CUtensorMap* m, uint64_t* bar, int x, int y,
                                                 uint64_t policy) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.mbarrier::complete_tx::bytes.L2::cache_hint"
      " [%0], [%1, {%3, %4}], [%2], %5;"
      ::"r"(smem_u32(smem_dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(y), "l"(policy)
      : "memory");
}
__device__ __forceinline__ uint64_t l2_policy_evict_first() {
  uint64_t p;
  asm volatile("createpolicy.fractional.L2::evict_first.b64 %0, 1.0;" : "=l"(p));
  return p;
}
__device__ __forceinline__ uint64_t l2_policy_evict_last() {
  uint64_t p;
  asm volatile("createpolicy.fractional.L2::evict_last.b64 %0, 1.0;" : "=l"(p));
  return p;
}

// ---- tcgen05 / TMEM -------------------------------------------------------------------
__device__ __forceinline__ void tmem_alloc(uint32_t* smem_slot, uint32_t cols) {
  asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(smem_slot)),
               "r"(cols)
               : "memory");
}
__device__ __forceinline__ void tmem_relinquish() {
  asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
}
__device__ __forceinline__ void tmem_dealloc(uint32_t taddr, uint32_t cols) {
  asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(taddr), "r"(cols) : "memory");
}
__device__ __forceinline__ void tc_fence_before() { asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory"); }
__device__ __forceinline__ void tc_fence_after() { asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory"); }
// Arrives on the mbarrier once every previously issued tcgen05.mma of this thread is done.
__device__ __forceinline__ void tc_commit(uint64_t* bar) {
  asm volatile("tcgen05.commit.cta_group::1.mbarrier::arrive::one.shared::cluster.b64 [%0];" ::"r"(smem_u32(bar))
               : "memory");
}
// D[tmem] (+)= A[smem desc] * B[smem desc], bf16/f16 inputs, fp32 accumulate.
__device__ __forceinline__ void tc_mma_f16(uint32_t d_tmem, uint64_t a_desc, uint64_t b_desc, uint32_t idesc,
                                           uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
      ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}
// 32 lanes x 16 consecutive 32-bit columns: thread t of the warp receives lane
// (taddr.lane + t), columns taddr.col .. +15.
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 "
      "{%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
}
__device__ __forceinline__ void tmem_ld_wait() { asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory"); }
// One column: thread t of the warp receives lane (taddr.lane + t).
__device__ __forceinline__ void tmem_ld1(uint32_t taddr, uint32_t& r) {
  asm volatile("tcgen05.ld.sync.aligned.32x32b.x1.b32 {%0}, [%1];" : "=r"(r) : "r"(taddr) : "memory");
}
// Store counterpart: thread t writes lane (taddr.lane + t), columns taddr.col .. +15.
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]),
        "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
// D[tmem] (+)= A[tmem] * B[smem desc]: the A operand (M lanes x K 16-bit elements, two per
// 32-bit column) is read from tensor memory.
__device__ __forceinline__ void tc_mma_f16_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc,
                                              uint32_t accumulate) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(accumulate)
      : "memory");
}

// Shared-memory matrix descriptor for a K-major bf16 tile whose rows are 128 bytes
// (64 elements) and stored with the 128-byte swizzle TMA produces: 8-row groups are
// 1024 bytes apart (stride byte offset), version 1 (Blackwell), layout type 2.
__device__ __forceinline__ uint64_t umma_desc_sw128(uint32_t smem_addr) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)1 << 16;            // leading byte offset (unused for swizzled K-major)
  d |= (uint64_t)(1024 >> 4) << 32;  // stride byte offset
  d |= (uint64_t)1 << 46;            // descriptor version
  d |= (uint64_t)2 << 61;            // SWIZZLE_128B
  return d;
}
// MN-major bf16 tile with the 128-byte swizzle: rows are 64 elements along M/N (128 bytes), one
// row per K index; 8-row groups along K are 1024 bytes apart (stride byte offset) and the next
// 64 elements along M/N start lbo_bytes further on (leading byte offset).
__device__ __forceinline__ uint64_t umma_desc_sw128_mn(uint32_t smem_addr, uint32_t lbo_bytes) {
  uint64_t d = 0;
  d |= (uint64_t)((smem_addr & 0x3FFFFu) >> 4);
  d |= (uint64_t)((lbo_bytes >> 4) & 0x3FFFu) << 16;
  d |= (uint64_t)(1024 >> 4) << 32;
  d |= (uint64_t)1 << 46;
  d |= (uint64_t)2 << 61;
  return d;
}
constexpr uint32_t UMMA_B_MN_MAJOR = 1u << 16;  // instruction-descriptor bit: B operand is MN-major
// Instruction descriptor: bf16 x bf16 -> fp32, both operands K-major, M x N tile.
__host__ __device__ constexpr uint32_t umma_idesc_bf16(int m, int n) {
  return (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(m >> 4) << 24);
}

// ---- host-side declarations shared between translation units -------------------------
// Cached CUtensorMap of a [rows, cols] bf16 row-major matrix with row stride ld (elements) and a
// box of box_rows x 64 elements, 128-byte swizzle (defined in gemm_tcgen05.cu).
int prism_get_tensor_map(const void* ptr, unsigned long long rows, unsigned long long cols, unsigned long long ld,
                         unsigned box_rows, CUtensorMap* out);
// [tokens][heads][head_dim] view, box = box_rows tokens x 1 head x 64 columns (columns past
// head_dim read as zeros); see gemm_tcgen05.cu.
int prism_make_head_tensor_map(const void* ptr, unsigned long long tokens, unsigned heads, unsigned head_dim,
                               unsigned long long ld, unsigned box_rows, CUtensorMap* out);
struct PrismLaunch {
  cudaStream_t stream;
  int pdl;  // 1: launch with programmatic stream serialization
};

template <typename... KArgs, typename... Args>
static inline cudaError_t prism_launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                       bool pdl, Args&&... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, static_cast<KArgs>(args)...);
}
