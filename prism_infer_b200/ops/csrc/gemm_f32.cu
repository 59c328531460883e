// True 32-bit projections (fp32 operands, fp32 fused multiply-adds, no reduced-precision mode): the arithmetic of
// an engine built with dtype "float32".  One 64 x 64 output tile per CTA, 4 x 4 outputs per thread, operands staged
// through shared memory 16 columns at a time.  out[t][m] = act_i(alpha_i * (W x_t)[m] + bias[m]), sections as in the
// tcgen05 GEMM.
#include "common.cuh"

PRISM_DEFINE_TU_STATUS(gemm_f32)

namespace {

constexpr int TM = 64, TN = 64, TK = 16;

struct F32Args {
  const float* w;   // [M][ldw]
  const float* x;   // [T][ldx]
  float* out;       // [T][ldo]
  const float* bias;
  int M, T, K;
  long long ldw, ldx, ldo;
  PrismSections sec;
};

__device__ __forceinline__ float act_f32(float v, int act, float cap) {
  switch (act) {
    case PRISM_ACT_GELU_TANH: return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    case PRISM_ACT_GELU_ERF: return gelu_erf(v);
    case PRISM_ACT_SIGMOID: return 1.0f / (1.0f + expf(-v));
    case PRISM_ACT_SOFTCAP: return cap * tanhf(v / cap);
    default: return v;
  }
}

__global__ void __launch_bounds__(256) gemm_f32_kernel(const F32Args a) {
  __shared__ float ws[TK][TM + 4];
  __shared__ float xs[TK][TN + 4];
  const int m0 = blockIdx.x * TM, t0 = blockIdx.y * TN;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  pdl_launch_dependents();
  pdl_wait();
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += TK) {
    for (int i = threadIdx.x; i < TM * TK; i += 256) {
      const int r = i / TK, k = i % TK;
      ws[k][r] = (m0 + r < a.M && k0 + k < a.K) ? a.w[(size_t)(m0 + r) * a.ldw + k0 + k] : 0.0f;
      xs[k][r] = (t0 + r < a.T && k0 + k < a.K) ? a.x[(size_t)(t0 + r) * a.ldx + k0 + k] : 0.0f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < TK; ++k) {
      float w[4], x[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        w[i] = ws[k][tx + 16 * i];
        x[i] = xs[k][ty + 16 * i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], w[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const int m = m0 + tx + 16 * j;
    if (m >= a.M) continue;
    float alpha = 1.0f;
    int act = 0;
    if (a.sec.n > 0) prism_section_of(a.sec, m, alpha, act);
    const float b = a.bias != nullptr ? a.bias[m] : 0.0f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = t0 + ty + 16 * i;
      if (t < a.T) a.out[(size_t)t * a.ldo + m] = act_f32(acc[i][j] * alpha + b, act, a.sec.cap);
    }
  }
}

}  // namespace

PRISM_API int prism_gemm_f32(const void* W, const void* X, void* out, int M, int T, int K, long long ldw, long long ldx,
                             long long ldo, const void* bias, int n_sections, const void* row_end, const void* alpha,
                             const void* act, float cap, void* stream, int pdl) {
  if (M <= 0 || T <= 0 || K <= 0) return -1;
  F32Args a;
  a.sec.n = 0;
  a.sec.cap = cap;
  if (n_sections > 0 && !prism_fill_sections(a.sec, n_sections, (const int*)row_end, (const float*)alpha, (const int*)act, cap, M))
    return -9;
  a.w = (const float*)W;
  a.x = (const float*)X;
  a.out = (float*)out;
  a.bias = (const float*)bias;
  a.M = M;
  a.T = T;
  a.K = K;
  a.ldw = ldw;
  a.ldx = ldx;
  a.ldo = ldo;
  const dim3 grid((M + TM - 1) / TM, (T + TN - 1) / TN);
  return (int)prism_launch(gemm_f32_kernel, grid, dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}
