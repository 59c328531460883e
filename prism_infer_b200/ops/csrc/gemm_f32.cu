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
  // Grouped form: tile blockIdx.y is groups[y] = (expert, first row, rows, -); expert e's weights start at row e * M.
  const int4* groups;
  const int* n_groups;
  const int* row_token;  // x row of every output row (null: the output row itself)
};

__device__ __forceinline__ float act_f32(float v, int act, float cap) {
  switch (act) {
    case PRISM_ACT_GELU_TANH: return 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v)));
    case PRISM_ACT_GELU_ERF: return gelu_erf(v);
    case PRISM_ACT_SIGMOID: return 1.0f / (1.0f + expf(-v));
    case PRISM_ACT_SOFTCAP: return cap * tanhf(v / cap);
    case PRISM_ACT_DECAY: return decay_of(v);
    default: return v;
  }
}

__global__ void __launch_bounds__(256) gemm_f32_kernel(const F32Args a) {
  __shared__ float ws[TK][TM + 4];
  __shared__ float xs[TK][TN + 4];
  const int m0 = blockIdx.x * TM;
  int t0 = blockIdx.y * TN, t_end = a.T;
  const float* w_base = a.w;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  pdl_launch_dependents();
  pdl_wait();
  if (a.groups != nullptr) {
    if ((int)blockIdx.y >= *a.n_groups) return;
    const int4 g = a.groups[blockIdx.y];
    t0 = g.y;
    t_end = min(a.T, g.y + g.z);
    w_base += (size_t)g.x * a.M * a.ldw;
  }
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += TK) {
    for (int i = threadIdx.x; i < TM * TK; i += 256) {
      const int r = i / TK, k = i % TK;
      ws[k][r] = (m0 + r < a.M && k0 + k < a.K) ? w_base[(size_t)(m0 + r) * a.ldw + k0 + k] : 0.0f;
      float x = 0.0f;
      if (t0 + r < t_end && k0 + k < a.K) x = a.x[(size_t)(a.row_token ? a.row_token[t0 + r] : t0 + r) * a.ldx + k0 + k];
      xs[k][r] = x;
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
      if (t < t_end) a.out[(size_t)t * a.ldo + m] = act_f32(acc[i][j] * alpha + b, act, a.sec.cap);
    }
  }
}

// out[n][i] = the gated unit of gu[n][i] and gu[n][F + i]
__global__ void __launch_bounds__(256) glu_f32_kernel(const float* gu, float* out, long long total, int F, int act, float limit) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const long long n = i / F;
  float z = gu[n * 2 * F + (i - n * F)], u = gu[n * 2 * F + F + (i - n * F)];
  if (act == PRISM_GLU_BOUNDED) {
    z = fminf(z, limit);
    u = fminf(fmaxf(u, -limit), limit) + 1.0f;
    z /= 1.0f + expf(-PRISM_GLU_SLOPE * z);
  } else {
    z = act == PRISM_GLU_GELU_TANH ? act_f32(z, PRISM_ACT_GELU_TANH, 0.0f) : z / (1.0f + expf(-z));
  }
  out[i] = z * u;
}

}  // namespace

// act: 1 silu, 2 gelu (tanh form), 3 bounded by `limit`
PRISM_API int prism_glu_f32(const void* gu, void* out, int N, int F, int act, float limit, void* stream, int pdl) {
  if (N <= 0) return 0;
  if (F <= 0 || act < PRISM_GLU_SILU || act > PRISM_GLU_BOUNDED) return -1;
  const long long total = (long long)N * F;
  return (int)prism_launch(glu_f32_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
                           pdl != 0, (const float*)gu, (float*)out, total, F, act, limit);
}

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
  a.groups = nullptr;
  a.n_groups = a.row_token = nullptr;
  const dim3 grid((M + TM - 1) / TM, (T + TN - 1) / TN);
  return (int)prism_launch(gemm_f32_kernel, grid, dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

// Experts' projections: output rows [first, first + rows) of groups[i] = (expert, first, rows, -) (at most 64 rows each) are
// W_expert x, W [experts * M][ldw], x row row_token[n] (null: n).  N output rows, X_rows rows of x.
PRISM_API int prism_gemm_f32_grouped(const void* W, const void* X, void* out, int M, int N, int K, long long ldw, long long ldx,
                                     long long ldo, const void* groups, int max_groups, const void* n_groups, const void* row_token,
                                     int X_rows, int experts, void* stream, int pdl) {
  if (M <= 0 || N <= 0 || K <= 0 || max_groups <= 0 || X_rows <= 0 || experts <= 0 || !groups || !n_groups) return -1;
  if (row_token == nullptr && X_rows < N) return -2;
  F32Args a;
  a.sec.n = 0;
  a.sec.cap = 0.0f;
  a.w = (const float*)W;
  a.x = (const float*)X;
  a.out = (float*)out;
  a.bias = nullptr;
  a.M = M;
  a.T = N;
  a.K = K;
  a.ldw = ldw;
  a.ldx = ldx;
  a.ldo = ldo;
  a.groups = (const int4*)groups;
  a.n_groups = (const int*)n_groups;
  a.row_token = (const int*)row_token;
  return (int)prism_launch(gemm_f32_kernel, dim3((M + TM - 1) / TM, max_groups), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
                           pdl != 0, a);
}
