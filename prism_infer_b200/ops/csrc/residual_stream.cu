// The 32-bit residual stream of models whose sublayers are gated and added in one step.
//
// One kernel (one CTA per token row) covers every place where the stream changes:
//   start     x = table[id]                                     (embedding)
//   pass      x = sum of the loop projection's slabs + step     (input of a looped section)
//   layer     x += mult * (gate_a * a + gate_b * b)             (two parallel sublayers, either may be absent)
// and what the next operation reads of it: the RMS-normalised row (gains are scalars that the next
// GEMM's epilogue applies), or the row itself (the loop projection's input, with the embedding beside it).
// a and b come as fp32 split-K slabs, summed here in a fixed order, or as rows of the compute type.
#include "common.cuh"

PRISM_DEFINE_TU_STATUS(stream)

namespace {

typedef __nv_bfloat16 bf16;

struct F4 {
  float v[4];
};
__device__ __forceinline__ F4 load4(const float* p) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  return F4{{f.x, f.y, f.z, f.w}};
}
__device__ __forceinline__ F4 load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return F4{{a.x, a.y, b.x, b.y}};
}
__device__ __forceinline__ void store4(float* p, const F4& f) {
  *reinterpret_cast<float4*>(p) = make_float4(f.v[0], f.v[1], f.v[2], f.v[3]);
}
__device__ __forceinline__ void store4(bf16* p, const F4& f) {
  uint2 o;
  *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(f.v[0], f.v[1]);
  *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(f.v[2], f.v[3]);
  *reinterpret_cast<uint2*>(p) = o;
}

template <typename T>
struct Branch {
  const float* slabs;      // [P][T][W] fp32 (null: none)
  long long slab_stride;
  int P;
  const T* rows;           // [T][ld] (null: none)
  long long ld;
  const T* gate;           // [T][gate_ld] (null: one)
  long long gate_ld;
};

template <typename T>
struct StreamArgs {
  float* x;                // [T][W] the stream
  int keep;                // 1: add to it, 0: replace it
  const long long* ids;    // embedding lookup (null: none)
  const T* table;          // [vocab][W]
  long long vocab;
  Branch<T> a, b;
  float mult;
  const T* bias;           // [W] (null: none)
  T* norm_out;             // rows x / sqrt(mean(x^2) + eps) (null: not wanted)
  long long norm_ld;
  T* raw_out;              // rows x in the compute type
  long long raw_ld;
  T* embed_out;            // the embedding rows
  long long embed_ld;
  int W, W_real;           // padded and real width: the padding columns are zero and do not enter the mean
  float eps;
};

template <typename T>
__device__ __forceinline__ void add_branch(const Branch<T>& br, size_t t, int W, int i, float mult, F4& acc) {
  if (br.slabs == nullptr && br.rows == nullptr) return;
  F4 d;
  if (br.slabs != nullptr) {
    d = F4{{0.0f, 0.0f, 0.0f, 0.0f}};
    const float* p0 = br.slabs + t * W + i;
#pragma unroll 8
    for (int p = 0; p < br.P; ++p) {
      const float4 v = __ldcg(reinterpret_cast<const float4*>(p0 + (size_t)p * br.slab_stride));
      d.v[0] += v.x;
      d.v[1] += v.y;
      d.v[2] += v.z;
      d.v[3] += v.w;
    }
  } else {
    d = load4(br.rows + t * br.ld + i);
  }
  if (br.gate != nullptr) {
    const F4 g = load4(br.gate + t * br.gate_ld + i);
#pragma unroll
    for (int e = 0; e < 4; ++e) d.v[e] *= g.v[e];
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) acc.v[e] += mult * d.v[e];
}

template <typename T>
__global__ void __launch_bounds__(1024) stream_update_kernel(const StreamArgs<T> a) {
  extern __shared__ float row[];  // W floats
  __shared__ float red[32];
  const size_t t = blockIdx.x;
  pdl_launch_dependents();
  pdl_wait();
  const T* emb = nullptr;
  if (a.ids != nullptr) {
    const long long id = a.ids[t];
    if (id >= 0 && id < a.vocab) emb = a.table + (size_t)id * a.W;
    else if (threadIdx.x == 0) prism_report(PRISM_ERR_BOUNDS, 1);
  }
  float ss = 0.0f;
  for (int i = threadIdx.x * 4; i < a.W; i += blockDim.x * 4) {
    F4 acc{{0.0f, 0.0f, 0.0f, 0.0f}};
    add_branch(a.a, t, a.W, i, a.mult, acc);
    add_branch(a.b, t, a.W, i, a.mult, acc);
    if (a.keep) {
      const F4 x = load4(a.x + t * a.W + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc.v[e] += x.v[e];
    }
    if (a.bias != nullptr) {
      const F4 s = load4(a.bias + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc.v[e] += s.v[e];
    }
    if (emb != nullptr) {
      const F4 v = load4(emb + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc.v[e] += v.v[e];
      if (a.embed_out != nullptr) store4(a.embed_out + t * a.embed_ld + i, v);
    } else if (a.embed_out != nullptr) {
      store4(a.embed_out + t * a.embed_ld + i, F4{{0.0f, 0.0f, 0.0f, 0.0f}});
    }
    store4(a.x + t * a.W + i, acc);
    if (a.raw_out != nullptr) store4(a.raw_out + t * a.raw_ld + i, acc);
    store4(row + i, acc);
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += acc.v[e] * acc.v[e];
  }
  if (a.norm_out == nullptr) return;
  ss = warp_sum(ss);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = warp_sum(lane < nw ? red[lane] : 0.0f);
  const float inv = 1.0f / sqrtf(ss / (float)a.W_real + a.eps);
  for (int i = threadIdx.x * 4; i < a.W; i += blockDim.x * 4) {
    F4 v = load4(row + i);
#pragma unroll
    for (int e = 0; e < 4; ++e) v.v[e] *= inv;
    store4(a.norm_out + t * a.norm_ld + i, v);
  }
}

template <typename T>
int launch_stream(int T_rows, void* x, int keep, const void* ids, const void* table, long long vocab, const void* a_slabs,
                  long long a_stride, int a_P, const void* a_rows, long long a_ld, const void* a_gate, const void* b_slabs,
                  long long b_stride, int b_P, const void* b_rows, long long b_ld, const void* b_gate, long long gate_ld,
                  float mult, const void* bias, void* norm_out, long long norm_ld, void* raw_out, long long raw_ld,
                  void* embed_out, long long embed_ld, int W, int W_real, float eps, cudaStream_t stream, bool pdl) {
  StreamArgs<T> a;
  a.x = (float*)x;
  a.keep = keep;
  a.ids = (const long long*)ids;
  a.table = (const T*)table;
  a.vocab = vocab;
  a.a = Branch<T>{(const float*)a_slabs, a_stride, a_P, (const T*)a_rows, a_ld, (const T*)a_gate, gate_ld};
  a.b = Branch<T>{(const float*)b_slabs, b_stride, b_P, (const T*)b_rows, b_ld, (const T*)b_gate, gate_ld};
  a.mult = mult;
  a.bias = (const T*)bias;
  a.norm_out = (T*)norm_out;
  a.norm_ld = norm_ld;
  a.raw_out = (T*)raw_out;
  a.raw_ld = raw_ld;
  a.embed_out = (T*)embed_out;
  a.embed_ld = embed_ld;
  a.W = W;
  a.W_real = W_real;
  a.eps = eps;
  int threads = (W / 4 + 31) / 32 * 32;
  if (threads > 1024) threads = 1024;
  const size_t smem = (size_t)W * sizeof(float);
  if (smem > 48 * 1024) {
    cudaError_t e = cudaFuncSetAttribute(stream_update_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
  }
  return (int)prism_launch(stream_update_kernel<T>, dim3(T_rows), dim3(threads), smem, stream, pdl, a);
}

}  // namespace

// f32: 1 = table, rows, gates, bias and outputs are fp32, 0 = bf16.  W a multiple of 8; every row stride a
// multiple of 4 elements.
PRISM_API int prism_stream_update(int f32, int T, void* x, int keep, const void* ids, const void* table, long long vocab,
                                  const void* a_slabs, long long a_stride, int a_P, const void* a_rows, long long a_ld,
                                  const void* a_gate, const void* b_slabs, long long b_stride, int b_P, const void* b_rows,
                                  long long b_ld, const void* b_gate, long long gate_ld, float mult, const void* bias,
                                  void* norm_out, long long norm_ld, void* raw_out, long long raw_ld, void* embed_out,
                                  long long embed_ld, int W, int W_real, float eps, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (W <= 0 || W % 8 || W_real <= 0 || W_real > W || W > 32768) return -1;
  if ((a_ld | b_ld | gate_ld | norm_ld | raw_ld | embed_ld) % 4) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_stream<float>(T, x, keep, ids, table, vocab, a_slabs, a_stride, a_P, a_rows, a_ld, a_gate, b_slabs, b_stride,
                                    b_P, b_rows, b_ld, b_gate, gate_ld, mult, bias, norm_out, norm_ld, raw_out, raw_ld, embed_out,
                                    embed_ld, W, W_real, eps, s, pdl != 0)
             : launch_stream<bf16>(T, x, keep, ids, table, vocab, a_slabs, a_stride, a_P, a_rows, a_ld, a_gate, b_slabs, b_stride,
                                   b_P, b_rows, b_ld, b_gate, gate_ld, mult, bias, norm_out, norm_ld, raw_out, raw_ld, embed_out,
                                   embed_ld, W, W_real, eps, s, pdl != 0);
}
