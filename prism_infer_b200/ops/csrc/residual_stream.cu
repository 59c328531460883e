// The 32-bit residual stream of models whose sublayers are gated and added in one step.
//
// One kernel (one CTA per token row) covers every place where the stream changes:
//   start     x = table[id]                                     (embedding)
//   pass      x = sum of the loop projection's slabs + step     (input of a looped section)
//   layer     x += mult * (gate_a * a + gate_b * b)             (two parallel sublayers, either may be absent)
//   layer     x += norm(a) * w                                  (a norm behind the sublayer)
//   average   x = sum of weighted earlier results and this one  (depth average behind a layer)
// and what the next operation reads of it: the RMS-normalised row (with a weight, or with a scalar gain that the
// next GEMM's epilogue applies), or the row itself (the loop projection's input, with the embedding beside it).
// a and b come as fp32 split-K slabs, summed here in a fixed order, or as rows of the compute type; a may also be
// the weighted sum of several (token, expert) rows, and of the stream's own row.  In a decode step the normalised row may also
// pass through the causal convolution in front of the next mixer, whose earlier rows are in the sequence's state slot.
#include "common.cuh"

#include <type_traits>

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
  const int* pos;          // [T][K]: rows of slabs / rows whose weighted sum is the value (null: row t itself)
  const float* weight;     // [T][K]
  int K;
  const T* post_w;         // weight of the norm behind the sublayer (null: none)
  const float* self_w;     // [T]: weight of the stream's row in the sum (null: none)
};

// Causal convolution of one token per sequence over the normalised rows, channel by channel.  The rows carried on, oldest
// first, are in the slot's version of the tokens so far (version c & 1 at c tokens), from element `carry` on.
template <typename T>
struct ConvStep {
  const T* w;              // [taps][W], the last tap meets the row itself (null: no convolution)
  int taps;
  float* state;            // [slots][2][row]
  long long row;
  int num_slots, carry;
  const int* slots;        // [T], < 0: no state
  const int* kv_lens;      // [T] tokens up to and including this one
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
  float emb_mult;          // factor on the embedding rows
  float w_offset;          // added to the weights of both norms (1: weights stored around zero)
  const T* bias;           // [W] (null: none)
  const T* norm_w;         // [W] (null: one)
  T* norm_out;             // rows x / sqrt(mean(x^2) + eps) * norm_w (null: not wanted)
  long long norm_ld;
  T* raw_out;              // rows x in the compute type
  long long raw_ld;
  T* embed_out;            // the embedding rows
  long long embed_ld;
  int W, W_real;           // padded and real width: the padding columns are zero and do not enter the mean
  float eps;
  // Results of the layers so far [hist_n][T][W] at a stride of hist_stride; this one is stored behind them (null: none kept).
  float* hist;
  long long hist_stride;
  const float* hist_w;     // [hist_n + 1]: x becomes the weighted sum of all of them (null: x stays this one)
  int hist_n;
  ConvStep<T> conv;
};

// Columns i .. i + 3 of row r of a branch, slabs summed.
template <typename T>
__device__ __forceinline__ F4 branch_row(const Branch<T>& br, size_t r, int W, int i) {
  if (br.slabs == nullptr) return load4(br.rows + r * br.ld + i);
  F4 d{{0.0f, 0.0f, 0.0f, 0.0f}};
  const float* p0 = br.slabs + r * W + i;
#pragma unroll 8
  for (int p = 0; p < br.P; ++p) {
    const float4 v = __ldcg(reinterpret_cast<const float4*>(p0 + (size_t)p * br.slab_stride));
    d.v[0] += v.x;
    d.v[1] += v.y;
    d.v[2] += v.z;
    d.v[3] += v.w;
  }
  return d;
}

template <typename T>
__device__ __forceinline__ F4 branch_value(const Branch<T>& br, size_t t, int W, int i) {
  F4 d = branch_row(br, t, W, i);
  if (br.gate != nullptr) {
    const F4 g = load4(br.gate + t * br.gate_ld + i);
#pragma unroll
    for (int e = 0; e < 4; ++e) d.v[e] *= g.v[e];
  }
  return d;
}

template <typename T>
__device__ __forceinline__ void add_branch(const Branch<T>& br, size_t t, int W, int i, float mult, F4& acc) {
  if (br.slabs == nullptr && br.rows == nullptr) return;
  const F4 d = branch_value(br, t, W, i);
#pragma unroll
  for (int e = 0; e < 4; ++e) acc.v[e] += mult * d.v[e];
}

// Sum over the block; every thread returns it.  red: 32 floats, free for the next use after the caller's next barrier.
__device__ __forceinline__ float block_sum(float v, float* red) {
  v = warp_sum(v);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nw = blockDim.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  return warp_sum(lane < nw ? red[lane] : 0.0f);
}

// A thread holds U groups of four columns in registers from the first load to the last store.  DEEP: with earlier results or a
// convolution.
template <typename T, int U, bool DEEP>
__global__ void __launch_bounds__(U == 1 ? 1024 : 512, U == 4 ? 2 : 1) stream_update_kernel(const StreamArgs<T> a) {
  __shared__ float red[2][32];
  const size_t t = blockIdx.x;
  const int i0 = threadIdx.x * 4, step = blockDim.x * 4;
  pdl_launch_dependents();
  F4 acc[U], x[U];
  // A single token's carried rows were written by an earlier step: a few of them are fetched before the previous kernel has finished.
  constexpr int EARLY = DEEP && U == 1 ? 3 : 0;
  const F4 zero{{0.0f, 0.0f, 0.0f, 0.0f}};
  const float* carry_old = nullptr;
  float* carry_new = nullptr;
  F4 early[EARLY > 0 ? EARLY : 1];
  if (DEEP && a.conv.w != nullptr) {
    const int slot = a.conv.slots[t], end = a.conv.kv_lens[t];
    if (slot >= a.conv.num_slots) {
      if (threadIdx.x == 0) prism_report(PRISM_ERR_BOUNDS, 3);
    } else if (slot >= 0 && end > 0) {
      float* base = a.conv.state + (size_t)slot * 2 * a.conv.row + a.conv.carry;
      if (end > 1) carry_old = base + (size_t)((end - 1) & 1) * a.conv.row;
      carry_new = base + (size_t)(end & 1) * a.conv.row;
    }
#pragma unroll
    for (int j = 0; j < EARLY; ++j) early[j] = carry_old && j < a.conv.taps - 1 && i0 < a.W ? load4(carry_old + (size_t)j * a.W + i0) : zero;
  }
  pdl_wait();
  const T* emb = nullptr;
  if (a.ids != nullptr) {
    const long long id = a.ids[t];
    if (id >= 0 && id < a.vocab) emb = a.table + (size_t)id * a.W;
    else if (threadIdx.x == 0) prism_report(PRISM_ERR_BOUNDS, 1);
  }
  const bool has_a = a.a.slabs != nullptr || a.a.rows != nullptr;
  float bs = 0.0f;
  auto earlier_results = [&](int i) {                // weighted sum of the results before this one
    F4 sum = zero;
    const float* h0 = a.hist + t * a.W + i;
#pragma unroll 8
    for (int j = 0; j < a.hist_n; ++j) {
      const float w = __ldg(a.hist_w + j);
      const F4 h = load4(h0 + (size_t)j * a.hist_stride);
#pragma unroll
      for (int e = 0; e < 4; ++e) sum.v[e] = fmaf(w, h.v[e], sum.v[e]);
    }
    return sum;
  };
  F4 before = zero;
  if (DEEP && U == 1 && a.hist_w != nullptr && i0 < a.W) before = earlier_results(i0);
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int i = i0 + u * step;
    acc[u] = x[u] = F4{{0.0f, 0.0f, 0.0f, 0.0f}};
    if (i < a.W) {
      if (U == 1 && a.keep) x[u] = load4(a.x + t * a.W + i);
      if (has_a && a.a.pos == nullptr) acc[u] = branch_value(a.a, t, a.W, i);
    }
  }
  if (a.a.pos != nullptr) {  // all of a thread's columns of one row at a time
    for (int k = 0; k < a.a.K; ++k) {
      const int r = __ldg(a.a.pos + t * a.a.K + k);
      if (r < 0) continue;
      const float w = __ldg(a.a.weight + t * a.a.K + k);
#pragma unroll
      for (int u = 0; u < U; ++u) {
        if (i0 + u * step >= a.W) continue;
        const F4 v = branch_row(a.a, (size_t)r, a.W, i0 + u * step);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[u].v[e] += w * v.v[e];
      }
    }
  }
  if (a.a.self_w != nullptr) {
    const float w = __ldg(a.a.self_w + t);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (i0 + u * step >= a.W) continue;
      const F4 v = U == 1 && a.keep ? x[u] : load4(a.x + t * a.W + i0 + u * step);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u].v[e] += w * v.v[e];
    }
  }
#pragma unroll
  for (int u = 0; u < U; ++u)
#pragma unroll
    for (int e = 0; e < 4; ++e) bs += acc[u].v[e] * acc[u].v[e];
  if (a.a.post_w != nullptr) {  // the branch over its own root mean square
    const float post = a.mult / sqrtf(block_sum(bs, red[0]) / (float)a.W_real + a.eps);
#pragma unroll
    for (int u = 0; u < U; ++u) {
      if (i0 + u * step >= a.W) continue;
      const F4 w = load4(a.a.post_w + i0 + u * step);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u].v[e] *= post * (a.w_offset + w.v[e]);
    }
  } else if (has_a) {
#pragma unroll
    for (int u = 0; u < U; ++u)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u].v[e] *= a.mult;
  }
  float ss = 0.0f;
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int i = i0 + u * step;
    if (i >= a.W) continue;
    if (U > 1 && a.keep) x[u] = load4(a.x + t * a.W + i);
    add_branch(a.b, t, a.W, i, a.mult, acc[u]);
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[u].v[e] += x[u].v[e];
    if (a.bias != nullptr) {
      const F4 s = load4(a.bias + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u].v[e] += s.v[e];
    }
    if (emb != nullptr) {
      F4 v = load4(emb + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) v.v[e] *= a.emb_mult;
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[u].v[e] += v.v[e];
      if (a.embed_out != nullptr) store4(a.embed_out + t * a.embed_ld + i, v);
    } else if (a.embed_out != nullptr) {
      store4(a.embed_out + t * a.embed_ld + i, F4{{0.0f, 0.0f, 0.0f, 0.0f}});
    }
    if (DEEP && a.hist != nullptr) {
      store4(a.hist + (size_t)a.hist_n * a.hist_stride + t * a.W + i, acc[u]);
      if (a.hist_w != nullptr) {
        const float own = __ldg(a.hist_w + a.hist_n);
        const F4 sum = U == 1 ? before : earlier_results(i);
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[u].v[e] = fmaf(own, acc[u].v[e], sum.v[e]);
      }
    }
    store4(a.x + t * a.W + i, acc[u]);
    if (a.raw_out != nullptr) store4(a.raw_out + t * a.raw_ld + i, acc[u]);
#pragma unroll
    for (int e = 0; e < 4; ++e) ss += acc[u].v[e] * acc[u].v[e];
  }
  if (a.norm_out == nullptr) return;
  const float inv = 1.0f / sqrtf(block_sum(ss, red[1]) / (float)a.W_real + a.eps);
#pragma unroll
  for (int u = 0; u < U; ++u) {
    const int i = i0 + u * step;
    if (i >= a.W) continue;
    F4 v = acc[u];
#pragma unroll
    for (int e = 0; e < 4; ++e) v.v[e] *= inv;
    if (a.norm_w != nullptr) {
      const F4 w = load4(a.norm_w + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) v.v[e] *= a.w_offset + w.v[e];
    }
    if (DEEP && a.conv.w != nullptr) {     // what a row of the compute type would hold meets the taps
      const int last = a.conv.taps - 1;
      F4 o = load4(a.conv.w + (size_t)last * a.W + i);
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if (sizeof(T) == 2) v.v[e] = bf16_round(v.v[e]);
        o.v[e] = fmaf(o.v[e], v.v[e], v.v[e]);
      }
      auto tap = [&](int j, const F4& c) {
        const F4 w = load4(a.conv.w + (size_t)j * a.W + i);
#pragma unroll
        for (int e = 0; e < 4; ++e) o.v[e] = fmaf(w.v[e], c.v[e], o.v[e]);
        if (carry_new && j > 0) store4(carry_new + (size_t)(j - 1) * a.W + i, c);
      };
#pragma unroll
      for (int j = 0; j < EARLY; ++j)
        if (j < last) tap(j, early[j]);
      for (int j = EARLY; j < last; ++j) tap(j, carry_old ? load4(carry_old + (size_t)j * a.W + i) : zero);
      if (carry_new && last > 0) store4(carry_new + (size_t)(last - 1) * a.W + i, v);
      v = o;
    }
    store4(a.norm_out + t * a.norm_ld + i, v);
  }
}

// -------------------------------------------------------------------------------------------------
// g[t][d] = gelu_tanh(z[t][d]) * table[ids[t]][offset + d]: the gate of a per-token side table.
// -------------------------------------------------------------------------------------------------
template <typename T>
struct SideArgs {
  Branch<T> z;
  const T* table;
  long long vocab, table_ld, offset;
  const long long* ids;
  T* out;                  // [T][D]
  int D;
  long long total;         // T * D / 4
};

template <typename T>
__global__ void __launch_bounds__(256) token_side_gate_kernel(const SideArgs<T> a) {
  pdl_launch_dependents();
  const long long n = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (n >= a.total) return;
  const size_t t = (size_t)(n * 4 / a.D);
  const int d = (int)(n * 4 - (long long)t * a.D);
  const long long id = a.ids[t];
  F4 e{{0.0f, 0.0f, 0.0f, 0.0f}};  // the table does not depend on the previous kernel
  if (id >= 0 && id < a.vocab) e = load4(a.table + (size_t)id * a.table_ld + a.offset + d);
  else prism_report(PRISM_ERR_BOUNDS, 2);
  pdl_wait();
  F4 z = branch_value(a.z, t, a.D, d);
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    const float v = z.v[k];
    z.v[k] = 0.5f * v * (1.0f + tanhf(0.7978845608028654f * (v + 0.044715f * v * v * v))) * e.v[k];
  }
  store4(a.out + t * a.D + d, z);
}

template <typename T>
int launch_side(const void* slabs, long long slab_stride, int P, const void* rows, long long ld, const void* table, long long vocab,
                long long table_ld, long long offset, const void* ids, void* out, int T_rows, int D, cudaStream_t stream, bool pdl) {
  SideArgs<T> a{Branch<T>{(const float*)slabs, slab_stride, P, (const T*)rows, ld, nullptr, 0, nullptr, nullptr, 0, nullptr, nullptr},
                (const T*)table, vocab, table_ld, offset, (const long long*)ids, (T*)out, D, (long long)T_rows * D / 4};
  return (int)prism_launch(token_side_gate_kernel<T>, dim3((unsigned)((a.total + 255) / 256)), dim3(256), 0, stream, pdl, a);
}

template <typename T>
int launch_stream(int T_rows, void* x, int keep, const void* ids, const void* table, long long vocab, const void* a_slabs,
                  long long a_stride, int a_P, const void* a_rows, long long a_ld, const void* a_gate, const void* b_slabs,
                  long long b_stride, int b_P, const void* b_rows, long long b_ld, const void* b_gate, long long gate_ld,
                  const void* a_pos, const void* a_weight, int a_K, const void* a_post, const void* a_self, float mult,
                  float emb_mult, float w_offset, const void* bias, const void* norm_w, void* norm_out, long long norm_ld, void* raw_out, long long raw_ld,
                  void* embed_out, long long embed_ld, int W, int W_real, float eps, void* hist, long long hist_stride, const void* hist_w,
                  int hist_n, const void* conv_w, int taps, void* state, long long state_row, int num_slots, int carry, const void* slots,
                  const void* kv_lens, cudaStream_t stream, bool pdl) {
  StreamArgs<T> a;
  a.hist = (float*)hist;
  a.hist_stride = hist_stride;
  a.hist_w = (const float*)hist_w;
  a.hist_n = hist_n;
  a.conv = ConvStep<T>{(const T*)conv_w, taps, (float*)state, state_row, num_slots, carry, (const int*)slots, (const int*)kv_lens};
  a.x = (float*)x;
  a.keep = keep;
  a.ids = (const long long*)ids;
  a.table = (const T*)table;
  a.vocab = vocab;
  a.a = Branch<T>{(const float*)a_slabs, a_stride, a_P, (const T*)a_rows, a_ld, (const T*)a_gate, gate_ld,
                  (const int*)a_pos, (const float*)a_weight, a_K, (const T*)a_post,
                  (const float*)a_self};
  a.b = Branch<T>{(const float*)b_slabs, b_stride, b_P, (const T*)b_rows, b_ld, (const T*)b_gate, gate_ld, nullptr, nullptr, 0, nullptr, nullptr};
  a.mult = mult;
  a.emb_mult = emb_mult;
  a.w_offset = w_offset;
  a.bias = (const T*)bias;
  a.norm_w = (const T*)norm_w;
  a.norm_out = (T*)norm_out;
  a.norm_ld = norm_ld;
  a.raw_out = (T*)raw_out;
  a.raw_ld = raw_ld;
  a.embed_out = (T*)embed_out;
  a.embed_ld = embed_ld;
  a.W = W;
  a.W_real = W_real;
  a.eps = eps;
  // a few rows: as many threads as there are groups of four columns; many rows: several groups per thread
  const int groups = W / 4;
  const int U = groups <= 1024 && (T_rows < 256 || groups < 256) ? 1 : (groups <= 2048 ? 4 : (groups <= 4096 ? 8 : 16));
  const dim3 grid(T_rows), block(((groups + U - 1) / U + 31) / 32 * 32);
  auto run = [&](auto deep) -> int {
    constexpr bool DEEP = decltype(deep)::value;
    switch (U) {
      case 1: return (int)prism_launch(stream_update_kernel<T, 1, DEEP>, grid, block, 0, stream, pdl, a);
      case 4: return (int)prism_launch(stream_update_kernel<T, 4, DEEP>, grid, block, 0, stream, pdl, a);
      case 8: return (int)prism_launch(stream_update_kernel<T, 8, DEEP>, grid, block, 0, stream, pdl, a);
    }
    return (int)prism_launch(stream_update_kernel<T, 16, DEEP>, grid, block, 0, stream, pdl, a);
  };
  return hist != nullptr || conv_w != nullptr ? run(std::true_type()) : run(std::false_type());
}

}  // namespace

// f32: 1 = table, rows, gates, bias and outputs are fp32, 0 = bf16.  W a multiple of 8; every row stride a
// multiple of 4 elements.  a_self [T] (with a branch a): weight of the old stream row in it.  w_offset: added to norm weights.
// hist: fp32 results of hist_n layers so far at hist_stride elements from one another, this one goes behind them; hist_w
// [hist_n + 1] fp32: the stream becomes their weighted sum.  conv_w [taps][W] (with norm_out, one token per sequence): the
// convolution of the normalised row with the taps - 1 rows in the state slots [num_slots][2][state_row] from `carry` on.
PRISM_API int prism_stream_update(int f32, int T, void* x, int keep, const void* ids, const void* table, long long vocab,
                                  const void* a_slabs, long long a_stride, int a_P, const void* a_rows, long long a_ld,
                                  const void* a_gate, const void* b_slabs, long long b_stride, int b_P, const void* b_rows,
                                  long long b_ld, const void* b_gate, long long gate_ld, const void* a_pos,
                                  const void* a_weight, int a_K, const void* a_post, const void* a_self, float mult,
                                  float emb_mult, float w_offset, const void* bias,
                                  const void* norm_w, void* norm_out, long long norm_ld, void* raw_out, long long raw_ld, void* embed_out,
                                  long long embed_ld, int W, int W_real, float eps, void* hist, long long hist_stride, const void* hist_w,
                                  int hist_n, const void* conv_w, int taps, void* state, long long state_row, int num_slots, int carry,
                                  const void* slots, const void* kv_lens, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (hist != nullptr && (hist_n < 0 || hist_stride < (long long)T * W)) return -4;
  if (conv_w != nullptr && (!norm_out || taps < 1 || !state || !slots || !kv_lens || num_slots <= 0 || carry < 0 || carry % 4 || state_row % 4 ||
                            carry + (long long)(taps - 1) * W > state_row))
    return -5;
  if (W <= 0 || W % 8 || W_real <= 0 || W_real > W || W > 32768) return -1;
  if ((a_ld | b_ld | gate_ld | norm_ld | raw_ld | embed_ld) % 4) return -2;
  if ((a_pos != nullptr && (a_K <= 0 || !a_weight || a_gate)) || ((a_pos || a_post || a_self) && !a_slabs && !a_rows)) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_stream<float>(T, x, keep, ids, table, vocab, a_slabs, a_stride, a_P, a_rows, a_ld, a_gate, b_slabs, b_stride,
                                    b_P, b_rows, b_ld, b_gate, gate_ld, a_pos, a_weight, a_K, a_post, a_self, mult, emb_mult, w_offset, bias, norm_w, norm_out, norm_ld, raw_out, raw_ld, embed_out,
                                    embed_ld, W, W_real, eps, hist, hist_stride, hist_w, hist_n, conv_w, taps, state, state_row,
                                    num_slots, carry, slots, kv_lens, s, pdl != 0)
             : launch_stream<bf16>(T, x, keep, ids, table, vocab, a_slabs, a_stride, a_P, a_rows, a_ld, a_gate, b_slabs, b_stride,
                                   b_P, b_rows, b_ld, b_gate, gate_ld, a_pos, a_weight, a_K, a_post, a_self, mult, emb_mult, w_offset, bias, norm_w, norm_out, norm_ld, raw_out, raw_ld, embed_out,
                                   embed_ld, W, W_real, eps, hist, hist_stride, hist_w, hist_n, conv_w, taps, state, state_row,
                                    num_slots, carry, slots, kv_lens, s, pdl != 0);
}

// g [T][D] = gelu_tanh(z) * table[ids[t]][offset ..]; z as fp32 slabs or rows of the compute type.  D, table_ld and offset
// multiples of 4.
PRISM_API int prism_token_side_gate(int f32, const void* slabs, long long slab_stride, int P, const void* rows, long long ld,
                                    const void* table, long long vocab, long long table_ld, long long offset, const void* ids,
                                    void* out, int T, int D, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (D <= 0 || (D | table_ld | offset | ld) % 4 || offset + D > table_ld || (!slabs && !rows)) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_side<float>(slabs, slab_stride, P, rows, ld, table, vocab, table_ld, offset, ids, out, T, D, s, pdl != 0)
             : launch_side<bf16>(slabs, slab_stride, P, rows, ld, table, vocab, table_ld, offset, ids, out, T, D, s, pdl != 0);
}
