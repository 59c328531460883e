// Recurrent mixers with a matrix state per head, and what they read of the previous token.
//
// A sequence's state of one layer is a row of fp32 in a slot:  [heads][n][n] (key channel, value channel), then the last
// token's input row [W].  Every slot has two versions: a step that takes a sequence from c tokens to c' reads version c & 1
// and writes version c' & 1, so a step that is repeated finds what it read before.  A sequence without tokens (c = 0)
// starts from zero whatever its slot holds.
//
//   token_mix_kernel      five blends of a token's row with the previous token's, and the table of a grouped projection
//   tanh_split_kernel     tanh of a narrow projection as a sum of two numbers of the compute type
//   state_step_kernel     one token per sequence: decay, output, state update, norm per head, gate
//   state_scan_kernel     many tokens of a sequence: the state stays in registers, loader warps feed token blocks
//   head_norm_gate_kernel norm per head and gate behind the scan
//
// Per head, with r, k, v, the decay d = exp(-exp(z)) and the bonus u (all fp32):
//   o_t = (S + diag(u) k v^T)^T r,   S <- diag(d) S + k v^T.
#include "common.cuh"

PRISM_DEFINE_TU_STATUS(recurrence)

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  uint2 o;
  *reinterpret_cast<__nv_bfloat162*>(&o.x) = __floats2bfloat162_rn(v.x, v.y);
  *reinterpret_cast<__nv_bfloat162*>(&o.y) = __floats2bfloat162_rn(v.z, v.w);
  *reinterpret_cast<uint2*>(p) = o;
}

// A projection's result: fp32 split-K slabs [P][rows][ld] whose sum it is, or rows of the compute type.
template <typename T>
struct Proj {
  const float* slabs;
  long long slab_stride;
  int P;
  const T* rows;
  long long ld;
};
template <typename T>
__device__ __forceinline__ float4 proj4(const Proj<T>& p, size_t row, int c) {
  if (p.slabs == nullptr) return load4(p.rows + row * p.ld + c);
  float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
  const float* s = p.slabs + row * p.ld + c;
#pragma unroll 4
  for (int i = 0; i < p.P; ++i) {
    const float4 x = __ldcg(reinterpret_cast<const float4*>(s + (size_t)i * p.slab_stride));
    v.x += x.x;
    v.y += x.y;
    v.z += x.z;
    v.w += x.w;
  }
  return v;
}
template <typename T>
__device__ __forceinline__ float proj1(const Proj<T>& p, size_t row, int c) {
  if (p.slabs == nullptr) return to_f(p.rows[row * p.ld + c]);
  float v = 0.0f;
  const float* s = p.slabs + row * p.ld + c;
#pragma unroll 4
  for (int i = 0; i < p.P; ++i) v += __ldcg(s + (size_t)i * p.slab_stride);
  return v;
}

// The state slots of a layer and the sequences of a step.
struct StateArgs {
  float* state;            // [slots][2][row]
  long long row;           // elements of a version
  int num_slots;
  int carry;               // first element of the last token's row
  const int* slots;        // [S], < 0: no state, nothing is computed
  const int* cu_q;         // [S + 1] token offsets (null: sequence s is token s)
  const int* kv_lens;      // [S] tokens up to and including the step's last
  const float* x;          // [T][W] input rows of the step
  int S, W;
};
struct Span {
  int first, len, before;  // token offset, tokens in this step, tokens before it
  float* old_version;      // null: none before
  float* new_version;      // null: no slot
};
__device__ __forceinline__ Span span_of(const StateArgs& a, int s) {
  Span r;
  r.first = a.cu_q ? a.cu_q[s] : s;
  r.len = a.cu_q ? a.cu_q[s + 1] - r.first : 1;
  const int end = a.kv_lens[s], slot = a.slots[s];
  r.before = max(0, end - r.len);
  r.old_version = r.new_version = nullptr;
  if (slot < 0 || r.len <= 0) return r;
  if (slot >= a.num_slots) {
    prism_report(PRISM_ERR_BOUNDS, 1);
    return r;
  }
  float* base = a.state + (size_t)slot * 2 * a.row;
  if (r.before > 0) r.old_version = base + (size_t)(r.before & 1) * a.row;
  r.new_version = base + (size_t)(end & 1) * a.row;
  return r;
}

// =====================================================================================
// mixed[m][t] = x_t + (x_(t-1) - x_t) mu_m.  grid (tokens, column blocks); five blends of one row.
// =====================================================================================
constexpr int MIXES = 5;
template <typename T>
struct MixArgs {
  StateArgs st;
  const T* mu;             // [5][W]
  T* out;                  // [5][T][W]
  int T_rows;
  int4* groups;            // table of the grouped projection of the first four blends: (blend, first row, rows, 0)
  int* n_groups;
  int tile;
};

template <typename T>
__global__ void __launch_bounds__(256) token_mix_kernel(const MixArgs<T> a) {
  const StateArgs& st = a.st;
  const int t = blockIdx.x, W = st.W;
  pdl_launch_dependents();
  // the sequence of token t: the last one that starts at or before it and is not empty
  int s = t;
  if (st.cu_q != nullptr) {
    int lo = 0, hi = st.S - 1;
    while (lo < hi) {
      const int mid = (lo + hi + 1) >> 1;
      if (st.cu_q[mid] <= t) lo = mid;
      else hi = mid - 1;
    }
    s = lo;
  }
  const Span sp = span_of(st, s);
  pdl_wait();
  if (blockIdx.y == 0 && t == 0 && a.groups != nullptr) {
    const int per = (a.T_rows + a.tile - 1) / a.tile;
    for (int i = threadIdx.x; i < 4 * per; i += blockDim.x) {
      const int m = i / per, r = i % per * a.tile;
      a.groups[i] = make_int4(m, m * a.T_rows + r, min(a.tile, a.T_rows - r), 0);
    }
    if (threadIdx.x == 0) *a.n_groups = 4 * per;
  }
  const float* prev = t > sp.first ? st.x + (size_t)(t - 1) * W : (sp.old_version ? sp.old_version + st.carry : nullptr);
  for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * 4; c < W; c += gridDim.y * blockDim.x * 4) {
    const float4 x = load4(st.x + (size_t)t * W + c);
    const float4 p = prev ? load4(prev + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 d = make_float4(p.x - x.x, p.y - x.y, p.z - x.z, p.w - x.w);
#pragma unroll
    for (int m = 0; m < MIXES; ++m) {
      const float4 mu = load4(a.mu + (size_t)m * W + c);
      store4(a.out + ((size_t)m * a.T_rows + t) * W + c,
             make_float4(fmaf(d.x, mu.x, x.x), fmaf(d.y, mu.y, x.y), fmaf(d.z, mu.z, x.z), fmaf(d.w, mu.w, x.w)));
    }
  }
}

// out[t] = [hi, lo] with hi + lo = tanh(z_t) to about twice the type's precision: the next projection multiplies both.
template <typename T>
__global__ void __launch_bounds__(256) tanh_split_kernel(const Proj<T> z, T* out, int R, long long total) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i >= total) return;
  const long long t = i / R;
  const int c = (int)(i - t * R);
  const float v = tanhf(proj1(z, (size_t)t, c));
  T hi;
  put(&hi, v);
  out[t * 2 * R + c] = hi;
  put(out + t * 2 * R + R + c, v - to_f(hi));
}

// =====================================================================================
// One token per sequence.  grid (heads, sequences).  Thread (ty, tx) owns value columns 4 tx .. 4 tx + 3 of key rows
// ty, ty + rows, ...; up to NV of its state elements (float4) are fetched before the previous kernel has finished: they
// were written by an earlier step.
// =====================================================================================
template <typename T>
struct StepArgs {
  StateArgs st;
  Proj<T> p;               // r, k, v, gate: rows m * tokens + t, columns head * n
  Proj<T> w1;              // [tokens][rank] input of the decay's second projection, before tanh
  const T* w2;             // [heads * n][rank]
  const T* w0;             // [heads * n]
  const T* u;              // [heads * n]
  const T* norm;           // [heads * n]
  T* out;                  // [tokens][heads * n]
  int tokens, H, n, n_real, rank;
  float eps;
};

constexpr int STEP_THREADS = 256;

template <typename T, int NV>
__global__ void __launch_bounds__(STEP_THREADS) state_step_kernel(const StepArgs<T> a) {
  extern __shared__ float sm[];
  const int n = a.n, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, s = blockIdx.y;
  float *r_s = sm, *k_s = sm + n, *v_s = sm + 2 * n, *g_s = sm + 3 * n, *d_s = sm + 4 * n, *t_s = sm + 5 * n;
  float* o_s = t_s + a.rank;                      // [rows][n] partial outputs
  __shared__ float red[STEP_THREADS / 32], bonus_s;
  const int c4 = n >> 2, rows = STEP_THREADS / c4, tx = tid % c4, ty = tid / c4;
  pdl_launch_dependents();
  const Span sp = span_of(a.st, s);
  const size_t C = (size_t)a.H * n, hc = (size_t)h * n;
  T* out = a.out + (size_t)s * C + hc;
  if (sp.new_version == nullptr) {
    pdl_wait();
    for (int c = tid; c < n; c += STEP_THREADS) put(out + c, 0.0f);
    return;
  }
  const float* old_s = sp.old_version ? sp.old_version + (size_t)h * n * n : nullptr;
  float* new_s = sp.new_version + (size_t)h * n * n;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool active = ty < rows;
  float4 S[NV > 0 ? NV : 1];
  if (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int key = ty + i * rows;
      S[i] = active && key < n && old_s ? __ldcg(reinterpret_cast<const float4*>(old_s + (size_t)key * n) + tx) : zero;
    }
  }
  pdl_wait();
  // the projections' sums, and the narrow one's tanh
  for (int i = tid; i < 4 * c4 + a.rank; i += STEP_THREADS) {
    if (i < 4 * c4) {
      const int m = i / c4, c = (i % c4) * 4;
      store4(sm + m * n + c, proj4(a.p, (size_t)m * a.tokens + s, (int)hc + c));
    } else {
      t_s[i - 4 * c4] = tanhf(proj1(a.w1, (size_t)s, i - 4 * c4));
    }
  }
  __syncthreads();
  // decay: eight lanes per channel over the rank
  for (int c0 = 0; c0 < n; c0 += STEP_THREADS / 8) {
    const int c = c0 + (tid >> 3);
    float z = 0.0f;
    if (c < n)
      for (int j = (tid & 7) * 4; j < a.rank; j += 32) {
        const float4 w = load4(a.w2 + (hc + c) * a.rank + j), t = load4(t_s + j);
        z += w.x * t.x + w.y * t.y + w.z * t.z + w.w * t.w;
      }
    z += __shfl_xor_sync(0xffffffffu, z, 1);
    z += __shfl_xor_sync(0xffffffffu, z, 2);
    z += __shfl_xor_sync(0xffffffffu, z, 4);
    if (c < n && (tid & 7) == 0) d_s[c] = expf(-expf(z + to_f(a.w0[hc + c])));
  }
  float b = 0.0f;
  for (int c = tid; c < n; c += STEP_THREADS) b += r_s[c] * to_f(a.u[hc + c]) * k_s[c];
  b = warp_sum(b);
  if (lane == 0) red[warp] = b;
  __syncthreads();
  if (tid == 0) {
    float t = 0.0f;
    for (int i = 0; i < STEP_THREADS / 32; ++i) t += red[i];
    bonus_s = t;
  }
  if (active) {
    const float4 v = load4(v_s + 4 * tx);
    float4 o = zero;
    auto step = [&](int key, float4 st) {
      const float r = r_s[key], k = k_s[key], d = d_s[key];
      o.x = fmaf(r, st.x, o.x);
      o.y = fmaf(r, st.y, o.y);
      o.z = fmaf(r, st.z, o.z);
      o.w = fmaf(r, st.w, o.w);
      store4(new_s + (size_t)key * n + 4 * tx, make_float4(fmaf(d, st.x, k * v.x), fmaf(d, st.y, k * v.y), fmaf(d, st.z, k * v.z), fmaf(d, st.w, k * v.w)));
    };
    if (NV > 0) {
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (ty + i * rows < n) step(ty + i * rows, S[i]);
    } else {
#pragma unroll 8
      for (int key = ty; key < n; key += rows) step(key, old_s ? __ldcg(reinterpret_cast<const float4*>(old_s + (size_t)key * n) + tx) : zero);
    }
    store4(o_s + (size_t)ty * n + 4 * tx, o);
  }
  // the last token's row, a share per head
  for (int c = (h * STEP_THREADS + tid) * 4; c < a.st.W; c += a.H * STEP_THREADS * 4)
    store4(sp.new_version + a.st.carry + c, load4(a.st.x + (size_t)s * a.st.W + c));
  __syncthreads();
  float ss = 0.0f;
  for (int c = tid; c < n; c += STEP_THREADS) {
    float o = bonus_s * v_s[c];
    for (int i = 0; i < rows; ++i) o += o_s[(size_t)i * n + c];
    o_s[c] = o;                                   // column c is this thread's
    ss += o * o;
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = warp_sum(lane < STEP_THREADS / 32 ? red[lane] : 0.0f);
  const float inv = 1.0f / sqrtf(ss / (float)a.n_real + a.eps);
  for (int c = tid; c < n; c += STEP_THREADS) {
    const float g = g_s[c];
    put(out + c, o_s[c] * inv * to_f(a.norm[hc + c]) * (g / (1.0f + expf(-g))));
  }
}

// =====================================================================================
// Many tokens per sequence.  grid (heads x column blocks of 32, sequences).  Four warps hold the state: a lane owns one
// value column and every fourth group of four keys of it (KT keys in all), so a token costs KT / 4 times three 16-byte
// shared-memory reads and the products in registers.  Four more warps fill the next block of TB tokens: sums of the
// projections' slabs, decays, the bonus' scalar per token.
// =====================================================================================
constexpr int TB = 16;
constexpr int SCAN_COLS = 32;
constexpr int SCAN_THREADS = 256;

template <typename T>
struct ScanArgs {
  StateArgs st;
  Proj<T> p;               // r, k, v: rows m * tokens + t
  const float* z;          // [tokens][heads * n]: decay exp(-exp(z))
  const T* u;              // [heads * n]
  float* o;                // [tokens][heads * n]
  int tokens, H, n;
};

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
__device__ __forceinline__ unsigned long long pair_of(float lo, float hi) {
  unsigned long long d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(lo), "f"(hi));
  return d;
}
__device__ __forceinline__ float pair_sum(unsigned long long v) {
  float lo, hi;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
  return lo + hi;
}

template <typename T, int KT>
__global__ void __launch_bounds__(SCAN_THREADS) state_scan_kernel(const ScanArgs<T> a) {
  extern __shared__ __align__(16) float sm[];
  constexpr int NP = 4 * KT;                      // keys, padded to the lanes' share
  const int n = a.n, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blocks = (n + SCAN_COLS - 1) / SCAN_COLS, h = blockIdx.x / blocks, col0 = blockIdx.x % blocks * SCAN_COLS, s = blockIdx.y;
  // two buffers of [r | k | d][TB][NP], v [TB][32], bonus [TB]; then outputs [TB][32] of the block under way
  const int buf = 3 * TB * NP + TB * SCAN_COLS + TB;
  float* out_s = sm + 2 * buf;
  pdl_launch_dependents();
  const Span sp = span_of(a.st, s);
  const size_t C = (size_t)a.H * n, hc = (size_t)h * n;
  pdl_wait();
  if (sp.len <= 0) return;
  const int nb = (sp.len + TB - 1) / TB;
  if (sp.new_version == nullptr) {                // no slot: outputs are zero
    for (int i = threadIdx.x; i < sp.len * SCAN_COLS; i += SCAN_THREADS)
      if (col0 + i % SCAN_COLS < n) a.o[(size_t)(sp.first + i / SCAN_COLS) * C + hc + col0 + i % SCAN_COLS] = 0.0f;
    return;
  }
  auto fill = [&](int b, int w) {                 // one warp's tokens of block b
    float* dst = sm + (b & 1) * buf;
#pragma unroll
    for (int q = 0; q < TB / 4; ++q) {
      const int i = w + 4 * q, tok = b * TB + i;
      if (tok >= sp.len) continue;
      const size_t t = (size_t)(sp.first + tok);
      float bonus = 0.0f;
      for (int c = lane * 4; c < NP; c += 128) {
        float4 r = make_float4(0.f, 0.f, 0.f, 0.f), k = r, d = r;
        if (c < n) {
          r = proj4(a.p, t, (int)hc + c);
          k = proj4(a.p, (size_t)a.tokens + t, (int)hc + c);
          const float4 z = __ldcg(reinterpret_cast<const float4*>(a.z + t * C + hc + c)), u = load4(a.u + hc + c);
          d = make_float4(expf(-expf(z.x)), expf(-expf(z.y)), expf(-expf(z.z)), expf(-expf(z.w)));
          bonus += r.x * u.x * k.x + r.y * u.y * k.y + r.z * u.z * k.z + r.w * u.w * k.w;
        }
        store4(dst + i * NP + c, r);
        store4(dst + (TB + i) * NP + c, k);
        store4(dst + (2 * TB + i) * NP + c, d);
      }
      if (lane * 4 < SCAN_COLS)
        store4(dst + 3 * TB * NP + i * SCAN_COLS + lane * 4,
               col0 + lane * 4 < n ? proj4(a.p, (size_t)2 * a.tokens + t, (int)hc + col0 + lane * 4) : make_float4(0.f, 0.f, 0.f, 0.f));
      bonus = warp_sum(bonus);
      if (lane == 0) dst[3 * TB * NP + TB * SCAN_COLS + i] = bonus;
    }
  };
  const bool loader = warp >= 4;
  const int lk = lane & 3, col = (warp & 3) * 8 + (lane >> 2);     // column of the block
  const bool live = col0 + col < n;
  unsigned long long S[KT / 2];                   // keys 16 g + 4 lk + {0, 1}, {2, 3}
  if (loader) {
    fill(0, warp - 4);
  } else {
    const float* src = sp.old_version ? sp.old_version + (size_t)h * n * n + col0 + col : nullptr;
#pragma unroll
    for (int g = 0; g < KT / 4; ++g)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = 16 * g + 4 * lk + 2 * e;
        const bool in = live && src && key < n;   // n is a multiple of 16
        S[2 * g + e] = pair_of(in ? src[(size_t)key * n] : 0.0f, in ? src[(size_t)(key + 1) * n] : 0.0f);
      }
  }
  __syncthreads();
  for (int b = 0; b < nb; ++b) {
    if (loader) {
      if (b + 1 < nb) fill(b + 1, warp - 4);
    } else {
      const float* src = sm + (b & 1) * buf;
      const int cnt = min(TB, sp.len - b * TB);
#pragma unroll 2
      for (int i = 0; i < cnt; ++i) {
        const float v = src[3 * TB * NP + i * SCAN_COLS + col];
        const unsigned long long vv = pair_of(v, v);
        unsigned long long o0 = 0, o1 = 0;
#pragma unroll
        for (int g = 0; g < KT / 4; ++g) {
          const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(src + i * NP + 16 * g + 4 * lk);
          const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(src + (TB + i) * NP + 16 * g + 4 * lk);
          const ulonglong2 d = *reinterpret_cast<const ulonglong2*>(src + (2 * TB + i) * NP + 16 * g + 4 * lk);
          o0 = fma2(r.x, S[2 * g], o0);
          o1 = fma2(r.y, S[2 * g + 1], o1);
          S[2 * g] = fma2(d.x, S[2 * g], mul2(k.x, vv));
          S[2 * g + 1] = fma2(d.y, S[2 * g + 1], mul2(k.y, vv));
        }
        float o = pair_sum(o0) + pair_sum(o1);
        o += __shfl_xor_sync(0xffffffffu, o, 1);
        o += __shfl_xor_sync(0xffffffffu, o, 2);
        if (lk == 0) out_s[(b & 1) * TB * SCAN_COLS + i * SCAN_COLS + col] = fmaf(src[3 * TB * NP + TB * SCAN_COLS + i], v, o);
      }
      // a warp's eight columns of the block
      __syncwarp();
      for (int i = lane >> 1; i < cnt; i += 16) {
        const int c = (warp & 3) * 8 + (lane & 1) * 4;
        if (col0 + c < n)
          store4(a.o + (size_t)(sp.first + b * TB + i) * C + hc + col0 + c, load4(out_s + (b & 1) * TB * SCAN_COLS + i * SCAN_COLS + c));
      }
    }
    __syncthreads();
  }
  if (!loader) {
    float* dst = sp.new_version + (size_t)h * n * n + col0 + col;
#pragma unroll
    for (int g = 0; g < KT / 4; ++g)
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int key = 16 * g + 4 * lk + 2 * e;
        if (live && key < n) {
          float lo, hi;
          asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(S[2 * g + e]));
          dst[(size_t)key * n] = lo;
          dst[(size_t)(key + 1) * n] = hi;
        }
      }
  } else {                                        // the last token's row, a share per CTA
    const float* x = a.st.x + (size_t)(sp.first + sp.len - 1) * a.st.W;
    for (int c = (blockIdx.x * 128 + threadIdx.x - 128) * 4; c < a.st.W; c += gridDim.x * 512)
      store4(sp.new_version + a.st.carry + c, load4(x + c));
  }
}

// out = o / rms(o) * norm * silu(gate) per head; one warp per (token, head)
template <typename T>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* o, const Proj<T> p, const T* norm, T* out, int tokens, int H, int n,
                                                             int n_real, float eps) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= (long long)tokens * H) return;
  const int lane = threadIdx.x & 31;
  const size_t t = (size_t)(i / H);
  const int hc = (int)(i % H) * n;
  const float* row = o + t * (size_t)H * n + hc;
  float4 v[2];
  float ss = 0.0f;
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int c = (lane + 32 * e) * 4;
    v[e] = c < n ? __ldcg(reinterpret_cast<const float4*>(row + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += v[e].x * v[e].x + v[e].y * v[e].y + v[e].z * v[e].z + v[e].w * v[e].w;
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)n_real + eps);
#pragma unroll
  for (int e = 0; e < 2; ++e) {
    const int c = (lane + 32 * e) * 4;
    if (c >= n) continue;
    const float4 g = proj4(p, (size_t)3 * tokens + t, hc + c), w = load4(norm + hc + c);
    auto silu_f = [](float z) { return z / (1.0f + expf(-z)); };
    store4(out + t * (size_t)H * n + hc + c, make_float4(v[e].x * inv * w.x * silu_f(g.x), v[e].y * inv * w.y * silu_f(g.y),
                                                         v[e].z * inv * w.z * silu_f(g.z), v[e].w * inv * w.w * silu_f(g.w)));
  }
}

StateArgs state_args(void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q, const void* kv_lens,
                     const void* x, int S, int W) {
  return StateArgs{(float*)state, row, num_slots, carry, (const int*)slots, (const int*)cu_q, (const int*)kv_lens, (const float*)x, S, W};
}
int check_state(long long row, int num_slots, int carry, int S, int W) {
  return row <= 0 || row % 4 || num_slots <= 0 || carry < 0 || carry % 4 || S <= 0 || W <= 0 || W % 8 || carry + W > row ? -1 : 0;
}
template <typename T>
Proj<T> proj_of(const void* slabs, long long stride, int P, const void* rows, long long ld) {
  return Proj<T>{(const float*)slabs, stride, P, (const T*)rows, ld};
}

template <typename K>
int allow_smem(K kernel, size_t smem, size_t& configured) {
  if (smem > 227 * 1024) return -5;
  if (smem <= configured) return 0;
  const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  if (e == cudaSuccess) configured = smem;
  return (int)e;
}

template <typename T, int NV>
int launch_step(const StepArgs<T>& a, cudaStream_t stream, bool pdl) {
  const int rows = STEP_THREADS / (a.n / 4);
  const size_t smem = (size_t)(5 * a.n + a.rank + rows * a.n) * sizeof(float);
  static size_t configured = 48 * 1024;
  if (int rc = allow_smem(state_step_kernel<T, NV>, smem, configured)) return rc;
  return (int)prism_launch(state_step_kernel<T, NV>, dim3(a.H, a.st.S), dim3(STEP_THREADS), smem, stream, pdl, a);
}

template <typename T, int KT>
int launch_scan(const ScanArgs<T>& a, cudaStream_t stream, bool pdl) {
  const size_t smem = (size_t)(2 * (3 * TB * 4 * KT + TB * SCAN_COLS + TB) + 2 * TB * SCAN_COLS) * sizeof(float);
  static size_t configured = 48 * 1024;
  if (int rc = allow_smem(state_scan_kernel<T, KT>, smem, configured)) return rc;
  const dim3 grid(a.H * ((a.n + SCAN_COLS - 1) / SCAN_COLS), a.st.S);
  return (int)prism_launch(state_scan_kernel<T, KT>, grid, dim3(SCAN_THREADS), smem, stream, pdl, a);
}

template <typename T>
int launch_mix(const StateArgs& st, const void* mu, void* out, int T_rows, void* groups, void* n_groups, int tile, cudaStream_t stream,
               bool pdl) {
  MixArgs<T> a{st, (const T*)mu, (T*)out, T_rows, (int4*)groups, (int*)n_groups, tile};
  // few tokens: a thread per four columns
  const int by = T_rows <= 64 ? (st.W / 4 + 255) / 256 : 1;
  return (int)prism_launch(token_mix_kernel<T>, dim3(T_rows, by), dim3(256), 0, stream, pdl, a);
}

}  // namespace

// State slots: state [num_slots][2][row] fp32, a version being [H][n][n] and from `carry` on the last token's row [W].
// slots, kv_lens [S]; cu_q [S + 1] (null: one token per sequence); x [T][W] fp32.

// out [5][T][W] = x + (previous row - x) mu[m].  groups (null: none): the table of a grouped projection of the first four
// blends in tiles of at most `tile` rows.
PRISM_API int prism_token_mix(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q,
                              const void* kv_lens, const void* x, int S, int W, const void* mu, void* out, int T, void* groups,
                              void* n_groups, int tile, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (int rc = check_state(row, num_slots, carry, S, W)) return rc;
  if (groups != nullptr && (!n_groups || tile < 1)) return -2;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, cu_q, kv_lens, x, S, W);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_mix<float>(st, mu, out, T, groups, n_groups, tile, s, pdl != 0)
             : launch_mix<bf16>(st, mu, out, T, groups, n_groups, tile, s, pdl != 0);
}

// out [T][2 R] = [hi, lo], hi + lo = tanh(z).  z as fp32 slabs or rows of the compute type.
PRISM_API int prism_tanh_split(int f32, const void* slabs, long long slab_stride, int P, const void* rows, long long ld, void* out, int T,
                               int R, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (R <= 0 || (!slabs && !rows)) return -1;
  const long long total = (long long)T * R;
  const dim3 grid((unsigned)((total + 255) / 256));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? (int)prism_launch(tanh_split_kernel<float>, grid, dim3(256), 0, s, pdl != 0, proj_of<float>(slabs, slab_stride, P, rows, ld), (float*)out, R, total)
             : (int)prism_launch(tanh_split_kernel<bf16>, grid, dim3(256), 0, s, pdl != 0, proj_of<bf16>(slabs, slab_stride, P, rows, ld), (bf16*)out, R, total);
}

// One token per sequence (token s belongs to sequence s).  p: r, k, v, gate of all tokens one after another, fp32 slabs or
// rows; w1: the decay's narrow projection [S][rank] likewise.  out [S][H n].  n a multiple of 16, at most 256.
PRISM_API int prism_state_step(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* kv_lens,
                               const void* x, int S, int W, const void* p_slabs, long long p_stride, int p_P, const void* p_rows,
                               long long p_ld, const void* w1_slabs, long long w1_stride, int w1_P, const void* w1_rows, long long w1_ld,
                               const void* w2, const void* w0, const void* u, const void* norm, void* out, int H, int n, int n_real,
                               int rank, float eps, void* stream, int pdl) {
  if (S <= 0) return 0;
  if (int rc = check_state(row, num_slots, carry, S, W)) return rc;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || n_real <= 0 || n_real > n || rank <= 0 || rank % 4 || (long long)H * n * n > carry || S > 65535) return -2;
  if ((!p_slabs && !p_rows) || (!w1_slabs && !w1_rows) || p_ld % 4) return -3;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, nullptr, kv_lens, x, S, W);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    StepArgs<T> a{st, proj_of<T>(p_slabs, p_stride, p_P, p_rows, p_ld), proj_of<T>(w1_slabs, w1_stride, w1_P, w1_rows, w1_ld), (const T*)w2,
                  (const T*)w0, (const T*)u, (const T*)norm, (T*)out, S, H, n, n_real, rank, eps};
    const int rows = STEP_THREADS / (n / 4), nv = (n + rows - 1) / rows;
    if (nv <= 4) return launch_step<T, 4>(a, s, pdl != 0);
    if (nv <= 16) return launch_step<T, 16>(a, s, pdl != 0);
    return launch_step<T, 0>(a, s, pdl != 0);
  };
  return f32 ? run(float()) : run(bf16());
}

// Prompts and portions.  p: r, k, v (and the gate) of all T tokens one after another; z [T][H n] fp32; o [T][H n] fp32.
PRISM_API int prism_state_scan(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q,
                               const void* kv_lens, const void* x, int S, int W, const void* p_slabs, long long p_stride, int p_P,
                               const void* p_rows, long long p_ld, const void* z, const void* u, void* o, int T_rows, int H, int n,
                               void* stream, int pdl) {
  if (T_rows <= 0) return 0;
  if (int rc = check_state(row, num_slots, carry, S, W)) return rc;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || (long long)H * n * n > carry || !cu_q || S > 65535) return -2;
  if ((!p_slabs && !p_rows) || p_ld % 4) return -3;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, cu_q, kv_lens, x, S, W);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    ScanArgs<T> a{st, proj_of<T>(p_slabs, p_stride, p_P, p_rows, p_ld), (const float*)z, (const T*)u, (float*)o, T_rows, H, n};
    if (n <= 32) return launch_scan<T, 8>(a, s, pdl != 0);
    if (n <= 64) return launch_scan<T, 16>(a, s, pdl != 0);
    if (n <= 128) return launch_scan<T, 32>(a, s, pdl != 0);
    return launch_scan<T, 64>(a, s, pdl != 0);
  };
  return f32 ? run(float()) : run(bf16());
}

// out [T][H n] = o / rms(o) * norm * silu(gate) per head; the gate is block 3 of p.
PRISM_API int prism_head_norm_gate(int f32, const void* o, const void* p_slabs, long long p_stride, int p_P, const void* p_rows,
                                   long long p_ld, const void* norm, void* out, int T_rows, int H, int n, int n_real, float eps,
                                   void* stream, int pdl) {
  if (T_rows <= 0) return 0;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || n_real <= 0 || n_real > n || (!p_slabs && !p_rows) || p_ld % 4) return -1;
  const dim3 grid((unsigned)(((long long)T_rows * H + 7) / 8));
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? (int)prism_launch(head_norm_gate_kernel<float>, grid, dim3(256), 0, s, pdl != 0, (const float*)o,
                                 proj_of<float>(p_slabs, p_stride, p_P, p_rows, p_ld), (const float*)norm, (float*)out, T_rows, H, n, n_real, eps)
             : (int)prism_launch(head_norm_gate_kernel<bf16>, grid, dim3(256), 0, s, pdl != 0, (const float*)o,
                                 proj_of<bf16>(p_slabs, p_stride, p_P, p_rows, p_ld), (const bf16*)norm, (bf16*)out, T_rows, H, n, n_real, eps);
}
