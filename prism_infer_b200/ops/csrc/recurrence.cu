// Recurrent mixers with a matrix state per head, and what a layer reads of the tokens before.
//
// A sequence's state of one layer is a row of fp32 in a slot:  [heads][n][m] (key channel, value channel), then what it carries
// of the last tokens' input rows.  Every slot has two versions: a step that takes a sequence from c tokens to c' reads version
// c & 1 and writes version c' & 1, so a step that is repeated finds what it read before.  A sequence without tokens (c = 0)
// starts from zero whatever its slot holds.
//
//   token_mix_kernel      five blends of a token's row with the previous token's, and the table of a grouped projection
//   short_conv_kernel     a causal convolution over the last few rows of every channel
//   decay_project_kernel  decays of many tokens from the narrow projection's rows (bf16; fp32 takes the 32-bit GEMM)
//   state_step_kernel     one token per sequence: output, state update, norm per head, gate
//   state_scan_kernel     many tokens of a sequence: the state stays in registers, loader warps feed token blocks
//   head_norm_gate_kernel norm per head and gate behind the scan
//
// Per head, with r, k, v, a decay d and a weight b per key channel (all fp32):
//   o_t = S^T r + (b . 1) v,   S <- diag(d) S + k v^T.
// The rules (n = m in the first):
//   RULE_BONUS   r and k as projected, b = r u k, d = exp(-exp(z)): the token itself counts with the bonus u
//   RULE_FORGET  a gate f = l + (1 - l) sigmoid(z + c) per key channel decays and writes:  d = f, k = 1 - f, and with
//                q = silu(y) read behind the update r = q f, b = q k
#include "mma_sync.cuh"

#include <type_traits>

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
enum StateRule : int { RULE_BONUS = 0, RULE_FORGET = 1 };
__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
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

// The same in two steps, so that many loads are under way before the first value is needed: what memory holds, and its value.
__device__ __forceinline__ float4 raw_value(float4 r) { return r; }
__device__ __forceinline__ float4 raw_value(uint2 r) {
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&r);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  return make_float4(a.x, a.y, b.x, b.y);
}
template <typename T, bool SLABS>
struct RawProj {
  typedef typename std::conditional<SLABS || std::is_same<T, float>::value, float4, uint2>::type type;
  static __device__ __forceinline__ type zero() { return type{}; }
  static __device__ __forceinline__ type load(const Proj<T>& p, size_t row, int c) {
    if constexpr (SLABS) {
      const float* s = p.slabs + row * p.ld + c;
      float4 v = __ldcg(reinterpret_cast<const float4*>(s));
      for (int i = 1; i < p.P; ++i) {
        const float4 x = __ldcg(reinterpret_cast<const float4*>(s + (size_t)i * p.slab_stride));
        v.x += x.x;
        v.y += x.y;
        v.z += x.z;
        v.w += x.w;
      }
      return v;
    } else {
      return __ldcg(reinterpret_cast<const type*>(p.rows + row * p.ld + c));
    }
  }
};

// What RULE_FORGET makes of a channel's query y, gate z (bias added) and lower bound l.
struct Forget {
  float r, k, d, b;
};
template <typename T>
__device__ __forceinline__ Forget forget_of(float y, float z, float l) {
  float stay, q;                                  // stay: 1 - sigmoid(z), exact where the gate is all but open
  if (sizeof(T) == 2) {
    stay = __fdividef(1.0f, 1.0f + __expf(z));
    q = __fdividef(y, 1.0f + __expf(-y));
  } else {
    stay = 1.0f / (1.0f + expf(z));
    q = y / (1.0f + expf(-y));
  }
  Forget f;
  f.k = (1.0f - l) * stay;
  f.d = 1.0f - f.k;
  f.r = q * f.d;
  f.b = q * f.k;
  return f;
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

// =====================================================================================
// out_t = x_t + sum_j w_j x_(t - taps + 1 + j) on every channel, rows before the step's from the slot's carry (oldest first) and
// zeros before the sequence's start.  grid (chunks of a sequence, column blocks, sequences): a thread walks four columns through
// a chunk, two groups of rows under way while it works on a third.  A chunk is no shorter than the rows that are carried on, so only
// a sequence's first one reads the carry: it writes the new one too, after it has read the old (both may be the same version).  MT:
// taps, rounded up.
// =====================================================================================
constexpr int CONV_MIN_CHUNK = 16, CONV_THREADS = 128;
template <typename T>
struct ConvArgs {
  StateArgs st;            // x is not used
  const T* x;              // [T][W]
  const T* w;              // [taps][W]
  T* out;                  // [T][W]
  int taps, chunk;
};

// Four columns as two packed pairs.
struct Pairs {
  unsigned long long lo, hi;
};
__device__ __forceinline__ Pairs pairs_of(float4 v) { return Pairs{pair_of(v.x, v.y), pair_of(v.z, v.w)}; }

template <typename T, int MT>
__global__ void __launch_bounds__(CONV_THREADS, MT <= 4 ? 5 : 2) short_conv_kernel(const ConvArgs<T> a) {
  constexpr int ROWS = MT <= 4 && sizeof(T) == 2 ? 8 : 4;
  using Raw = RawProj<T, false>;
  using RawT = typename Raw::type;
  const int W = a.st.W, s = blockIdx.z, c = (blockIdx.y * CONV_THREADS + threadIdx.x) * 4, i0 = blockIdx.x * a.chunk;
  pdl_launch_dependents();
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  Pairs w[MT], h[MT];                             // aligned at the end: tap MT - 1 meets the row itself, whose one it takes in
#pragma unroll
  for (int k = 0; k < MT; ++k) {
    float4 v = k >= MT - a.taps && c < W ? load4(a.w + (size_t)(k - (MT - a.taps)) * W + c) : zero;
    if (k == MT - 1) v = make_float4(1.0f + v.x, 1.0f + v.y, 1.0f + v.z, 1.0f + v.w);
    w[k] = pairs_of(v);
  }
  const Span sp = span_of(a.st, s);
  if (i0 >= sp.len || c >= W) return;             // a row without a slot has a carry of zeros
  pdl_wait();
  const T* x = a.x + (size_t)sp.first * W + c;
  const int keep = a.taps - 1, n = min(a.chunk, sp.len - i0);
  const T* src = x + (size_t)i0 * W;              // the next row to fetch
  T* dst = a.out + (size_t)(sp.first + i0) * W + c;
  RawT raw[2][ROWS];
  auto fetch = [&](RawT (&r)[ROWS], int from) {
    if (from + ROWS <= n) {
#pragma unroll
      for (int q = 0; q < ROWS; ++q, src += W) r[q] = *reinterpret_cast<const RawT*>(src);
    } else {
#pragma unroll
      for (int q = 0; q < ROWS; ++q, src += W) r[q] = from + q < n ? *reinterpret_cast<const RawT*>(src) : Raw::zero();
    }
  };
  fetch(raw[0], 0);
#pragma unroll
  for (int k = 0; k < MT - 1; ++k) {
    const int p = i0 - (MT - 1) + k;              // row within the step's part of the sequence
    float4 v = zero;
    if (k >= MT - a.taps) {
      if (p >= 0) v = load4(x + (size_t)p * W);
      else if (sp.old_version) v = load4(sp.old_version + a.st.carry + (size_t)(keep + p) * W + c);
    }
    h[k] = pairs_of(v);
  }
  if (i0 == 0 && sp.new_version) {
    float* carry = sp.new_version + a.st.carry + c;
    float4 v[MT];
#pragma unroll
    for (int k = 0; k < MT - 1; ++k) {            // all of it is read before any of it is written
      const int p = sp.len - (MT - 1) + k;
      v[k] = zero;
      if (k < MT - a.taps) continue;
      if (p >= 0) v[k] = load4(x + (size_t)p * W);
      else if (sp.old_version) v[k] = load4(sp.old_version + a.st.carry + (size_t)(keep + p) * W + c);
    }
#pragma unroll
    for (int k = 0; k < MT - 1; ++k)
      if (k >= MT - a.taps) store4(carry + (size_t)(k - (MT - a.taps)) * W, v[k]);
  }
  fetch(raw[1], ROWS);
  auto row = [&](RawT r, bool live) {
    h[MT - 1] = pairs_of(raw_value(r));
    Pairs o{mul2(w[0].lo, h[0].lo), mul2(w[0].hi, h[0].hi)};
#pragma unroll
    for (int k = 1; k < MT; ++k) {
      o.lo = fma2(w[k].lo, h[k].lo, o.lo);
      o.hi = fma2(w[k].hi, h[k].hi, o.hi);
    }
#pragma unroll
    for (int k = 0; k < MT - 1; ++k) h[k] = h[k + 1];
    const float2 l = unpair(o.lo), u = unpair(o.hi);
    if (live) store4(dst, make_float4(l.x, l.y, u.x, u.y));
    dst += W;
  };
  auto work = [&](const RawT (&r)[ROWS], int from) {
    if (from + ROWS <= n) {
#pragma unroll
      for (int q = 0; q < ROWS; ++q) row(r[q], true);
    } else {
#pragma unroll
      for (int q = 0; q < ROWS; ++q) row(r[q], from + q < n);
    }
  };
  for (int from = 0; from < n; from += 2 * ROWS) {
    work(raw[0], from);
    fetch(raw[0], from + 2 * ROWS);
    work(raw[1], from + ROWS);
    fetch(raw[1], from + 3 * ROWS);
  }
}

// =====================================================================================
// decay[t][c] = exp(-exp(w0[c] + W2[c] . tanh(z_t))), the narrow rows z summed on the way in.  A CTA makes 64 tokens x
// `tiles` times 128 channels; tanh(z) enters the products as the sum of two bf16 numbers, so that only the weights' own rounding is left.
// =====================================================================================
constexpr int DP_TOKENS = 64, DP_COLS = 128, DP_K = 128;
struct DecayArgs {
  const float* z;          // [P][T][ld] slabs whose sum is the narrow projection
  long long stride, ld;
  int P;
  const bf16* w2;          // [C][R]
  const bf16* w0;          // [C]
  float* out;              // [T][C]
  int T, C, R, tiles;
};

// Place of a block's thread in a matrix of `groups` groups per row, 256 places on with every step.
struct Walk {
  int row, group, groups, rows_on, groups_on;
  __device__ __forceinline__ Walk(int i, int groups_) : row(i / groups_), group(i % groups_), groups(groups_), rows_on(256 / groups_), groups_on(256 % groups_) {}
  __device__ __forceinline__ void next() {
    row += rows_on;
    group += groups_on;
    if (group >= groups) {
      group -= groups;
      ++row;
    }
  }
};
// With the hardware's exponential: absolute errors of a few 2^-23.
__device__ __forceinline__ float tanh_exp(float x) { return 1.0f - __fdividef(2.0f, __expf(2.0f * x) + 1.0f); }
__device__ __forceinline__ float decay_fast(float x) { return __expf(-__expf(x)); }

__global__ void __launch_bounds__(256, 3) decay_project_kernel(const DecayArgs a) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int LD = min(DP_K, a.R) + 8;
  bf16* hi_s = reinterpret_cast<bf16*>(smem_raw);               // [64][LD]
  bf16* lo_s = hi_s + DP_TOKENS * LD;
  bf16* w_s = lo_s + DP_TOKENS * LD;                            // [128][LD]
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, t0 = blockIdx.y * DP_TOKENS;
  const int wt = (warp & 3) * 16, wc = (warp >> 2) * 64;        // the warp's tokens and channels
  pdl_launch_dependents();
  for (int tile = 0; tile < a.tiles; ++tile) {
    const int c0 = (blockIdx.x * a.tiles + tile) * DP_COLS;
    if (c0 >= a.C) break;
    float acc[8][4] = {};
    for (int k0 = 0; k0 < a.R; k0 += DP_K) {
      const int kn = min(DP_K, a.R - k0);                         // a multiple of 16
      if (tile + k0 > 0) __syncthreads();
      Walk w(tid, kn / 8);
      while (w.row < DP_COLS) {                   // four groups at a time, all their loads first
        uint4 v[4];
        int at[4];
#pragma unroll
        for (int q = 0; q < 4; ++q, w.next()) {
          at[q] = w.row < DP_COLS ? w.row * LD + w.group * 8 : -1;
          v[q] = __ldg(reinterpret_cast<const uint4*>(a.w2 + (size_t)min(c0 + w.row, a.C - 1) * a.R + k0 + w.group * 8));
        }
#pragma unroll
        for (int q = 0; q < 4; ++q)
          if (at[q] >= 0) *reinterpret_cast<uint4*>(w_s + at[q]) = v[q];   // channels past the end are not stored
      }
      if (tile + k0 == 0) pdl_wait();             // the weights do not depend on the previous kernel
      Walk z(tid, kn / 4);
      while ((tile == 0 || a.R > DP_K) && z.row < DP_TOKENS) {
        float4 v[4];
        int at[4];
        size_t src[4];
#pragma unroll
        for (int q = 0; q < 4; ++q, z.next()) {
          at[q] = z.row < DP_TOKENS ? z.row * LD + z.group * 4 : -1;
          src[q] = (size_t)min(t0 + z.row, a.T - 1) * a.ld + k0 + z.group * 4;   // rows past the end are not stored
          v[q] = make_float4(0.f, 0.f, 0.f, 0.f);
        }
#pragma unroll 2
        for (int p = 0; p < a.P; ++p) {
          const float* slab = a.z + (size_t)p * a.stride;
#pragma unroll
          for (int q = 0; q < 4; ++q) {
            const float4 x = __ldcg(reinterpret_cast<const float4*>(slab + src[q]));
            v[q].x += x.x;
            v[q].y += x.y;
            v[q].z += x.z;
            v[q].w += x.w;
          }
        }
#pragma unroll
        for (int q = 0; q < 4; ++q) {
          if (at[q] < 0) continue;
          const float4 x = make_float4(tanh_exp(v[q].x), tanh_exp(v[q].y), tanh_exp(v[q].z), tanh_exp(v[q].w));
          const float4 h = make_float4(bf16_round(x.x), bf16_round(x.y), bf16_round(x.z), bf16_round(x.w));
          store4(hi_s + at[q], h);
          store4(lo_s + at[q], make_float4(x.x - h.x, x.y - h.y, x.z - h.z, x.w - h.w));
        }
      }
      __syncthreads();
      const bf16* hp = hi_s + (wt + (lane & 15)) * LD + 8 * (lane >> 4);
      const bf16* lp = lo_s + (wt + (lane & 15)) * LD + 8 * (lane >> 4);
      const bf16* wp = w_s + (wc + (lane & 7) + 8 * (lane >> 4)) * LD + 8 * ((lane >> 3) & 1);
      for (int k = 0; k < kn; k += 16) {
        uint32_t h[4], l[4];
        ldsm_x4(h, smem_u32(hp + k));
        ldsm_x4(l, smem_u32(lp + k));
#pragma unroll
        for (int n = 0; n < 8; n += 2) {
          uint32_t b[4];
          ldsm_x4(b, smem_u32(wp + n * 8 * LD + k));
          mma_bf16(acc[n], h, b[0], b[1]);
          mma_bf16(acc[n], l, b[0], b[1]);
          mma_bf16(acc[n + 1], h, b[2], b[3]);
          mma_bf16(acc[n + 1], l, b[2], b[3]);
        }
      }
    }
#pragma unroll
    for (int n = 0; n < 8; ++n) {
      const int c = c0 + wc + n * 8 + (lane & 3) * 2;             // C is a multiple of 16
      if (c >= a.C) continue;
      const float b0 = to_f(a.w0[c]), b1 = to_f(a.w0[c + 1]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int t = t0 + wt + (lane >> 2) + 8 * e;
        if (t < a.T)
          *reinterpret_cast<float2*>(a.out + (size_t)t * a.C + c) = make_float2(decay_fast(acc[n][2 * e] + b0), decay_fast(acc[n][2 * e + 1] + b1));
      }
    }
  }
}

// out = tanh of the summed rows, fp32
__global__ void __launch_bounds__(256) tanh_f32_kernel(const Proj<float> z, float* out, int R, long long total) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
  if (i < total) out[i] = tanhf(proj1(z, (size_t)(i / R), (int)(i % R)));
}

// =====================================================================================
// One token per sequence.  grid (heads, sequences), NT threads.  Thread (ty, tx) owns value columns 4 tx .. 4 tx + 3 of key
// rows ty, ty + rows, ...; up to NV of its state elements (float4) are fetched before the previous kernel has finished:
// they were written by an earlier step.
// =====================================================================================
template <typename T>
struct StepArgs {
  StateArgs st;
  // RULE_BONUS: r, k, v, gate, rows m * tokens + t, columns head * n.  RULE_FORGET: a row per token, [queries | gates | values].
  Proj<T> p;
  Proj<T> w1;              // [tokens][rank] input of the decay's second projection, before tanh
  const T* w2;             // [heads * n][rank]
  const T* w0;             // [heads * n] decays' offsets; RULE_FORGET: gates' bias
  const T* u;              // [heads * n] bonus; RULE_FORGET: lower bounds
  const T* norm;           // [heads * m]; RULE_FORGET: [m], for every head
  T* out;                  // [tokens][heads * m]
  int tokens, H, n, m, m_real, rank;
  float eps;
};

template <typename T, int NV, int NT, int RULE>
__global__ void __launch_bounds__(NT, NV > 8 ? 1 : (NT == 128 ? 7 : 3)) state_step_kernel(const StepArgs<T> a) {
  extern __shared__ float sm[];
  const int n = a.n, m = a.m, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, h = blockIdx.x, s = blockIdx.y;
  float *r_s = sm, *k_s = sm + n, *d_s = sm + 2 * n, *b_s = sm + 3 * n, *v_s = sm + 4 * n, *g_s = v_s + m, *t_s = g_s + m;
  float* o_s = t_s + a.rank;                      // [rows][m] partial outputs
  __shared__ float red[NT / 32];
  const int c4 = m >> 2, rows = NT / c4, tx = tid % c4, ty = tid / c4;
  pdl_launch_dependents();
  const Span sp = span_of(a.st, s);
  const size_t C = (size_t)a.H * m, hn = (size_t)h * n, hm = (size_t)h * m;
  T* out = a.out + (size_t)s * C + hm;
  if (sp.new_version == nullptr) {
    pdl_wait();
    for (int c = tid; c < m; c += NT) put(out + c, 0.0f);
    return;
  }
  const float* old_s = sp.old_version ? sp.old_version + (size_t)h * n * m : nullptr;
  float* new_s = sp.new_version + (size_t)h * n * m;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const bool active = ty < rows;
  float4 S[NV > 0 ? NV : 1];
  if (NV > 0) {
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int key = ty + i * rows;
      S[i] = active && key < n && old_s ? __ldcs(reinterpret_cast<const float4*>(old_s + (size_t)key * m) + tx) : zero;
    }
  }
  if (RULE == RULE_BONUS) {
    for (int i = tid * 128; i < n * a.rank * (int)sizeof(T); i += NT * 128)   // the head's rows of the decay projection
      asm volatile("prefetch.global.L2 [%0];" ::"l"(reinterpret_cast<const char*>(a.w2 + hn * a.rank) + i));
    pdl_wait();
    // the projections' sums, and the narrow one's tanh
    for (int i = tid; i < 4 * c4 + a.rank; i += NT) {
      if (i < 4 * c4) {
        const int q = i / c4, c = (i - q * c4) * 4;
        float* dst = q == 0 ? r_s : (q == 1 ? k_s : (q == 2 ? v_s : g_s));
        store4(dst + c, proj4(a.p, (size_t)q * a.tokens + s, (int)hm + c));
      } else {
        t_s[i - 4 * c4] = tanhf(proj1(a.w1, (size_t)s, i - 4 * c4));
      }
    }
    __syncthreads();
    // decay and bonus: eight lanes per channel over the rank
#pragma unroll 4
    for (int c0 = 0; c0 < n; c0 += NT / 8) {
      const int c = c0 + (tid >> 3);
      float z = 0.0f;
      if (c < n)
        for (int j = (tid & 7) * 4; j < a.rank; j += 32) {
          const float4 w = load4(a.w2 + (hn + c) * a.rank + j), t = load4(t_s + j);
          z += w.x * t.x + w.y * t.y + w.z * t.z + w.w * t.w;
        }
      z += __shfl_xor_sync(0xffffffffu, z, 1);
      z += __shfl_xor_sync(0xffffffffu, z, 2);
      z += __shfl_xor_sync(0xffffffffu, z, 4);
      if (c < n && (tid & 7) == 0) {
        d_s[c] = decay_of(z + to_f(a.w0[hn + c]));
        b_s[c] = r_s[c] * to_f(a.u[hn + c]) * k_s[c];
      }
    }
  } else {
    pdl_wait();
    const int n4 = n >> 2, Hn = a.H * n;
    for (int i = tid; i < n4 + c4; i += NT) {
      if (i < n4) {
        const int c = i * 4;
        const float4 y = proj4(a.p, (size_t)s, (int)hn + c), z = proj4(a.p, (size_t)s, Hn + (int)hn + c);
        const float4 bias = load4(a.w0 + hn + c), low = load4(a.u + hn + c);
        const Forget f[4] = {forget_of<float>(y.x, z.x + bias.x, low.x), forget_of<float>(y.y, z.y + bias.y, low.y),
                             forget_of<float>(y.z, z.z + bias.z, low.z), forget_of<float>(y.w, z.w + bias.w, low.w)};
        store4(r_s + c, make_float4(f[0].r, f[1].r, f[2].r, f[3].r));
        store4(k_s + c, make_float4(f[0].k, f[1].k, f[2].k, f[3].k));
        store4(d_s + c, make_float4(f[0].d, f[1].d, f[2].d, f[3].d));
        store4(b_s + c, make_float4(f[0].b, f[1].b, f[2].b, f[3].b));
      } else {
        const int c = (i - n4) * 4;
        store4(v_s + c, proj4(a.p, (size_t)s, 2 * Hn + (int)hm + c));
      }
    }
  }
  __syncthreads();
  if (active) {
    const float4 v = load4(v_s + 4 * tx);
    float4 o = zero;
    auto step = [&](int key, float4 st) {
      const float r = r_s[key], k = k_s[key], d = d_s[key], b = b_s[key];
      o.x = fmaf(b, v.x, fmaf(r, st.x, o.x));
      o.y = fmaf(b, v.y, fmaf(r, st.y, o.y));
      o.z = fmaf(b, v.z, fmaf(r, st.z, o.z));
      o.w = fmaf(b, v.w, fmaf(r, st.w, o.w));
      __stcs(reinterpret_cast<float4*>(new_s + (size_t)key * m) + tx,
             make_float4(fmaf(d, st.x, k * v.x), fmaf(d, st.y, k * v.y), fmaf(d, st.z, k * v.z), fmaf(d, st.w, k * v.w)));
    };
    if (NV > 0) {
#pragma unroll
      for (int i = 0; i < NV; ++i)
        if (ty + i * rows < n) step(ty + i * rows, S[i]);
    } else {
#pragma unroll 8
      for (int key = ty; key < n; key += rows) step(key, old_s ? __ldcs(reinterpret_cast<const float4*>(old_s + (size_t)key * m) + tx) : zero);
    }
    store4(o_s + (size_t)ty * m + 4 * tx, o);
  }
  if (RULE == RULE_BONUS)                         // the last token's row, a share per head
    for (int c = (h * NT + tid) * 4; c < a.st.W; c += a.H * NT * 4)
      store4(sp.new_version + a.st.carry + c, load4(a.st.x + (size_t)s * a.st.W + c));
  __syncthreads();
  float ss = 0.0f;
  for (int c = tid; c < m; c += NT) {
    float o = 0.0f;
#pragma unroll 8
    for (int i = 0; i < rows; ++i) o += o_s[(size_t)i * m + c];
    o_s[c] = o;                                   // column c is this thread's
    ss += o * o;
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  ss = warp_sum(lane < NT / 32 ? red[lane] : 0.0f);
  const float inv = 1.0f / sqrtf(ss / (float)a.m_real + a.eps);
  for (int c = tid; c < m; c += NT) {
    const float o = o_s[c] * inv * to_f(a.norm[RULE == RULE_BONUS ? hm + c : c]);
    put(out + c, RULE == RULE_BONUS ? o * silu_f(g_s[c]) : o);
  }
}

// =====================================================================================
// Many tokens per sequence.  grid (heads x column blocks of 32, sequences).  Four warps hold the state: a lane owns KL keys of
// four value columns, sixteen lanes the keys of a column, so that a token costs a lane three 16-byte shared-memory reads per
// four keys and one for the values; the lanes' partial outputs of four tokens are summed by one reduce-scatter.  Four more
// warps feed blocks of TB tokens: while a block is worked on they turn the next one's raw rows, already in registers, into
// what the products need (fp32, the scalar b . 1 per token) and fetch rows of the blocks behind it.
// =====================================================================================
constexpr int SCAN_COLS = 32;
constexpr int SCAN_THREADS = 256;

template <typename T>
struct ScanArgs {
  StateArgs st;
  Proj<T> p;               // RULE_BONUS: r, k, v, rows m * tokens + t.  RULE_FORGET: a row per token, [queries | gates | values]
  const float* d;          // [tokens][heads * n] decays (RULE_BONUS)
  const T* u;              // [heads * n] bonus; RULE_FORGET: lower bounds
  const T* bias;           // [heads * n] of the gates (RULE_FORGET)
  float* o;                // [tokens][heads * m]
  int tokens, H, n, m;
};

template <int KL>
struct ScanTile {
  static constexpr int TB = KL == 4 ? 32 : 16;                  // tokens of a block
  static constexpr int NP = 16 * KL;                            // keys, padded to the lanes' share
  static constexpr int G = NP / 4;                              // groups of four keys
  static constexpr int ITEMS = TB * G / 128;                    // (token, group) items of a loader thread
  static constexpr int PARTS = G > 32 ? G / 32 : 1;             // warps that share a token's bonus
  static constexpr int K = TB * NP, D = 2 * TB * NP, V = 3 * TB * NP, BONUS = V + TB * SCAN_COLS;
  static constexpr int FLOATS = BONUS + TB * PARTS;             // one buffer: [r | k | d][TB][NP], v [TB][32], bonus
};

template <typename T, int KL, bool SLABS, int RULE>
__global__ void __launch_bounds__(SCAN_THREADS) state_scan_kernel(const ScanArgs<T> a) {
  extern __shared__ __align__(16) float sm[];                   // two buffers, then outputs [2][TB][32]
  using Tile = ScanTile<KL>;
  constexpr int TB = Tile::TB, NP = Tile::NP, G = Tile::G, ITEMS = Tile::ITEMS;
  const int n = a.n, m = a.m, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int blocks = (m + SCAN_COLS - 1) / SCAN_COLS, h = blockIdx.x / blocks, col0 = blockIdx.x % blocks * SCAN_COLS, s = blockIdx.y;
  float* out_s = sm + 2 * Tile::FLOATS;
  pdl_launch_dependents();
  const Span sp = span_of(a.st, s);
  const size_t C = (size_t)a.H * m, D = (size_t)a.H * n, hc = (size_t)h * n, hm = (size_t)h * m;
  pdl_wait();
  if (sp.len <= 0) return;
  const int nb = (sp.len + TB - 1) / TB;
  if (sp.new_version == nullptr) {                // no slot: outputs are zero
    for (int i = threadIdx.x; i < sp.len * SCAN_COLS; i += SCAN_THREADS)
      if (col0 + i % SCAN_COLS < m) a.o[(size_t)(sp.first + i / SCAN_COLS) * C + hm + col0 + i % SCAN_COLS] = 0.0f;
    return;
  }
  if (warp >= 4) {
    // ------------------------------ loaders ------------------------------
    const int tid = threadIdx.x - 128, g = tid % G, c = g * 4;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool in = c < n;
    const float4 u = in ? load4(a.u + hc + c) : zero, bias = RULE == RULE_FORGET && in ? load4(a.bias + hc + c) : zero;
    const int vi = tid >> 3, vc = (tid & 7) * 4;                // a token in sixteen, a group of value columns
    const bool v_in = col0 + vc < m;
    using Raw = RawProj<T, SLABS>;
    struct Rows {                                               // of one block (k: the gates under RULE_FORGET)
      typename Raw::type r[ITEMS], k[ITEMS], v[TB / 16];
      float4 d[RULE == RULE_BONUS ? ITEMS : 1];
    };
    constexpr int AHEAD = ITEMS <= 4 ? 2 : 1;                   // blocks held in registers
    Rows held[AHEAD];
    auto fetch = [&](Rows& x, int b) {
      if (b >= nb) return;
#pragma unroll
      for (int q = 0; q < ITEMS; ++q) {
        const int tok = b * TB + tid / G + q * (128 / G);
        x.r[q] = x.k[q] = Raw::zero();
        if constexpr (RULE == RULE_BONUS) {
          x.d[q] = zero;
          if (tok >= sp.len) x.d[q].x = x.d[q].y = x.d[q].z = x.d[q].w = 1.0f;   // past the end: no decay, nothing added
        }
        if (tok < sp.len && in) {
          const size_t t = (size_t)(sp.first + tok);
          x.r[q] = Raw::load(a.p, t, (int)hc + c);
          if constexpr (RULE == RULE_BONUS) {
            x.k[q] = Raw::load(a.p, (size_t)a.tokens + t, (int)hc + c);
            x.d[q] = __ldcg(reinterpret_cast<const float4*>(a.d + t * D + hc + c));
          } else {
            x.k[q] = Raw::load(a.p, t, (int)(D + hc) + c);
          }
        }
      }
#pragma unroll
      for (int q = 0; q < TB / 16; ++q) {
        const int tok = b * TB + vi + 16 * q;
        const size_t row = RULE == RULE_BONUS ? (size_t)2 * a.tokens + sp.first + tok : (size_t)(sp.first + tok);
        x.v[q] = v_in && tok < sp.len ? Raw::load(a.p, row, (int)(RULE == RULE_BONUS ? hm : 2 * D + hm) + col0 + vc) : Raw::zero();
      }
    };
    auto store = [&](const Rows& x, int b) {
      if (b >= nb) return;
      float* dst = sm + (b & 1) * Tile::FLOATS;
#pragma unroll
      for (int q = 0; q < ITEMS; ++q) {
        const int i = tid / G + q * (128 / G);
        const float4 rq = raw_value(x.r[q]), kq = raw_value(x.k[q]);
        float bonus;
        if constexpr (RULE == RULE_BONUS) {
          store4(dst + i * NP + c, rq);
          store4(dst + Tile::K + i * NP + c, kq);
          store4(dst + Tile::D + i * NP + c, x.d[q]);
          bonus = rq.x * u.x * kq.x + rq.y * u.y * kq.y + rq.z * u.z * kq.z + rq.w * u.w * kq.w;
        } else {
          // past the sequence's end, and in columns past the head's: no decay, nothing added
          const bool live = in && b * TB + i < sp.len;
          const float4 low = live ? u : make_float4(1.f, 1.f, 1.f, 1.f);
          const Forget f[4] = {forget_of<T>(rq.x, kq.x + bias.x, low.x), forget_of<T>(rq.y, kq.y + bias.y, low.y),
                               forget_of<T>(rq.z, kq.z + bias.z, low.z), forget_of<T>(rq.w, kq.w + bias.w, low.w)};
          store4(dst + i * NP + c, make_float4(f[0].r, f[1].r, f[2].r, f[3].r));
          store4(dst + Tile::K + i * NP + c, make_float4(f[0].k, f[1].k, f[2].k, f[3].k));
          store4(dst + Tile::D + i * NP + c, make_float4(f[0].d, f[1].d, f[2].d, f[3].d));
          bonus = f[0].b + f[1].b + f[2].b + f[3].b;
        }
#pragma unroll
        for (int o = (G < 32 ? G : 32) / 2; o > 0; o >>= 1) bonus += __shfl_xor_sync(0xffffffffu, bonus, o);
        if (g % 32 == 0) dst[Tile::BONUS + i * Tile::PARTS + g / 32] = bonus;
      }
#pragma unroll
      for (int q = 0; q < TB / 16; ++q) store4(dst + Tile::V + (vi + 16 * q) * SCAN_COLS + vc, raw_value(x.v[q]));
    };
#pragma unroll
    for (int e = 0; e < AHEAD; ++e) fetch(held[e], e);
    store(held[0], 0);
    fetch(held[0], AHEAD);
    __syncthreads();
    for (int b0 = 0; b0 < nb; b0 += AHEAD) {
#pragma unroll
      for (int e = 0; e < AHEAD; ++e) {
        const int b = b0 + e;
        if (b >= nb) break;
        store(held[(e + 1) % AHEAD], b + 1);
        fetch(held[(e + 1) % AHEAD], b + 1 + AHEAD);
        __syncthreads();
      }
    }
    if (RULE == RULE_BONUS) {                     // the last token's row, a share per CTA
      const float* last = a.st.x + (size_t)(sp.first + sp.len - 1) * a.st.W;
      for (int i = (blockIdx.x * 128 + tid) * 4; i < a.st.W; i += gridDim.x * 512) store4(sp.new_version + a.st.carry + i, load4(last + i));
    }
    return;
  }
  // ------------------------------ state ------------------------------
  const int kl = lane & 15, col = warp * 8 + (lane >> 4) * 4;    // first of the lane's columns in the block
  const bool live = col0 + col < m;
  unsigned long long S[KL / 2][4];                // keys 64 g + 4 kl + {0, 1}, {2, 3}
  {
    const float* src = sp.old_version ? sp.old_version + (size_t)h * n * m + col0 + col : nullptr;
#pragma unroll
    for (int p = 0; p < KL / 2; ++p) {
      const int key = 64 * (p >> 1) + 4 * kl + 2 * (p & 1);
      float4 lo = make_float4(0.f, 0.f, 0.f, 0.f), hi = lo;
      if (live && src && key < n) {               // n is a multiple of 16
        lo = load4(src + (size_t)key * m);
        hi = load4(src + (size_t)(key + 1) * m);
      }
      S[p][0] = pair_of(lo.x, hi.x);
      S[p][1] = pair_of(lo.y, hi.y);
      S[p][2] = pair_of(lo.z, hi.z);
      S[p][3] = pair_of(lo.w, hi.w);
    }
  }
  __syncthreads();
  for (int b = 0; b < nb; ++b) {
    const float* __restrict__ src = sm + (b & 1) * Tile::FLOATS;
    const float* __restrict__ rp = src + 4 * kl;
    const int cnt = min(TB, sp.len - b * TB);
    float* __restrict__ out_b = out_s + (b & 1) * TB * SCAN_COLS;
    // partial outputs [token][column] of four tokens, and of the four before them, whose sum over the lanes goes on meanwhile
    float x[16], done[16];
    auto tokens4 = [&](int i0) {
#pragma unroll
      for (int q = 0; q < 4; ++q) {
        const int i = i0 + q;
        const float4 v = load4(src + Tile::V + i * SCAN_COLS + col);
        const unsigned long long vv[4] = {pair_of(v.x, v.x), pair_of(v.y, v.y), pair_of(v.z, v.z), pair_of(v.w, v.w)};
        unsigned long long o[4];
#pragma unroll
        for (int g = 0; g < KL / 4; ++g) {
          const ulonglong2 r = *reinterpret_cast<const ulonglong2*>(rp + i * NP + 64 * g);
          const ulonglong2 k = *reinterpret_cast<const ulonglong2*>(rp + Tile::K + i * NP + 64 * g);
          const ulonglong2 d = *reinterpret_cast<const ulonglong2*>(rp + Tile::D + i * NP + 64 * g);
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            o[c] = g == 0 ? mul2(r.x, S[0][c]) : fma2(r.x, S[2 * g][c], o[c]);
            S[2 * g][c] = fma2(d.x, S[2 * g][c], mul2(k.x, vv[c]));
          }
#pragma unroll
          for (int c = 0; c < 4; ++c) {
            o[c] = fma2(r.y, S[2 * g + 1][c], o[c]);
            S[2 * g + 1][c] = fma2(d.y, S[2 * g + 1][c], mul2(k.y, vv[c]));
          }
        }
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          const float2 f = unpair(o[c]);
          x[4 * q + c] = f.x + f.y;
        }
      }
    };
    auto finish4 = [&](int i0) {                  // sixteen lanes, sixteen sums: lane kl ends up with value kl
      const int i = i0 + (kl >> 2), c = col + (kl & 3);
      float bonus = src[Tile::BONUS + i * Tile::PARTS];
#pragma unroll
      for (int e = 1; e < Tile::PARTS; ++e) bonus += src[Tile::BONUS + i * Tile::PARTS + e];
      const float v = src[Tile::V + i * SCAN_COLS + c];
#pragma unroll
      for (int m = 8; m > 0; m >>= 1) {
        const bool up = (kl & m) != 0;
#pragma unroll
        for (int e = 0; e < m; ++e) {
          const float send = up ? done[e] : done[e + m], own = up ? done[e + m] : done[e];
          done[e] = own + __shfl_xor_sync(0xffffffffu, send, m);
        }
      }
      out_b[i * SCAN_COLS + c] = fmaf(bonus, v, done[0]);
    };
    auto keep = [&]() {
#pragma unroll
      for (int e = 0; e < 16; ++e) done[e] = x[e];
    };
    tokens4(0);
    keep();
    if (cnt > TB - 4) {
#pragma unroll
      for (int i0 = 4; i0 < TB; i0 += 4) {
        tokens4(i0);
        finish4(i0 - 4);
        keep();
      }
      finish4(TB - 4);
    } else {
      int i0 = 4;
      for (; i0 < cnt; i0 += 4) {                 // tokens past the end leave the state as it is
        finish4(i0 - 4);
        tokens4(i0);
        keep();
      }
      finish4(i0 - 4);
    }
    // a warp's eight columns of the block
    __syncwarp();
    for (int i = lane >> 1; i < cnt; i += 16) {
      const int c = warp * 8 + (lane & 1) * 4;
      if (col0 + c < m) store4(a.o + (size_t)(sp.first + b * TB + i) * C + hm + col0 + c, load4(out_b + i * SCAN_COLS + c));
    }
    __syncthreads();
  }
  if (!live) return;
  float* dst = sp.new_version + (size_t)h * n * m + col0 + col;
#pragma unroll
  for (int p = 0; p < KL / 2; ++p) {
    const int key = 64 * (p >> 1) + 4 * kl + 2 * (p & 1);
    if (key >= n) continue;
    const float2 f0 = unpair(S[p][0]), f1 = unpair(S[p][1]), f2 = unpair(S[p][2]), f3 = unpair(S[p][3]);
    store4(dst + (size_t)key * m, make_float4(f0.x, f1.x, f2.x, f3.x));
    store4(dst + (size_t)(key + 1) * m, make_float4(f0.y, f1.y, f2.y, f3.y));
  }
}

// out = o / rms(o) * norm * silu(gate) per head (GATE: none, rows or slabs; without one the norm's weights are those of a head,
// for every head).  A lane holds eight columns, L lanes a head; four rows of a warp at a time.
enum GateKind : int { GATE_NONE = 0, GATE_ROWS = 1, GATE_SLABS = 2 };
template <typename T, int L, int GATE>
__global__ void __launch_bounds__(256) head_norm_gate_kernel(const float* o, const Proj<T> p, const T* norm, T* out, int tokens, int H, int n,
                                                             int n_real, float eps) {
  constexpr int ROWS = 4;
  const int lane = threadIdx.x & 31, c = (lane % L) * 8;
  const long long total = (long long)tokens * H, first = ((long long)blockIdx.x * 8 + (threadIdx.x >> 5)) * (32 / L) * ROWS + lane / L;
  pdl_launch_dependents();
  pdl_wait();
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  using Raw = RawProj<T, GATE == GATE_SLABS>;
  float4 v[ROWS][2];
  typename Raw::type g[ROWS][2];
  long long t[ROWS];
  int hc[ROWS];
  bool in[ROWS];
#pragma unroll
  for (int q = 0; q < ROWS; ++q) {
    const long long i = first + q * (32 / L);
    in[q] = i < total && c < n;
    t[q] = in[q] ? i / H : 0;
    hc[q] = in[q] ? (int)(i - t[q] * H) * n + c : 0;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      v[q][e] = in[q] ? __ldcg(reinterpret_cast<const float4*>(o + t[q] * (size_t)H * n + hc[q] + 4 * e)) : zero;
      if (GATE != GATE_NONE) g[q][e] = in[q] ? Raw::load(p, (size_t)3 * tokens + t[q], hc[q] + 4 * e) : Raw::zero();
    }
  }
#pragma unroll
  for (int q = 0; q < ROWS; ++q) {
    float ss = 0.0f;
#pragma unroll
    for (int e = 0; e < 2; ++e) ss += v[q][e].x * v[q][e].x + v[q][e].y * v[q][e].y + v[q][e].z * v[q][e].z + v[q][e].w * v[q][e].w;
#pragma unroll
    for (int x = L / 2; x > 0; x >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, x);
    const float inv = 1.0f / sqrtf(ss / (float)n_real + eps);
    if (!in[q]) continue;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const float4 w = load4(norm + (GATE != GATE_NONE ? hc[q] : c) + 4 * e), x = v[q][e];
      float4 y = make_float4(x.x * inv * w.x, x.y * inv * w.y, x.z * inv * w.z, x.w * inv * w.w);
      if (GATE != GATE_NONE) {
        const float4 z = raw_value(g[q][e]);
        y = make_float4(y.x * silu_f(z.x), y.y * silu_f(z.y), y.z * silu_f(z.z), y.w * silu_f(z.w));
      }
      store4(out + t[q] * (size_t)H * n + hc[q] + 4 * e, y);
    }
  }
}

StateArgs state_args(void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q, const void* kv_lens,
                     const void* x, int S, int W) {
  return StateArgs{(float*)state, row, num_slots, carry, (const int*)slots, (const int*)cu_q, (const int*)kv_lens, (const float*)x, S, W};
}
// W columns in each of `rows` rows that are carried on
int check_state(long long row, int num_slots, int carry, int S, int W, int rows = 1) {
  return row <= 0 || row % 4 || num_slots <= 0 || carry < 0 || carry % 4 || S <= 0 || W <= 0 || W % 8 || carry + (long long)rows * W > row ? -1 : 0;
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

template <typename T, int NV, int NT, int RULE>
int launch_step(const StepArgs<T>& a, cudaStream_t stream, bool pdl) {
  const int rows = NT / (a.m / 4);
  const size_t smem = (size_t)(4 * a.n + 2 * a.m + a.rank + rows * a.m) * sizeof(float);
  static size_t configured = 48 * 1024;
  if (int rc = allow_smem(state_step_kernel<T, NV, NT, RULE>, smem, configured)) return rc;
  return (int)prism_launch(state_step_kernel<T, NV, NT, RULE>, dim3(a.H, a.st.S), dim3(NT), smem, stream, pdl, a);
}
// As many float4s of the state per thread as its key rows need.
template <typename T, int RULE>
int launch_step_sized(const StepArgs<T>& a, cudaStream_t stream, bool pdl) {
  auto rows_of = [&](int threads) { return threads / (a.m / 4); };
  if (rows_of(128) * 8 >= a.n) return launch_step<T, 8, 128, RULE>(a, stream, pdl);
  if (rows_of(256) * 16 >= a.n) return launch_step<T, 16, 256, RULE>(a, stream, pdl);
  return launch_step<T, 0, 256, RULE>(a, stream, pdl);
}

template <typename T, int KL, bool SLABS, int RULE>
int launch_scan(const ScanArgs<T>& a, cudaStream_t stream, bool pdl) {
  const size_t smem = (size_t)(2 * ScanTile<KL>::FLOATS + 2 * ScanTile<KL>::TB * SCAN_COLS) * sizeof(float);
  static size_t configured = 48 * 1024;
  if (int rc = allow_smem(state_scan_kernel<T, KL, SLABS, RULE>, smem, configured)) return rc;
  const dim3 grid(a.H * ((a.m + SCAN_COLS - 1) / SCAN_COLS), a.st.S);
  return (int)prism_launch(state_scan_kernel<T, KL, SLABS, RULE>, grid, dim3(SCAN_THREADS), smem, stream, pdl, a);
}
template <typename T, int RULE>
int launch_scan_sized(const ScanArgs<T>& a, cudaStream_t stream, bool pdl) {
  auto sized = [&](auto slabs) -> int {
    constexpr bool SLABS = decltype(slabs)::value;
    if (a.n <= 64) return launch_scan<T, 4, SLABS, RULE>(a, stream, pdl);
    if (a.n <= 128) return launch_scan<T, 8, SLABS, RULE>(a, stream, pdl);
    return launch_scan<T, 16, SLABS, RULE>(a, stream, pdl);
  };
  return a.p.slabs ? sized(std::true_type()) : sized(std::false_type());
}

template <typename T>
int launch_conv(const StateArgs& st, const void* x, const void* w, void* out, int taps, int max_len, cudaStream_t stream, bool pdl) {
  ConvArgs<T> a{st, (const T*)x, (const T*)w, (T*)out, taps, CONV_MIN_CHUNK};
  const int across = (st.W / 4 + CONV_THREADS - 1) / CONV_THREADS;
  // longer chunks while the device stays full
  while (a.chunk < 64 && (long long)max_len / (2 * a.chunk) * across * st.S >= 6 * 148) a.chunk *= 2;
  const dim3 grid((max_len + a.chunk - 1) / a.chunk, across, st.S), block(CONV_THREADS);
  if (taps <= 4) return (int)prism_launch(short_conv_kernel<T, 4>, grid, block, 0, stream, pdl, a);
  if (taps <= 8) return (int)prism_launch(short_conv_kernel<T, 8>, grid, block, 0, stream, pdl, a);
  return (int)prism_launch(short_conv_kernel<T, 16>, grid, block, 0, stream, pdl, a);
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

// bf16: decay [T][C] fp32 = exp(-exp(w0 + W2 tanh(z))), z the sum of P fp32 slabs [T][ld] of R columns, w2 [C][R].  R and C
// multiples of 16.
PRISM_API int prism_decay_project(const void* slabs, long long slab_stride, int P, long long ld, const void* w2, const void* w0, void* out,
                                  int T, int C, int R, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (C <= 0 || C % 16 || R <= 0 || R % 16 || !slabs || P < 1 || ld % 4 || ld < R || (reinterpret_cast<uintptr_t>(w2) & 15)) return -1;
  DecayArgs a{(const float*)slabs, slab_stride, ld, P, (const bf16*)w2, (const bf16*)w0, (float*)out, T, C, R, 1};
  const int col_tiles = (C + DP_COLS - 1) / DP_COLS, token_tiles = (T + DP_TOKENS - 1) / DP_TOKENS;
  const int across = 3 * 148 / token_tiles;       // CTAs side by side: three per SM, and no second wave, where that is possible
  a.tiles = (col_tiles + (across > 1 ? across : 1) - 1) / (across > 1 ? across : 1);
  const size_t smem = (size_t)(2 * DP_TOKENS + DP_COLS) * ((R < DP_K ? R : DP_K) + 8) * sizeof(bf16);
  static size_t configured = 48 * 1024;
  if (int rc = allow_smem(decay_project_kernel, smem, configured)) return rc;
  const dim3 grid((col_tiles + a.tiles - 1) / a.tiles, token_tiles);
  return (int)prism_launch(decay_project_kernel, grid, dim3(256), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

// out [T][R] = tanh(z), fp32
PRISM_API int prism_tanh_f32(const void* slabs, long long slab_stride, int P, void* out, int T, int R, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (R <= 0 || !slabs) return -1;
  const long long total = (long long)T * R;
  return (int)prism_launch(tanh_f32_kernel, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream),
                           pdl != 0, proj_of<float>(slabs, slab_stride, P, nullptr, R), (float*)out, R, total);
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
                  (const T*)w0, (const T*)u, (const T*)norm, (T*)out, S, H, n, n, n_real, rank, eps};
    return launch_step_sized<T, RULE_BONUS>(a, s, pdl != 0);
  };
  return f32 ? run(float()) : run(bf16());
}

// The forget rule, one token per sequence: p [S][ld] = [H n queries | H n gates | H m values] as fp32 slabs or rows; bias and lower
// [H n] of the gates, norm [m]; out [S][H m].  n and m multiples of 16, at most 256.
PRISM_API int prism_forget_step(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* kv_lens, int S,
                                const void* p_slabs, long long p_stride, int p_P, const void* p_rows, long long p_ld, const void* bias,
                                const void* lower, const void* norm, void* out, int H, int n, int m, int m_real, float eps, void* stream, int pdl) {
  if (S <= 0) return 0;
  if (int rc = check_state(row, num_slots, carry, S, 8, 0)) return rc;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || m <= 0 || m % 16 || m > 256 || m_real <= 0 || m_real > m || (long long)H * n * m > carry || S > 65535) return -2;
  if ((!p_slabs && !p_rows) || p_ld % 4 || p_ld < (long long)H * (2 * n + m)) return -3;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, nullptr, kv_lens, nullptr, S, 0);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    StepArgs<T> a{st, proj_of<T>(p_slabs, p_stride, p_P, p_rows, p_ld), Proj<T>{}, nullptr, (const T*)bias, (const T*)lower, (const T*)norm, (T*)out,
                  S, H, n, m, m_real, 0, eps};
    return launch_step_sized<T, RULE_FORGET>(a, s, pdl != 0);
  };
  return f32 ? run(float()) : run(bf16());
}

// Prompts and portions.  p: r, k, v (and the gate) of all T tokens one after another; decay [T][H n] and o [T][H n] fp32.
PRISM_API int prism_state_scan(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q,
                               const void* kv_lens, const void* x, int S, int W, const void* p_slabs, long long p_stride, int p_P,
                               const void* p_rows, long long p_ld, const void* decay, const void* u, void* o, int T_rows, int H, int n,
                               void* stream, int pdl) {
  if (T_rows <= 0) return 0;
  if (int rc = check_state(row, num_slots, carry, S, W)) return rc;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || (long long)H * n * n > carry || !cu_q || S > 65535) return -2;
  if ((!p_slabs && !p_rows) || p_ld % 4) return -3;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, cu_q, kv_lens, x, S, W);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    ScanArgs<T> a{st, proj_of<T>(p_slabs, p_stride, p_P, p_rows, p_ld), (const float*)decay, (const T*)u, nullptr, (float*)o, T_rows, H, n, n};
    return launch_scan_sized<T, RULE_BONUS>(a, s, pdl != 0);
  };
  return f32 ? run(float()) : run(bf16());
}

// The forget rule over prompts and portions; p [T][ld], bias and lower as in prism_forget_step, o [T][H m] fp32.
PRISM_API int prism_forget_scan(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q,
                                const void* kv_lens, int S, const void* p_slabs, long long p_stride, int p_P, const void* p_rows, long long p_ld,
                                const void* bias, const void* lower, void* o, int T_rows, int H, int n, int m, void* stream, int pdl) {
  if (T_rows <= 0) return 0;
  if (int rc = check_state(row, num_slots, carry, S, 8, 0)) return rc;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || m <= 0 || m % 16 || m > 256 || (long long)H * n * m > carry || !cu_q || S > 65535) return -2;
  if ((!p_slabs && !p_rows) || p_ld % 4 || p_ld < (long long)H * (2 * n + m)) return -3;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, cu_q, kv_lens, nullptr, S, 0);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    ScanArgs<T> a{st, proj_of<T>(p_slabs, p_stride, p_P, p_rows, p_ld), nullptr, (const T*)lower, (const T*)bias, (float*)o, T_rows, H, n, m};
    return launch_scan_sized<T, RULE_FORGET>(a, s, pdl != 0);
  };
  return f32 ? run(float()) : run(bf16());
}

// out [T][W] = x + causal convolution of x with w [taps][W] on every channel, for prompts and portions (max_len: the most tokens of
// a sequence).  The state's carry is taps - 1 rows of W fp32, oldest first.  taps at most 16.
PRISM_API int prism_short_conv(int f32, void* state, long long row, int num_slots, int carry, const void* slots, const void* cu_q,
                               const void* kv_lens, int S, int W, const void* x, const void* w, void* out, int taps, int max_len, void* stream,
                               int pdl) {
  if (max_len <= 0) return 0;
  if (taps < 1 || taps > 16 || !cu_q || S > 65535) return -2;
  if (int rc = check_state(row, num_slots, carry, S, W, taps - 1)) return rc;
  const StateArgs st = state_args(state, row, num_slots, carry, slots, cu_q, kv_lens, nullptr, S, W);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_conv<float>(st, x, w, out, taps, max_len, s, pdl != 0) : launch_conv<bf16>(st, x, w, out, taps, max_len, s, pdl != 0);
}

// out [T][H n] = o / rms(o) * norm * silu(gate) per head; the gate is block 3 of p.  Without p: no gate, and norm
// [n] holds for every head.
PRISM_API int prism_head_norm_gate(int f32, const void* o, const void* p_slabs, long long p_stride, int p_P, const void* p_rows,
                                   long long p_ld, const void* norm, void* out, int T_rows, int H, int n, int n_real, float eps,
                                   void* stream, int pdl) {
  if (T_rows <= 0) return 0;
  if (H <= 0 || n <= 0 || n % 16 || n > 256 || n_real <= 0 || n_real > n || p_ld % 4) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type, auto lanes) -> int {
    using T = decltype(type);
    constexpr int L = decltype(lanes)::value, PER_CTA = 8 * (32 / L) * 4;
    const dim3 grid((unsigned)(((long long)T_rows * H + PER_CTA - 1) / PER_CTA));
    auto* kernel = p_slabs ? head_norm_gate_kernel<T, L, GATE_SLABS> : (p_rows ? head_norm_gate_kernel<T, L, GATE_ROWS> : head_norm_gate_kernel<T, L, GATE_NONE>);
    return (int)prism_launch(kernel, grid, dim3(256), 0, s, pdl != 0,
                             (const float*)o, proj_of<T>(p_slabs, p_stride, p_P, p_rows, p_ld), (const T*)norm, (T*)out, T_rows, H, n, n_real, eps);
  };
  auto sized = [&](auto type) -> int {
    if (n <= 32) return run(type, std::integral_constant<int, 4>());
    if (n <= 64) return run(type, std::integral_constant<int, 8>());
    if (n <= 128) return run(type, std::integral_constant<int, 16>());
    return run(type, std::integral_constant<int, 32>());
  };
  return f32 ? sized(float()) : sized(bf16());
}
