// Windowed grouped-query attention over a paged cache with one row per token,
//   row = [key heads x maps x dq | value heads x dv],
// plain (one map) or differential (two maps: every head has two queries and two keys over one value; the outputs
// are combined as (a1 - lam a2) over its root mean square, times a constant).  A query at position i sees key j when
// j <= i and (i - j < window or j < keep).  Scores may be bounded (cap tanh(s / cap)) and a sink per head may take part in
// the denominator of the softmax.
//
//   window_prepare_kernel      bias, norm over the whole query and key rows or over each head, rotation, page store (values:
//                              columns of their own, or the keys as projected), head gates
//   window_decode_kernel       one query token per sequence: mma.sync over key tiles of 64, key range split over CTAs,
//                              the last CTA of a (sequence, value head) merges the splits and combines maps / gates
//   window_prefill_tc_kernel   128 query rows on tcgen05, two softmax streams per CTA (the two maps of a head, two
//                              heads of a group, or two query tiles), key and value tiles by TMA straight from the pages
//   window_simple_kernel       any sizes, fp32 (true 32-bit) or bf16
//
// Head widths are padded with zeros to multiples of 16.
#include "mma_sync.cuh"

PRISM_DEFINE_TU_STATUS(window)

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
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
}

// =====================================================================================
// Projection outputs -> rotated queries, cache rows, gates.  One CTA per token.
// =====================================================================================
template <typename T>
struct PrepareArgs {
  const float* slabs;      // [P][T][M] fp32 (null: rows)
  long long slab_stride;
  int P;
  const T* rows;           // [T][ld]
  long long ld;
  const T* bias;           // [M] (null: none)
  const T* q_w;            // norm weights over the whole query / key row, or of one head (null: no norm)
  const T* k_w;
  const float* freq;       // [rot / 2]
  const int* positions;
  const long long* slots;  // flat slot, < 0: not stored
  long long num_slots;
  T* q_out;                // [T][nq]
  T* cache;                // [slots][nk + nv]
  float* gate;             // [T][H] (null: no gates)
  int M, nq, nk, nv, H, dq, rot, q_real, k_real;
  int v_col, gate_col;     // first column of the values and of the gates (tied values: the keys' first column)
  float eps;
  int shift;               // 2^shift unit places per map
};

template <typename T>
__device__ __forceinline__ float4 projected4(const PrepareArgs<T>& a, size_t t, int c) {
  float4 v;
  if (a.slabs != nullptr) {
    v = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* p0 = a.slabs + t * a.M + c;
#pragma unroll 4
    for (int p = 0; p < a.P; ++p) {
      const float4 s = __ldcg(reinterpret_cast<const float4*>(p0 + (size_t)p * a.slab_stride));
      v.x += s.x;
      v.y += s.y;
      v.z += s.z;
      v.w += s.w;
    }
  } else {
    v = load4(a.rows + t * a.ld + c);
  }
  if (a.bias != nullptr) {
    const float4 b = load4(a.bias + c);
    v.x += b.x;
    v.y += b.y;
    v.z += b.z;
    v.w += b.w;
  }
  return v;
}

// A unit is four columns of a map of a head and, inside the rotated part, their four partners half the rotated width on.
// Units are numbered with 2^shift places per map, so that a unit's map and place come without a division.
struct PrepareUnit {
  int c, d;      // column of q | k (< 0: an unused place), and inside the map
  bool pair;
};
template <typename T>
__device__ __forceinline__ PrepareUnit prepare_unit(const PrepareArgs<T>& a, int u) {
  const int pairs = a.rot >> 3, map = u >> a.shift, r = u & ((1 << a.shift) - 1);
  PrepareUnit p;
  p.pair = r < pairs;
  p.d = p.pair ? r * 4 : a.rot + (r - pairs) * 4;
  p.c = p.d < a.dq && map * a.dq < a.nq + a.nk ? map * a.dq + p.d : -1;
  return p;
}
__device__ __forceinline__ float sum_sq(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 mul4(float4 v, float f, float4 w) { return make_float4(v.x * f * w.x, v.y * f * w.y, v.z * f * w.z, v.w * f * w.w); }

constexpr int PREP_PARTS = 4;
__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire.aligned;" ::: "memory"); }
__device__ __forceinline__ float cluster_load(const float* own, int rank) {
  float v;
  asm volatile(
      "{\n\t.reg .b32 a;\n\t"
      "mapa.shared::cluster.u32 a, %1, %2;\n\t"
      "ld.shared::cluster.f32 %0, [a];\n\t}"
      : "=f"(v)
      : "r"(smem_u32(own)), "r"(rank)
      : "memory");
  return v;
}

// Threads keep their first U units in registers between the norm's sum and the rotation; others are read again.
// PARTS CTAs (a cluster) per token; FEW tokens: norm weights fetched before the previous kernel has finished; HEAD: norms
// per head.  Widths whose rotated half is not a multiple of four go element by element.
template <typename T, int PARTS, bool FEW, bool HEAD>
__device__ __forceinline__ void prepare_token(const PrepareArgs<T>& a) {
  constexpr int U = 2;
  extern __shared__ float cs[];          // [rot / 2] cosines, then sines, then the heads' norm factors where they are not
                                         // formed in registers
  __shared__ float red[2][16], part_s[2];
  const size_t t = blockIdx.x / PARTS;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = a.rot >> 1;
  const int part = blockIdx.x % PARTS, tid = part * blockDim.x + threadIdx.x, nt = PARTS * blockDim.x;  // threads of the token
  pdl_launch_dependents();
  const float pos = (float)a.positions[t];
  for (int i = threadIdx.x; i < half; i += blockDim.x) sincosf(pos * a.freq[i], &cs[half + i], &cs[i]);
  const int nqk = a.nq + a.nk;
  const bool vec = (half & 3) == 0, any_norm = a.q_w != nullptr, norm = any_norm && !HEAD;
  const bool seg = HEAD && any_norm && vec && a.shift <= 5;  // the units of a head are neighbouring lanes
  const int units = vec ? (nqk / a.dq) << a.shift : 0;
  float* hinv = cs + 2 * half;
  PrepareUnit pu[U];
  float4 w_lo[FEW ? U : 1], w_hi[FEW ? U : 1];
  auto weight4 = [&](const PrepareUnit& p, int o) {
    if (HEAD) return load4((p.c < a.nq ? a.q_w : a.k_w) + p.d + o);
    return p.c < a.nq ? load4(a.q_w + p.c + o) : load4(a.k_w + p.c + o - a.nq);
  };
  // 1 / root mean square of a unit's head from the sums of squares of its units (every lane of the warp)
  auto segment_inv = [&](float ss) {
    for (int o = 1; o < 1 << a.shift; o <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    return 1.0f / sqrtf(ss / (float)a.q_real + a.eps);
  };
#pragma unroll
  for (int k = 0; k < U; ++k) {
    const int u = tid + k * nt;
    pu[k].c = -1;
    if (u < units) pu[k] = prepare_unit(a, u);
    if (FEW && any_norm && pu[k].c >= 0) {
      w_lo[k] = weight4(pu[k], 0);
      if (pu[k].pair) w_hi[k] = weight4(pu[k], half);
    }
  }
  pdl_wait();
  long long slot = a.slots[t];
  if (slot >= a.num_slots) {
    if (tid == 0) prism_report(PRISM_ERR_BOUNDS, 3);
    slot = -1;
  }
  T* page_row = slot >= 0 ? a.cache + (size_t)slot * (a.nk + a.nv) : nullptr;
  float4 lo[U], hi[U];
#pragma unroll
  for (int k = 0; k < U; ++k) {
    lo[k] = hi[k] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (pu[k].c >= 0) {
      lo[k] = projected4(a, t, pu[k].c);
      if (pu[k].pair) hi[k] = projected4(a, t, pu[k].c + half);
    }
  }
  if (page_row)
    for (int c = tid * 4; c < a.nv; c += nt * 4) store4(page_row + a.nk + c, projected4(a, t, a.v_col + c));
  if (a.gate != nullptr)
    for (int h = tid; h * 4 < a.H; h += nt) {
      const float4 v = projected4(a, t, a.gate_col + 4 * h);
      const float z[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (4 * h + e < a.H) a.gate[t * a.H + 4 * h + e] = 1.0f / (1.0f + expf(-z[e]));
    }
  float iq = 1.0f, ik = 1.0f, unit_inv[U];
  if (seg) {
#pragma unroll
    for (int k = 0; k < U; ++k) unit_inv[k] = segment_inv(sum_sq(lo[k]) + sum_sq(hi[k]));
  } else if (HEAD && any_norm) {
    for (int h = warp; h < nqk / a.dq; h += blockDim.x >> 5) {
      float ss = 0.0f;
      for (int c = lane * 4; c < a.dq; c += 128) ss += sum_sq(projected4(a, t, h * a.dq + c));
      ss = warp_sum(ss);
      if (lane == 0) hinv[h] = 1.0f / sqrtf(ss / (float)a.q_real + a.eps);
    }
  }
  if (norm) {
    float sq = 0.0f, sk = 0.0f;
    if (vec) {
#pragma unroll
      for (int k = 0; k < U; ++k) (pu[k].c < a.nq ? sq : sk) += sum_sq(lo[k]) + sum_sq(hi[k]);
      for (int u = tid + U * nt; u < units; u += nt) {
        const PrepareUnit p = prepare_unit(a, u);
        if (p.c < 0) continue;
        float ss = sum_sq(projected4(a, t, p.c));
        if (p.pair) ss += sum_sq(projected4(a, t, p.c + half));
        (p.c < a.nq ? sq : sk) += ss;
      }
    } else {
      for (int c = tid * 4; c < nqk; c += nt * 4) (c < a.nq ? sq : sk) += sum_sq(projected4(a, t, c));
    }
    sq = warp_sum(sq);
    sk = warp_sum(sk);
    if (lane == 0) {
      red[0][warp] = sq;
      red[1][warp] = sk;
    }
  }
  __syncthreads();
  if (norm) {
    const int nw = blockDim.x >> 5;
    float sq = warp_sum(lane < nw ? red[0][lane] : 0.0f), sk = warp_sum(lane < nw ? red[1][lane] : 0.0f);
    if (PARTS > 1) {                     // the parts of a token add up through distributed shared memory, in their order
      if (threadIdx.x == 0) {
        part_s[0] = sq;
        part_s[1] = sk;
      }
      __syncwarp();
      cluster_arrive();
      cluster_wait();
      sq = sk = 0.0f;
#pragma unroll
      for (int r = 0; r < PARTS; ++r) {
        sq += cluster_load(&part_s[0], r);
        sk += cluster_load(&part_s[1], r);
      }
      cluster_arrive();                  // a part leaves only after the others have read its sums
    }
    iq = 1.0f / sqrtf(sq / (float)a.q_real + a.eps);
    ik = 1.0f / sqrtf(sk / (float)a.k_real + a.eps);
  }
  auto write4 = [&](int c, float4 v) {
    if (c < a.nq) store4(a.q_out + t * a.nq + c, v);
    else if (page_row) store4(page_row + c - a.nq, v);
  };
  if (vec) {
    auto finish = [&](const PrepareUnit& p, float4 x, float4 y, float4 wx, float4 wy, float own) {
      if (any_norm) {
        const float inv = !HEAD ? (p.c < a.nq ? iq : ik) : (seg ? own : hinv[p.c / a.dq]);
        x = mul4(x, inv, wx);
        if (p.pair) y = mul4(y, inv, wy);
      }
      if (p.pair) {
        const float4 co = load4(cs + p.d), si = load4(cs + half + p.d);
        write4(p.c, make_float4(x.x * co.x - y.x * si.x, x.y * co.y - y.y * si.y, x.z * co.z - y.z * si.z, x.w * co.w - y.w * si.w));
        write4(p.c + half, make_float4(y.x * co.x + x.x * si.x, y.y * co.y + x.y * si.y, y.z * co.z + x.z * si.z, y.w * co.w + x.w * si.w));
      } else {
        write4(p.c, x);
      }
    };
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int k = 0; k < U; ++k)
      if (pu[k].c >= 0) {
        if (FEW) finish(pu[k], lo[k], hi[k], w_lo[k], w_hi[k], unit_inv[k]);
        else finish(pu[k], lo[k], hi[k], any_norm ? weight4(pu[k], 0) : zero, any_norm && pu[k].pair ? weight4(pu[k], half) : zero, unit_inv[k]);
      }
    for (int u0 = tid - (HEAD ? lane : 0) + U * nt; u0 < units; u0 += nt) {  // per head whole warps: segment_inv takes every lane
      const int u = u0 + (HEAD ? lane : 0);
      PrepareUnit p{-1, 0, false};
      if (u < units) p = prepare_unit(a, u);
      if (!HEAD && p.c < 0) continue;
      float4 x = zero, y = zero;
      if (p.c >= 0) {
        x = projected4(a, t, p.c);
        if (p.pair) y = projected4(a, t, p.c + half);
      }
      const float own = seg ? segment_inv(sum_sq(x) + sum_sq(y)) : 1.0f;
      if (p.c >= 0) finish(p, x, y, any_norm ? weight4(p, 0) : zero, any_norm && p.pair ? weight4(p, half) : zero, own);
    }
  } else {
    auto value = [&](int c) {
      const float4 v = projected4(a, t, c & ~3);
      const float f = (c & 2) ? ((c & 1) ? v.w : v.z) : ((c & 1) ? v.y : v.x);
      if (HEAD && any_norm) return f * hinv[c / a.dq] * to_f((c < a.nq ? a.q_w : a.k_w)[c % a.dq]);
      return norm ? f * (c < a.nq ? iq * to_f(a.q_w[c]) : ik * to_f(a.k_w[c - a.nq])) : f;
    };
    for (int c = tid; c < nqk; c += nt) {
      const int d = c % a.dq;
      float o = value(c);
      if (d < half) o = o * cs[d] - value(c + half) * cs[half + d];
      else if (d < a.rot) o = o * cs[d - half] + value(c - half) * cs[d];
      if (c < a.nq) put(a.q_out + t * a.nq + c, o);
      else if (page_row) put(page_row + c - a.nq, o);
    }
  }
  if (PARTS > 1 && norm) {
    __syncwarp();
    cluster_wait();
  }
}

template <typename T, bool HEAD>
__global__ void __cluster_dims__(PREP_PARTS, 1, 1) __launch_bounds__(256) window_prepare_few_kernel(const PrepareArgs<T> a) {
  prepare_token<T, PREP_PARTS, true, HEAD>(a);
}
template <typename T, bool HEAD>
__global__ void __launch_bounds__(512) window_prepare_mid_kernel(const PrepareArgs<T> a) {
  prepare_token<T, 1, true, HEAD>(a);
}
template <typename T, bool HEAD>
__global__ void __launch_bounds__(256, 4) window_prepare_kernel(const PrepareArgs<T> a) {
  prepare_token<T, 1, false, HEAD>(a);
}

// =====================================================================================
// What the attention kernels share.
// =====================================================================================
template <typename T>
struct WinArgs {
  const T* q;               // [tokens][H * maps * dq]
  const T* cache;           // [blocks][page][R]
  const int* block_tables;  // [S][max_blocks], < 0: hole
  const int* cu_q;          // [S + 1] token offsets; null: sequence s is token s
  const int* kv_lens;       // [S] keys up to and including the sequence's last token
  const float* gate;        // [tokens][H] (null: one)
  const float* sink;        // [H] (null: none); one map only
  T* out;                   // [tokens][out_ld]
  long long out_ld;
  float* part_o;            // decode partials [CTA group][nsplit][rows][dv]
  float* part_ml;           // [CTA group][nsplit][rows][2]
  int* counters;            // [CTA groups], zero-initialised, self-resetting
  int H, G, maps, dq, dv, vdim, R, page, max_blocks, num_blocks, window, keep, nsplit;
  float scale, lam, gain, eps, cap;  // cap 0: scores are not bounded
};

// cap tanh(s scale / cap) times log2(e), as 1 - 2 / (exp(2x) + 1): a = 2 scale log2(e) / cap, b = cap log2(e).  The absolute
// error is a few 2^-24 of cap.
__device__ __forceinline__ float capped_log2(float s, float a, float b) { return b - __fdividef(2.0f * b, ex2_fast(s * a) + 1.0f); }

// The same by tanh's power series up to x^9, all on the multiply-add pipe: cap tanh(x) log2(e) with x = s scale / cap.  For
// |x| < CAP_SERIES the first term left out is below 4e-7 of cap.
constexpr float CAP_SERIES = 0.4f;
struct CapSeries {
  unsigned long long a0, a1, a2, a3, a4;   // the same value in both halves
  __device__ __forceinline__ CapSeries(float scale, float cap) {
    const float x = cap > 0.0f ? scale / cap : 0.0f, q = x * x, f = cap * 1.4426950408889634f * x;
    auto both = [](float v) { return pair_of(v, v); };
    a0 = both(f);
    a1 = both(f * q * (-1.0f / 3.0f));
    a2 = both(f * q * q * (2.0f / 15.0f));
    a3 = both(f * q * q * q * (-17.0f / 315.0f));
    a4 = both(f * q * q * q * q * (62.0f / 2835.0f));
  }
  __device__ __forceinline__ void operator()(float& u, float& v) const {
    const unsigned long long s = pair_of(u, v), q = mul2(s, s);
    const float2 r = unpair(mul2(s, fma2(q, fma2(q, fma2(q, fma2(q, a4, a3), a2), a1), a0)));
    u = r.x;
    v = r.y;
  }
};

// Factor on accumulated values whose weights sum to l relative to 2^m: one over the denominator, with the sink's part in it.
__device__ __forceinline__ float softmax_factor(float l, float m, const float* sink, int h) {
  if (!(l > 0.0f)) return 0.0f;
  if (sink == nullptr) return 1.0f / l;
  const float s = sink[h] * 1.4426950408889634f;
  if (s <= m) return 1.0f / (l + ex2_fast(s - m));
  const float f = ex2_fast(m - s);
  return f / (l * f + 1.0f);
}

// Key tiles a query range [p_first, p_last] touches: the kept tiles before the window's first tile, then the window's.
struct TileList {
  int kept, first, count;
  __device__ __forceinline__ int id(int t) const { return t < kept ? t : first + t - kept; }
};
__device__ __forceinline__ TileList tile_list(int p_first, int p_last, int window, int keep, int tile) {
  TileList l;
  const int lo = window > p_first ? 0 : p_first - window + 1;
  l.first = lo / tile;
  l.kept = min((keep + tile - 1) / tile, l.first);
  l.count = p_last < 0 ? 0 : l.kept + p_last / tile - l.first + 1;
  return l;
}

// =====================================================================================
// Decode.  Rows of a CTA: up to 16 MT (head, map) pairs of one value head; a row's query sits in its own map's
// columns of a maps x dq wide row and is zero elsewhere, so both maps are scored by one product with the concatenated
// keys and weight the same values.  Each of the four warps owns 16 keys of every 64-key tile and streams their rows by
// bulk copies (one per lane: 16 key rows, 16 value rows) through its own ring; the warps meet only at the end.  Tiles
// that hold only keys of earlier steps are fetched before the previous kernel has finished.
// =====================================================================================
constexpr int DEC_TILE = 64;

// `bytes` (a multiple of 16) from global to shared memory, completing on `bar`.
__device__ __forceinline__ void bulk_row(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// KS: 16-element steps of the query kept in registers (0: read from shared memory every tile)
template <int MT, int DVT, int KS>
__global__ void __launch_bounds__(128) window_decode_kernel(const WinArgs<bf16> a, const int stages) {
  extern __shared__ __align__(128) uint8_t smem_raw[];
  const int KD = a.maps * a.dq, LDQ = KD + 8, LDR = KD + a.dv + 8;  // an odd number of 16-byte steps: no bank conflicts
  constexpr int BM = 16 * MT;
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);                   // [BM][LDQ]
  bf16* ring = q_s + BM * LDQ;                                      // [4 warps][stages][16][LDR]
  __shared__ float m_s[4][BM], l_s[4][BM], f_s[4][BM], L_s[BM], M_s[BM];
  __shared__ __align__(8) uint64_t bars[4][4];
  __shared__ int last_s;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int share = a.H / a.G, rows_all = share * a.maps, blocks = (rows_all + BM - 1) / BM;
  const int seq = blockIdx.x, kvh = blockIdx.y / blocks, rb = blockIdx.y % blocks, split = blockIdx.z;
  const int row0 = rb * BM, rows = min(BM, rows_all - row0);       // BM is a multiple of maps: heads stay whole
  const int head0 = kvh * share + row0 / a.maps;
  pdl_launch_dependents();
  const int ctx = clamp_context(a.kv_lens[seq], a.max_blocks, a.page);
  const int pos = ctx - 1;
  const TileList tl = tile_list(pos, pos, a.window, a.keep, DEC_TILE);
  const int per = (tl.count + a.nsplit - 1) / a.nsplit;
  const int tb = min(tl.count, split * per), te = min(tl.count, tb + per);
  const int* bt = a.block_tables + (size_t)seq * a.max_blocks;
  const int lo = pos - a.window;                                    // keys after lo are inside the window
  bf16* my = ring + (size_t)warp * stages * 16 * LDR;
  if (lane < stages) mbar_init(&bars[warp][lane], 1);
  fence_barrier_init();
  __syncwarp();

  auto issue = [&](int t) {                                         // this warp's 16 keys of list entry t
    if (t >= te) return;
    const int st = (t - tb) % stages, r = lane & 15;
    const int key = tl.id(t) * DEC_TILE + warp * 16 + r;
    const int blk = key < ctx ? checked_page(bt[key / a.page], a.num_blocks) : -1;
    const bool ok = blk >= 0, is_k = lane < 16;
    const unsigned live = __ballot_sync(0xffffffffu, ok) & 0xffffu;
    if (lane == 0) mbar_expect_tx(&bars[warp][st], (uint32_t)__popc(live) * (uint32_t)(KD + a.dv) * 2u);
    bf16* dst = my + ((size_t)st * 16 + r) * LDR + (is_k ? 0 : KD);
    const int n = is_k ? KD : a.dv;
    if (ok) {
      const bf16* src = a.cache + ((size_t)blk * a.page + key % a.page) * a.R + (is_k ? kvh * KD : a.G * KD + kvh * a.dv);
      fence_proxy_async();
      bulk_row(dst, src, (uint32_t)n * 2u, &bars[warp][st]);
    } else {                                                        // past the end, or a hole: zeros
      for (int c = 0; c < n; c += 8) *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
    }
  };
  // the newest key was written by the kernel before this one, all others in earlier steps
  auto is_old = [&](int t) { return t < te && tl.id(t) * DEC_TILE + DEC_TILE <= pos; };
  int ahead = 0;
  while (ahead < stages - 1 && is_old(tb + ahead)) issue(tb + ahead++);
  pdl_wait();
  while (ahead < stages - 1) issue(tb + ahead++);

  for (int i = tid; i < BM * (LDQ / 8); i += 128) {
    const int r = i / (LDQ / 8), c = (i % (LDQ / 8)) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (r < rows && c < KD) {
      const int m = (row0 + r) % a.maps, h = head0 + r / a.maps;
      if (c / a.dq == m) v = *reinterpret_cast<const uint4*>(a.q + ((size_t)seq * a.H + h) * KD + c);
    }
    *reinterpret_cast<uint4*>(q_s + r * LDQ + c) = v;
  }
  __syncthreads();

  float o[MT][DVT][4], m_run[MT][2], l_run[MT][2];
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    m_run[m][0] = m_run[m][1] = -INFINITY;
    l_run[m][0] = l_run[m][1] = 0.0f;
#pragma unroll
    for (int n = 0; n < DVT; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.0f;
  }
  const float sl2 = a.scale * 1.4426950408889634f;
  const float cap_a = a.cap > 0.0f ? 2.0f * sl2 / a.cap : 0.0f, cap_b = a.cap * 1.4426950408889634f;
  const int dvt = a.dv >> 3, ksteps = KD >> 4;
  const bf16* qp = q_s + (lane & 15) * LDQ + 8 * (lane >> 4);
  uint32_t qr[MT][KS > 0 ? KS : 1][4];
  if (KS > 0) {
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int k = 0; k < KS; ++k)
        if (k < ksteps) ldsm_x4(qr[m][k], smem_u32(qp + m * 16 * LDQ + k * 16));
  }
  for (int t = tb; t < te; ++t) {
    const int i = t - tb;
    issue(t + stages - 1);
    (void)mbar_wait(&bars[warp][i % stages], (i / stages) & 1, 51);
    __syncwarp();
    const bf16* kv = my + (size_t)(i % stages) * 16 * LDR;
    float s[MT][2][4] = {};
    const bf16* kp = kv + ((lane & 7) + 8 * (lane >> 4)) * LDR + 8 * ((lane >> 3) & 1);
    if (KS > 0) {
#pragma unroll
      for (int k = 0; k < KS; ++k)
        if (k < ksteps) {
          uint32_t kb[4];
          ldsm_x4(kb, smem_u32(kp + k * 16));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(s[m][0], qr[m][k], kb[0], kb[1]);
            mma_bf16(s[m][1], qr[m][k], kb[2], kb[3]);
          }
        }
    } else {
#pragma unroll 4
      for (int k = 0; k < ksteps; ++k) {
        uint32_t kb[4];
        ldsm_x4(kb, smem_u32(kp + k * 16));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          uint32_t qf[4];
          ldsm_x4(qf, smem_u32(qp + m * 16 * LDQ + k * 16));
          mma_bf16(s[m][0], qf, kb[0], kb[1]);
          mma_bf16(s[m][1], qf, kb[2], kb[3]);
        }
      }
    }
    const int j0 = tl.id(t) * DEC_TILE + warp * 16;
    const bool whole = j0 + 15 <= pos && (j0 > lo || j0 + 16 <= a.keep);  // every key of the warp is visible
    uint32_t pf[MT][4];
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int j = j0 + n * 8 + t4 * 2 + (e & 1);
          const bool ok = whole || (j <= pos && (j > lo || j < a.keep));
          const float z = a.cap > 0.0f ? capped_log2(s[m][n][e], cap_a, cap_b) : s[m][n][e] * sl2;
          s[m][n][e] = ok ? z : -INFINITY;
          mx[e >> 1] = fmaxf(mx[e >> 1], s[m][n][e]);
        }
      float use[2], corr[2], sum[2] = {0.0f, 0.0f};
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
        mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
        // the reference only rises when a tile exceeds it by more than 2^8: the weights stay below 256
        const float mn = mx[r] > m_run[m][r] + 8.0f ? mx[r] : m_run[m][r];
        use[r] = mn == -INFINITY ? 0.0f : mn;
        corr[r] = ex2_fast(m_run[m][r] - use[r]);  // 0 before the first visible key
        m_run[m][r] = mn;
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          s[m][n][e] = ex2_fast(s[m][n][e] - use[e >> 1]);
          sum[e >> 1] += s[m][n][e];
        }
#pragma unroll
      for (int r = 0; r < 2; ++r) l_run[m][r] = l_run[m][r] * corr[r] + sum[r];  // this thread's keys; the quad adds up at the end
      if (__any_sync(0xffffffffu, corr[0] != 1.0f || corr[1] != 1.0f)) {
#pragma unroll
        for (int n = 0; n < DVT; ++n) {
          o[m][n][0] *= corr[0];
          o[m][n][1] *= corr[0];
          o[m][n][2] *= corr[1];
          o[m][n][3] *= corr[1];
        }
      }
      pf[m][0] = pack_bf16(s[m][0][0], s[m][0][1]);
      pf[m][1] = pack_bf16(s[m][0][2], s[m][0][3]);
      pf[m][2] = pack_bf16(s[m][1][0], s[m][1][1]);
      pf[m][3] = pack_bf16(s[m][1][2], s[m][1][3]);
    }
    const bf16* vp = kv + (lane & 15) * LDR + KD + 8 * (lane >> 4);
#pragma unroll
    for (int n = 0; n < DVT; n += 2) {
      if (n < dvt) {                                                // dv is a multiple of 16: tiles come in pairs
        uint32_t vb[4];
        ldsm_x4_t(vb, smem_u32(vp + n * 8));
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          mma_bf16(o[m][n], pf[m], vb[0], vb[1]);
          mma_bf16(o[m][n + 1], pf[m], vb[2], vb[3]);
        }
      }
    }
    __syncwarp();
  }
  __syncthreads();                                                  // every row that was issued has been waited for

  // ---- the four warps meet: accumulators, maxima and sums in shared memory
  float* acc_s = reinterpret_cast<float*>(smem_raw);                // [4][BM][dv + 4]
  const int LDA = a.dv + 4;
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int row = m * 16 + g + 8 * r;
      float l = l_run[m][r];
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if (t4 == 0) {
        m_s[warp][row] = m_run[m][r];
        l_s[warp][row] = l;
      }
      if (row < rows) {
#pragma unroll
        for (int n = 0; n < DVT; ++n)
          if (n < dvt)
            *reinterpret_cast<float2*>(acc_s + ((size_t)warp * BM + row) * LDA + n * 8 + t4 * 2) = make_float2(o[m][n][2 * r], o[m][n][2 * r + 1]);
      }
    }
  __syncthreads();
  const int group = seq * gridDim.y + blockIdx.y, per_row4 = a.dv >> 2;
  const size_t base = ((size_t)group * a.nsplit + split) * BM;
  if (tid < BM) {
    float mx = -INFINITY, l = 0.0f;
#pragma unroll
    for (int v = 0; v < 4; ++v) mx = fmaxf(mx, m_s[v][tid]);
#pragma unroll
    for (int v = 0; v < 4; ++v) {
      const float f = m_s[v][tid] == -INFINITY ? 0.0f : ex2_fast(m_s[v][tid] - mx);
      f_s[v][tid] = f;
      l += l_s[v][tid] * f;
    }
    L_s[tid] = l;
    M_s[tid] = mx;
    if (a.nsplit > 1 && tid < rows) *reinterpret_cast<float2*>(a.part_ml + (base + tid) * 2) = make_float2(mx, l);
  }
  __syncthreads();
  for (int i = tid; i < rows * per_row4; i += 128) {
    const int r = i / per_row4, c = (i % per_row4) * 4;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float f = f_s[w][r];
      const float4 p = load4(acc_s + ((size_t)w * BM + r) * LDA + c);
      v.x += f * p.x;
      v.y += f * p.y;
      v.z += f * p.z;
      v.w += f * p.w;
    }
    if (a.nsplit == 1) store4(acc_s + r * LDA + c, v);              // read by this thread only
    else if (tb < te) store4(a.part_o + (base + r) * a.dv + c, v);
  }
  if (a.nsplit > 1) {
    __threadfence();
    __syncthreads();
    if (tid == 0) {
      const int old = atomicAdd(&a.counters[group], 1);
      last_s = old == a.nsplit - 1;
      if (last_s) a.counters[group] = 0;
    }
    __syncthreads();
    if (!last_s) return;
    __threadfence();
    // ---- the last CTA merges all splits: coefficients first, then independent loads
    float* coef = acc_s + BM * LDA;                                 // [BM][nsplit]
    for (int r = warp; r < rows; r += 4) {
      float2 ml = make_float2(-INFINITY, 0.0f);
      if (lane < a.nsplit) ml = __ldcg(reinterpret_cast<const float2*>(a.part_ml + (((size_t)group * a.nsplit + lane) * BM + r) * 2));
      const float mx = warp_max(ml.x);
      const float f = ml.x == -INFINITY ? 0.0f : ex2_fast(ml.x - mx);
      const float l = warp_sum(f * ml.y);
      if (lane < a.nsplit) coef[r * a.nsplit + lane] = f;
      if (lane == 0) {
        L_s[r] = l;
        M_s[r] = mx;
      }
    }
    __syncthreads();
    for (int i = tid; i < rows * per_row4; i += 128) {
      const int r = i / per_row4, c = (i % per_row4) * 4;
      float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
      const float* src = a.part_o + ((size_t)group * a.nsplit * BM + r) * a.dv + c;
#pragma unroll 8
      for (int s = 0; s < a.nsplit; ++s) {
        const float f = coef[r * a.nsplit + s];
        // an empty split's rows were never written
        const float4 p = f > 0.0f ? __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * BM * a.dv)) : make_float4(0.f, 0.f, 0.f, 0.f);
        v.x += f * p.x;
        v.y += f * p.y;
        v.z += f * p.z;
        v.w += f * p.w;
      }
      store4(acc_s + r * LDA + c, v);
    }
  }
  __syncthreads();
  // ---- combine maps, gate, store: one head per warp
  for (int hh = warp; hh < rows / a.maps; hh += 4) {
    const int r = hh * a.maps, h = head0 + hh;
    const float i1 = softmax_factor(L_s[r], M_s[r], a.sink, h);
    float f1 = i1, f2 = 0.0f, post = 1.0f;
    if (a.maps == 2) {
      f2 = L_s[r + 1] > 0.0f ? a.lam / L_s[r + 1] : 0.0f;
      float ss = 0.0f;
      for (int c = lane; c < a.dv; c += 32) {
        const float v = acc_s[r * LDA + c] * f1 - acc_s[(r + 1) * LDA + c] * f2;
        ss += v * v;
      }
      post = a.gain / sqrtf(warp_sum(ss) / (float)a.vdim + a.eps);
    }
    if (a.gate != nullptr) post *= a.gate[(size_t)seq * a.H + h];
    bf16* dst = a.out + (size_t)seq * a.out_ld + (size_t)h * a.dv;
    for (int c = lane * 2; c < a.dv; c += 64) {
      float v0 = acc_s[r * LDA + c] * f1, v1 = acc_s[r * LDA + c + 1] * f1;
      if (a.maps == 2) {
        v0 -= acc_s[(r + 1) * LDA + c] * f2;
        v1 -= acc_s[(r + 1) * LDA + c + 1] * f2;
      }
      *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16(v0 * post, v1 * post);
    }
  }
}

// =====================================================================================
// Prompts on tcgen05.  A CTA runs two streams of 128 query rows with a softmax warpgroup each:
//   two maps            the two maps of one head: own queries and keys, shared values
//   one map, even group two heads of one value head: shared keys and values
//   one map, odd group  two consecutive query tiles of one head: shared keys and values
// Warp 0 streams key and value tiles of 64 rows from the pages by TMA, one thread of warp 1 issues the MMAs of stream 0
// and one of warp 10 those of stream 1; warps 2 - 5 and 6 - 9 are the streams' softmax, one thread per query row.
//   S[s][b] = Q_s K^T (two buffers per stream), P written over S as bf16, O_s += P V with P read from TMEM.
// A tile that no row of a stream sees is skipped for that stream; every role derives the same list.
// TMEM: S 4 x 64 columns, O 2 x 128.  Every wait is bounded; on a timeout the roles unwind and TMEM is freed.
// =====================================================================================
constexpr int PT = 128;          // query rows per stream
constexpr int PKT = 64;          // keys per tile
constexpr int PRE_THREADS = 352;
constexpr int Q_ATOM = PT * 128, KV_ATOM = PKT * 128;   // bytes of a 64-column atom
constexpr int TM_O = 256;

struct PrefillArgs {
  WinArgs<bf16> w;
  int pair_heads;   // one map: streams are two heads (1) or two query tiles (0)
  int stages, box;  // ring depth; key rows per TMA box (divides the page)
  int k_maps;       // key tiles per stage (maps)
  int total_rows;   // rows of the cache: a coordinate past them reads zeros
};

__device__ __forceinline__ void named_bar(int id, int threads) {
  asm volatile("bar.sync %0, %1;" ::"r"(id), "r"(threads) : "memory");
}

template <bool CAPPED>
__global__ void __launch_bounds__(PRE_THREADS, 1)
window_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                         const __grid_constant__ CUtensorMap tmV, const PrefillArgs p) {
  extern __shared__ uint8_t pre_raw[];
  const WinArgs<bf16>& a = p.w;
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(pre_raw) + 1023) & ~uintptr_t(1023));
  const int qa = (a.dq + 63) >> 6, va = a.dv > 64 ? 2 : 1;           // 64-column atoms of a key / value head
  const int q_bytes = qa * Q_ATOM, k_bytes = qa * KV_ATOM, v_bytes = va * KV_ATOM;
  const int stage_bytes = p.k_maps * k_bytes + v_bytes;
  uint8_t* q_s = smem;                                               // [2 streams][qa][128 rows]
  uint8_t* ring = smem + 2 * q_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(ring + (size_t)p.stages * stage_bytes);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;      // [stream][buffer] MMA -> softmax
  uint64_t* p_full = bars + 5;      // [stream][buffer] softmax -> MMA, 128 arrivals
  uint64_t* pv_done = bars + 9;     // [stream][buffer] P V accumulated
  uint64_t* kv_full = bars + 13;    // [stages]
  uint64_t* kv_empty = kv_full + 4; // [stages]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(kv_empty + 4);
  float* xch = reinterpret_cast<float*>(tmem_slot + 4);              // [2][128] row sums, then [2][128] sums of squares

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int seq = blockIdx.z, qt = gridDim.x - 1 - blockIdx.x;       // late tiles first
  const int share = a.H / a.G;
  const bool tiles2 = a.maps == 1 && !p.pair_heads;                  // the streams are two query tiles
  const int head0 = p.pair_heads ? blockIdx.y * 2 : blockIdx.y, kvh = head0 / share;

  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 4; ++i) {
      mbar_init(&s_full[i], 1);
      mbar_init(&p_full[i], 128);
      mbar_init(&pv_done[i], 1);
      mbar_init(&kv_full[i], 1);
      mbar_init(&kv_empty[i], 2);
    }
    fence_barrier_init();
    tma_prefetch_desc(&tmQ);
    tma_prefetch_desc(&tmK);
    tma_prefetch_desc(&tmV);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents();
  pdl_wait();

  const int q_start = a.cu_q[seq], q_len = a.cu_q[seq + 1] - q_start;
  const int kv_len = max(clamp_context(a.kv_lens[seq], a.max_blocks, a.page), q_len);
  const int pos_off = kv_len - q_len;
  const int q0 = qt * (tiles2 ? 2 * PT : PT);
  const bool live = q0 < q_len;                                      // uniform over the CTA
  // first and last query position of each stream; a stream without rows has last < first
  const int row_0 = q0, row_1 = tiles2 ? q0 + PT : q0;
  const int pf0 = pos_off + row_0, pl0 = pos_off + min(row_0 + PT, q_len) - 1;
  const int pf1 = pos_off + row_1, pl1 = pos_off + min(row_1 + PT, q_len) - 1;
  TileList tl{0, 0, 0};
  if (live) tl = tile_list(pf0, max(pl0, pl1), a.window, a.keep, PKT);
  const int n_tiles = tl.count;
  auto active = [&](int s, int t) {
    const int j0 = tl.id(t) * PKT, pf = s ? pf1 : pf0, pl = s ? pl1 : pl0;
    return pl >= pf && j0 <= pl && (j0 + PKT - 1 > pf - a.window || j0 < a.keep);
  };

  if (warp == 0) {
    if (lane == 0 && live) {
      // ------------------------------ TMA producer ------------------------------
      const bool two_q = !tiles2 || row_1 < q_len;
      mbar_expect_tx(q_full, (two_q ? 2 : 1) * q_bytes);
      for (int s = 0; s < (two_q ? 2 : 1); ++s) {
        const int h = a.maps == 2 ? head0 * 2 + s : (p.pair_heads ? head0 + s : head0);
        for (int c = 0; c < qa; ++c) tma_load_3d(q_s + s * q_bytes + c * Q_ATOM, &tmQ, q_full, c * 64, h, q_start + (s ? row_1 : row_0));
      }
      const int* bt = a.block_tables + (size_t)seq * a.max_blocks;
      bool ok = true;
      int issued = 0;
      for (int t = 0; t < n_tiles && ok; ++t) {
        const int st = t % p.stages;
        if (t >= p.stages) {
          ok = mbar_wait(&kv_empty[st], ((t / p.stages) - 1) & 1, 41);
          if (!ok) break;
        }
        uint8_t* dst = ring + (size_t)st * stage_bytes;
        mbar_expect_tx(&kv_full[st], stage_bytes);
        for (int r = 0; r < PKT; r += p.box) {
          const int key = tl.id(t) * PKT + r;
          const int blk = key < kv_len ? checked_page(bt[key / a.page], a.num_blocks) : -1;
          const int row = blk >= 0 ? blk * a.page + key % a.page : p.total_rows;
          for (int m = 0; m < p.k_maps; ++m)
            for (int c = 0; c < qa; ++c)
              tma_load_3d(dst + m * k_bytes + c * KV_ATOM + r * 128, &tmK, &kv_full[st], c * 64, kvh * p.k_maps + m, row);
          for (int c = 0; c < va; ++c) tma_load_3d(dst + p.k_maps * k_bytes + c * KV_ATOM + r * 128, &tmV, &kv_full[st], c * 64, kvh, row);
        }
        issued = t + 1;
      }
      if (!ok)
        for (int t = max(0, issued - p.stages); t < issued; ++t) (void)mbar_wait(&kv_full[t % p.stages], (t / p.stages) & 1, 42);
    }
  } else if (warp == 1 || warp == 10) {
    if (lane == 0 && live) {
      // ------------------------------ MMA issuer of one stream ------------------------------
      const int s = warp == 1 ? 0 : 1;
      const uint32_t idesc_s = umma_idesc_bf16(PT, PKT);
      const uint32_t idesc_o = umma_idesc_bf16(PT, a.dv) | UMMA_B_MN_MAJOR;
      const int ksteps = a.dq >> 4;
      // descriptors of stage 0; a stage further on is stage_bytes / 16 higher
      const uint64_t q_desc = umma_desc_sw128(smem_u32(q_s + s * q_bytes));
      const uint64_t k_desc = umma_desc_sw128(smem_u32(ring + (p.k_maps == 2 ? s * k_bytes : 0)));
      const uint64_t v_desc = umma_desc_sw128_mn(smem_u32(ring + p.k_maps * k_bytes), KV_ATOM);
      const uint32_t s_tmem = tmem_base + s * 2 * PKT, o_tmem = tmem_base + TM_O + s * 128;
      int sc = 0, pc = 0, st_next = 0, st = 0;
      uint32_t ph_next = 0;
      bool ok = mbar_wait(q_full, 0, 43);
      auto score = [&](int t) {  // S of tile t, which is in stage st_next
        if (active(s, t)) {
          const uint64_t kd = k_desc + (uint64_t)((uint32_t)(st_next * stage_bytes) >> 4);
          const uint32_t d = s_tmem + (sc & 1) * PKT;
#pragma unroll
          for (int k = 0; k < 12; ++k)
            if (k < ksteps)
              tc_mma_f16(d, q_desc + ((k >> 2) * (Q_ATOM >> 4) + 2 * (k & 3)), kd + ((k >> 2) * (KV_ATOM >> 4) + 2 * (k & 3)), idesc_s, k != 0);
          tc_commit(&s_full[s * 2 + (sc & 1)]);
          ++sc;
        }
        if (++st_next == p.stages) {
          st_next = 0;
          ph_next ^= 1;
        }
      };
      if (ok) ok = mbar_wait(&kv_full[0], 0, 44);
      if (ok) {
        tc_fence_after();
        score(0);
      }
      for (int t = 0; t < n_tiles && ok; ++t) {
        if (t + 1 < n_tiles) {
          ok = mbar_wait(&kv_full[st_next], ph_next, 45);
          if (!ok) break;
          tc_fence_after();
          score(t + 1);  // into the buffer whose P V was issued before: it is read first
        }
        if (active(s, t)) {
          const int b = pc & 1;
          ok = mbar_wait(&p_full[s * 2 + b], (pc >> 1) & 1, 46);
          if (!ok) break;
          tc_fence_after();
          const uint64_t vd = v_desc + (uint64_t)((uint32_t)(st * stage_bytes) >> 4);
#pragma unroll
          for (int k = 0; k < PKT / 16; ++k) tc_mma_f16_ts(o_tmem, s_tmem + b * PKT + k * 8, vd + k * (2048 >> 4), idesc_o, (pc | k) != 0);
          tc_commit(&pv_done[s * 2 + b]);
          ++pc;
        }
        tc_commit(&kv_empty[st]);  // one arrival per stream
        if (++st == p.stages) st = 0;
      }
    }
  } else if (live) {
    // ------------------------------ softmax warps ------------------------------
    const int s = (warp - 2) >> 2, q4 = warp & 3;
    const int r_local = q4 * 32 + lane, row = (s ? row_1 : row_0) + r_local;
    const int last_key = min(pos_off + row, kv_len - 1);
    const int low = last_key - a.window;                             // keys after low are inside the window
    const uint32_t lanes = tmem_base + ((uint32_t)(q4 * 32) << 16);
    const float scale2 = a.scale * 1.4426950408889634f, sl2 = CAPPED ? 1.0f : scale2;  // capped scores are in powers of two already
    const float cap_a = CAPPED ? 2.0f * scale2 / a.cap : 0.0f, cap_b = a.cap * 1.4426950408889634f;
    const CapSeries series(a.scale, CAPPED ? a.cap : 0.0f);
    const float small = CAPPED ? CAP_SERIES * a.cap / a.scale : 0.0f;
    constexpr float RAISE = 8.0f;  // the reference maximum rises only when a tile exceeds it by 2^8
    float m_ref = -INFINITY, l_run = 0.0f;
    bool ok = true;
    int c = 0;
    for (int t = 0; t < n_tiles; ++t) {
      if (!active(s, t)) continue;
      const int b = c & 1, j0 = tl.id(t) * PKT;
      if (ok) ok = mbar_wait(&s_full[s * 2 + b], (c >> 1) & 1, 47);
      ok = __all_sync(0xffffffffu, ok);  // the TMEM accesses below are warp-wide
      if (!ok) break;
      tc_fence_after();
      float v[PKT];
      {
        uint32_t(&r0)[16] = *reinterpret_cast<uint32_t(*)[16]>(&v[0]);
        uint32_t(&r1)[16] = *reinterpret_cast<uint32_t(*)[16]>(&v[16]);
        uint32_t(&r2)[16] = *reinterpret_cast<uint32_t(*)[16]>(&v[32]);
        uint32_t(&r3)[16] = *reinterpret_cast<uint32_t(*)[16]>(&v[48]);
        const uint32_t src = lanes + (s * 2 + b) * PKT;
        tmem_ld16(src, r0);
        tmem_ld16(src + 16, r1);
        tmem_ld16(src + 32, r2);
        tmem_ld16(src + 48, r3);
        tmem_ld_wait();
      }
      if (CAPPED) {
        float h4[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int i = 0; i < PKT; ++i) h4[i & 3] = fmaxf(h4[i & 3], fabsf(v[i]));
        if (__all_sync(0xffffffffu, fmaxf(fmaxf(h4[0], h4[1]), fmaxf(h4[2], h4[3])) < small)) {
#pragma unroll
          for (int i = 0; i < PKT; i += 2) series(v[i], v[i + 1]);
        } else {
#pragma unroll
          for (int i = 0; i < PKT; ++i) v[i] = capped_log2(v[i], cap_a, cap_b);
        }
      }
      if (j0 + PKT - 1 > last_key || !(j0 > low || j0 + PKT <= a.keep)) {
#pragma unroll
        for (int i = 0; i < PKT; ++i) {
          const int j = j0 + i;
          if (j > last_key || (j <= low && j >= a.keep)) v[i] = -INFINITY;
        }
      }
      float m4[4] = {v[0], v[1], v[2], v[3]};
#pragma unroll
      for (int i = 4; i < PKT; ++i) m4[i & 3] = fmaxf(m4[i & 3], v[i]);
      const float mx = fmaxf(fmaxf(m4[0], m4[1]), fmaxf(m4[2], m4[3])) * sl2;  // scale > 0: the scaled maximum
      if (c == 0) {
        m_ref = mx;
      } else {
        const bool raise = mx > m_ref + RAISE;
        if (__any_sync(0xffffffffu, raise)) {
          ok = __all_sync(0xffffffffu, mbar_wait(&pv_done[s * 2 + (b ^ 1)], ((c - 1) >> 1) & 1, 48));
          if (!ok) break;
          tc_fence_after();
          float f = 1.0f;
          if (raise) {
            f = m_ref == -INFINITY ? 0.0f : ex2_fast(m_ref - mx);
            m_ref = mx;
            l_run *= f;
          }
          for (int k = 0; k < a.dv / 16; ++k) {
            uint32_t r[16];
            tmem_ld16(lanes + TM_O + s * 128 + k * 16, r);
            tmem_ld_wait();
#pragma unroll
            for (int i = 0; i < 16; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * f);
            tmem_st16(lanes + TM_O + s * 128 + k * 16, r);
          }
        }
      }
      const float m_use = m_ref == -INFINITY ? 0.0f : m_ref;
      float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
      for (int k = 0; k < PKT / 32; ++k) {
        uint32_t packed[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float p0 = ex2_fast(fmaf(v[k * 32 + 2 * i], sl2, -m_use)), p1 = ex2_fast(fmaf(v[k * 32 + 2 * i + 1], sl2, -m_use));
          sum0 += p0;
          sum1 += p1;
          packed[i] = pack_bf16(p0, p1);
        }
        tmem_st16(lanes + (s * 2 + b) * PKT + k * 16, packed);
      }
      l_run += sum0 + sum1;
      tmem_st_wait();
      tc_fence_before();
      mbar_arrive(&p_full[s * 2 + b]);
      ++c;
    }
    const bool rows_here = c > 0;
    if (ok && rows_here) ok = mbar_wait(&pv_done[s * 2 + ((c - 1) & 1)], ((c - 1) >> 1) & 1, 49);
    const bool store = row < q_len;
    const int chunks = a.dv / 16;
    if (a.maps == 2) {
      // both threads of a row need both accumulators: the barrier follows each stream's last product
      xch[s * PT + r_local] = l_run;
      ok = __all_sync(0xffffffffu, ok);
      tc_fence_before();
      named_bar(1, 256);
      tc_fence_after();
      const float l1 = xch[r_local], l2 = xch[PT + r_local];
      const float f1 = l1 > 0.0f ? 1.0f / l1 : 0.0f, f2 = l2 > 0.0f ? a.lam / l2 : 0.0f;
      const int c_lo = s ? (chunks + 1) / 2 : 0, c_hi = s ? chunks : (chunks + 1) / 2;
      float o[4][16], ss = 0.0f;
#pragma unroll
      for (int k = 0; k < 4; ++k) {
        if (ok && c_lo + k < c_hi) {
          uint32_t r1[16], r2[16];
          tmem_ld16(lanes + TM_O + (c_lo + k) * 16, r1);
          tmem_ld16(lanes + TM_O + 128 + (c_lo + k) * 16, r2);
          tmem_ld_wait();
#pragma unroll
          for (int i = 0; i < 16; ++i) {
            o[k][i] = __uint_as_float(r1[i]) * f1 - __uint_as_float(r2[i]) * f2;
            ss += o[k][i] * o[k][i];
          }
        }
      }
      xch[(2 + s) * PT + r_local] = ss;
      named_bar(1, 256);
      if (ok && store) {
        ss = xch[2 * PT + r_local] + xch[3 * PT + r_local];
        const float post = a.gain / sqrtf(ss / (float)a.vdim + a.eps);
        bf16* dst = a.out + (size_t)(q_start + row) * a.out_ld + (size_t)head0 * a.dv;
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (c_lo + k < c_hi) {
            uint4 w[2];
            uint32_t* u = reinterpret_cast<uint32_t*>(w);
#pragma unroll
            for (int e = 0; e < 8; ++e) u[e] = pack_bf16(o[k][2 * e] * post, o[k][2 * e + 1] * post);
            *reinterpret_cast<uint4*>(dst + (c_lo + k) * 16) = w[0];
            *reinterpret_cast<uint4*>(dst + (c_lo + k) * 16 + 8) = w[1];
          }
      }
    } else if (__all_sync(0xffffffffu, ok) && rows_here) {
      tc_fence_after();
      const int h = p.pair_heads ? head0 + s : head0;
      float f = softmax_factor(l_run, m_ref, a.sink, h);
      if (a.gate != nullptr && store) f *= a.gate[(size_t)(q_start + row) * a.H + h];
      bf16* dst = a.out + (size_t)(q_start + row) * a.out_ld + (size_t)h * a.dv;
      for (int k = 0; k < chunks; ++k) {
        uint32_t r[16];
        tmem_ld16(lanes + TM_O + s * 128 + k * 16, r);
        tmem_ld_wait();
        uint4 w[2];
        uint32_t* u = reinterpret_cast<uint32_t*>(w);
#pragma unroll
        for (int e = 0; e < 8; ++e) u[e] = pack_bf16(__uint_as_float(r[2 * e]) * f, __uint_as_float(r[2 * e + 1]) * f);
        if (store) {
          *reinterpret_cast<uint4*>(dst + k * 16) = w[0];
          *reinterpret_cast<uint4*>(dst + k * 16 + 8) = w[1];
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem_base, 512);
}

// =====================================================================================
// Any sizes, fp32 or bf16 storage, all arithmetic in fp32.  One CTA per (query row, head); its four warps take every
// fourth visible key and merge at the end.  Lanes hold every 32nd element: up to 32 RL elements per row.
// =====================================================================================
template <typename T, int RL>
__global__ void __launch_bounds__(128) window_simple_kernel(const WinArgs<T> a) {
  extern __shared__ float o_s[];  // [4 warps][maps][dv]
  __shared__ float m_s[4][2], l_s[4][2], red[4];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, seq = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const int q_start = a.cu_q ? a.cu_q[seq] : seq;
  const int q_len = a.cu_q ? a.cu_q[seq + 1] - q_start : 1;
  const int tok = blockIdx.x / a.H, h = blockIdx.x % a.H;
  if (tok >= q_len) return;
  const int kv_len = clamp_context(a.kv_lens[seq], a.max_blocks, a.page);
  const int pos = kv_len - q_len + tok, kvh = h / (a.H / a.G);
  const int lo = max(0, pos - a.window + 1), kept = min(a.keep, lo);   // keys [0, kept) and [lo, pos]
  const int count = pos < 0 ? 0 : kept + pos - lo + 1;
  const size_t row = (size_t)q_start + tok;
  float q[2][RL], o[2][RL], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
#pragma unroll
  for (int mp = 0; mp < 2; ++mp)
#pragma unroll
    for (int e = 0; e < RL; ++e) {
      const int i = lane + 32 * e;
      q[mp][e] = mp < a.maps && i < a.dq ? to_f(a.q[((row * a.H + h) * a.maps + mp) * a.dq + i]) : 0.0f;
      o[mp][e] = 0.0f;
    }
  for (int n = warp; n < count; n += 4) {
    const int j = n < kept ? n : lo + n - kept;
    const int blk = checked_page(a.block_tables[(size_t)seq * a.max_blocks + j / a.page], a.num_blocks);
    if (blk < 0) continue;
    const T* src = a.cache + ((size_t)blk * a.page + j % a.page) * a.R;
    const T* k = src + (size_t)kvh * a.maps * a.dq;
    const T* vsrc = src + (size_t)a.G * a.maps * a.dq + (size_t)kvh * a.dv;
    float v[RL];
#pragma unroll
    for (int e = 0; e < RL; ++e) {
      const int i = lane + 32 * e;
      v[e] = i < a.dv ? to_f(vsrc[i]) : 0.0f;
    }
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
      if (mp >= a.maps) continue;
      float s = 0.0f;
#pragma unroll
      for (int e = 0; e < RL; ++e) {
        const int i = lane + 32 * e;
        if (i < a.dq) s = fmaf(q[mp][e], to_f(k[mp * a.dq + i]), s);
      }
      s = warp_sum(s) * a.scale;
      if (a.cap > 0.0f) s = a.cap * tanhf(s / a.cap);
      if (s > m[mp]) {
        const float f = expf(m[mp] - s);  // 0 for the first key
        m[mp] = s;
        l[mp] *= f;
#pragma unroll
        for (int e = 0; e < RL; ++e) o[mp][e] *= f;
      }
      const float w = expf(s - m[mp]);
      l[mp] += w;
#pragma unroll
      for (int e = 0; e < RL; ++e) o[mp][e] = fmaf(w, v[e], o[mp][e]);
    }
  }
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    if (mp >= a.maps) continue;
    if (lane == 0) {
      m_s[warp][mp] = m[mp];
      l_s[warp][mp] = l[mp];
    }
#pragma unroll
    for (int e = 0; e < RL; ++e) {
      const int i = lane + 32 * e;
      if (i < a.dv) o_s[((size_t)warp * a.maps + mp) * a.dv + i] = o[mp][e];
    }
  }
  __syncthreads();
  float f[2][4];
#pragma unroll
  for (int mp = 0; mp < 2; ++mp) {
    if (mp >= a.maps) continue;
    float mx = -INFINITY, sum = 0.0f;
    for (int w = 0; w < 4; ++w)
      if (l_s[w][mp] > 0.0f) mx = fmaxf(mx, m_s[w][mp]);
    if (a.sink != nullptr && mx > -INFINITY) {
      mx = fmaxf(mx, a.sink[h]);
      sum = expf(a.sink[h] - mx);
    }
    for (int w = 0; w < 4; ++w) {
      f[mp][w] = l_s[w][mp] > 0.0f ? expf(m_s[w][mp] - mx) : 0.0f;
      sum += f[mp][w] * l_s[w][mp];
    }
    const float inv = sum > 0.0f ? (mp == 0 ? 1.0f : -a.lam) / sum : 0.0f;
    for (int w = 0; w < 4; ++w) f[mp][w] *= inv;
  }
  float ss = 0.0f;
  __shared__ float post_s;
  for (int i = threadIdx.x; i < a.dv; i += 128) {
    float v = 0.0f;
    for (int mp = 0; mp < a.maps; ++mp)
      for (int w = 0; w < 4; ++w) v += f[mp][w] * o_s[((size_t)w * a.maps + mp) * a.dv + i];
    o_s[i] = v;  // column i of every partial is read by this thread only
    ss += v * v;
  }
  ss = warp_sum(ss);
  if (lane == 0) red[warp] = ss;
  __syncthreads();
  if (threadIdx.x == 0) {
    float post = 1.0f;
    if (a.maps == 2) post = a.gain / sqrtf((red[0] + red[1] + red[2] + red[3]) / (float)a.vdim + a.eps);
    if (a.gate != nullptr) post *= a.gate[row * a.H + h];
    post_s = post;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < a.dv; i += 128) put(a.out + row * a.out_ld + (size_t)h * a.dv + i, o_s[i] * post_s);
}

template <typename T>
WinArgs<T> win_args(const void* q, const void* cache, const void* block_tables, const void* cu_q, const void* kv_lens,
                    const void* gate, const void* sink, void* out, long long out_ld, int H, int G, int maps, int dq, int dv, int vdim,
                    int R, int page, int max_blocks, int num_blocks, int window, int keep, float scale, float lam, float gain, float eps,
                    float cap) {
  return WinArgs<T>{(const T*)q, (const T*)cache, (const int*)block_tables, (const int*)cu_q, (const int*)kv_lens, (const float*)gate,
                    (const float*)sink, (T*)out, out_ld, nullptr, nullptr, nullptr, H, G, maps, dq, dv, vdim, R, page, max_blocks, num_blocks,
                    window, keep, 1, scale, lam, gain, eps, cap};
}

int check_sizes(int H, int G, int maps, int dq, int dv, int vdim, int R, int page, int max_blocks, int window, int keep, const void* sink,
                float cap) {
  if ((sink != nullptr && maps != 1) || !(cap >= 0.0f)) return -7;
  if (H <= 0 || G <= 0 || H % G || maps < 1 || maps > 2 || page <= 0 || max_blocks <= 0 || window < 1 || keep < 0) return -1;
  if (dq <= 0 || dq % 16 || dv <= 0 || dv % 16 || vdim <= 0 || vdim > dv || R != G * (maps * dq + dv)) return -2;
  return 0;
}

template <int MT, int DVT, int KS>
int launch_decode(const WinArgs<bf16>& a, int S, int blocks, cudaStream_t stream, bool pdl) {
  const int ldq = a.maps * a.dq + 8, ldr = ldq + a.dv;
  const size_t q_bytes = (size_t)16 * MT * ldq * 2, stage = (size_t)4 * 16 * ldr * 2;
  const size_t merge = (size_t)16 * MT * (4 * (a.dv + 4) + a.nsplit) * 4;
  int stages = q_bytes + 3 * stage <= 72 * 1024 ? 3 : 2;  // three CTAs per SM where they fit
  size_t smem = q_bytes + stages * stage;
  if (smem < merge) smem = merge;
  if (smem > 227 * 1024) return -5;
  static size_t configured = 40 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(window_decode_kernel<MT, DVT, KS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return (int)prism_launch(window_decode_kernel<MT, DVT, KS>, dim3(S, a.G * blocks, a.nsplit), dim3(128), smem, stream, pdl, a, stages);
}

template <typename T>
int launch_simple(const WinArgs<T>& a, int S, int max_q_len, cudaStream_t stream, bool pdl) {
  const dim3 grid((unsigned)max_q_len * a.H, S);
  const size_t smem = (size_t)4 * a.maps * a.dv * sizeof(float);
  const int widest = a.dq > a.dv ? a.dq : a.dv;
  if (widest <= 64) return (int)prism_launch(window_simple_kernel<T, 2>, grid, dim3(128), smem, stream, pdl, a);
  if (widest <= 128) return (int)prism_launch(window_simple_kernel<T, 4>, grid, dim3(128), smem, stream, pdl, a);
  if (widest <= 256) return (int)prism_launch(window_simple_kernel<T, 8>, grid, dim3(128), smem, stream, pdl, a);
  if (widest <= 512) return (int)prism_launch(window_simple_kernel<T, 16>, grid, dim3(128), smem, stream, pdl, a);
  return -4;
}

template <typename T>
int launch_prepare(const void* slabs, long long slab_stride, int P, const void* rows, long long ld, const void* bias, const void* q_w,
                   const void* k_w, const void* freq, const void* positions, const void* slots, long long num_slots, void* q_out,
                   void* cache, void* gate, int tokens, int M, int nq, int nk, int nv, int H, int dq, int rot, int q_real, int k_real,
                   int head_norm, int tied, float eps, cudaStream_t s, bool pdl) {
  PrepareArgs<T> a{(const float*)slabs, slab_stride, P, (const T*)rows, ld, (const T*)bias, (const T*)q_w, (const T*)k_w,
                   (const float*)freq, (const int*)positions, (const long long*)slots, num_slots, (T*)q_out, (T*)cache, (float*)gate,
                   M, nq, nk, nv, H, dq, rot, q_real, k_real, tied ? nq : nq + nk, nq + nk + (tied ? 0 : nv), eps, 0};
  while ((1 << a.shift) < rot / 8 + (dq - rot) / 4) ++a.shift;
  const size_t smem = (size_t)(rot + 4 + (head_norm ? (nq + nk) / dq : 0)) * sizeof(float);
  if (smem > 48 * 1024) return -5;
  // with a norm the cluster's exchange costs more than it spreads from a few dozen tokens on
  if (tokens <= (q_w != nullptr && !head_norm ? 48 : 256))
    return (int)prism_launch(head_norm ? window_prepare_few_kernel<T, true> : window_prepare_few_kernel<T, false>, dim3(tokens * PREP_PARTS),
                             dim3(M >= 4096 ? 256 : 128), smem, s, pdl, a);
  if (tokens <= 256)
    return (int)prism_launch(head_norm ? window_prepare_mid_kernel<T, true> : window_prepare_mid_kernel<T, false>, dim3(tokens),
                             dim3(M >= 4096 ? 512 : 256), smem, s, pdl, a);
  return (int)prism_launch(head_norm ? window_prepare_kernel<T, true> : window_prepare_kernel<T, false>, dim3(tokens), dim3(256), smem, s, pdl, a);
}

}  // namespace

// Stacked projection (fp32 slabs or rows of the compute type) -> queries, cache rows, sigmoid gates.  Columns: nq queries,
// nk keys, nv values (tied: none, the nv = nk values are the keys before norm and rotation), then (gate != null) one gate per
// head; dq columns per map of a head, the first rot of them rotated.  head_norm: q_w and k_w [dq] hold for every head of
// q_real = k_real columns.  nk = nv = 0: queries only.
PRISM_API int prism_window_prepare(int f32, const void* slabs, long long slab_stride, int P, const void* rows, long long ld,
                                   const void* bias, const void* q_w, const void* k_w, const void* freq, const void* positions,
                                   const void* slots, long long num_slots, void* q_out, void* cache, void* gate, int tokens, int M,
                                   int nq, int nk, int nv, int H, int dq, int rot, int q_real, int k_real, int head_norm, int tied,
                                   float eps, void* stream, int pdl) {
  if (tokens <= 0) return 0;
  if (dq <= 0 || dq % 16 || nq % dq || nk % dq || nv % 16 || M % 16 || M < nq + nk + (tied ? 0 : nv) + (gate ? H : 0)) return -1;
  if ((tied && nv != nk) || (head_norm && q_real != k_real)) return -3;
  if (rot < 0 || rot % 2 || rot > dq || (q_w != nullptr) != (k_w != nullptr) || (!slabs && (!rows || ld % 4))) return -2;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_prepare<float>(slabs, slab_stride, P, rows, ld, bias, q_w, k_w, freq, positions, slots, num_slots, q_out, cache, gate,
                                     tokens, M, nq, nk, nv, H, dq, rot, q_real, k_real, head_norm, tied, eps, s, pdl != 0)
             : launch_prepare<bf16>(slabs, slab_stride, P, rows, ld, bias, q_w, k_w, freq, positions, slots, num_slots, q_out, cache, gate,
                                    tokens, M, nq, nk, nv, H, dq, rot, q_real, k_real, head_norm, tied, eps, s, pdl != 0);
}

// One query token per sequence.  mt: 16-row tiles per CTA (1 or 2); nsplit > 1 needs the partial buffers
// ([S * G * blocks][nsplit][16 mt][dv] and [...][2] floats) and zeroed counters [S * G * blocks].
PRISM_API int prism_window_decode(const void* q, const void* cache, const void* block_tables, const void* cu_q, const void* kv_lens,
                                  const void* gate, const void* sink, void* out, long long out_ld, void* part_o, void* part_ml, void* counters, int S,
                                  int H, int G, int maps, int dq, int dv, int vdim, int R, int page, int max_blocks, int num_blocks,
                                  int window, int keep, int mt, int nsplit, float scale, float lam, float gain, float eps, float cap,
                                  void* stream, int pdl) {
  if (S <= 0) return 0;
  if (int rc = check_sizes(H, G, maps, dq, dv, vdim, R, page, max_blocks, window, keep, sink, cap)) return rc;
  if (maps * dq > 512 || dv > 256 || (mt != 1 && mt != 2) || (mt == 2 && dv > 128) || out_ld % 2 || cu_q != nullptr) return -3;
  if (nsplit < 1 || nsplit > 32 || (nsplit > 1 && (!part_o || !part_ml || !counters))) return -4;
  WinArgs<bf16> a = win_args<bf16>(q, cache, block_tables, cu_q, kv_lens, gate, sink, out, out_ld, H, G, maps, dq, dv, vdim, R, page, max_blocks,
                                   num_blocks, window, keep, scale, lam, gain, eps, cap);
  a.part_o = (float*)part_o;
  a.part_ml = (float*)part_ml;
  a.counters = (int*)counters;
  a.nsplit = nsplit;
  const int blocks = (H / G * maps + 16 * mt - 1) / (16 * mt);
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const bool p = pdl != 0;
  const bool regs = maps * dq <= 256;
  if (dv <= 64)
    return mt == 2 ? launch_decode<2, 8, 0>(a, S, blocks, s, p)
                   : (regs ? launch_decode<1, 8, 16>(a, S, blocks, s, p) : launch_decode<1, 8, 0>(a, S, blocks, s, p));
  if (dv <= 128)
    return mt == 2 ? launch_decode<2, 16, 0>(a, S, blocks, s, p)
                   : (regs ? launch_decode<1, 16, 16>(a, S, blocks, s, p) : launch_decode<1, 16, 0>(a, S, blocks, s, p));
  return launch_decode<1, 32, 0>(a, S, blocks, s, p);
}

// Prompts and portions (cu_q: token offsets of the sequences), values up to 128 wide, keys up to 128 (one map: 192), pages of a
// multiple of 8 rows.
PRISM_API int prism_window_prefill_tc(const void* q, const void* cache, const void* block_tables, const void* cu_q, const void* kv_lens,
                                      const void* gate, const void* sink, void* out, long long out_ld, int T, int S, int max_q_len, int H, int G, int maps,
                                      int dq, int dv, int vdim, int R, int page, int max_blocks, int num_blocks, int window, int keep,
                                      float scale, float lam, float gain, float eps, float cap, void* stream, int pdl) {
  if (T <= 0 || S <= 0 || max_q_len <= 0) return 0;
  if (int rc = check_sizes(H, G, maps, dq, dv, vdim, R, page, max_blocks, window, keep, sink, cap)) return rc;
  if (dq > (maps == 1 ? 192 : 128) || dv > 128 || page % 8 || !cu_q || num_blocks <= 0 || !(scale > 0.0f) || out_ld % 8 || (reinterpret_cast<uintptr_t>(out) & 15)) return -3;
  PrefillArgs p;
  p.w = win_args<bf16>(q, cache, block_tables, cu_q, kv_lens, gate, sink, out, out_ld, H, G, maps, dq, dv, vdim, R, page, max_blocks, num_blocks,
                       window, keep, scale, lam, gain, eps, cap);
  p.k_maps = maps;
  p.pair_heads = maps == 1 && (H / G) % 2 == 0;
  p.box = 64;
  while (page % p.box) p.box >>= 1;
  const long long rows = (long long)num_blocks * page;
  if (rows > 0x7ffffff0ll) return -6;
  p.total_rows = (int)rows;
  CUtensorMap tq, tk, tv;
  const bf16* base = (const bf16*)cache;
  int rc = prism_make_head_tensor_map(q, (unsigned long long)T, (unsigned)(H * maps), (unsigned)dq, (unsigned long long)H * maps * dq, PT, &tq);
  if (rc) return rc;
  rc = prism_make_head_tensor_map(base, (unsigned long long)rows, (unsigned)(G * maps), (unsigned)dq, (unsigned long long)R, (unsigned)p.box, &tk);
  if (rc) return rc;
  rc = prism_make_head_tensor_map(base + (size_t)G * maps * dq, (unsigned long long)rows, (unsigned)G, (unsigned)dv, (unsigned long long)R,
                                  (unsigned)p.box, &tv);
  if (rc) return rc;
  const int qa = (dq + 63) / 64, va = dv > 64 ? 2 : 1;
  const size_t fixed = 1024 + (size_t)2 * qa * Q_ATOM + 21 * 8 + 16 + 4 * PT * sizeof(float);
  const size_t stage = (size_t)(maps * qa + va) * KV_ATOM;
  p.stages = 4;
  while (p.stages > 2 && fixed + p.stages * stage > 227 * 1024) --p.stages;
  const size_t smem = fixed + p.stages * stage;
  void (*kernel)(const CUtensorMap, const CUtensorMap, const CUtensorMap, const PrefillArgs) =
      cap > 0.0f ? window_prefill_tc_kernel<true> : window_prefill_tc_kernel<false>;
  static size_t configured[2] = {0, 0};
  if (smem > configured[cap > 0.0f]) {
    cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured[cap > 0.0f] = smem;
  }
  const int rows_per_cta = maps == 1 && !p.pair_heads ? 2 * PT : PT;
  const dim3 grid((max_q_len + rows_per_cta - 1) / rows_per_cta, p.pair_heads ? H / 2 : H, S);
  return (int)prism_launch(kernel, grid, dim3(PRE_THREADS), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, tq, tk,
                           tv, p);
}

// Any sizes up to 512 elements per head, decode (cu_q null) and prompts, fp32 or bf16 storage.
PRISM_API int prism_window_attention_simple(int f32, const void* q, const void* cache, const void* block_tables, const void* cu_q,
                                            const void* kv_lens, const void* gate, const void* sink, void* out, long long out_ld, int S, int max_q_len,
                                            int H, int G, int maps, int dq, int dv, int vdim, int R, int page, int max_blocks,
                                            int num_blocks, int window, int keep, float scale, float lam, float gain, float eps, float cap,
                                            void* stream, int pdl) {
  if (S <= 0 || max_q_len <= 0) return 0;
  if (int rc = check_sizes(H, G, maps, dq, dv, vdim, R, page, max_blocks, window, keep, sink, cap)) return rc;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (f32)
    return launch_simple<float>(win_args<float>(q, cache, block_tables, cu_q, kv_lens, gate, sink, out, out_ld, H, G, maps, dq, dv, vdim, R, page,
                                                max_blocks, num_blocks, window, keep, scale, lam, gain, eps, cap),
                                S, max_q_len, s, pdl != 0);
  return launch_simple<bf16>(win_args<bf16>(q, cache, block_tables, cu_q, kv_lens, gate, sink, out, out_ld, H, G, maps, dq, dv, vdim, R, page,
                                            max_blocks, num_blocks, window, keep, scale, lam, gain, eps, cap),
                             S, max_q_len, s, pdl != 0);
}
