// Latent attention: every head's keys and values are linear in one shared latent row c per token,
// k_h = U_h c and v_h = V_h c, and only c is cached (one row per token and layer run, paged).
//
// Absorbed form (decode steps, short portions of a prompt): with q~_h = U_h^T q_h the score is q~_h . c and the
// head's output V_h (sum_j p_j c_j), so attention runs over the latents themselves, all heads of a token sharing
// every latent row it reads.
//   latent_absorb_kernel     q~ for every (token, head), and, from extra CTAs of the same launch, the RMS-normalised
//                            latent of every new token written to its page
//   latent_attention_kernel  16 or 32 (token, head) rows against tiles of 64 latents (32 above 512 elements), the
//                            key range split over CTAs; mma.sync, scores and softmax in 32-bit
//   latent_out_kernel        merges the splits, multiplies by V_h and by the output gate
// Expanded form (whole prompts): the visible latents are gathered from their pages (gather_latents_kernel), one
// GEMM makes keys and values of all heads, and the tcgen05 kernel of attention_tcgen05.cu attends over them.
// The *_f32 kernels are the absorbed form in true 32-bit.
//
// Rotated columns.  A row may hold, behind the latent, a rotated key part that all heads share; a head's query then has a
// rotated part of its own.  With an identity block in U_h for those columns, q~_h holds the rotated query beside U_h^T q_h, so
// that scores are still q~_h . row and explicit keys still U_h row; values take the row's first Rv elements only.
//   latent_prepare_kernel    norms of the query latent and of the key latent, rotation and page store of the shared key part
//   latent_rotate_kernel     rotation of the queries where no absorb kernel does it (explicit keys, 32-bit)
// A query may see a window of the newest rows only: tiles outside it are not visited.
//
// Latent rows are padded with zeros to Rc elements (a multiple of 64), heads to dq / dv elements (multiples of 8).
#include "mma_sync.cuh"

PRISM_DEFINE_TU_STATUS(latent)

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

// -------------------------------------------------------------------------------------------------
// RMS norm of the projected latent and its store: one warp per token.
// -------------------------------------------------------------------------------------------------
template <typename T>
struct NormStoreArgs {
  const T* raw;            // [tokens][ld_raw]
  long long ld_raw;
  const T* weight;         // [R]
  T* cache;                // [blocks][page][Rc]
  const long long* slots;  // [tokens] flat slot, < 0: not stored
  long long num_slots;
  T* rows;                 // [tokens][Rc] contiguous copy (null: none)
  int tokens, R, Rc;
  float eps;
  int vec;                 // 1: raw rows and the weight start on 16-byte boundaries
};

struct F8 {
  float v[8];
};
__device__ __forceinline__ F8 load8(const float* p) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  return F8{{a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w}};
}
__device__ __forceinline__ F8 load8(const bf16* p) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
  F8 f;
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const float2 t = __bfloat1622float2(h[e]);
    f.v[2 * e] = t.x;
    f.v[2 * e + 1] = t.y;
  }
  return f;
}
__device__ __forceinline__ void store8(float* p, const F8& f) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f.v[0], f.v[1], f.v[2], f.v[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f.v[4], f.v[5], f.v[6], f.v[7]);
}
__device__ __forceinline__ void store8(bf16* p, const F8& f) {
  uint4 o;
  uint32_t* w = reinterpret_cast<uint32_t*>(&o);
#pragma unroll
  for (int e = 0; e < 4; ++e) w[e] = pack_bf16(f.v[2 * e], f.v[2 * e + 1]);
  *reinterpret_cast<uint4*>(p) = o;
}

constexpr int NORM_VEC = 4;  // 8-element pieces per lane: rows of up to 1024 elements

// A last piece that is not whole (and every piece of unaligned rows) is read element by element.
template <typename T>
__device__ __forceinline__ void norm_store_token(const NormStoreArgs<T>& a, int t, int lane) {
  const T* src = a.raw + (size_t)t * a.ld_raw;
  F8 x[NORM_VEC];
  float ss = 0.0f;
#pragma unroll
  for (int k = 0; k < NORM_VEC; ++k) {
    const int i = (lane + 32 * k) * 8;
    if (a.vec && i + 8 <= a.R) {
      x[k] = load8(src + i);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) x[k].v[e] = i + e < a.R ? to_f(src[i + e]) : 0.0f;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) ss += x[k].v[e] * x[k].v[e];
  }
  const float inv = 1.0f / sqrtf(warp_sum(ss) / (float)a.R + a.eps);
  long long slot = a.slots[t];
  if (slot >= a.num_slots) {
    if (lane == 0) prism_report(PRISM_ERR_BOUNDS, 3);
    slot = -1;
  }
  T* page_row = slot >= 0 ? a.cache + (size_t)slot * a.Rc : nullptr;
  T* row = a.rows ? a.rows + (size_t)t * a.Rc : nullptr;
#pragma unroll
  for (int k = 0; k < NORM_VEC; ++k) {
    const int i = (lane + 32 * k) * 8;
    if (i >= a.Rc) continue;
    F8 w;
    if (a.vec && i + 8 <= a.R) {
      w = load8(a.weight + i);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) w.v[e] = i + e < a.R ? to_f(a.weight[i + e]) : 0.0f;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) w.v[e] *= x[k].v[e] * inv;
    if (page_row) store8(page_row + i, w);
    if (row) store8(row + i, w);
  }
}

template <typename T>
__global__ void __launch_bounds__(256) latent_norm_store_kernel(const NormStoreArgs<T> a) {
  pdl_launch_dependents();
  pdl_wait();
  const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
  if (t < a.tokens) norm_store_token(a, t, threadIdx.x & 31);
}

// -------------------------------------------------------------------------------------------------
// Rotation of neighbouring columns: the pair (u, v) number i of a row at position p turns by p * freq[i].
// -------------------------------------------------------------------------------------------------
struct Rotation {
  const float* freq;       // [dims / 2] (null: nothing turns)
  const int* positions;    // [tokens]
  float amplitude;         // factor on sine and cosine
  int start, dims;         // columns start .. start + dims - 1
};
// Columns c .. c + 3 (c and start multiples of 4) of a row whose position is pos.
__device__ __forceinline__ void rotate4(float (&v)[4], const Rotation& r, float pos, int c) {
#pragma unroll
  for (int e = 0; e < 4; e += 2) {
    const int i = c + e - r.start;
    if (i < 0 || i >= r.dims) continue;
    float sn, cs;
    sincosf(pos * r.freq[i >> 1], &sn, &cs);
    sn *= r.amplitude;
    cs *= r.amplitude;
    const float a = v[e], b = v[e + 1];
    v[e] = a * cs - b * sn;
    v[e + 1] = b * cs + a * sn;
  }
}

// Rows of a projection: fp32 split-K slabs [P][tokens][ld] whose sum they are, or rows of the compute type.
template <typename T>
struct Source {
  const float* slabs;
  long long slab_stride;
  int P;
  const T* rows;
  long long ld;
};
__device__ __forceinline__ void get4(float (&v)[4], const float* p) {
  const float4 f = *reinterpret_cast<const float4*>(p);
  v[0] = f.x;
  v[1] = f.y;
  v[2] = f.z;
  v[3] = f.w;
}
__device__ __forceinline__ void get4(float (&v)[4], const bf16* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
  const float2 a = __bfloat1622float2(h[0]), b = __bfloat1622float2(h[1]);
  v[0] = a.x;
  v[1] = a.y;
  v[2] = b.x;
  v[3] = b.y;
}
__device__ __forceinline__ void put4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void put4(bf16* p, const float (&v)[4]) {
  uint2 o;
  o.x = pack_bf16(v[0], v[1]);
  o.y = pack_bf16(v[2], v[3]);
  *reinterpret_cast<uint2*>(p) = o;
}
template <typename T>
__device__ __forceinline__ void source4(float (&v)[4], const Source<T>& s, size_t row, int c) {
  if (s.slabs == nullptr) {
    get4(v, s.rows + row * s.ld + c);
    return;
  }
  v[0] = v[1] = v[2] = v[3] = 0.0f;
  const float* src = s.slabs + row * s.ld + c;
#pragma unroll 8
  for (int p = 0; p < s.P; ++p) {
    const float4 f = __ldcg(reinterpret_cast<const float4*>(src + (size_t)p * s.slab_stride));
    v[0] += f.x;
    v[1] += f.y;
    v[2] += f.z;
    v[3] += f.w;
  }
}

// -------------------------------------------------------------------------------------------------
// The stacked projection [query latent | key latent | shared key part] of a token, one CTA per token: the query latent over
// its root mean square times a weight, and the token's cache row.  Sections start at multiples of 16 columns and their padding
// is zero, so that sums over padded columns are sums over real ones.
// -------------------------------------------------------------------------------------------------
template <typename T>
struct PrepareArgs {
  Source<T> y;
  const T* q_w;            // [Qp]
  const T* c_w;            // [Cp]
  T* q_out;                // [tokens][Qp]
  T* cache;                // [blocks][page][Rc]
  const long long* slots;  // flat slot, < 0: not stored
  long long num_slots;
  int Q, Qp, R, Cp, Rc;    // real and padded widths of the latents (Cp = 0: queries only), cache row
  float eps;
  Rotation rot;            // start: Cp, in columns of the cache row
};

constexpr int PREP_GROUPS = 4;  // groups of four columns a thread holds

template <typename T>
__global__ void __launch_bounds__(512) latent_prepare_kernel(const PrepareArgs<T> a) {
  __shared__ float red[2][16];
  const size_t t = blockIdx.x;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, nw = blockDim.x >> 5;
  pdl_launch_dependents();
  pdl_wait();
  const int total = a.Cp > 0 ? a.Qp + a.Rc : a.Qp, filled = a.Cp > 0 ? a.Qp + a.Cp + (a.rot.dims + 3) / 4 * 4 : a.Qp;
  float v[PREP_GROUPS][4], sq = 0.0f, sc = 0.0f;
#pragma unroll
  for (int u = 0; u < PREP_GROUPS; ++u) {
    const int c = (tid + u * blockDim.x) * 4;
    v[u][0] = v[u][1] = v[u][2] = v[u][3] = 0.0f;
    if (c < filled) source4(v[u], a.y, t, c);
    const float ss = v[u][0] * v[u][0] + v[u][1] * v[u][1] + v[u][2] * v[u][2] + v[u][3] * v[u][3];
    if (c < a.Qp) sq += ss;
    else if (c < a.Qp + a.Cp) sc += ss;
  }
  sq = warp_sum(sq);
  sc = warp_sum(sc);
  if (lane == 0) {
    red[0][warp] = sq;
    red[1][warp] = sc;
  }
  __syncthreads();
  sq = warp_sum(lane < nw ? red[0][lane] : 0.0f);
  sc = warp_sum(lane < nw ? red[1][lane] : 0.0f);
  const float iq = 1.0f / sqrtf(sq / (float)a.Q + a.eps), ic = 1.0f / sqrtf(sc / (float)max(a.R, 1) + a.eps);
  T* row = nullptr;
  float pos = 0.0f;
  if (a.Cp > 0) {
    const long long slot = a.slots[t];
    if (slot >= a.num_slots) {
      if (tid == 0) prism_report(PRISM_ERR_BOUNDS, 5);
    } else if (slot >= 0) {
      row = a.cache + (size_t)slot * a.Rc;
    }
    if (a.rot.dims > 0) pos = (float)a.rot.positions[t];
  }
#pragma unroll
  for (int u = 0; u < PREP_GROUPS; ++u) {
    const int c = (tid + u * blockDim.x) * 4;
    if (c >= total) continue;
    if (c < a.Qp) {
      float w[4];
      get4(w, a.q_w + c);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[u][e] *= iq * w[e];
      put4(a.q_out + t * a.Qp + c, v[u]);
      continue;
    }
    if (row == nullptr) continue;
    const int r = c - a.Qp;
    if (r < a.Cp) {
      float w[4];
      get4(w, a.c_w + r);
#pragma unroll
      for (int e = 0; e < 4; ++e) v[u][e] *= ic * w[e];
    } else {
      rotate4(v[u], a.rot, pos, r);
    }
    put4(row + r, v[u]);
  }
}

// -------------------------------------------------------------------------------------------------
// Queries [tokens][H * dq] with the rotated columns of every head turned.  In place only those columns are touched.
// -------------------------------------------------------------------------------------------------
template <typename T>
struct RotateArgs {
  Source<T> q;
  T* out;                  // [tokens][ldo]
  long long ldo;
  int tokens, H, dq, per;  // per: groups of four columns of a head that are handled
  int first;               // first of them
  Rotation rot;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_rotate_kernel(const RotateArgs<T> a) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 256 + threadIdx.x, per_token = (long long)a.H * a.per;
  if (i >= a.tokens * per_token) return;
  const size_t t = (size_t)(i / per_token);
  const int k = (int)(i - (long long)t * per_token), h = k / a.per, c = a.first + (k - h * a.per) * 4;
  float v[4];
  source4(v, a.q, t, h * a.dq + c);
  if (a.rot.dims > 0) rotate4(v, a.rot, (float)a.rot.positions[t], c);
  put4(a.out + t * a.ldo + (size_t)h * a.dq + c, v);
}

// -------------------------------------------------------------------------------------------------
// q~ = U_h^T q_h for a tile of 16 tokens, one head and 128 latent elements per CTA.  The CTAs with
// blockIdx.y == H (if the launch has them) run the norm and store instead, one token per warp.  Queries that are rotated, or
// that come as slabs, are rounded once, on their way into shared memory.
// -------------------------------------------------------------------------------------------------
constexpr int ABS_N = 128, ABS_LDW = ABS_N + 8;

struct AbsorbArgs {
  const bf16* q;           // [tokens][ldq], head h at column h * dq
  long long ldq;
  const bf16* uk;          // [H * dq][Rc]
  bf16* out;               // [tokens][H][Rc]
  int H, dq, dk16;         // dk16: dq rounded up to 16
  NormStoreArgs<bf16> ns;
  Source<bf16> src;        // the queries where they are not taken as they are (slabs or rows null otherwise)
  Rotation rot;            // columns of a head
};

__global__ void __launch_bounds__(128) latent_absorb_kernel(const AbsorbArgs a) {
  extern __shared__ uint8_t smem_raw[];
  bf16* w_s = reinterpret_cast<bf16*>(smem_raw);          // [dk16][ABS_LDW]
  bf16* q_s = w_s + (size_t)a.dk16 * ABS_LDW;             // [16][dk16 + 8]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.z * 16, Rc = a.ns.Rc;
  pdl_launch_dependents();
  if ((int)blockIdx.y == a.H) {
    pdl_wait();
    for (int t = t0 + blockIdx.x * 4 + warp; t < min(t0 + 16, a.ns.tokens); t += 4 * gridDim.x) norm_store_token(a.ns, t, lane);
    return;
  }
  const int h = blockIdx.y, n0 = blockIdx.x * ABS_N, ldq_s = a.dk16 + 8;
  for (int i = threadIdx.x; i < a.dk16 * (ABS_N / 8); i += 128) {  // weights do not depend on the previous kernel
    const int k = i / (ABS_N / 8), c = (i % (ABS_N / 8)) * 8;
    const bool ok = k < a.dq && n0 + c < Rc;
    cp_async16(w_s + k * ABS_LDW + c, ok ? a.uk + ((size_t)h * a.dq + k) * Rc + n0 + c : a.uk, ok);
  }
  pdl_wait();
  if (a.src.slabs != nullptr || a.src.rows != nullptr) {
    for (int i = threadIdx.x; i < 16 * (a.dk16 / 4); i += 128) {
      const int r = i / (a.dk16 / 4), c = (i % (a.dk16 / 4)) * 4;
      float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
      if (t0 + r < a.ns.tokens && c < a.dq) {
        source4(v, a.src, (size_t)(t0 + r), h * a.dq + c);
        if (a.rot.dims > 0) rotate4(v, a.rot, (float)a.rot.positions[t0 + r], c);
      }
      put4(q_s + r * ldq_s + c, v);
    }
  } else {
    for (int i = threadIdx.x; i < 16 * (a.dk16 / 8); i += 128) {
      const int r = i / (a.dk16 / 8), c = (i % (a.dk16 / 8)) * 8;
      const bool ok = t0 + r < a.ns.tokens && c < a.dq;
      cp_async16(q_s + r * ldq_s + c, ok ? a.q + (size_t)(t0 + r) * a.ldq + (size_t)h * a.dq + c : a.q, ok);
    }
  }
  cp_async_commit();
  cp_async_wait_all();
  __syncthreads();
  float acc[4][4] = {};
  for (int kk = 0; kk < a.dk16; kk += 16) {
    uint32_t qf[4];
    ldsm_x4(qf, smem_u32(q_s + (lane & 15) * ldq_s + kk + 8 * (lane >> 4)));
#pragma unroll
    for (int np = 0; np < 2; ++np) {
      uint32_t wb[4];
      ldsm_x4_t(wb, smem_u32(w_s + (kk + (lane & 15)) * ABS_LDW + warp * 32 + np * 16 + 8 * (lane >> 4)));
      mma_bf16(acc[2 * np], qf, wb[0], wb[1]);
      mma_bf16(acc[2 * np + 1], qf, wb[2], wb[3]);
    }
  }
#pragma unroll
  for (int n = 0; n < 4; ++n) {
    const int col = n0 + warp * 32 + n * 8 + 2 * (lane & 3);
    if (col >= Rc) continue;
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = t0 + (lane >> 2) + 8 * half;
      if (t < a.ns.tokens)
        *reinterpret_cast<uint32_t*>(a.out + ((size_t)t * a.H + h) * Rc + col) = pack_bf16(acc[n][2 * half], acc[n][2 * half + 1]);
    }
  }
}

// -------------------------------------------------------------------------------------------------
// Attention of (token, head) rows over paged latents.
// -------------------------------------------------------------------------------------------------
struct LatentAttnArgs {
  const bf16* q;            // [tokens][H][Rc]
  const bf16* cache;        // [blocks][page][Rc]
  const int* block_tables;  // [S][max_blocks], < 0: hole
  const int* cu_q;          // [S + 1] token offsets; null: sequence s is token s
  const int* kv_lens;       // [S] visible latents of the sequence's last token
  float* part_o;            // [tokens * H][nsplit][Rv]  (nsplit > 1)
  float* part_ml;           // [tokens * H][nsplit][2]   maximum (base 2, scaled) and sum
  bf16* out;                // [tokens * H][Rv] normalised (nsplit == 1)
  int H, Rc, Rv, page, max_blocks, num_blocks, nsplit;
  int window;               // a query sees that many newest rows, its own among them
  float scale;
};

// One row of a tile: `bytes` (a multiple of 16) from global to shared memory, completing on `bar`.
__device__ __forceinline__ void bulk_row(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(src), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// Shared-memory bytes of a launch (the kernel lays its buffers out in this order).
template <int MT, int BN>
__host__ __device__ constexpr size_t latent_smem_bytes(int Rc) {
  return (size_t)(16 * MT + 2 * BN) * (Rc + 8) * 2 + (size_t)(8 / (BN / 16)) * 16 * MT * (BN + 4) * 4 + (size_t)16 * MT * (BN + 8) * 2 +
         4 * 16 * MT * 4 + 3 * 8;
}

// BM = 16 MT rows of one sequence against its latents in tiles of BN keys.  Eight warps:
//   scores    warp (kg, kh) takes 16 keys and one of KH slices of the latent; its query fragments stay in registers
//             for the whole kernel where they fit (QREG), the slices are added when the softmax reads them
//   softmax   BM / 8 rows per warp; a row's reference maximum is only raised when a tile exceeds it by more than
//             2^8 (the weights stay below 256), so the accumulators are rarely rescaled
//   output    every warp accumulates Rv / 8 columns of P C in registers
// Latent rows come by one bulk copy each, issued by one thread per row, two tiles in flight.  Tiles that hold only
// latents of earlier steps are fetched before the previous kernel has finished.  Rv is at most 64 NT, Rc at most 64 QN.
template <int MT, int NT, int QN, int BN>
__global__ void __launch_bounds__(256, 1) latent_attention_kernel(const LatentAttnArgs a) {
  constexpr int BM = 16 * MT;
  constexpr int KG = BN / 16, KH = 8 / KG;
  constexpr bool QREG = QN <= 8 || (QN <= 10 && MT == 1);
  constexpr int QS = QREG ? QN * 4 / KH : 1;              // 16-element steps of a warp's slice (compile-time bound)
  constexpr int LDS = BN + 4, LDP = BN + 8;
  extern __shared__ __align__(128) uint8_t smem_raw[];
  const int Rc = a.Rc, LD = Rc + 8, nt = a.Rv >> 6;       // nt: 8-column tiles of the output per warp
  bf16* q_s = reinterpret_cast<bf16*>(smem_raw);           // [BM][LD]
  bf16* kv_s = q_s + (size_t)BM * LD;                      // [2][BN][LD]
  float* s_s = reinterpret_cast<float*>(kv_s + (size_t)2 * BN * LD);  // [KH][BM][LDS]
  bf16* p_s = reinterpret_cast<bf16*>(s_s + KH * BM * LDS);  // [BM][LDP]
  float* fac_s = reinterpret_cast<float*>(p_s + BM * LDP); // [BM] rescale of the accumulator
  float* m_s = fac_s + BM;                                 // [BM] running maximum
  float* l_s = m_s + BM;                                   // [BM] running sum
  int* lim_s = reinterpret_cast<int*>(l_s + BM);           // [BM] keys a row sees
  uint64_t* bars = reinterpret_cast<uint64_t*>(lim_s + BM);  // two tiles, then the queries
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int seq = blockIdx.z, split = blockIdx.y;
  pdl_launch_dependents();
  const int q_start = a.cu_q ? a.cu_q[seq] : seq;
  const int q_len = a.cu_q ? a.cu_q[seq + 1] - q_start : 1;
  const int n_rows = q_len * a.H, row0 = blockIdx.x * BM;
  if (row0 >= n_rows) return;                              // uniform over the CTA
  const int kv_len = clamp_context(a.kv_lens[seq], a.max_blocks, a.page);
  const int last_t = min(row0 + BM, n_rows) - 1;
  const int kv_end = max(0, min(kv_len, kv_len - q_len + last_t / a.H + 1));
  // the first row any query of the tile sees, in whole tiles
  const int t_first = max(0, kv_len - q_len + row0 / a.H + 1 - a.window) / BN;
  const int tiles = (kv_end + BN - 1) / BN, per = (max(0, tiles - t_first) + a.nsplit - 1) / a.nsplit;
  const int tb = t_first + split * per, te = min(tiles, tb + per);
  const size_t out_row0 = (size_t)q_start * a.H + row0;
  const int* bt = a.block_tables + (size_t)seq * a.max_blocks;
  const uint32_t row_bytes = (uint32_t)Rc * 2;

  if (tid == 0) {
    mbar_init(&bars[0], BN);
    mbar_init(&bars[1], BN);
    mbar_init(&bars[2], BM);
    fence_barrier_init();
  }
  __syncthreads();

  auto page_of = [&](int j) {                              // threads 0 .. BN - 1: the page of one latent row of tile j
    const int key = j * BN + tid;
    return tid < BN && j < te && key < kv_end ? bt[key / a.page] : -1;
  };
  auto issue = [&](int j, int page_id) {
    if (tid < BN && j < te) {
      const int stage = (j - tb) & 1, key = j * BN + tid;
      bf16* dst = kv_s + ((size_t)stage * BN + tid) * LD;
      const int blk = checked_page(page_id, a.num_blocks);
      if (blk >= 0) {
        fence_proxy_async();
        mbar_expect_tx(&bars[stage], row_bytes);
        bulk_row(dst, a.cache + ((size_t)blk * a.page + key % a.page) * Rc, row_bytes, &bars[stage]);
      } else {                                             // past the end, or a hole: zeros
        for (int c = 0; c < Rc; c += 8) *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
        fence_proxy_async();
        mbar_arrive(&bars[stage]);
      }
    }
  };
  const int old_tiles = max(0, kv_len - q_len) / BN;       // tiles that hold latents of earlier steps only
  const bool pre0 = tb < old_tiles, pre1 = tb + 1 < old_tiles;
  const int page0 = page_of(tb), page1 = page_of(tb + 1);
  if (pre0) issue(tb, page0);
  if (pre1) issue(tb + 1, page1);
  if (tid < BM) {
    const int row = row0 + tid;
    m_s[tid] = -INFINITY;
    l_s[tid] = 0.0f;
    lim_s[tid] = row < n_rows ? kv_len - q_len + row / a.H + 1 : 0;
  }
  pdl_wait();
  if (tb < te && tid < BM) {
    bf16* dst = q_s + (size_t)tid * LD;
    if (row0 + tid < n_rows) {
      mbar_expect_tx(&bars[2], row_bytes);
      bulk_row(dst, a.q + (out_row0 + tid) * Rc, row_bytes, &bars[2]);
    } else {
      for (int c = 0; c < Rc; c += 8) *reinterpret_cast<uint4*>(dst + c) = make_uint4(0, 0, 0, 0);
      mbar_arrive(&bars[2]);
    }
  }
  if (!pre0) issue(tb, page0);
  if (!pre1) issue(tb + 1, page1);

  float acc[MT][NT][4];
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int n = 0; n < NT; ++n) acc[m][n][0] = acc[m][n][1] = acc[m][n][2] = acc[m][n][3] = 0.0f;
  const float sl2 = a.scale * 1.4426950408889634f;
  const int kg = warp % KG, kh = warp / KG, steps = (Rc >> 4) / KH, k0 = kh * steps * 16;
  const bf16* q_frag = q_s + (size_t)(lane & 15) * LD + k0 + 8 * (lane >> 4);
  uint32_t qf[MT][QS][4];
  if (tb < te) {
    (void)mbar_wait(&bars[2], 0, 31);
    if (QREG) {
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int k = 0; k < QS; ++k)
          if (k < steps) ldsm_x4(qf[m][k], smem_u32(q_frag + (size_t)m * 16 * LD + k * 16));
    }
  }

  for (int j = tb; j < te; ++j) {
    const int stage = (j - tb) & 1;
    const int next_page = page_of(j + 2);
    (void)mbar_wait(&bars[stage], ((j - tb) >> 1) & 1, 32 + stage);
    const bf16* kv = kv_s + (size_t)stage * BN * LD;
    {
      float s[MT][2][4] = {};
      const bf16* kp = kv + (size_t)(kg * 16 + (lane & 7) + 8 * (lane >> 4)) * LD + k0 + 8 * ((lane >> 3) & 1);
      if (QREG) {
#pragma unroll
        for (int k = 0; k < QS; ++k)
          if (k < steps) {
            uint32_t kb[4];
            ldsm_x4(kb, smem_u32(kp + k * 16));
#pragma unroll
            for (int m = 0; m < MT; ++m) {
              mma_bf16(s[m][0], qf[m][k], kb[0], kb[1]);
              mma_bf16(s[m][1], qf[m][k], kb[2], kb[3]);
            }
          }
      } else {
#pragma unroll 4
        for (int k = 0; k < steps; ++k) {
          uint32_t kb[4];
          ldsm_x4(kb, smem_u32(kp + k * 16));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            uint32_t q[4];
            ldsm_x4(q, smem_u32(q_frag + (size_t)m * 16 * LD + k * 16));
            mma_bf16(s[m][0], q, kb[0], kb[1]);
            mma_bf16(s[m][1], q, kb[2], kb[3]);
          }
        }
      }
#pragma unroll
      for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          float* d = s_s + ((size_t)kh * BM + m * 16 + (lane >> 2)) * LDS + kg * 16 + n * 8 + 2 * (lane & 3);
          *reinterpret_cast<float2*>(d) = make_float2(s[m][n][0], s[m][n][1]);
          *reinterpret_cast<float2*>(d + 8 * LDS) = make_float2(s[m][n][2], s[m][n][3]);
        }
    }
    __syncthreads();
    // online softmax, BM / 8 rows per warp
#pragma unroll
    for (int i = 0; i < BM / 8; ++i) {
      const int r = warp * (BM / 8) + i;
      const int limit = lim_s[r] - j * BN, low = limit - a.window;
      float v[BN / 32], mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < BN / 32; ++e) {
        const int c = lane + 32 * e;
        float t = s_s[r * LDS + c];
#pragma unroll
        for (int h = 1; h < KH; ++h) t += s_s[(h * BM + r) * LDS + c];
        v[e] = c < limit && c >= low ? t * sl2 : -INFINITY;
        mx = fmaxf(mx, v[e]);
      }
      mx = warp_max(mx);
      const float m_old = m_s[r], m_new = mx > m_old + 8.0f ? mx : m_old;
      const float m_use = m_new == -INFINITY ? 0.0f : m_new;
      float sum = 0.0f;
#pragma unroll
      for (int e = 0; e < BN / 32; ++e) {
        const float p = ex2_fast(v[e] - m_use);
        sum += p;
        p_s[r * LDP + lane + 32 * e] = __float2bfloat16_rn(p);
      }
      sum = warp_sum(sum);
      __syncwarp();
      if (lane == 0) {
        const float f = ex2_fast(m_old - m_use);  // 0 while nothing has been seen
        fac_s[r] = f;
        m_s[r] = m_new;
        l_s[r] = l_s[r] * f + sum;
      }
    }
    __syncthreads();
    // accumulate P C, columns warp * Rc / 8 ..
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      const float f0 = fac_s[m * 16 + (lane >> 2)], f1 = fac_s[m * 16 + (lane >> 2) + 8];
      if (__any_sync(0xffffffffu, f0 != 1.0f || f1 != 1.0f)) {
#pragma unroll
        for (int n = 0; n < NT; ++n) {
          acc[m][n][0] *= f0;
          acc[m][n][1] *= f0;
          acc[m][n][2] *= f1;
          acc[m][n][3] *= f1;
        }
      }
    }
    const int col0 = warp * nt * 8;
#pragma unroll
    for (int kk = 0; kk < BN; kk += 16) {
      uint32_t pf[MT][4];
#pragma unroll
      for (int m = 0; m < MT; ++m) ldsm_x4(pf[m], smem_u32(p_s + (m * 16 + (lane & 15)) * LDP + kk + 8 * (lane >> 4)));
      const bf16* vrow = kv + (size_t)(kk + (lane & 15)) * LD + col0 + 8 * (lane >> 4);
#pragma unroll
      for (int n = 0; n < NT; n += 2) {
        if (n < nt) {                // a last odd tile loads its neighbour (or the row's padding) and ignores it
          uint32_t vb[4];
          ldsm_x4_t(vb, smem_u32(vrow + n * 8));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16(acc[m][n], pf[m], vb[0], vb[1]);
            if (n + 1 < nt) mma_bf16(acc[m][n + 1], pf[m], vb[2], vb[3]);
          }
        }
      }
    }
    __syncthreads();                 // every warp is done with this tile: its buffer takes the tile after the next
    issue(j + 2, next_page);
  }
  __syncthreads();
  if (a.nsplit > 1 && tid < BM && row0 + tid < n_rows) {
    float* ml = a.part_ml + ((out_row0 + tid) * a.nsplit + split) * 2;
    ml[0] = m_s[tid];
    ml[1] = l_s[tid];
  }
  if (a.nsplit > 1 && tb >= te) return;  // an empty split has no partial rows
#pragma unroll
  for (int m = 0; m < MT; ++m)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int r = m * 16 + (lane >> 2) + 8 * half;
      if (row0 + r >= n_rows) continue;
      const float l = l_s[r], inv = a.nsplit > 1 ? 1.0f : (l > 0.0f ? 1.0f / l : 0.0f);
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        if (n >= nt) continue;
        const int col = warp * nt * 8 + n * 8 + 2 * (lane & 3);
        const float v0 = acc[m][n][2 * half] * inv, v1 = acc[m][n][2 * half + 1] * inv;
        if (a.nsplit > 1)
          *reinterpret_cast<float2*>(a.part_o + ((out_row0 + r) * a.nsplit + split) * a.Rv + col) = make_float2(v0, v1);
        else
          *reinterpret_cast<uint32_t*>(a.out + (out_row0 + r) * a.Rv + col) = pack_bf16(v0, v1);
      }
    }
}

// -------------------------------------------------------------------------------------------------
// o_h = gate * V_h (merged latent output): a tile of 16 tokens, one head, 64 output elements per CTA.
// -------------------------------------------------------------------------------------------------
constexpr int OUT_N = 64, OUT_THREADS = 256, MAX_SPLITS = 64;

struct LatentOutArgs {
  const float* part_o;
  const float* part_ml;
  const bf16* lat;         // [tokens * H][Rc] (nsplit == 1)
  const bf16* uv;          // [H * dv][ldw]
  long long ldw;
  const bf16* gate;        // [tokens][gate_ld], head h at column h * dv (null: one)
  long long gate_ld;
  bf16* out;               // [tokens][ld_out]
  long long ld_out;
  int tokens, H, dv, Rc, nsplit;
};

// Weighted sum of the splits for 16 tokens of one head, as bf16 rows in shared memory.  A thread keeps ITEMS x BATCH
// independent 16-byte loads in flight.
template <int ITEMS, int BATCH>
__device__ __forceinline__ void merge_splits(const LatentOutArgs& a, bf16* a_s, int LD, const float (*wgt)[MAX_SPLITS], const int* used,
                                             int t0, int h) {
  const int per_row = a.Rc >> 2, total = 16 * per_row;
  for (int i0 = threadIdx.x; i0 < total; i0 += OUT_THREADS * ITEMS) {
    float4 v[ITEMS];
    int r[ITEMS], c[ITEMS], n_max = 0;
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
      const int i = min(i0 + k * OUT_THREADS, total - 1);
      r[k] = i / per_row;
      c[k] = (i - r[k] * per_row) * 4;
      v[k] = make_float4(0.f, 0.f, 0.f, 0.f);
      n_max = max(n_max, used[r[k]]);
    }
    for (int s0 = 0; s0 < n_max; s0 += BATCH) {
      float4 p[ITEMS][BATCH];
#pragma unroll
      for (int k = 0; k < ITEMS; ++k) {
        const float* src = a.part_o + (((size_t)(t0 + r[k]) * a.H + h) * a.nsplit + s0) * a.Rc + c[k];
#pragma unroll
        for (int s = 0; s < BATCH; ++s)  // an empty split's rows were never written: weight zero, not read
          p[k][s] = (s0 + s < used[r[k]] && wgt[r[k]][s0 + s] > 0.0f) ? __ldcg(reinterpret_cast<const float4*>(src + (size_t)s * a.Rc))
                                                                      : make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll
      for (int k = 0; k < ITEMS; ++k)
#pragma unroll
        for (int s = 0; s < BATCH; ++s) {
          const float w = s0 + s < used[r[k]] ? wgt[r[k]][s0 + s] : 0.0f;
          v[k].x += w * p[k][s].x;
          v[k].y += w * p[k][s].y;
          v[k].z += w * p[k][s].z;
          v[k].w += w * p[k][s].w;
        }
    }
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
      if (i0 + k * OUT_THREADS >= total) continue;
      uint2 o;
      o.x = pack_bf16(v[k].x, v[k].y);
      o.y = pack_bf16(v[k].z, v[k].w);
      *reinterpret_cast<uint2*>(a_s + (size_t)r[k] * LD + c[k]) = o;
    }
  }
}

__global__ void __launch_bounds__(OUT_THREADS) latent_out_kernel(const LatentOutArgs a) {
  extern __shared__ __align__(128) uint8_t smem_raw[];
  const int Rc = a.Rc, LD = Rc + 8;
  bf16* w_s = reinterpret_cast<bf16*>(smem_raw);   // [OUT_N][LD]
  bf16* a_s = w_s + (size_t)OUT_N * LD;            // [16][LD]
  __shared__ float wgt[16][MAX_SPLITS];
  __shared__ int used[16];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int n0 = blockIdx.x * OUT_N, h = blockIdx.y, t0 = blockIdx.z * 16;
  pdl_launch_dependents();
  for (int r = warp; r < OUT_N; r += OUT_THREADS / 32) {
    const bool ok = n0 + r < a.dv;
    const bf16* src = ok ? a.uv + ((size_t)h * a.dv + n0 + r) * a.ldw : a.uv;
    for (int c = lane * 8; c < Rc; c += 256) cp_async16(w_s + (size_t)r * LD + c, ok ? src + c : src, ok);
  }
  cp_async_commit();
  pdl_wait();
  const int rows = min(16, a.tokens - t0);
  if (a.nsplit > 1) {
    for (int r = warp; r < 16; r += OUT_THREADS / 32) {  // weights of the splits: 2^(m_s - m) / l
      float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
      if (r < rows) {
        const float2* ml = reinterpret_cast<const float2*>(a.part_ml) + ((size_t)(t0 + r) * a.H + h) * a.nsplit;
#pragma unroll
        for (int e = 0; e < 2; ++e)
          if (lane + 32 * e < a.nsplit) {
            const float2 v = ml[lane + 32 * e];
            m[e] = v.y > 0.0f ? v.x : -INFINITY;
            l[e] = v.y;
          }
      }
      const float mx = warp_max(fmaxf(m[0], m[1]));
      const float f0 = l[0] > 0.0f ? ex2_fast(m[0] - mx) : 0.0f, f1 = l[1] > 0.0f ? ex2_fast(m[1] - mx) : 0.0f;
      const float sum = warp_sum(f0 * l[0] + f1 * l[1]);
      const float inv = sum > 0.0f ? 1.0f / sum : 0.0f;
      wgt[r][lane] = f0 * inv;
      wgt[r][lane + 32] = f1 * inv;
      const unsigned b0 = __ballot_sync(0xffffffffu, f0 > 0.0f), b1 = __ballot_sync(0xffffffffu, f1 > 0.0f);
      if (lane == 0) used[r] = b1 ? 64 - __clz(b1) : (b0 ? 32 - __clz(b0) : 0);
    }
    __syncthreads();
    if (a.nsplit <= 4) merge_splits<4, 4>(a, a_s, LD, wgt, used, t0, h);
    else if (a.nsplit <= 16) merge_splits<2, 16>(a, a_s, LD, wgt, used, t0, h);
    else merge_splits<1, 32>(a, a_s, LD, wgt, used, t0, h);
  } else {
    for (int r = warp; r < 16; r += OUT_THREADS / 32) {
      const bool ok = r < rows;
      const bf16* src = ok ? a.lat + ((size_t)(t0 + r) * a.H + h) * Rc : a.lat;
      for (int c = lane * 8; c < Rc; c += 256) cp_async16(a_s + (size_t)r * LD + c, ok ? src + c : src, ok);
    }
    cp_async_commit();
  }
  cp_async_wait<0>();
  __syncthreads();
  float acc[2][4] = {};                              // even and odd steps: two independent chains, 8 columns per warp
#pragma unroll 4
  for (int kk = 0; kk < Rc; kk += 32) {
    uint32_t a0[4], a1[4], wb[4];
    ldsm_x4(wb, smem_u32(w_s + (size_t)(warp * 8 + (lane & 7)) * LD + kk + 8 * (lane >> 3)));
    ldsm_x4(a0, smem_u32(a_s + (size_t)(lane & 15) * LD + kk + 8 * (lane >> 4)));
    ldsm_x4(a1, smem_u32(a_s + (size_t)(lane & 15) * LD + kk + 16 + 8 * (lane >> 4)));
    mma_bf16(acc[0], a0, wb[0], wb[1]);
    mma_bf16(acc[1], a1, wb[2], wb[3]);
  }
  const int col = n0 + warp * 8 + 2 * (lane & 3);
  if (col >= a.dv) return;
#pragma unroll
  for (int half = 0; half < 2; ++half) {
    const int r = (lane >> 2) + 8 * half;
    if (r >= rows) continue;
    float v0 = acc[0][2 * half] + acc[1][2 * half], v1 = acc[0][2 * half + 1] + acc[1][2 * half + 1];
    if (a.gate) {
      const float2 g = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(a.gate + (size_t)(t0 + r) * a.gate_ld + (size_t)h * a.dv + col));
      v0 *= g.x;
      v1 *= g.y;
    }
    *reinterpret_cast<uint32_t*>(a.out + (size_t)(t0 + r) * a.ld_out + (size_t)h * a.dv + col) = pack_bf16(v0, v1);
  }
}

// -------------------------------------------------------------------------------------------------
// Visible latents of every sequence, page by page, as contiguous rows.  One warp per row.
// -------------------------------------------------------------------------------------------------
struct GatherLatentArgs {
  const uint8_t* cache;
  const int* block_tables;
  const int* cu_kv;        // [S + 1]
  uint8_t* rows;           // [total][row_bytes]
  int max_blocks, num_blocks, page, row_bytes;
  int total;
};

__global__ void __launch_bounds__(256) gather_latents_kernel(const GatherLatentArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.y, lane = threadIdx.x & 31, j = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int start = a.cu_kv[seq];
  const int len = clamp_context(a.cu_kv[seq + 1] - start, a.max_blocks, a.page);
  if (j >= len) return;
  const long long dst = (long long)start + j;
  if (dst < 0 || dst >= a.total) {
    if (lane == 0) prism_report(PRISM_ERR_BOUNDS, 4);
    return;
  }
  const int blk = checked_page(a.block_tables[(size_t)seq * a.max_blocks + j / a.page], a.num_blocks);
  const uint4* src = reinterpret_cast<const uint4*>(a.cache + ((size_t)max(blk, 0) * a.page + j % a.page) * a.row_bytes);
  uint4* out = reinterpret_cast<uint4*>(a.rows + (size_t)dst * a.row_bytes);
  for (int i = lane; i < a.row_bytes / 16; i += 32) out[i] = blk >= 0 ? src[i] : make_uint4(0, 0, 0, 0);
}

// Pages of every sequence from first[s] on, one behind the other from scratch page base[s] on; rows past the sequence's end and
// holes are zero.  One warp per row.
struct GatherPagesArgs {
  const uint8_t* cache;
  const int* block_tables;
  const int* kv_lens;
  const int* first;        // [S]
  const int* base;         // [S + 1]
  uint8_t* rows;           // [base[S] * page][row_bytes]
  int max_blocks, num_blocks, page, row_bytes, total;
};

__global__ void __launch_bounds__(256) gather_latent_pages_kernel(const GatherPagesArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int seq = blockIdx.y, lane = threadIdx.x & 31, j = blockIdx.x * 8 + (threadIdx.x >> 5);
  const int base = a.base[seq];
  if (j >= (a.base[seq + 1] - base) * a.page) return;
  const long long dst = (long long)base * a.page + j;
  if (dst < 0 || dst >= a.total) {
    if (lane == 0) prism_report(PRISM_ERR_BOUNDS, 6);
    return;
  }
  const int page_no = a.first[seq] + j / a.page, key = page_no * a.page + j % a.page;
  const bool in = key < a.kv_lens[seq] && page_no < a.max_blocks;
  const int blk = in ? checked_page(a.block_tables[(size_t)seq * a.max_blocks + page_no], a.num_blocks) : -1;
  const uint4* src = reinterpret_cast<const uint4*>(a.cache + ((size_t)max(blk, 0) * a.page + j % a.page) * a.row_bytes);
  uint4* out = reinterpret_cast<uint4*>(a.rows + (size_t)dst * a.row_bytes);
  for (int i = lane; i < a.row_bytes / 16; i += 32) out[i] = blk >= 0 ? src[i] : make_uint4(0, 0, 0, 0);
}

// -------------------------------------------------------------------------------------------------
// True 32-bit forms.
// -------------------------------------------------------------------------------------------------
// out[t][h * n_out + n] = gate * sum_k x[t][h * kx + k] w(h, k, n): w is [H * kx][ldw] (transposed = 0, n along the
// row) or [H * n_out][ldw] (transposed = 1, k along the row).
struct HeadwiseArgs {
  const float* x;
  long long ldx;
  const float* w;
  long long ldw;
  const float* gate;
  long long gate_ld;
  float* out;
  long long ldo;
  int H, kx, n_out, transposed;
};

__global__ void __launch_bounds__(128) headwise_f32_kernel(const HeadwiseArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int n = blockIdx.x * 128 + threadIdx.x, h = blockIdx.y;
  const size_t t = blockIdx.z;
  if (n >= a.n_out) return;
  const float* x = a.x + t * a.ldx + (size_t)h * a.kx;
  float v = 0.0f;
  if (a.transposed) {
    const float* w = a.w + ((size_t)h * a.n_out + n) * a.ldw;
    for (int k = 0; k < a.kx; ++k) v = fmaf(x[k], w[k], v);
  } else {
    const float* w = a.w + (size_t)h * a.kx * a.ldw + n;
    for (int k = 0; k < a.kx; ++k) v = fmaf(x[k], w[(size_t)k * a.ldw], v);
  }
  if (a.gate) v *= a.gate[t * a.gate_ld + (size_t)h * a.n_out + n];
  a.out[t * a.ldo + (size_t)h * a.n_out + n] = v;
}

struct LatentF32Args {
  const float* q;           // [tokens][H][Rc]
  const float* cache;       // [blocks][page][Rc]
  const int* block_tables;
  const int* cu_q;
  const int* kv_lens;
  float* out;               // [tokens][H][Rc]
  int H, Rc, page, max_blocks, num_blocks, window;
  float scale;
};

// One CTA per (token, head) row; its four warps take every fourth key and merge at the end.
template <int RL>
__global__ void __launch_bounds__(128) latent_attention_f32_kernel(const LatentF32Args a) {
  __shared__ float m_s[4], l_s[4];
  extern __shared__ float o_s[];  // [4][Rc]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, seq = blockIdx.y;
  pdl_launch_dependents();
  pdl_wait();
  const int q_start = a.cu_q ? a.cu_q[seq] : seq;
  const int q_len = a.cu_q ? a.cu_q[seq + 1] - q_start : 1;
  const int row = blockIdx.x;
  if (row >= q_len * a.H) return;
  const int kv_len = clamp_context(a.kv_lens[seq], a.max_blocks, a.page);
  const int limit = min(kv_len, kv_len - q_len + row / a.H + 1);
  const size_t r = (size_t)q_start * a.H + row;
  float q[RL], o[RL];
#pragma unroll
  for (int e = 0; e < RL; ++e) {
    const int i = lane + 32 * e;
    q[e] = i < a.Rc ? a.q[r * a.Rc + i] : 0.0f;
    o[e] = 0.0f;
  }
  float m = -INFINITY, l = 0.0f;
  for (int j = max(0, limit - a.window) + warp; j < limit; j += 4) {
    const int blk = checked_page(a.block_tables[(size_t)seq * a.max_blocks + j / a.page], a.num_blocks);
    if (blk < 0) continue;
    const float* c = a.cache + ((size_t)blk * a.page + j % a.page) * a.Rc;
    float k[RL], s = 0.0f;
#pragma unroll
    for (int e = 0; e < RL; ++e) {
      const int i = lane + 32 * e;
      k[e] = i < a.Rc ? c[i] : 0.0f;
      s = fmaf(q[e], k[e], s);
    }
    s = warp_sum(s) * a.scale;
    if (s > m) {
      const float f = expf(m - s);  // 0 for the first key
      m = s;
      l *= f;
#pragma unroll
      for (int e = 0; e < RL; ++e) o[e] *= f;
    }
    const float p = expf(s - m);
    l += p;
#pragma unroll
    for (int e = 0; e < RL; ++e) o[e] = fmaf(p, k[e], o[e]);
  }
  if (lane == 0) {
    m_s[warp] = m;
    l_s[warp] = l;
  }
#pragma unroll
  for (int e = 0; e < RL; ++e) {
    const int i = lane + 32 * e;
    if (i < a.Rc) o_s[warp * a.Rc + i] = o[e];
  }
  __syncthreads();
  float mx = -INFINITY;
  for (int w = 0; w < 4; ++w)
    if (l_s[w] > 0.0f) mx = fmaxf(mx, m_s[w]);
  float f[4], sum = 0.0f;
  for (int w = 0; w < 4; ++w) {
    f[w] = l_s[w] > 0.0f ? expf(m_s[w] - mx) : 0.0f;
    sum += f[w] * l_s[w];
  }
  for (int i = threadIdx.x; i < a.Rc; i += 128) {
    float v = 0.0f;
    for (int w = 0; w < 4; ++w) v += f[w] * o_s[w * a.Rc + i];
    a.out[r * a.Rc + i] = sum > 0.0f ? v / sum : 0.0f;
  }
}

template <int MT, int NT, int QN, int BN>
int launch_latent(const LatentAttnArgs& a, int row_tiles, int S, cudaStream_t stream, bool pdl) {
  const size_t smem = latent_smem_bytes<MT, BN>(a.Rc);
  static size_t configured = 0;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_attention_kernel<MT, NT, QN, BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  return (int)prism_launch(latent_attention_kernel<MT, NT, QN, BN>, dim3(row_tiles, a.nsplit, S), dim3(256), smem, stream, pdl, a);
}

template <typename T>
NormStoreArgs<T> norm_store_args(const void* raw, long long ld_raw, const void* weight, void* cache, const void* slots,
                                 long long num_slots, void* rows, int tokens, int R, int Rc, float eps) {
  return NormStoreArgs<T>{(const T*)raw, ld_raw, (const T*)weight, (T*)cache, (const long long*)slots, num_slots, (T*)rows,
                          tokens, R, Rc, eps,
                          ld_raw * sizeof(T) % 16 == 0 && ((reinterpret_cast<uintptr_t>(raw) | reinterpret_cast<uintptr_t>(weight)) & 15) == 0};
}

}  // namespace

// Latent rows of the new tokens: RMS norm over R elements with a weight, zero padding up to Rc, stored at flat slots
// (block * page + offset) and, when rows is given, contiguously.
PRISM_API int prism_latent_norm_store(int f32, const void* raw, long long ld_raw, const void* weight, void* cache,
                                      const void* slots, long long num_slots, void* rows, int tokens, int R, int Rc, float eps,
                                      void* stream, int pdl) {
  if (tokens <= 0) return 0;
  if (R <= 0 || R > Rc || Rc % 64 || Rc > 1024) return -1;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((tokens + 7) / 8);
  if (f32)
    return (int)prism_launch(latent_norm_store_kernel<float>, grid, dim3(256), 0, s, pdl != 0,
                             norm_store_args<float>(raw, ld_raw, weight, cache, slots, num_slots, rows, tokens, R, Rc, eps));
  return (int)prism_launch(latent_norm_store_kernel<bf16>, grid, dim3(256), 0, s, pdl != 0,
                           norm_store_args<bf16>(raw, ld_raw, weight, cache, slots, num_slots, rows, tokens, R, Rc, eps));
}

// q~ [tokens][H][Rc] = U_h^T q_h (bf16), with the norm and store of the same tokens' latents in the same launch (raw null:
// without).  Queries: rows q, or q_slabs [P][tokens][ldq] fp32 whose sum they are; freq (null: none): columns rot_start ..
// rot_start + rot - 1 of every head are rotated first.
PRISM_API int prism_latent_absorb(const void* q, const void* q_slabs, long long q_stride, int q_P, long long ldq, const void* freq,
                                  const void* positions, float amplitude, int rot_start, int rot, const void* uk, void* out, const void* raw,
                                  long long ld_raw, const void* weight, void* cache, const void* slots, long long num_slots, int tokens, int H,
                                  int dq, int R, int Rc, float eps, void* stream, int pdl) {
  if (tokens <= 0) return 0;
  if (R <= 0 || R > Rc || Rc % 64 || H <= 0 || dq % 8 || ldq % 8 || Rc > 1024 || (!q && !q_slabs)) return -1;
  if (freq != nullptr && (!positions || rot_start < 0 || rot_start % 4 || rot < 0 || rot % 2 || rot_start + rot > dq)) return -3;
  AbsorbArgs a;
  a.q = (const bf16*)q;
  a.ldq = ldq;
  a.uk = (const bf16*)uk;
  a.out = (bf16*)out;
  a.H = H;
  a.dq = dq;
  a.dk16 = (dq + 15) / 16 * 16;
  a.ns = norm_store_args<bf16>(raw, ld_raw, weight, cache, slots, num_slots, nullptr, tokens, R, Rc, eps);
  a.src = Source<bf16>{(const float*)q_slabs, q_stride, q_P, freq != nullptr ? (const bf16*)q : nullptr, ldq};
  a.rot = Rotation{(const float*)freq, (const int*)positions, amplitude, rot_start, freq != nullptr ? rot : 0};
  const size_t smem = ((size_t)a.dk16 * ABS_LDW + 16 * (a.dk16 + 8)) * 2;
  if (smem > 220 * 1024) return -2;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_absorb_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  const dim3 grid((Rc + ABS_N - 1) / ABS_N, raw != nullptr ? H + 1 : H, (tokens + 15) / 16);
  return (int)prism_launch(latent_absorb_kernel, grid, dim3(128), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

// Causal attention of q~ over the paged latents, the newest `window` of them.  nsplit > 1: unnormalised fp32 partials and their
// maxima / sums; nsplit == 1: normalised bf16 rows in out.  Rows of Rc elements, of which the first Rv are summed up; both
// multiples of 64, Rc at most 1024.
PRISM_API int prism_latent_attention(const void* q, const void* cache, const void* block_tables, const void* cu_q,
                                     const void* kv_lens, void* part_o, void* part_ml, void* out, int S, int max_q_len, int H,
                                     int Rc, int Rv, int page, int max_blocks, int num_blocks, int nsplit, int window, float scale,
                                     void* stream, int pdl) {
  if (S <= 0 || max_q_len <= 0) return 0;
  if (H <= 0 || Rc % 64 || Rc <= 0 || Rc > 1024 || Rv % 64 || Rv <= 0 || Rv > Rc || page <= 0 || max_blocks <= 0 || window < 1) return -1;
  if (nsplit < 1 || nsplit > MAX_SPLITS || (nsplit > 1 ? (!part_o || !part_ml) : !out)) return -2;
  LatentAttnArgs a{(const bf16*)q, (const bf16*)cache, (const int*)block_tables, (const int*)cu_q, (const int*)kv_lens,
                   (float*)part_o, (float*)part_ml, (bf16*)out, H, Rc, Rv, page, max_blocks, num_blocks, nsplit, window, scale};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const long long rows = (long long)max_q_len * H;
  // 16-row tiles read the latents once per 16 heads instead of 32: worth it while they still fit the device in one wave
  const bool narrow = rows <= 16 || (rows + 15) / 16 * nsplit * S <= 148;
  const int tiles = (int)((rows + (narrow ? 15 : 31)) / (narrow ? 16 : 32));
  const bool p = pdl != 0;
#define PRISM_LATENT_CASE(NT_, QN_, BN_)                                         \
  return narrow ? launch_latent<1, NT_, QN_, BN_>(a, tiles, S, s, p) : launch_latent<2, NT_, QN_, BN_>(a, tiles, S, s, p);
  if (Rc <= 128) PRISM_LATENT_CASE(2, 2, 64)
  if (Rc <= 256) PRISM_LATENT_CASE(4, 4, 64)
  if (Rc <= 512) PRISM_LATENT_CASE(8, 8, 64)
  if (Rc <= 640 && Rv <= 512) PRISM_LATENT_CASE(8, 10, 64)
  PRISM_LATENT_CASE(16, 16, 32)
#undef PRISM_LATENT_CASE
}

// out [tokens][ld_out] (head h at column h * dv) = gate * V_h o~_h, o~ merged from the splits of prism_latent_attention.  Rc: the
// elements that were summed up; uv rows ldw apart.
PRISM_API int prism_latent_out(const void* part_o, const void* part_ml, const void* lat, const void* uv, long long ldw, const void* gate,
                               long long gate_ld, void* out, long long ld_out, int tokens, int H, int dv, int Rc, int nsplit,
                               void* stream, int pdl) {
  if (tokens <= 0) return 0;
  if (H <= 0 || dv % 8 || Rc % 64 || Rc <= 0 || Rc > 1024 || nsplit < 1 || nsplit > MAX_SPLITS || gate_ld % 2 || ld_out % 2 || ldw < Rc || ldw % 8) return -1;
  LatentOutArgs a{(const float*)part_o, (const float*)part_ml, (const bf16*)lat, (const bf16*)uv, ldw, (const bf16*)gate, gate_ld,
                  (bf16*)out, ld_out, tokens, H, dv, Rc, nsplit};
  const size_t smem = (size_t)(OUT_N + 16) * (Rc + 8) * 2;
  static size_t configured = 40 * 1024;
  if (smem > configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) return (int)e;
    configured = smem;
  }
  const dim3 grid((dv + OUT_N - 1) / OUT_N, H, (tokens + 15) / 16);
  return (int)prism_launch(latent_out_kernel, grid, dim3(OUT_THREADS), smem, reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

// Stacked projection [tokens][ld] (fp32 slabs or rows of the compute type) with Qp columns of a query latent (Q real ones), Cp of
// a key latent (R real ones) and rot of the shared key part -> q_out [tokens][Qp], normed, and cache rows of Rc elements
// [Cp | rot | zeros].  Cp = 0: queries only.  Qp and Cp multiples of 16.
PRISM_API int prism_latent_prepare(int f32, const void* slabs, long long slab_stride, int P, const void* rows, long long ld, const void* q_w,
                                   const void* c_w, void* q_out, void* cache, const void* slots, long long num_slots, const void* freq,
                                   const void* positions, float amplitude, int tokens, int Q, int Qp, int R, int Cp, int rot, int Rc, float eps,
                                   void* stream, int pdl) {
  if (tokens <= 0) return 0;
  if (Q <= 0 || Q > Qp || Qp % 16 || Cp < 0 || Cp % 16 || rot < 0 || rot % 2 || ld % 4 || (!slabs && !rows)) return -1;
  if (Cp > 0 && (R <= 0 || R > Cp || Rc % 64 || Cp + rot > Rc || !cache || !slots || (rot > 0 && (!freq || !positions)))) return -2;
  const int groups = (Qp + (Cp > 0 ? Rc : 0)) / 4, per = tokens <= 256 ? 1 : PREP_GROUPS;
  int threads = ((groups + per - 1) / per + 31) / 32 * 32;
  if (threads > 512) threads = 512;
  if (groups > threads * PREP_GROUPS) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    PrepareArgs<T> a{Source<T>{(const float*)slabs, slab_stride, P, (const T*)rows, ld}, (const T*)q_w, (const T*)c_w, (T*)q_out, (T*)cache,
                     (const long long*)slots, num_slots, Q, Qp, R, Cp, Rc, eps,
                     Rotation{(const float*)freq, (const int*)positions, amplitude, Cp, Cp > 0 ? rot : 0}};
    return (int)prism_launch(latent_prepare_kernel<T>, dim3(tokens), dim3(threads), 0, s, pdl != 0, a);
  };
  return f32 ? run(float()) : run(bf16());
}

// Queries as slabs or rows [tokens][ld] -> out [tokens][ldo], columns rot_start .. rot_start + rot - 1 of every head rotated.  rows ==
// out: only those are touched.
PRISM_API int prism_latent_rotate(int f32, const void* slabs, long long slab_stride, int P, const void* rows, long long ld, void* out,
                                  long long ldo, const void* freq, const void* positions, float amplitude, int tokens, int H, int dq,
                                  int rot_start, int rot, void* stream, int pdl) {
  if (tokens <= 0) return 0;
  if (H <= 0 || dq <= 0 || dq % 8 || ld % 4 || ldo % 4 || rot_start < 0 || rot_start % 4 || rot < 0 || rot % 2 || rot_start + rot > dq) return -1;
  if ((!slabs && !rows) || (rot > 0 && (!freq || !positions))) return -2;
  const bool in_place = !slabs && rows == out;
  const int first = in_place ? rot_start : 0, per = in_place ? (rot + 3) / 4 : dq / 4;
  if (per == 0) return 0;
  const long long total = (long long)tokens * H * per;
  if ((total + 255) / 256 > 0x7fffffffll) return -3;
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  auto run = [&](auto type) -> int {
    using T = decltype(type);
    RotateArgs<T> a{Source<T>{(const float*)slabs, slab_stride, P, (const T*)rows, ld}, (T*)out, ldo, tokens, H, dq, per, first,
                    Rotation{(const float*)freq, (const int*)positions, amplitude, rot_start, rot}};
    return (int)prism_launch(latent_rotate_kernel<T>, dim3((unsigned)((total + 255) / 256)), dim3(256), 0, s, pdl != 0, a);
  };
  return f32 ? run(float()) : run(bf16());
}

// rows [total][row_bytes]: the latents each sequence sees (cu_kv), gathered from their pages.
PRISM_API int prism_gather_latents(const void* cache, const void* block_tables, const void* cu_kv, void* rows, int S,
                                   int max_kv_len, int total, int max_blocks, int num_blocks, int page, int row_bytes,
                                   void* stream, int pdl) {
  if (S <= 0 || max_kv_len <= 0 || total <= 0) return 0;
  if (row_bytes % 16 || page <= 0 || max_blocks <= 0) return -1;
  GatherLatentArgs a{(const uint8_t*)cache, (const int*)block_tables, (const int*)cu_kv, (uint8_t*)rows,
                     max_blocks, num_blocks, page, row_bytes, total};
  return (int)prism_launch(gather_latents_kernel, dim3((max_kv_len + 7) / 8, S), dim3(256), 0,
                           reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

// rows [total][row_bytes]: of every sequence the pages first[s] .. as scratch pages base[s] .. base[s + 1] - 1, each of `page`
// rows; max_pages: the most pages of a sequence.
PRISM_API int prism_gather_latent_pages(const void* cache, const void* block_tables, const void* kv_lens, const void* first, const void* base,
                                        void* rows, int S, int max_pages, int total, int max_blocks, int num_blocks, int page, int row_bytes,
                                        void* stream, int pdl) {
  if (S <= 0 || max_pages <= 0 || total <= 0) return 0;
  if (row_bytes % 16 || page <= 0 || max_blocks <= 0 || S > 65535) return -1;
  GatherPagesArgs a{(const uint8_t*)cache, (const int*)block_tables, (const int*)kv_lens, (const int*)first, (const int*)base, (uint8_t*)rows,
                    max_blocks, num_blocks, page, row_bytes, total};
  return (int)prism_launch(gather_latent_pages_kernel, dim3((unsigned)(((long long)max_pages * page + 7) / 8), S), dim3(256), 0,
                           reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

PRISM_API int prism_headwise_f32(const void* x, long long ldx, const void* w, long long ldw, const void* gate, long long gate_ld,
                                 void* out, long long ldo, int tokens, int H, int kx, int n_out, int transposed, void* stream,
                                 int pdl) {
  if (tokens <= 0) return 0;
  if (H <= 0 || kx <= 0 || n_out <= 0 || tokens > 65535) return -1;
  HeadwiseArgs a{(const float*)x, ldx, (const float*)w, ldw, (const float*)gate, gate_ld, (float*)out, ldo, H, kx, n_out, transposed};
  return (int)prism_launch(headwise_f32_kernel, dim3((n_out + 127) / 128, H, tokens), dim3(128), 0,
                           reinterpret_cast<cudaStream_t>(stream), pdl != 0, a);
}

PRISM_API int prism_latent_attention_f32(const void* q, const void* cache, const void* block_tables, const void* cu_q,
                                         const void* kv_lens, void* out, int S, int max_q_len, int H, int Rc, int page,
                                         int max_blocks, int num_blocks, int window, float scale, void* stream, int pdl) {
  if (S <= 0 || max_q_len <= 0) return 0;
  if (H <= 0 || Rc % 64 || Rc <= 0 || Rc > 1024 || page <= 0 || max_blocks <= 0 || window < 1) return -1;
  LatentF32Args a{(const float*)q, (const float*)cache, (const int*)block_tables, (const int*)cu_q, (const int*)kv_lens,
                  (float*)out, H, Rc, page, max_blocks, num_blocks, window, scale};
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  const dim3 grid((unsigned)max_q_len * H, S);
  const size_t smem = (size_t)4 * Rc * sizeof(float);
  if (Rc <= 128) return (int)prism_launch(latent_attention_f32_kernel<4>, grid, dim3(128), smem, s, pdl != 0, a);
  if (Rc <= 256) return (int)prism_launch(latent_attention_f32_kernel<8>, grid, dim3(128), smem, s, pdl != 0, a);
  if (Rc <= 512) return (int)prism_launch(latent_attention_f32_kernel<16>, grid, dim3(128), smem, s, pdl != 0, a);
  return (int)prism_launch(latent_attention_f32_kernel<32>, grid, dim3(128), smem, s, pdl != 0, a);
}
