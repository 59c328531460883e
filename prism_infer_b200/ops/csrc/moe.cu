// Routing and dispatch of a mixture of experts.
//
// Every token has `top` routed slots and `always` more that name experts E .. E + always - 1.  Pairs (token, slot) get a
// row each, sorted by expert and, within one, by token: the grouped GEMMs then read an expert's tokens as consecutive
// rows.  The order is a function of the routing alone.
//
//   moe_route_kernel   one CTA per chunk of tokens: sum of the router's split-K slabs, top-k (one warp per token), softmax
//                      over the chosen logits, count per expert and rank of each pair within its chunk and expert.  With a
//                      single chunk it also places the pairs.  Scored form: the softmax is over all outputs, a correction
//                      enters the choice only, which is among the best groups of neighbours; outputs E .. choices - 1 stand
//                      for the token's own row (their weights are summed up for the kernel that adds the branch).  Scores
//                      may be the outputs' own sigmoids, and a group as good as the sum of its two best.
//   moe_place_kernel   one CTA per chunk: first row of every expert, then rows of the chunk's pairs
//   moe_gather_kernel  copies a token's row to the rows of its pairs
#include "common.cuh"

PRISM_DEFINE_TU_STATUS(moe)

namespace {

typedef __nv_bfloat16 bf16;

constexpr int ROUTE_THREADS = 1024, ROUTE_WARPS = ROUTE_THREADS / 32;
constexpr int MAX_EXPERTS = 1024;  // routed and always-on together: one thread each in the prefix sums

struct RouteArgs {
  const float* logits;     // [P][T][ld] fp32 slabs
  long long slab_stride, ld;
  int P;
  const long long* slots;  // cache slot of each token, < 0: takes no part
  int* expert;             // [T][K] expert of each pair (-1: none)
  int* pos;                // [T][K] rank within chunk and expert, then the pair's row (-1: none)
  float* weight;           // [T][K]
  int* row_token;          // [T * K]
  int* counts;             // [chunks][E + always]
  int4* groups;            // (expert, first row, rows, 0)
  int max_groups;
  int* n_groups;
  int T, top, E, always, chunk, tile;
  // scored form (correction != null)
  const float* correction;  // [choices]
  float* self_weight;       // [T] weight of the token's own row
  int choices;              // outputs that can be chosen, the E experts first; E without the scored form
  int sets, keep;           // the best `keep` of `sets` equal runs of neighbours are open to choice
  int always_col;           // logit whose sigmoid weighs the always-on experts (-1: weight one)
  float scale;
  int sigmoid;              // 1: the scores are the logits' sigmoids, not divided by their sum
  int group_best;           // a group's score is its best output's (1) or the sum of its two best (2)
};

// Exclusive prefix sum over the block of one value per thread; *total gets the sum.
__device__ __forceinline__ int block_scan(int v, int* warp_sums, int* total) {
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  int x = v;
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const int y = __shfl_up_sync(0xffffffffu, x, o);
    if (lane >= o) x += y;
  }
  if (lane == 31) warp_sums[warp] = x;
  __syncthreads();
  if (warp == 0) {
    int s = warp_sums[lane];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int y = __shfl_up_sync(0xffffffffu, s, o);
      if (lane >= o) s += y;
    }
    warp_sums[lane] = s;
  }
  __syncthreads();
  const int before = warp > 0 ? warp_sums[warp - 1] : 0;
  *total = warp_sums[31];
  __syncthreads();
  return before + x - v;
}

// Rows of a chunk's pairs from the experts' first rows, and (writer) the table of tiles.  count: pairs of expert
// threadIdx.x over all tokens, before: those in earlier chunks.
__device__ __forceinline__ void place(const RouteArgs& a, int t0, int n, int count, int before, bool writer, int* scan_s, int* base_s) {
  const int e = threadIdx.x, all = a.E + a.always, K = a.top + a.always;
  int total;
  const int first = block_scan(e < all ? count : 0, scan_s, &total);
  if (e < all) base_s[e] = first + before;
  const int tiles = e < all ? (count + a.tile - 1) / a.tile : 0;
  int n_tiles;
  const int g0 = block_scan(tiles, scan_s, &n_tiles);
  if (writer) {
    for (int i = 0; i < tiles; ++i)
      if (g0 + i < a.max_groups) a.groups[g0 + i] = make_int4(e, first + i * a.tile, min(a.tile, count - i * a.tile), 0);
    if (e == 0) {
      *a.n_groups = min(n_tiles, a.max_groups);
      if (n_tiles > a.max_groups) prism_report(PRISM_ERR_BOUNDS, 1);
    }
  }
  __syncthreads();
  for (int i = threadIdx.x; i < n * K; i += blockDim.x) {
    const size_t pair = (size_t)t0 * K + i;
    const int x = a.expert[pair];
    if (x < 0) continue;
    const int row = base_s[x] + a.pos[pair];
    a.pos[pair] = row;
    a.row_token[row] = t0 + i / K;
  }
}

// choice [C]: lane l's values of outputs l, l + 32, ...  Outputs outside the best groups become -inf.
template <int C>
__device__ __forceinline__ void keep_best_groups(float (&choice)[C], const RouteArgs& a, int lane) {
  const int size = a.choices / a.sets;
  int of[C];                       // group of each of the lane's outputs
#pragma unroll
  for (int c = 0; c < C; ++c) of[c] = (c * 32 + lane) / size;
  float best[C];                   // lane l: scores of groups l, l + 32, ...
#pragma unroll
  for (int c = 0; c < C; ++c) best[c] = -INFINITY;
  for (int g = 0; g < a.sets; ++g) {
    float m = -INFINITY, second = -INFINITY;
#pragma unroll
    for (int c = 0; c < C; ++c)
      if (of[c] == g) {
        second = fmaxf(second, fminf(m, choice[c]));
        m = fmaxf(m, choice[c]);
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float om = __shfl_xor_sync(0xffffffffu, m, o), os = __shfl_xor_sync(0xffffffffu, second, o);
      second = fmaxf(fmaxf(second, os), fminf(m, om));
      m = fmaxf(m, om);
    }
    if (a.group_best == 2 && second > -INFINITY) m += second;
#pragma unroll
    for (int c = 0; c < C; ++c)
      if (c * 32 + lane == g) best[c] = m;
  }
  unsigned open = 0;
  for (int k = 0; k < a.keep; ++k) {
    float bv = -INFINITY;
    int bg = MAX_EXPERTS;
#pragma unroll
    for (int c = 0; c < C; ++c)
      if (best[c] > bv) {
        bv = best[c];
        bg = c * 32 + lane;
      }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
      const int og = __shfl_xor_sync(0xffffffffu, bg, o);
      if (ov > bv || (ov == bv && og < bg)) {
        bv = ov;
        bg = og;
      }
    }
#pragma unroll
    for (int c = 0; c < C; ++c) {
      if (of[c] == bg) open |= 1u << c;
      if (c * 32 + lane == bg) best[c] = -INFINITY;
    }
  }
#pragma unroll
  for (int c = 0; c < C; ++c)
    if (!(open >> c & 1u)) choice[c] = -INFINITY;
}

// C: groups of 32 outputs
template <int C, bool SCORED>
__global__ void __launch_bounds__(ROUTE_THREADS) moe_route_kernel(const RouteArgs a) {
  extern __shared__ int expert_s[];            // [chunk * K]
  __shared__ int count_s[MAX_EXPERTS], base_s[MAX_EXPERTS], scan_s[32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t0 = blockIdx.x * a.chunk, n = min(a.chunk, a.T - t0), all = a.E + a.always, K = a.top + a.always;
  pdl_launch_dependents();
  pdl_wait();
  for (int i = warp; i < n; i += ROUTE_WARPS) {
    const size_t t = (size_t)t0 + i;
    const bool live = a.slots[t] >= 0;
    // lane l holds experts l, l + 32, ...: the next best is found by a maximum over (value, lowest expert)
    float v[C];
#pragma unroll
    for (int c = 0; c < C; ++c) {
      const int e = c * 32 + lane;
      float s = 0.0f;
      if (e < a.choices) {
#pragma unroll 16
        for (int p = 0; p < a.P; ++p) s += __ldcg(a.logits + (size_t)p * a.slab_stride + t * a.ld + e);
      }
      v[c] = e < a.choices ? s : -INFINITY;
    }
    float always_w = 1.0f, score[SCORED ? C : 1];
    if (SCORED) {
      if (a.always_col >= 0) {
        float s = 0.0f;
#pragma unroll 16
        for (int p = 0; p < a.P; ++p) s += __ldcg(a.logits + (size_t)p * a.slab_stride + t * a.ld + a.always_col);
        always_w = 1.0f / (1.0f + expf(-s));
      }
      float total = 1.0f;
      if (a.sigmoid) {
#pragma unroll
        for (int c = 0; c < C; ++c) score[c] = 1.0f / (1.0f + expf(-v[c]));
      } else {
        float m = v[0];
#pragma unroll
        for (int c = 1; c < C; ++c) m = fmaxf(m, v[c]);
        m = warp_max(m);
        total = 0.0f;
#pragma unroll
        for (int c = 0; c < C; ++c) total += score[c] = expf(v[c] - m);
        total = 1.0f / warp_sum(total);
      }
#pragma unroll
      for (int c = 0; c < C; ++c) {
        score[c] *= total;
        if (c * 32 + lane < a.choices) v[c] = score[c] + a.correction[c * 32 + lane];
      }
      if (a.sets > a.keep) keep_best_groups(v, a, lane);
    }
    float best0 = 0.0f, sum = 0.0f, self = 0.0f;
    for (int k = 0; k < a.top; ++k) {
      float bv = -INFINITY;
      int be = MAX_EXPERTS;
#pragma unroll
      for (int c = 0; c < C; ++c)
        if (v[c] > bv) {
          bv = v[c];
          be = c * 32 + lane;
        }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
        const int oe = __shfl_xor_sync(0xffffffffu, be, o);
        if (ov > bv || (ov == bv && oe < be)) {
          bv = ov;
          be = oe;
        }
      }
      if (be >= a.choices) be = 0;             // no finite logit left: any expert, weight from its own logit
#pragma unroll
      for (int c = 0; c < C; ++c)
        if (be == c * 32 + lane) v[c] = -INFINITY;
      float w;
      if (SCORED) {
        float mine = 0.0f;
#pragma unroll
        for (int c = 0; c < C; ++c)
          if (be == c * 32 + lane) mine = score[c];
        w = __shfl_sync(0xffffffffu, mine, be & 31);
        if (be >= a.E) self += w;
      } else {
        if (k == 0) best0 = bv;
        w = expf(bv - best0);
      }
      sum += w;
      if (lane == 0) {
        expert_s[i * K + k] = live && be < a.E ? be : -1;
        a.weight[t * K + k] = be < a.E ? w : 0.0f;
      }
    }
    __syncwarp();
    const float inv = SCORED ? (a.sigmoid ? a.scale : a.scale / (sum + 1e-20f)) : 1.0f / sum;
    for (int k = lane; k < K; k += 32) {
      if (k >= a.top) expert_s[i * K + k] = live ? a.E + k - a.top : -1;
      a.weight[t * K + k] = live ? (k < a.top ? a.weight[t * K + k] * inv : always_w) : 0.0f;
    }
    if (SCORED && lane == 0) a.self_weight[t] = live ? self * inv : 0.0f;
  }
  __syncthreads();
  // count and rank: one warp per expert looks at 32 pairs at a time
  for (int e = warp; e < all; e += ROUTE_WARPS) {
    int c = 0;
    for (int i0 = 0; i0 < n * K; i0 += 32) {
      const int i = i0 + lane;
      const bool hit = i < n * K && expert_s[i] == e;
      const unsigned m = __ballot_sync(0xffffffffu, hit);
      if (hit) a.pos[(size_t)t0 * K + i] = c + __popc(m & ((1u << lane) - 1));
      c += __popc(m);
    }
    if (lane == 0) count_s[e] = c;
  }
  for (int i = threadIdx.x; i < n * K; i += ROUTE_THREADS) {
    a.expert[(size_t)t0 * K + i] = expert_s[i];
    if (expert_s[i] < 0) a.pos[(size_t)t0 * K + i] = -1;
  }
  __syncthreads();
  if (gridDim.x > 1) {
    for (int e = threadIdx.x; e < all; e += ROUTE_THREADS) a.counts[(size_t)blockIdx.x * all + e] = count_s[e];
    return;
  }
  place(a, t0, n, (int)threadIdx.x < all ? count_s[threadIdx.x] : 0, 0, true, scan_s, base_s);
}

__global__ void __launch_bounds__(ROUTE_THREADS) moe_place_kernel(const RouteArgs a) {
  __shared__ int base_s[MAX_EXPERTS], scan_s[32];
  const int t0 = blockIdx.x * a.chunk, n = min(a.chunk, a.T - t0), all = a.E + a.always;
  pdl_launch_dependents();
  pdl_wait();
  int count = 0, before = 0;
  if ((int)threadIdx.x < all)
    for (int c = 0; c < (int)gridDim.x; ++c) {
      const int v = a.counts[(size_t)c * all + threadIdx.x];
      count += v;
      if (c < (int)blockIdx.x) before += v;
    }
  place(a, t0, n, count, before, blockIdx.x == 0, scan_s, base_s);
}

// grid (tokens): row t of x to every row of its pairs
__global__ void __launch_bounds__(256) moe_gather_kernel(const bf16* x, long long ldx, const int* pos, bf16* rows, int K, int W, int N) {
  pdl_launch_dependents();
  pdl_wait();
  const size_t t = blockIdx.x;
  const uint4* src = reinterpret_cast<const uint4*>(x + t * ldx);
  for (int i = threadIdx.x; i < W / 8; i += 256) {
    const uint4 v = src[i];
    for (int k = 0; k < K; ++k) {
      const int r = pos[t * K + k];
      if (r >= 0 && r < N) reinterpret_cast<uint4*>(rows + (size_t)r * W)[i] = v;
    }
  }
}

int check_route(const RouteArgs& a) {
  if (a.top < 1 || a.top > a.choices || a.choices < a.E || a.choices > MAX_EXPERTS || a.always < 0 || a.E + a.always > MAX_EXPERTS || a.chunk < 1 || a.tile < 1 || a.max_groups < 1) return -1;
  if ((long long)a.T * (a.top + a.always) > 0x7fffffffll || a.chunk * (a.top + a.always) > 10240) return -2;
  if (a.correction != nullptr && (!a.self_weight || a.sets < 1 || a.choices % a.sets || a.keep < 1 || a.keep > a.sets || a.group_best < 1 || a.group_best > 2)) return -3;
  return 0;
}

template <int C>
int launch_route(const RouteArgs& a, size_t smem, cudaStream_t st, bool pdl) {
  const dim3 grid((a.T + a.chunk - 1) / a.chunk), block(ROUTE_THREADS);
  return (int)(a.correction != nullptr ? prism_launch(moe_route_kernel<C, true>, grid, block, smem, st, pdl, a)
                                       : prism_launch(moe_route_kernel<C, false>, grid, block, smem, st, pdl, a));
}

}  // namespace

// logits: P fp32 slabs [T][ld] of E columns.  expert, pos, weight [T][top + always]; row_token [T * (top + always)]; counts
// [chunks][E + always]; groups [max_groups] int4 and n_groups: tiles of at most `tile` rows of one expert.  With more than
// one chunk prism_moe_place must follow.  correction != null: the scored form, with the logits of `choices` outputs (the E
// experts, then those that stand for the token's own row, whose weight goes to self_weight [T]) and, at column always_col if
// that is not negative, the one whose sigmoid weighs the always-on experts; sigmoid and group_best as in RouteArgs.
PRISM_API int prism_moe_route(const void* logits, long long slab_stride, long long ld, int P, const void* slots, void* expert, void* pos,
                              void* weight, void* row_token, void* counts, void* groups, int max_groups, void* n_groups, int T, int top,
                              int E, int always, int chunk, int tile, const void* correction, void* self_weight, int choices,
                              int sets, int keep, int always_col, float scale, int sigmoid, int group_best, void* stream, int pdl) {
  if (T <= 0) return 0;
  RouteArgs a{(const float*)logits, slab_stride, ld, P, (const long long*)slots, (int*)expert, (int*)pos, (float*)weight, (int*)row_token,
              (int*)counts, (int4*)groups, max_groups, (int*)n_groups, T, top, E, always, chunk, tile, (const float*)correction,
              (float*)self_weight, choices, sets, keep, always_col, scale, sigmoid, group_best};
  if (int rc = check_route(a)) return rc;
  const size_t smem = (size_t)chunk * (top + always) * sizeof(int);
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (choices <= 32) return launch_route<1>(a, smem, st, pdl != 0);
  if (choices <= 64) return launch_route<2>(a, smem, st, pdl != 0);
  if (choices <= 128) return launch_route<4>(a, smem, st, pdl != 0);
  if (choices <= 256) return launch_route<8>(a, smem, st, pdl != 0);
  return launch_route<MAX_EXPERTS / 32>(a, smem, st, pdl != 0);
}

PRISM_API int prism_moe_place(void* expert, void* pos, void* weight, void* row_token, void* counts, void* groups, int max_groups,
                              void* n_groups, int T, int top, int E, int always, int chunk, int tile, void* stream, int pdl) {
  if (T <= 0) return 0;
  RouteArgs a{nullptr, 0, 0, 0, nullptr, (int*)expert, (int*)pos, (float*)weight, (int*)row_token, (int*)counts, (int4*)groups, max_groups,
              (int*)n_groups, T, top, E, always, chunk, tile, nullptr, nullptr, top > E ? top : E, 1, 1, -1, 1.0f, 0, 1};
  if (int rc = check_route(a)) return rc;
  return (int)prism_launch(moe_place_kernel, dim3((T + chunk - 1) / chunk), dim3(ROUTE_THREADS), 0, reinterpret_cast<cudaStream_t>(stream),
                           pdl != 0, a);
}

// rows [T * K][W] (bf16, W a multiple of 8): x[t] at every pos[t][k] >= 0.
PRISM_API int prism_moe_gather(const void* x, long long ldx, const void* pos, void* rows, int T, int K, int W, void* stream, int pdl) {
  if (T <= 0) return 0;
  if (K <= 0 || W <= 0 || W % 8 || ldx % 8) return -1;
  return (int)prism_launch(moe_gather_kernel, dim3(T), dim3(256), 0, reinterpret_cast<cudaStream_t>(stream), pdl != 0, (const bf16*)x, ldx,
                           (const int*)pos, (bf16*)rows, K, W, T * K);
}
