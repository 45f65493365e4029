// Routed feed-forward (mixture of experts): the router, the grouping of (token, expert) pairs by
// expert, and the experts' two products as grouped matrix products.
//
//   router:   z = W_r x (float32 sums; in this kernel, or handed in as float32 logits), score = sigmoid(z) (or softmax over the experts); experts lie in
//             `groups` equal groups of neighbours; a group's score is the sum of its `group_top` best
//             choice scores; only experts of the best `keep` groups can be chosen; the `top` best of those are
//             the token's experts, weighted by their scores (optionally divided by their sum);
//             a choice bias per expert may be added to the scores for the choice alone (the weights are the
//             scores without it); the weights may be multiplied by a constant
//   identity: router outputs beyond the experts that have matrices stand for the input itself: their pairs
//             get no tiles, and the combine kernel takes the token's input row in place of a product
//   pairs:    pair p = token * top + k; `order` lists the pairs expert by expert, `tile_expert` /
//             `tile_begin` / `tile_rows` cut every expert's pairs into tiles of up to 64 rows
//   products: up:   act[p, :]  = f(W_up[e]   x[token(p), :])      f = activation
//             down: y[p, :]    =   W_down[e] act[p, :]
//   combine:  out[t, :] = sum_k weight[t, k] * y[t * top + k, :] (+ shared[t, :], times sigmoid(gate_t) where
//             the shared expert has a gate), k in order
//
// A pair's results do not depend on which other pairs share its tile or on the order within the
// expert's list: every output element is one thread's sum over k in a fixed order.  All sums are float32.
// bfloat16 operands go through mma.sync (m16n8k16, float32 accumulators); float32 operands through
// FFMA only; steps of a handful of pairs stream the chosen experts' weights through FFMA in both types.
#include "common.cuh"

namespace rl {

enum { ACT_NONE = 0, ACT_RELU_SQ = 1, ACT_GELU_ERF = 2, ACT_SILU = 3, ACT_GELU_TANH = 4, ACT_CLAMPED_SWISH = 6 };

__device__ __forceinline__ float moe_activate(float z, int mode) {
  switch (mode) {
    case ACT_RELU_SQ: { const float r = fmaxf(z, 0.f); return r * r; }
    case ACT_GELU_ERF: return 0.5f * z * (1.f + erff(z * 0.70710678118654752f));
    case ACT_SILU: return z / (1.f + expf(-z));
    case ACT_GELU_TANH: return 0.5f * z * (1.f + tanhf(0.79788456080286536f * (z + 0.044715f * z * z * z)));
    default: return z;
  }
}

// ------------------------------------------------------------------ router
// One warp per token.  Scores live in shared memory (experts floats per warp).  The largest score wins,
// the lower index among equals.
struct ArgMax {
  float v;
  int i;
};
__device__ __forceinline__ ArgMax warp_argmax(ArgMax a) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const float v = __shfl_xor_sync(0xffffffffu, a.v, o);
    const int i = __shfl_xor_sync(0xffffffffu, a.i, o);
    if (v > a.v || (v == a.v && i < a.i)) {
      a.v = v;
      a.i = i;
    }
  }
  return a;
}

struct RouteArgs {
  int ld, tokens, width, experts, groups, keep, group_top, top, softmax, renorm;
  const float* bias;
  const float* choice_bias;
  float weight_scale, renorm_floor;
};

// One token's choice by one warp; `score` points to 2 * experts + 2 * groups floats of the warp's own.
template <typename TA, typename TW>
__device__ __forceinline__ void route_token(const RouteArgs& a, const TA* __restrict__ xr, const TW* __restrict__ router,
                                            int t, float* score, int32_t* choice, float* weight) {
  const int lane = threadIdx.x & 31;
  const int width = a.width, experts = a.experts, groups = a.groups, keep = a.keep, group_top = a.group_top, top = a.top;
  const float *bias = a.bias, *choice_bias = a.choice_bias;
  float* work = score + experts;           // [experts] scores, [experts] working copy, 2 x [groups]
  float* gscore = work + experts;
  float* gsel = gscore + groups;
  if (router == nullptr) {
    // x holds the logits themselves [tokens, experts] (a matrix product before this kernel made them)
    for (int e = lane; e < experts; e += 32) score[e] = to_float(xr[e]);
  } else {
    for (int e = 0; e < experts; ++e) {
      const TW* w = router + static_cast<size_t>(e) * width;
      float s = 0.f;
      for (int c = lane; c < width; c += 32) s = fmaf(to_float(xr[c]), to_float(w[c]), s);
      s = warp_sum(s);
      if (lane == 0) score[e] = s;
    }
  }
  __syncwarp();
  if (bias != nullptr) {            // a bias of the router's logits
    for (int e = lane; e < experts; e += 32) score[e] += bias[e];
    __syncwarp();
  }
  if (a.softmax) {
    float mx = -INFINITY;
    for (int e = lane; e < experts; e += 32) mx = fmaxf(mx, score[e]);
    mx = warp_max(mx);
    float l = 0.f;
    for (int e = lane; e < experts; e += 32) l += expf(score[e] - mx);
    l = warp_sum(l);
    for (int e = lane; e < experts; e += 32) score[e] = expf(score[e] - mx) / l;
  } else {
    for (int e = lane; e < experts; e += 32) score[e] = 1.f / (1.f + expf(-score[e]));
  }
  __syncwarp();
  for (int e = lane; e < experts; e += 32) work[e] = score[e] + (choice_bias != nullptr ? choice_bias[e] : 0.f);
  __syncwarp();
  const int per = experts / groups;
  if (groups > 1 && keep < groups) {
    // a group's score: the sum of its group_top best choice scores
    for (int g = lane; g < groups; g += 32) {
      float total = 0.f;
      int taken_a = -1;                    // (group_top is small: the best, then the best of the rest, ...)
      float last = INFINITY;
      for (int k = 0; k < group_top && k < per; ++k) {
        float best = -INFINITY;
        int bi = -1;
        for (int e = 0; e < per; ++e) {
          const float v = work[g * per + e];
          // next in the order (value descending, index ascending) after (last, taken_a)
          const bool after = v < last || (v == last && e > taken_a);
          if (after && (v > best || bi < 0)) {
            best = v;
            bi = e;
          }
        }
        total += best;
        last = best;
        taken_a = bi;
      }
      gscore[g] = total;
    }
    __syncwarp();
    // the best `keep` groups stay (the lower index among equals); the others' experts cannot be chosen
    for (int g = lane; g < groups; g += 32) gsel[g] = 0.f;
    __syncwarp();
    for (int k = 0; k < keep; ++k) {
      ArgMax a = {-INFINITY, 0x7fffffff};
      for (int g = lane; g < groups; g += 32) {
        const float v = gscore[g];
        if (gsel[g] == 0.f && (a.i == 0x7fffffff || v > a.v)) {
          a.v = v;
          a.i = g;
        }
      }
      a = warp_argmax(a);
      __syncwarp();
      if (lane == 0 && a.i < groups) gsel[a.i] = 1.f;
      __syncwarp();
    }
    for (int e = lane; e < experts; e += 32)
      if (gsel[e / per] == 0.f) work[e] = -INFINITY;
    __syncwarp();
  }
  float total = 0.f;
  for (int k = 0; k < top; ++k) {
    ArgMax a = {-INFINITY, 0x7fffffff};
    for (int e = lane; e < experts; e += 32) {
      const float v = work[e];
      if (v > a.v || (v == a.v && e < a.i)) {
        a.v = v;
        a.i = e;
      }
    }
    a = warp_argmax(a);
    __syncwarp();
    const bool found = a.i < experts;              // (false only if fewer experts are allowed than asked for)
    if (lane == 0) {
      choice[static_cast<size_t>(t) * top + k] = found ? a.i : 0;
      weight[static_cast<size_t>(t) * top + k] = found ? score[a.i] : 0.f;
      if (found) work[a.i] = -INFINITY;
    }
    if (found) total += score[a.i];
    __syncwarp();
  }
  if (lane == 0 && (a.renorm || a.weight_scale != 1.f)) {
    for (int k = 0; k < top; ++k) {
      float wk = weight[static_cast<size_t>(t) * top + k];
      if (a.renorm) wk /= total + a.renorm_floor;
      weight[static_cast<size_t>(t) * top + k] = wk * a.weight_scale;
    }
  }
}

template <typename TA, typename TW>
__global__ void moe_route_kernel(const TA* __restrict__ x, const TW* __restrict__ router, const RouteArgs a,
                                 int32_t* __restrict__ choice, float* __restrict__ weight) {
  pdl_launch();
  pdl_wait();
  extern __shared__ float sm[];
  const int warps = blockDim.x >> 5, warp = threadIdx.x >> 5;
  const int t = blockIdx.x * warps + warp;
  if (t >= a.tokens) return;
  route_token(a, x + static_cast<size_t>(t) * a.ld, router, t, sm + warp * (2 * a.experts + 2 * a.groups), choice, weight);
}

// ------------------------------------------------------------------ pairs grouped by expert
// One CTA.  counts -> offsets -> order (an expert's pairs in ascending order); then the tiles.  meta: [0] number of
// tiles.
constexpr int kTileRows = 64;
constexpr int kGroupThreads = 1024;

// Offsets of the experts' lists and their tiles from the counts; by one warp (running sums, 32 experts at a time;
// experts from `tiled` on have no matrices and get no tiles).
__device__ __forceinline__ void group_offsets(const int32_t* cnt, int experts, int tiled, int32_t* off, int32_t* first,
                                              int32_t* __restrict__ meta) {
  const int lane = threadIdx.x & 31;
  int at = 0, tiles = 0;
  for (int e0 = 0; e0 < experts; e0 += 32) {
    const int e = e0 + lane, n = e < experts ? cnt[e] : 0;
    const int nt = e < tiled ? (n + kTileRows - 1) / kTileRows : 0;
    int s = n, st = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, s, o), v = __shfl_up_sync(0xffffffffu, st, o);
      if (lane >= o) {
        s += u;
        st += v;
      }
    }
    if (e < experts) {
      off[e] = at + s - n;
      first[e] = tiles + st - nt;
    }
    at += __shfl_sync(0xffffffffu, s, 31);
    tiles += __shfl_sync(0xffffffffu, st, 31);
  }
  if (lane == 0) meta[0] = tiles;
}
__device__ __forceinline__ void group_tiles(const int32_t* cnt, const int32_t* off, const int32_t* first, int experts,
                                            int tiled, int32_t* __restrict__ tile_expert, int32_t* __restrict__ tile_begin,
                                            int32_t* __restrict__ tile_rows) {
  for (int e = threadIdx.x; e < experts && e < tiled; e += blockDim.x)
    for (int r = 0, i = first[e]; r < cnt[e]; r += kTileRows, ++i) {
      tile_expert[i] = e;
      tile_begin[i] = off[e] + r;
      tile_rows[i] = min(kTileRows, cnt[e] - r);
    }
}

// Every warp counts the experts of a run of pairs of its own (`rows` warps share the work: as many as their
// counters fit in shared memory); the runs' counts are summed in order, and a pair's place is its expert's offset,
// the counts of the runs before, and its rank within the run (pairs of one expert among 32 find each other by a
// warp-wide match).
__global__ void __launch_bounds__(kGroupThreads)
moe_group_kernel(const int32_t* __restrict__ choice, int pairs, int experts, int tiled, int rows,
                 int32_t* __restrict__ order, int32_t* __restrict__ tile_expert,
                 int32_t* __restrict__ tile_begin, int32_t* __restrict__ tile_rows, int32_t* __restrict__ meta) {
  pdl_launch();
  pdl_wait();
  extern __shared__ int32_t cnt[];          // [experts] counts, offsets, first tiles; [rows][experts] the runs' counts
  int32_t *off = cnt + experts, *first = off + experts, *hist = first + experts;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int i = threadIdx.x; i < rows * experts; i += blockDim.x) hist[i] = 0;
  __syncthreads();
  const int run = ((pairs + rows - 1) / rows + 31) / 32 * 32;
  int32_t* mine = hist + warp * experts;
  const int begin = warp * run, end = min(pairs, begin + run);
  if (warp < rows)
    for (int p0 = begin; p0 < end; p0 += 32) {
      const int p = p0 + lane;
      const int e = p < end ? choice[p] : -1;
      const unsigned same = __match_any_sync(0xffffffffu, e);
      if (e >= 0 && lane == __ffs(same) - 1) mine[e] += __popc(same);
      __syncwarp();
    }
  __syncthreads();
  for (int e = threadIdx.x; e < experts; e += blockDim.x) {
    int sum = 0;
    for (int w = 0; w < rows; ++w) {
      const int n = hist[w * experts + e];
      hist[w * experts + e] = sum;
      sum += n;
    }
    cnt[e] = sum;
  }
  __syncthreads();
  if (warp == 0) group_offsets(cnt, experts, tiled, off, first, meta);
  __syncthreads();
  group_tiles(cnt, off, first, experts, tiled, tile_expert, tile_begin, tile_rows);
  if (warp < rows)
    for (int p0 = begin; p0 < end; p0 += 32) {
      const int p = p0 + lane;
      const int e = p < end ? choice[p] : -1;
      const unsigned same = __match_any_sync(0xffffffffu, e);
      if (e >= 0) order[off[e] + mine[e] + __popc(same & ((1u << lane) - 1))] = p;
      __syncwarp();
      if (e >= 0 && lane == __ffs(same) - 1) mine[e] += __popc(same);
      __syncwarp();
    }
}

// Router and grouping of a step of few tokens in one CTA, a warp per token (float32 logits; every pair gets its
// place as in moe_group_kernel).
__global__ void __launch_bounds__(512)
moe_route_group_kernel(const float* __restrict__ x, const RouteArgs a, int tiled, int32_t* choice, float* weight,
                       int32_t* __restrict__ order, int32_t* __restrict__ tile_expert, int32_t* __restrict__ tile_begin,
                       int32_t* __restrict__ tile_rows, int32_t* __restrict__ meta) {
  pdl_launch();
  pdl_wait();
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, nwarps = blockDim.x >> 5;
  const int per = 2 * a.experts + 2 * a.groups, pairs = a.tokens * a.top;
  int32_t* chosen = reinterpret_cast<int32_t*>(sm + nwarps * per);      // [pairs], then [experts] counts, offsets, first tiles
  int32_t* cnt = chosen + pairs;
  int32_t* off = cnt + a.experts;
  int32_t* first = off + a.experts;
  for (int t = warp; t < a.tokens; t += nwarps) {
    route_token<float, float>(a, x + static_cast<size_t>(t) * a.ld, nullptr, t, sm + warp * per, choice, weight);
    __syncwarp();
    for (int k = lane; k < a.top; k += 32) chosen[t * a.top + k] = choice[static_cast<size_t>(t) * a.top + k];
  }
  __syncthreads();
  for (int e = threadIdx.x; e < a.experts; e += blockDim.x) {
    int n = 0;
    for (int p = 0; p < pairs; ++p) n += chosen[p] == e;
    cnt[e] = n;
  }
  __syncthreads();
  if (warp == 0) group_offsets(cnt, a.experts, tiled, off, first, meta);
  __syncthreads();
  group_tiles(cnt, off, first, a.experts, tiled, tile_expert, tile_begin, tile_rows);
  for (int p = threadIdx.x; p < pairs; p += blockDim.x) {
    const int e = chosen[p];
    int before = 0;
    for (int q = 0; q < p; ++q) before += chosen[q] == e;
    order[off[e] + before] = p;
  }
}

// ------------------------------------------------------------------ grouped products
// One CTA per (tile of up to 64 pairs of one expert, 64 output features).  Row r of the tile is pair
// order[begin + r]; its input row is src[pair / src_div] (src_div = top for the first product, whose
// input is the token's row; 1 for the second, whose input is the pair's own row); its output row is
// dst[pair].  W is [experts, n, k].
template <typename TA, typename TW>
__global__ void __launch_bounds__(128)
moe_gemm_simt_kernel(const TA* __restrict__ src, int ld_src, int src_div, const TW* __restrict__ w, int n, int k,
                     TA* __restrict__ dst, int ld_dst, const int32_t* __restrict__ order,
                     const int32_t* __restrict__ tile_expert, const int32_t* __restrict__ tile_begin,
                     const int32_t* __restrict__ tile_rows, const int32_t* __restrict__ meta, int act) {
  pdl_launch();
  pdl_wait();
  constexpr int BM = kTileRows, BN = 64, BK = 32, RPT = BM / 8;
  __shared__ float As[BM][BK + 1];
  __shared__ float Ws[BN][BK + 1];
  __shared__ int32_t pair_of[BM];
  const int tile = blockIdx.x;
  if (tile >= meta[0]) return;
  const int e = tile_expert[tile], begin = tile_begin[tile], rows = tile_rows[tile];
  const int n0 = blockIdx.y * BN;
  const TW* we = w + static_cast<size_t>(e) * n * k;
  if (threadIdx.x < BM) pair_of[threadIdx.x] = threadIdx.x < rows ? order[begin + threadIdx.x] : -1;
  __syncthreads();
  // thread (ty, tx): rows ty * 8 .. + 7 (8 groups), columns tx, tx + 16, tx + 32, tx + 48
  const int ty = threadIdx.x / 16, tx = threadIdx.x % 16;
  float acc[RPT][4];
#pragma unroll
  for (int i = 0; i < RPT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  for (int k0 = 0; k0 < k; k0 += BK) {
    __syncthreads();
    for (int i = threadIdx.x; i < BM * BK; i += 128) {
      const int r = i / BK, c = i - r * BK;
      const int p = pair_of[r];
      As[r][c] = (p >= 0 && k0 + c < k) ? to_float(src[static_cast<size_t>(p / src_div) * ld_src + k0 + c]) : 0.f;
    }
    for (int i = threadIdx.x; i < BN * BK; i += 128) {
      const int r = i / BK, c = i - r * BK;
      Ws[r][c] = (n0 + r < n && k0 + c < k) ? to_float(we[static_cast<size_t>(n0 + r) * k + k0 + c]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int c = 0; c < BK; ++c) {
      float av[RPT], wv[4];
#pragma unroll
      for (int i = 0; i < RPT; ++i) av[i] = As[ty * RPT + i][c];
#pragma unroll
      for (int j = 0; j < 4; ++j) wv[j] = Ws[tx + 16 * j][c];
#pragma unroll
      for (int i = 0; i < RPT; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
  }
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int p = pair_of[ty * RPT + i];
    if (p < 0) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int col = n0 + tx + 16 * j;
      if (col < n) dst[static_cast<size_t>(p) * ld_dst + col] = from_float<TA>(moe_activate(acc[i][j], act));
    }
  }
}

// The tile on the tensor cores for bfloat16: 64 pairs x 128 output features per CTA, eight warps in a
// 2 x 4 grid (32 rows x 32 features each: 2 x 4 MMAs per 16 of k).  A (the pairs' rows) and W blocks of 64 k
// come by asynchronous copies into a ring of three stages, two of which are on their way while the MMAs of the
// third run; fragments by ldmatrix.  mma.sync.m16n8k16, float32 accumulators, k ascending.
__device__ __forceinline__ void mma_bf16_16816(float* d, const uint32_t* a, const uint32_t* b) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__device__ __forceinline__ void ldmatrix4(uint32_t* r, unsigned addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// 16 bytes on their way, or zeros
__device__ __forceinline__ void async_piece(unsigned dst, const void* src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0));
}

constexpr int kMmaCols = 128, kMmaK = 64, kMmaStages = 3, kMmaLd = kMmaK + 8;      // 144-byte rows: ldmatrix hits distinct banks
constexpr int kMmaStage = (kTileRows + kMmaCols) * kMmaLd;                         // elements of a stage: A rows, then W rows
constexpr int kMmaSmem = kMmaStages * kMmaStage * 2;

__global__ void __launch_bounds__(256, 2)
moe_gemm_mma_kernel(const bf16* __restrict__ src, int ld_src, int src_div, const bf16* __restrict__ w, int n, int k,
                    bf16* __restrict__ dst, int ld_dst, const int32_t* __restrict__ order,
                    const int32_t* __restrict__ tile_expert, const int32_t* __restrict__ tile_begin,
                    const int32_t* __restrict__ tile_rows, const int32_t* __restrict__ meta, int act) {
  pdl_launch();
  pdl_wait();
  constexpr int BM = kTileRows, BN = kMmaCols, BK = kMmaK, LD = kMmaLd;
  extern __shared__ __align__(16) bf16 ring[];
  __shared__ int32_t pair_of[BM];
  const int tile = blockIdx.x;
  if (tile >= meta[0]) return;
  const int e = tile_expert[tile], begin = tile_begin[tile], rows = tile_rows[tile];
  const int n0 = blockIdx.y * BN;
  const bf16* we = w + static_cast<size_t>(e) * n * k;
  if (threadIdx.x < BM) pair_of[threadIdx.x] = threadIdx.x < rows ? order[begin + threadIdx.x] : -1;
  __syncthreads();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int gid = lane >> 2, tig = lane & 3;
  const int wm = warp & 1, wn = warp >> 1;            // this warp's 32 rows and 32 features
  float acc[2][4][4];
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int f = 0; f < 4; ++f) acc[i][j][f] = 0.f;
  // this thread's pieces of a k block: rows (tid / 8) + 32 i of A (i < 2) and of W (i < 4), piece tid % 8
  const int pr = threadIdx.x >> 3, pc = (threadIdx.x & 7) * 8;
  const bf16* a_src[2];
  const bf16* w_src[4];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int p = pair_of[pr + 32 * i];
    a_src[i] = p >= 0 ? src + static_cast<size_t>(p / src_div) * ld_src + pc : nullptr;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = n0 + pr + 32 * i;
    w_src[i] = r < n ? we + static_cast<size_t>(r) * k + pc : nullptr;
  }
  const unsigned base = static_cast<unsigned>(__cvta_generic_to_shared(ring));
  auto fetch = [&](int stage, int k0) {
    const unsigned at = base + static_cast<unsigned>(stage * kMmaStage + pr * LD + pc) * 2;
    const bool in = k0 + pc < k;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const bool ok = in && a_src[i] != nullptr;
      async_piece(at + 32 * i * LD * 2, ok ? a_src[i] + k0 : src, ok);
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const bool ok = in && w_src[i] != nullptr;
      async_piece(at + (BM + 32 * i) * LD * 2, ok ? w_src[i] + k0 : w, ok);
    }
  };
  const int blocks = (k + BK - 1) / BK;
#pragma unroll
  for (int s = 0; s < kMmaStages - 1; ++s) {
    if (s < blocks) fetch(s, s * BK);
    asm volatile("cp.async.commit_group;" ::: "memory");
  }
  // where this lane's ldmatrix rows begin: A rows (16 x 16 tiles), W rows (two tiles of 8 features x 16 k)
  const unsigned a_row = (wm * 32 + (lane & 15)) * LD + (lane >> 4) * 8;
  const unsigned w_row = (BM + wn * 32 + (lane & 7) + (lane & 16 ? 8 : 0)) * LD + (lane & 8 ? 8 : 0);
  int stage = 0;
  for (int b = 0; b < blocks; ++b) {
    asm volatile("cp.async.wait_group %0;" ::"n"(kMmaStages - 2) : "memory");
    __syncthreads();                                  // block b has arrived for all; block b - 1 has been read by all
    const int ahead = b + kMmaStages - 1;
    if (ahead < blocks) fetch(stage == 0 ? kMmaStages - 1 : stage - 1, ahead * BK);
    asm volatile("cp.async.commit_group;" ::: "memory");
    const unsigned at = base + static_cast<unsigned>(stage * kMmaStage) * 2;
#pragma unroll
    for (int kk = 0; kk < BK; kk += 16) {
      uint32_t fa[2][4], fb[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) ldmatrix4(fa[i], at + (a_row + i * 16 * LD + kk) * 2);
#pragma unroll
      for (int j = 0; j < 2; ++j) ldmatrix4(fb[j], at + (w_row + j * 16 * LD + kk) * 2);
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) mma_bf16_16816(acc[i][j], fa[i], &fb[j >> 1][(j & 1) * 2]);
    }
    stage = stage == kMmaStages - 1 ? 0 : stage + 1;
  }
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int p = pair_of[wm * 32 + i * 16 + gid + half * 8];
      if (p < 0) continue;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = n0 + wn * 32 + j * 8 + tig * 2;
        const float v0 = moe_activate(acc[i][j][half * 2], act), v1 = moe_activate(acc[i][j][half * 2 + 1], act);
        bf16* d = dst + static_cast<size_t>(p) * ld_dst + col;
        if (col + 1 < n && (ld_dst % 2 == 0)) {
          *reinterpret_cast<__nv_bfloat162*>(d) = __floats2bfloat162_rn(v0, v1);
        } else {
          if (col < n) d[0] = __float2bfloat16_rn(v0);
          if (col + 1 < n) d[1] = __float2bfloat16_rn(v1);
        }
      }
    }
}

__device__ __forceinline__ uint4 stream16(const void* p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}

// For a handful of pairs (single-token steps) the products are bound by the stream of the chosen experts'
// weights: one CTA per (tile, 16 output features), a warp takes four features at once and streams their
// weight rows in 16-byte pieces, up to four of the tile's rows at a time (their input rows come from L1).
// GATED: an expert has 2 n rows, gate rows and then up rows, and the result is act(gate) * up (two features and
// their four rows at once; gate and up rounded to the activation type first, as when they are stored).
template <typename T, bool GATED>
__global__ void __launch_bounds__(128)
moe_gemv_kernel(const T* __restrict__ src, int ld_src, int src_div, const T* __restrict__ w, int n, int k,
                T* __restrict__ dst, int ld_dst, const int32_t* __restrict__ order,
                const int32_t* __restrict__ tile_expert, const int32_t* __restrict__ tile_begin,
                const int32_t* __restrict__ tile_rows, const int32_t* __restrict__ meta, int act, float limit,
                float slope) {
  pdl_launch();
  pdl_wait();
  constexpr int VEC = Vec16<T>::N, NF = 4, NR = 4, OF = GATED ? NF / 2 : NF;      // OF: output features of a warp
  const int tile = blockIdx.x;
  if (tile >= meta[0]) return;
  const int e = tile_expert[tile], begin = tile_begin[tile], rows = tile_rows[tile];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int f0 = (blockIdx.y * 4 + warp) * OF;
  if (f0 >= n) return;
  const T* we = w + static_cast<size_t>(e) * (GATED ? 2 * n : n) * k;
  const T* wr[NF];                               // (a feature beyond n: the last one's row, its result is not stored)
#pragma unroll
  for (int f = 0; f < NF; ++f)
    wr[f] = we + (static_cast<size_t>(min(f0 + f % OF, n - 1)) + (f >= OF ? n : 0)) * k;
  const bool vec = (k % VEC == 0) && (ld_src % VEC == 0) && (reinterpret_cast<uintptr_t>(src) % 16 == 0) &&
                   (reinterpret_cast<uintptr_t>(w) % 16 == 0);
  for (int r0 = 0; r0 < rows; r0 += NR) {
    const int nr = min(NR, rows - r0);
    int pair[NR];
    const T* xr[NR];
#pragma unroll
    for (int r = 0; r < NR; ++r) {
      pair[r] = r < nr ? order[begin + r0 + r] : 0;
      xr[r] = src + static_cast<size_t>(pair[r] / src_div) * ld_src;
    }
    float acc[NF][NR];
#pragma unroll
    for (int f = 0; f < NF; ++f)
#pragma unroll
      for (int r = 0; r < NR; ++r) acc[f][r] = 0.f;
    if (vec) {
      // (the next pieces of the weight rows are asked for before the sums over the present ones)
      uint4 cur[NF];
      int c = lane * VEC;
#pragma unroll
      for (int f = 0; f < NF; ++f) cur[f] = c < k ? stream16(wr[f] + c) : make_uint4(0, 0, 0, 0);
      for (; c < k; c += 32 * VEC) {
        uint4 nxt[NF];
        const int cn = c + 32 * VEC;
#pragma unroll
        for (int f = 0; f < NF; ++f) nxt[f] = cn < k ? stream16(wr[f] + cn) : make_uint4(0, 0, 0, 0);
        float wv[NF][VEC];
#pragma unroll
        for (int f = 0; f < NF; ++f) load16(reinterpret_cast<const T*>(&cur[f]), wv[f]);
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          if (r < nr) {
            float xv[VEC];
            load16(xr[r] + c, xv);
#pragma unroll
            for (int f = 0; f < NF; ++f)
#pragma unroll
              for (int i = 0; i < VEC; ++i) acc[f][r] = fmaf(wv[f][i], xv[i], acc[f][r]);
          }
        }
#pragma unroll
        for (int f = 0; f < NF; ++f) cur[f] = nxt[f];
      }
    } else {
      for (int c = lane; c < k; c += 32) {
#pragma unroll
        for (int r = 0; r < NR; ++r) {
          const float xv = r < nr ? to_float(xr[r][c]) : 0.f;
#pragma unroll
          for (int f = 0; f < NF; ++f)
            acc[f][r] = fmaf(to_float(wr[f][c]), xv, acc[f][r]);
        }
      }
    }
#pragma unroll
    for (int f = 0; f < OF; ++f)
#pragma unroll
      for (int r = 0; r < NR; ++r) {
        float v = warp_sum(acc[f][r]);
        if (GATED) {
          const float up = to_float(from_float<T>(warp_sum(acc[f + NF - OF][r])));
          v = to_float(from_float<T>(v));
          if (act == ACT_CLAMPED_SWISH) {
            const float g = fminf(v, limit);
            v = g / (1.f + expf(-slope * g)) * (fminf(fmaxf(up, -limit), limit) + 1.f);
          } else {
            v = moe_activate(v, act) * up;
          }
        } else {
          v = moe_activate(v, act);
        }
        if (lane == 0 && r < nr && f0 + f < n) dst[static_cast<size_t>(pair[r]) * ld_dst + f0 + f] = from_float<T>(v);
      }
  }
}

// ------------------------------------------------------------------ combine
// out[t, c] = sum_k weight[t, k] * y[t * top + k, c] (+ shared[t, c])
template <typename TA>
__global__ void moe_combine_kernel(const TA* __restrict__ y, const float* __restrict__ weight,
                                   const TA* __restrict__ shared, TA* __restrict__ out, int width, int top,
                                   const int32_t* __restrict__ choice, int real_experts, const TA* __restrict__ x,
                                   int ld_x, const float* __restrict__ shared_gate, int ld_gate) {
  pdl_launch();
  pdl_wait();
  const int t = blockIdx.y;
  const float sg = shared_gate != nullptr ? 1.f / (1.f + expf(-shared_gate[static_cast<size_t>(t) * ld_gate])) : 1.f;
  for (int c = blockIdx.x * blockDim.x + threadIdx.x; c < width; c += gridDim.x * blockDim.x) {
    float s = 0.f;
    for (int k = 0; k < top; ++k) {
      const size_t pair = static_cast<size_t>(t) * top + k;
      // (an identity expert's pair has no product: its term is the token's input row)
      const bool same = choice != nullptr && choice[pair] >= real_experts;
      s = fmaf(weight[pair], same ? to_float(x[static_cast<size_t>(t) * ld_x + c]) : to_float(y[pair * width + c]), s);
    }
    if (shared != nullptr) s = fmaf(sg, to_float(shared[static_cast<size_t>(t) * width + c]), s);
    out[static_cast<size_t>(t) * width + c] = from_float<TA>(s);
  }
}

}  // namespace rl

using namespace rl;

extern "C" {

int rl_moe_tile_rows() { return kTileRows; }

int rl_moe_route(const void* x, int act_dtype, int ld, const void* router, int w_dtype, int tokens, int width,
                 int experts, int groups, int keep, int group_top, int top, int softmax, int renorm, const float* bias,
                 const float* choice_bias, float weight_scale, float renorm_floor, int32_t* choice, float* weight,
                 cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const int warps = 4;
  const size_t smem = static_cast<size_t>(warps) * (2 * experts + 2 * groups) * sizeof(float);
  dim3 grid((tokens + warps - 1) / warps), block(warps * 32);
  const RouteArgs a{ld, tokens, width, experts, groups, keep, group_top, top, softmax, renorm, bias, choice_bias,
                    weight_scale, renorm_floor};
#define RL_CASE(TA, TW)                                                                                            \
  launch_kernel(moe_route_kernel<TA, TW>, grid, block, smem, stream, static_cast<const TA*>(x),                    \
                static_cast<const TW*>(router), a, choice, weight)
  if (act_dtype == 0) RL_CASE(float, float);
  else if (w_dtype == 0) RL_CASE(bf16, float);
  else RL_CASE(bf16, bf16);
#undef RL_CASE
  RL_LAUNCH_END();
}

// Router (from float32 logits) and grouping in one launch; tokens * top at most 256.
int rl_moe_route_group(const float* logits, int ld, int tokens, int experts, int groups, int keep, int group_top, int top,
                       int softmax, int renorm, const float* bias, const float* choice_bias, float weight_scale,
                       float renorm_floor, int tiled, int32_t* choice, float* weight, int32_t* order,
                       int32_t* tile_expert, int32_t* tile_begin, int32_t* tile_rows, int32_t* meta,
                       cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (tokens * top > 256) return static_cast<int>(cudaErrorInvalidValue);
  const int warps = max(4, min(16, tokens));
  const size_t smem = (static_cast<size_t>(warps) * (2 * experts + 2 * groups) + tokens * top + 3 * experts) * sizeof(float);
  if (smem > 48 * 1024) return static_cast<int>(cudaErrorInvalidValue);
  const RouteArgs a{ld, tokens, 0, experts, groups, keep, group_top, top, softmax, renorm, bias, choice_bias,
                    weight_scale, renorm_floor};
  launch_kernel(moe_route_group_kernel, dim3(1), dim3(warps * 32), smem, stream, logits, a, tiled, choice, weight, order,
                tile_expert, tile_begin, tile_rows, meta);
  RL_LAUNCH_END();
}

int rl_moe_group(const int32_t* choice, int pairs, int experts, int tiled, int32_t* order, int32_t* tile_expert,
                 int32_t* tile_begin, int32_t* tile_rows, int32_t* meta, cudaStream_t stream) {
  if (pairs <= 0) return 0;
  // as many runs as there are warps' worth of pairs and as fit 48 KB of counters
  int rows = max(1, min(kGroupThreads / 32, (pairs + 31) / 32));
  while (rows > 1 && (3 + rows) * experts * sizeof(int32_t) > 48 * 1024) rows /= 2;
  const size_t smem = (3 + static_cast<size_t>(rows)) * experts * sizeof(int32_t);
  if (smem > 48 * 1024) return static_cast<int>(cudaErrorInvalidValue);
  launch_kernel(moe_group_kernel, dim3(1), dim3(min(kGroupThreads, max(128, rows * 32))), smem, stream, choice, pairs,
                experts, tiled, rows, order, tile_expert, tile_begin, tile_rows, meta);
  RL_LAUNCH_END();
}

// max_tiles: the most tiles the grouping can have made (pairs / 64 + experts); CTAs beyond the real
// number leave at once.  few_pairs: the weight-streaming kernel for a handful of pairs (single-token steps), which
// can also form act(gate) * up from an expert's 2 n rows (gated).
int rl_moe_gemm(int act_dtype, const void* src, int ld_src, int src_div, const void* w, int n, int k, void* dst,
                int ld_dst, const int32_t* order, const int32_t* tile_expert, const int32_t* tile_begin,
                const int32_t* tile_rows, const int32_t* meta, int max_tiles, int few_pairs, int act, int gated,
                float limit, float slope, cudaStream_t stream) {
  if (max_tiles <= 0) return 0;
  if (gated && !few_pairs) return static_cast<int>(cudaErrorInvalidValue);
  if (few_pairs) {
    dim3 g(max_tiles, (n + (gated ? 7 : 15)) / (gated ? 8 : 16));
#define RL_CASE(T, G)                                                                                              \
  launch_kernel(moe_gemv_kernel<T, G>, g, dim3(128), 0, stream, static_cast<const T*>(src), ld_src, src_div,      \
                static_cast<const T*>(w), n, k, static_cast<T*>(dst), ld_dst, order, tile_expert, tile_begin,     \
                tile_rows, meta, act, limit, slope)
    if (act_dtype == 0) {
      if (gated) RL_CASE(float, true); else RL_CASE(float, false);
    } else {
      if (gated) RL_CASE(bf16, true); else RL_CASE(bf16, false);
    }
#undef RL_CASE
    RL_LAUNCH_END();
  }
  dim3 grid(max_tiles, (n + 63) / 64);
  if (act_dtype == 0) {
    launch_kernel(moe_gemm_simt_kernel<float, float>, grid, dim3(128), 0, stream, static_cast<const float*>(src),
                  ld_src, src_div, static_cast<const float*>(w), n, k, static_cast<float*>(dst), ld_dst, order,
                  tile_expert, tile_begin, tile_rows, meta, act);
  } else if (k % 8 == 0 && ld_src % 8 == 0 && (reinterpret_cast<uintptr_t>(src) % 16 == 0) &&
             (reinterpret_cast<uintptr_t>(w) % 16 == 0)) {
    static bool raised = false;
    if (!raised) {
      const cudaError_t e = cudaFuncSetAttribute(moe_gemm_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kMmaSmem);
      if (e != cudaSuccess) return static_cast<int>(e);
      raised = true;
    }
    launch_kernel(moe_gemm_mma_kernel, dim3(max_tiles, (n + kMmaCols - 1) / kMmaCols), dim3(256), kMmaSmem, stream,
                  static_cast<const bf16*>(src), ld_src, src_div,
                  static_cast<const bf16*>(w), n, k, static_cast<bf16*>(dst), ld_dst, order, tile_expert, tile_begin,
                  tile_rows, meta, act);
  } else {
    launch_kernel(moe_gemm_simt_kernel<bf16, bf16>, grid, dim3(128), 0, stream, static_cast<const bf16*>(src), ld_src,
                  src_div, static_cast<const bf16*>(w), n, k, static_cast<bf16*>(dst), ld_dst, order, tile_expert,
                  tile_begin, tile_rows, meta, act);
  }
  RL_LAUNCH_END();
}

int rl_moe_combine(int act_dtype, const void* y, const float* weight, const void* shared, void* out, int tokens,
                   int width, int top, const int32_t* choice, int real_experts, const void* x, int ld_x,
                   const float* shared_gate, int ld_gate, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  dim3 grid(min((width + 255) / 256, 32), tokens);
  if (act_dtype == 0)
    launch_kernel(moe_combine_kernel<float>, grid, dim3(256), 0, stream, static_cast<const float*>(y), weight,
                  static_cast<const float*>(shared), static_cast<float*>(out), width, top, choice, real_experts,
                  static_cast<const float*>(x), ld_x, shared_gate, ld_gate);
  else
    launch_kernel(moe_combine_kernel<bf16>, grid, dim3(256), 0, stream, static_cast<const bf16*>(y), weight,
                  static_cast<const bf16*>(shared), static_cast<bf16*>(out), width, top, choice, real_experts,
                  static_cast<const bf16*>(x), ld_x, shared_gate, ld_gate);
  RL_LAUNCH_END();
}

}  // extern "C"
