// Attention over a cached latent: what lies between the projections and the attention kernel, and the
// per-head products around it.
//
// A token's projection row holds, per head, a query [n | r] (n unrotated entries, r rotated ones) and, behind
// the queries, [c' | k_r]: the raw latent of `rank` entries and one rotated key part of r entries that all
// heads share.  Keys and values of head h are W_uk,h c and W_uv,h c with c = c' / rms(c') * w, so
//     q_n . (W_uk,h c) = (W_uk,h^T q_n) . c      and      sum_j p_j W_uv,h c_j = W_uv,h (sum_j p_j c_j):
// attention runs over the cached rows [c | k_r] themselves, one key head for all query heads, with the query
// [W_uk,h^T q_n | q_r] and the row's first `rank` entries as the value; W_uv,h is applied to its result.
//
// The queries may come from a latent of their own (RMS-normed, then a product), and a layer may attend over
// the rows another layer has cached; the three jobs of latent_prep can then be asked for one by one.
//
//   latent_prep   per token: c (RMS norm in float32, weight w), k_r and every head's q_r turned by the
//                 token's position (entry i with entry i + dims/2 of the first `dims` rotated entries, or
//                 neighbours, cos and sin from tables), [c | k_r] into the paged cache, q_r into the
//                 attention's query rows; the norm of the queries' latent
//   head_linear   y[t, h, :] = W_h x[t, h, :] for every head h, W [heads, n, k], float32 sums, times
//                 sigmoid(gate[t, h, :]) where a gate is given; the heads' rotated query parts may go along; FFMA for float32, mma.sync.m16n8k16 for bfloat16
//                 operands whose sizes allow it, and a kernel that streams the weights for up to 16 tokens
#include "common.cuh"

namespace rl {

struct LatentPrepArgs {
  int q_src_ld;      // row length of the buffer the queries lie in
  int c_ld;          // row length of the buffer the raw latent lies in
  int heads, dn, dr, rank, rot_dims;
  int q_ld;          // row length of the attention's query buffer: heads * (rank + dr)
  float eps;
  int page_size;
  long long num_slots;
  int max_pos;       // rows of the tables
  int pairs;         // rotated entries 2i and 2i + 1 turn together (else i and i + rot_dims / 2)
  int dq_ld, dq_rank, dq_out_ld;     // a latent of the queries, normed for the product behind it
};

// Entry d of a rotated part, turned.
template <typename TA>
__device__ __forceinline__ float rotated(const TA* __restrict__ src, int d, int rot_dims, int pairs,
                                         const float* __restrict__ cs, const float* __restrict__ sn) {
  const float v = to_float(src[d]);
  if (d >= rot_dims) return v;
  const int half = rot_dims / 2;
  const bool first = pairs ? (d & 1) == 0 : d < half;
  const int i = pairs ? d >> 1 : (first ? d : d - half), gap = pairs ? 1 : half;
  return first ? v * cs[i] - to_float(src[d + gap]) * sn[i] : v * cs[i] + to_float(src[d - gap]) * sn[i];
}

// One CTA per token; each of the three jobs is done where its buffers are given: the heads' rotated query
// parts (q), the norm of the queries' latent (dq), the latent and the shared key part into the cache (craw and
// slots).  A position beyond the tables sets bit 1 of *status, a slot beyond the pool bit 2 (negative slot: no
// write).
template <typename TA, typename TW>
__global__ void __launch_bounds__(128)
latent_prep_kernel(const TA* __restrict__ q, const TA* __restrict__ craw, const int32_t* __restrict__ positions,
                   const TW* __restrict__ w, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                   TA* __restrict__ qa, const int32_t* __restrict__ slots, TA* __restrict__ cache,
                   const TA* __restrict__ dq, const TW* __restrict__ dq_w, TA* __restrict__ dq_out, int* status,
                   const LatentPrepArgs a) {
  pdl_launch();
  pdl_wait();
  __shared__ float scratch[32];
  const int t = blockIdx.x;
  const int half = a.rot_dims / 2;
  int pos = positions[t];
  if (a.dr > 0 && (pos < 0 || pos >= a.max_pos)) {
    if (threadIdx.x == 0) atomicOr(status, 2);
    pos = 0;
  }
  const float* cs = cos_t + static_cast<size_t>(pos) * half;
  const float* sn = sin_t + static_cast<size_t>(pos) * half;
  if (q != nullptr) {
    // ---- the heads' rotated query parts
    const TA* row = q + static_cast<size_t>(t) * a.q_src_ld;
    TA* qrow = qa + static_cast<size_t>(t) * a.q_ld;
    for (int i = threadIdx.x; i < a.heads * a.dr; i += blockDim.x) {
      const int h = i / a.dr, d = i - h * a.dr;
      qrow[h * (a.rank + a.dr) + a.rank + d] =
          from_float<TA>(rotated(row + h * (a.dn + a.dr) + a.dn, d, a.rot_dims, a.pairs, cs, sn));
    }
  }
  if (dq != nullptr) {
    // ---- the queries' latent, normed
    const TA* src = dq + static_cast<size_t>(t) * a.dq_ld;
    float ss = 0.f;
    for (int i = threadIdx.x; i < a.dq_rank; i += blockDim.x) {
      const float v = to_float(src[i]);
      ss += v * v;
    }
    const float r = rsqrtf(block_sum(ss, scratch) / static_cast<float>(a.dq_rank) + a.eps);
    TA* dst = dq_out + static_cast<size_t>(t) * a.dq_out_ld;
    for (int i = threadIdx.x; i < a.dq_rank; i += blockDim.x) dst[i] = from_float<TA>(to_float(src[i]) * r * to_float(dq_w[i]));
  }
  if (craw == nullptr || slots == nullptr) return;
  // ---- the latent and the shared key part into the cache
  const TA* c = craw + static_cast<size_t>(t) * a.c_ld;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) {
    const float v = to_float(c[i]);
    ss += v * v;
  }
  const float r = rsqrtf(block_sum(ss, scratch) / static_cast<float>(a.rank) + a.eps);
  const int slot = slots[t];
  if (slot < 0) return;
  if (slot >= a.num_slots) {
    if (threadIdx.x == 0) atomicOr(status, 4);
    return;
  }
  TA* dst = cache + static_cast<size_t>(slot) * (a.rank + a.dr);     // one key head: [pages, 1, page, rank + dr]
  for (int i = threadIdx.x; i < a.rank; i += blockDim.x) dst[i] = from_float<TA>(to_float(c[i]) * r * to_float(w[i]));
  for (int d = threadIdx.x; d < a.dr; d += blockDim.x)
    dst[a.rank + d] = from_float<TA>(rotated(c + a.rank, d, a.rot_dims, a.pairs, cs, sn));
}

// ------------------------------------------------------------------ per-head products
// y[t, y_col + h * y_head + j] = sum_k W[h, j, k] x[t, x_col + h * x_head + k]
// and, with turn.dims > 0, the rotated part of every head's row goes along: y[t, y_col + h * y_head + turn.y + d] =
// entry d of the part at x[t, x_col + h * x_head + turn.x], turned by the token's position (see `rotated`).
struct Turn {
  int dims, rot_dims, pairs, x, y, max_pos;      // dims: entries of the part, of which the first rot_dims turn
  const float *cos_t, *sin_t;                    // [max_pos, rot_dims / 2]
  const int32_t* positions;
  int* status;
};
struct HeadLinearArgs {
  int tokens, heads, n, k;
  int x_ld, x_col, x_head;
  int y_ld, y_col, y_head;
  Turn turn;
  const void* gate;        // [tokens, heads * n] in rows of gate_ld entries of the activation type, or null
  int gate_ld;
};

// The factor of output j of head h for token t.
template <typename TA>
__device__ __forceinline__ float gate_of(const HeadLinearArgs& a, int t, int h, int j) {
  if (a.gate == nullptr) return 1.f;
  const float g = to_float(static_cast<const TA*>(a.gate)[static_cast<size_t>(t) * a.gate_ld + h * a.n + j]);
  return 1.f / (1.f + expf(-g));
}

// The rotated parts of tokens t0 .. t0 + rows - 1 of head h, by all threads of a CTA.
template <typename TA>
__device__ __forceinline__ void turn_parts(const TA* __restrict__ x, TA* __restrict__ y, const HeadLinearArgs& a, int t0,
                                           int rows, int h) {
  const Turn& r = a.turn;
  for (int i = threadIdx.x; i < rows * r.dims; i += blockDim.x) {
    const int t = t0 + i / r.dims, d = i % r.dims;
    if (t >= a.tokens) return;
    int pos = r.positions[t];
    if (pos < 0 || pos >= r.max_pos) {
      atomicOr(r.status, 2);
      pos = 0;
    }
    const size_t at = static_cast<size_t>(pos) * (r.rot_dims / 2);
    y[static_cast<size_t>(t) * a.y_ld + a.y_col + h * a.y_head + r.y + d] = from_float<TA>(
        rotated(x + static_cast<size_t>(t) * a.x_ld + a.x_col + h * a.x_head + r.x, d, r.rot_dims, r.pairs, r.cos_t + at,
                r.sin_t + at));
  }
}

constexpr int kHlRows = 16, kHlCols = 128, kHlK = 32;

// CUDA cores: a CTA takes 16 tokens x 128 outputs of one head; thread j owns output column j for all 16 tokens.
template <typename TA, typename TW, bool TURN>
__global__ void __launch_bounds__(kHlCols)
head_linear_kernel(const TA* __restrict__ x, const TW* __restrict__ w, TA* __restrict__ y, const HeadLinearArgs a) {
  pdl_launch();
  pdl_wait();
  __shared__ float xs[kHlRows][kHlK];
  __shared__ float wsm[kHlK][kHlCols + 1];
  const int t0 = blockIdx.x * kHlRows, j0 = blockIdx.y * kHlCols, h = blockIdx.z;
  if (TURN && blockIdx.y == gridDim.y - 1) {          // the last row of CTAs turns the rotated parts
    turn_parts(x, y, a, t0, kHlRows, h);
    return;
  }
  const int j = j0 + threadIdx.x;
  const TW* wh = w + static_cast<size_t>(h) * a.n * a.k;
  float acc[kHlRows];
#pragma unroll
  for (int r = 0; r < kHlRows; ++r) acc[r] = 0.f;
  for (int k0 = 0; k0 < a.k; k0 += kHlK) {
    __syncthreads();
    for (int i = threadIdx.x; i < kHlRows * kHlK; i += kHlCols) {
      const int r = i / kHlK, kk = i - r * kHlK;
      xs[r][kk] = (t0 + r < a.tokens && k0 + kk < a.k)
                      ? to_float(x[static_cast<size_t>(t0 + r) * a.x_ld + a.x_col + h * a.x_head + k0 + kk])
                      : 0.f;
    }
    for (int i = threadIdx.x; i < kHlCols * kHlK; i += kHlCols) {
      const int c = i / kHlK, kk = i - c * kHlK;
      wsm[kk][c] = (j0 + c < a.n && k0 + kk < a.k) ? to_float(wh[static_cast<size_t>(j0 + c) * a.k + k0 + kk]) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int kk = 0; kk < kHlK; ++kk) {
      const float wv = wsm[kk][threadIdx.x];
#pragma unroll
      for (int r = 0; r < kHlRows; ++r) acc[r] = fmaf(xs[r][kk], wv, acc[r]);
    }
  }
  if (j < a.n) {
#pragma unroll
    for (int r = 0; r < kHlRows; ++r)
      if (t0 + r < a.tokens)
        y[static_cast<size_t>(t0 + r) * a.y_ld + a.y_col + h * a.y_head + j] =
            from_float<TA>(acc[r] * gate_of<TA>(a, t0 + r, h, j));
  }
}

// Tensor cores for bfloat16: a CTA of four warps takes 64 tokens x 64 outputs of one head, a warp 16 tokens;
// A fragments (x) and B fragments (W rows are the MMA's columns: W is [n, k] row-major, which is the "col"
// operand) come straight from global memory; k ascending in steps of 16.  Needs k % 16 == 0, n % 8 == 0 and
// even strides and columns (4-byte loads and stores).
__device__ __forceinline__ void hl_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

constexpr int kHmRows = 64, kHmCols = 64;

template <bool TURN, bool GATE>
__global__ void __launch_bounds__(128)
head_linear_mma_kernel(const bf16* __restrict__ x, const bf16* __restrict__ w, bf16* __restrict__ y,
                       const HeadLinearArgs a) {
  pdl_launch();
  pdl_wait();
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gid = lane >> 2, tig = lane & 3;
  const int t0 = blockIdx.x * kHmRows + warp * 16, j0 = blockIdx.y * kHmCols, h = blockIdx.z;
  if (TURN && blockIdx.y == gridDim.y - 1) {
    turn_parts(x, y, a, blockIdx.x * kHmRows, kHmRows, h);
    return;
  }
  if (t0 >= a.tokens) return;
  const int r0 = t0 + gid, r1 = r0 + 8;
  const bool ok0 = r0 < a.tokens, ok1 = r1 < a.tokens;
  const bf16* x0 = x + static_cast<size_t>(ok0 ? r0 : t0) * a.x_ld + a.x_col + h * a.x_head + tig * 2;
  const bf16* x1 = x + static_cast<size_t>(ok1 ? r1 : t0) * a.x_ld + a.x_col + h * a.x_head + tig * 2;
  const bf16* wh = w + static_cast<size_t>(h) * a.n * a.k;
  // (the gates are asked for ahead of the product; their pairs start on 4-byte boundaries as y's do)
  uint32_t gates[GATE ? kHmCols / 8 : 1][2];
  if (GATE) {
    const bf16* g = static_cast<const bf16*>(a.gate) + h * a.n + j0 + tig * 2;
#pragma unroll
    for (int nt = 0; nt < kHmCols / 8; ++nt) {
      const bool in = j0 + nt * 8 < a.n;
      gates[GATE ? nt : 0][0] = in && ok0 ? *reinterpret_cast<const uint32_t*>(g + static_cast<size_t>(r0) * a.gate_ld + nt * 8) : 0u;
      gates[GATE ? nt : 0][1] = in && ok1 ? *reinterpret_cast<const uint32_t*>(g + static_cast<size_t>(r1) * a.gate_ld + nt * 8) : 0u;
    }
  }
  float acc[kHmCols / 8][4];
#pragma unroll
  for (int nt = 0; nt < kHmCols / 8; ++nt) acc[nt][0] = acc[nt][1] = acc[nt][2] = acc[nt][3] = 0.f;
#pragma unroll 4
  for (int k0 = 0; k0 < a.k; k0 += 16) {
    uint32_t af[4];
    af[0] = *reinterpret_cast<const uint32_t*>(x0 + k0);
    af[1] = *reinterpret_cast<const uint32_t*>(x1 + k0);
    af[2] = *reinterpret_cast<const uint32_t*>(x0 + k0 + 8);
    af[3] = *reinterpret_cast<const uint32_t*>(x1 + k0 + 8);
#pragma unroll
    for (int nt = 0; nt < kHmCols / 8; ++nt) {
      const int j = j0 + nt * 8 + gid;
      if (j0 + nt * 8 < a.n) {               // (n is a multiple of 8: a group of 8 columns is in or out as a whole)
        const bf16* wr = wh + static_cast<size_t>(j) * a.k + k0 + tig * 2;
        hl_mma(acc[nt], af, *reinterpret_cast<const uint32_t*>(wr), *reinterpret_cast<const uint32_t*>(wr + 8));
      }
    }
  }
#pragma unroll
  for (int nt = 0; nt < kHmCols / 8; ++nt) {
    const int j = j0 + nt * 8 + tig * 2;
    if (j0 + nt * 8 >= a.n) continue;
    if (GATE) {
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const uint32_t g = gates[GATE ? nt : 0][e >> 1];
        acc[nt][e] = __fdividef(acc[nt][e], 1.f + __expf(-__uint_as_float(e & 1 ? g & 0xFFFF0000u : g << 16)));
      }
    }
    if (ok0)
      *reinterpret_cast<__nv_bfloat162*>(y + static_cast<size_t>(r0) * a.y_ld + a.y_col + h * a.y_head + j) =
          __floats2bfloat162_rn(acc[nt][0], acc[nt][1]);
    if (ok1)
      *reinterpret_cast<__nv_bfloat162*>(y + static_cast<size_t>(r1) * a.y_ld + a.y_col + h * a.y_head + j) =
          __floats2bfloat162_rn(acc[nt][2], acc[nt][3]);
  }
}

// A few tokens (single-token steps): the product is bound by the stream of the heads' matrices, and CTAs of the
// kernel above would be few and each walk all of k.  A warp takes four output features of one head and streams
// their rows in 16-byte pieces, lanes side by side, up to eight tokens at a time; the lanes' sums meet by
// shuffles.  Needs k % 8 == 0 and rows on 16-byte boundaries.
constexpr int kHfTokens = 8, kHfCols = 4;
template <bool TURN>
__global__ void __launch_bounds__(128)
head_linear_few_kernel(const bf16* x, const bf16* __restrict__ w, bf16* __restrict__ y, const HeadLinearArgs a) {
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, t0 = blockIdx.z * kHfTokens;
  pdl_launch();
  if (TURN && blockIdx.x == gridDim.x - 1) {
    pdl_wait();
    turn_parts(x, y, a, t0, kHfTokens, h);
    return;
  }
  const int j0 = (blockIdx.x * 4 + warp) * kHfCols;
  if (j0 >= a.n) return;
  const bf16* wr[kHfCols];
#pragma unroll
  for (int f = 0; f < kHfCols; ++f) wr[f] = w + (static_cast<size_t>(h) * a.n + min(j0 + f, a.n - 1)) * a.k;
  float acc[kHfCols][kHfTokens];
#pragma unroll
  for (int f = 0; f < kHfCols; ++f)
#pragma unroll
    for (int t = 0; t < kHfTokens; ++t) acc[f][t] = 0.f;
  const int nt = min(kHfTokens, a.tokens - t0);
  const bf16* xr = x + static_cast<size_t>(t0) * a.x_ld + a.x_col + h * a.x_head;
  // lane 8 f + t writes output f of token t
  static_assert(kHfCols * kHfTokens == 32, "a lane per output");
  const int my_f = lane / kHfTokens, my_t = lane % kHfTokens;
  const bool mine = my_t < nt && j0 + my_f < a.n;
  float factor = 1.f, sum = 0.f;
  for (int c0 = 0; c0 < a.k; c0 += 256) {
    const int c = c0 + lane * 8;
    const bool in = c < a.k;
    float wv[kHfCols][8];
#pragma unroll
    for (int f = 0; f < kHfCols; ++f) {
      if (in) load16(wr[f] + c, wv[f]);
      else {
#pragma unroll
        for (int i = 0; i < 8; ++i) wv[f][i] = 0.f;
      }
    }
    if (c0 == 0) {                             // (the matrices come from no earlier kernel of the step)
      pdl_wait();
      if (mine) factor = gate_of<bf16>(a, t0 + my_t, h, j0 + my_f);
    }
#pragma unroll
    for (int t = 0; t < kHfTokens; ++t) {
      if (t < nt && in) {
        float xv[8];
        load16(xr + static_cast<size_t>(t) * a.x_ld + c, xv);
#pragma unroll
        for (int f = 0; f < kHfCols; ++f)
#pragma unroll
          for (int i = 0; i < 8; ++i) acc[f][t] = fmaf(wv[f][i], xv[i], acc[f][t]);
      }
    }
  }
#pragma unroll
  for (int f = 0; f < kHfCols; ++f)
#pragma unroll
    for (int t = 0; t < kHfTokens; ++t) {
      const float v = warp_sum(acc[f][t]);
      if (f == my_f && t == my_t) sum = v;
    }
  if (mine)
    y[static_cast<size_t>(t0 + my_t) * a.y_ld + a.y_col + h * a.y_head + j0 + my_f] = __float2bfloat16_rn(sum * factor);
}

}  // namespace rl

using namespace rl;

extern "C" {

int rl_latent_prep(int act_dtype, int w_dtype, const void* q, int q_src_ld, const void* craw, int c_ld,
                   const int32_t* positions, int tokens, int heads, int dn, int dr, int rank, int rot_dims, int pairs,
                   const void* w, float eps, const float* cos_t, const float* sin_t, int max_pos, void* qa, int q_ld,
                   const int32_t* slots, void* cache, int page_size, long long num_slots, const void* dq, int dq_ld,
                   int dq_rank, const void* dq_w, void* dq_out, int dq_out_ld, int* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  LatentPrepArgs a;
  a.q_src_ld = q_src_ld;
  a.c_ld = c_ld;
  a.heads = heads;
  a.dn = dn;
  a.dr = dr;
  a.rank = rank;
  a.rot_dims = rot_dims;
  a.q_ld = q_ld;
  a.eps = eps;
  a.page_size = page_size;
  a.num_slots = num_slots;
  a.max_pos = max_pos;
  a.pairs = pairs;
  a.dq_ld = dq_ld;
  a.dq_rank = dq_rank;
  a.dq_out_ld = dq_out_ld;
#define RL_CASE(TA, TW)                                                                                            \
  launch_kernel(latent_prep_kernel<TA, TW>, dim3(tokens), dim3(128), 0, stream, static_cast<const TA*>(q),         \
                static_cast<const TA*>(craw), positions, static_cast<const TW*>(w), cos_t, sin_t,                  \
                static_cast<TA*>(qa), slots, static_cast<TA*>(cache), static_cast<const TA*>(dq),                  \
                static_cast<const TW*>(dq_w), static_cast<TA*>(dq_out), status, a)
  if (act_dtype == 0) RL_CASE(float, float);
  else if (w_dtype == 0) RL_CASE(bf16, float);
  else RL_CASE(bf16, bf16);
#undef RL_CASE
  RL_LAUNCH_END();
}

// impl 0: the form that fits (few tokens, tensor cores, CUDA cores); 1: CUDA cores; 2: tensor cores where they apply.
int rl_head_linear(int act_dtype, int w_dtype, const void* x, int x_ld, int x_col, int x_head, const void* w, int heads,
                   int n, int k, void* y, int y_ld, int y_col, int y_head, int tokens, int impl, int turn_dims,
                   int rot_dims, int pairs, int turn_x, int turn_y, const float* cos_t, const float* sin_t, int max_pos,
                   const int32_t* positions, int* status, const void* gate, int gate_ld, cudaStream_t stream) {
  if (tokens <= 0 || heads <= 0 || n <= 0) return 0;
  if (gate != nullptr && turn_dims > 0) return static_cast<int>(cudaErrorInvalidValue);
  HeadLinearArgs a;
  a.gate = gate;
  a.gate_ld = gate_ld;
  a.tokens = tokens;
  a.heads = heads;
  a.n = n;
  a.k = k;
  a.x_ld = x_ld;
  a.x_col = x_col;
  a.x_head = x_head;
  a.y_ld = y_ld;
  a.y_col = y_col;
  a.y_head = y_head;
  a.turn = Turn{turn_dims, rot_dims, pairs, turn_x, turn_y, max_pos, cos_t, sin_t, positions, status};
  const bool even = ((x_ld | x_col | x_head | y_ld | y_col | y_head) & 1) == 0 &&
                    reinterpret_cast<uintptr_t>(x) % 4 == 0 && reinterpret_cast<uintptr_t>(y) % 4 == 0 &&
                    reinterpret_cast<uintptr_t>(w) % 4 == 0 && (gate == nullptr || (gate_ld % 2 == 0 && reinterpret_cast<uintptr_t>(gate) % 4 == 0));
  const int turning = turn_dims > 0 ? 1 : 0;
  const bool pieces = act_dtype == 1 && w_dtype == 1 && k % 8 == 0 && x_ld % 8 == 0 && x_col % 8 == 0 && x_head % 8 == 0 &&
                      reinterpret_cast<uintptr_t>(x) % 16 == 0 && reinterpret_cast<uintptr_t>(w) % 16 == 0;
  if (impl == 0 && pieces && tokens <= 2 * kHfTokens) {
    const dim3 grid((n + 4 * kHfCols - 1) / (4 * kHfCols) + turning, heads, (tokens + kHfTokens - 1) / kHfTokens);
    if (turning) launch_kernel(head_linear_few_kernel<true>, grid, dim3(128), 0, stream, static_cast<const bf16*>(x), static_cast<const bf16*>(w), static_cast<bf16*>(y), a);
    else launch_kernel(head_linear_few_kernel<false>, grid, dim3(128), 0, stream, static_cast<const bf16*>(x), static_cast<const bf16*>(w), static_cast<bf16*>(y), a);
    RL_LAUNCH_END();
  }
  if (act_dtype == 1 && w_dtype == 1 && impl != 1 && k % 16 == 0 && n % 8 == 0 && even) {
    const dim3 grid((tokens + kHmRows - 1) / kHmRows, (n + kHmCols - 1) / kHmCols + turning, heads);
    if (turning) launch_kernel(head_linear_mma_kernel<true, false>, grid, dim3(128), 0, stream, static_cast<const bf16*>(x), static_cast<const bf16*>(w), static_cast<bf16*>(y), a);
    else if (gate != nullptr) launch_kernel(head_linear_mma_kernel<false, true>, grid, dim3(128), 0, stream, static_cast<const bf16*>(x), static_cast<const bf16*>(w), static_cast<bf16*>(y), a);
    else launch_kernel(head_linear_mma_kernel<false, false>, grid, dim3(128), 0, stream, static_cast<const bf16*>(x), static_cast<const bf16*>(w), static_cast<bf16*>(y), a);
    RL_LAUNCH_END();
  }
  dim3 grid((tokens + kHlRows - 1) / kHlRows, (n + kHlCols - 1) / kHlCols + turning, heads);
#define RL_CASE(TA, TW)                                                                                          \
  do {                                                                                                           \
    if (turning)                                                                                                 \
      launch_kernel(head_linear_kernel<TA, TW, true>, grid, dim3(kHlCols), 0, stream, static_cast<const TA*>(x), \
                    static_cast<const TW*>(w), static_cast<TA*>(y), a);                                          \
    else                                                                                                         \
      launch_kernel(head_linear_kernel<TA, TW, false>, grid, dim3(kHlCols), 0, stream,                           \
                    static_cast<const TA*>(x), static_cast<const TW*>(w), static_cast<TA*>(y), a);               \
  } while (0)
  if (act_dtype == 0) RL_CASE(float, float);
  else if (w_dtype == 0) RL_CASE(bf16, float);
  else RL_CASE(bf16, bf16);
#undef RL_CASE
  RL_LAUNCH_END();
}

}  // extern "C"
