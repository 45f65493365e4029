// Linear attention with a decaying state, as a recurrence over a state kept per request.  Per head, S [D, DV]
// in float32:
//
//   one decay per head           S_t = a_h S_(t-1) + k_t v_t^T,            o_t = S_t^T q_t
//   a decay per token and key    o_t = S_(t-1)^T q_t + (sum_i q_i u_i k_i) v_t,
//   channel, with a bonus        S_t = diag(a_t) S_(t-1) + k_t v_t^T,      a_t = exp(-exp(z_t + b))
//   a decay per token (state     S_t = exp(-exp(A_h) d_t) S_(t-1) + d_t k_t v_t^T,   d_t = softplus(z_t + b_h),
//   space), with a skip          o_t = S_t^T q_t + D_h v_t;   neighbouring heads share their q and k
//
// (the second form's read-out sees the token's own write through the bonus u only).  The third form is a module of
// its own (compiled with -DRL_LIN_TOKEN=1).  One kernel serves prompt
// portions and single tokens: a CTA takes one sequence of the step, one head and a block of value columns.
// Columns of S never mix.  A thread keeps four neighbouring columns of a group of eight rows in registers, as
// pairs of rows (fma.rn.f32x2: two rows per instruction, each rounded as a single fma); the G = 1 to 32 groups
// of a column lie in one warp and their partial read-outs meet by shuffles that leave each lane with a column
// of its own.  The state is read from the request's slot at the start and written back at the end.
//
// q, k, v, the gate (in the activation type), the decays' projections and the rotation's table rows of eight
// tokens at a time are copied to shared memory asynchronously, into one of two buffers while the tokens of the
// other are worked on; there q, k and v become float32 (every v twice in a row: an operand for two rows), and q
// and k may be
//   rotated   entry i of the first 2 * rot_pairs with entry i + rot_pairs, cosines and sines from tables,
//   scaled    k by a constant,
// and the decays are formed.  The state, the decays, the sums are float32.
//
// Output: float32 o; or, where one CTA covers all columns of a head, the finished heads right away:
// y = o / sqrt(mean over the head (o^2) + eps) (* weight) (* act(gate)) in the activation type
// (linear_output_kernel does the same from a float32 o where a head is spread over several CTAs).
//
// Long portions are cut in three passes so that a sequence is not one serial chain: (1) every chunk of C
// tokens sums its own contribution to the state from zero (and the product of its decays), (2) the chunks'
// states are chained, S_c = A_c S_(c-1) + dS_c, (3) every chunk replays its tokens from its starting state.
// A chunk's starting state is rounded no differently from the serial recurrence's except in the order of the
// sums.
#include "common.cuh"

#ifndef RL_LIN_DIM
#error "compile with -DRL_LIN_DIM=<key size>"
#endif

namespace rl {

constexpr int kD = RL_LIN_DIM;
static_assert(kD >= 1 && kD <= 256, "key size out of range");
constexpr int kRows = 8;                                               // rows of a group
constexpr int kGroups = kD <= 8 ? 1 : (kD <= 16 ? 2 : (kD <= 32 ? 4 : (kD <= 64 ? 8 : (kD <= 128 ? 16 : 32))));
constexpr int kStride = kRows + 4;                                     // floats between groups in shared memory (spreads the banks)
constexpr int kSm = kGroups * kStride;                                 // floats of one staged vector
constexpr int kCols = 4;                                               // columns of a thread
constexpr int kSlots = 32 / kGroups;                                   // column quadruples of a warp
constexpr int kTok = 8;                                                // tokens staged at a time
constexpr int kMaxThreads = 256;
constexpr int kTcMinTokens = 16, kTcMaxCols = 128;                     // blocks of tokens on the tensor cores: from so many on

enum { GATE_NONE = 0, GATE_SIGMOID = 1, GATE_SILU = 2 };
enum { PER_HEAD = 0, PER_CHANNEL = 1, PER_TOKEN = 2 };                 // the kind of decay

template <typename T>
struct LinArgs {
  const T *q, *k, *v;            // head h of token t: q + t * q_ld + h * D, k likewise, v + t * v_ld + h * DV
  int q_ld, k_ld, v_ld;
  float k_scale;
  const float *cos_t, *sin_t;    // [max_pos, rot_pairs]
  const int32_t* positions;
  int rot_pairs, max_pos;
  const int32_t* seq_of_token;   // [tokens]
  const int32_t* state_slot;     // [sequences]
  const float* decay;            // [heads], or (per channel) z [tokens, heads * D]
  const float* decay_bias;       // per channel: b [heads * D]
  const float* bonus;            // per channel: u [heads * D]
  float* state;                  // [slots] x [heads, D, DV]
  long long slot_stride;         // floats from one slot to the next
  float* out;                    // [tokens, heads * DV] float32 (with y: scratch)
  T* y;                          // the finished heads (one CTA per head's columns), or null
  int y_ld;
  const T* gate;
  int gate_ld, gate_mode;
  const float* norm_w;           // [heads * DV] or null
  float eps;
  float* chunk_state;            // [sequences, chunks, heads, D, DV] (chunked passes only)
  float* chunk_decay;            // per channel: [sequences, chunks, heads, D]
  int* status;
  const T* steps;                // per token: z, head h of token t at steps + t * steps_ld + h
  int steps_ld, qk_heads;        // heads of q and k (head h reads h / (heads / qk_heads))
  const float *step_bias, *a_log, *skip;         // per token: b, A and D of every head
  int tokens, heads, dv, chunk, max_chunks;
  int quads_ok;                  // column quadruples of the state start on 16-byte boundaries
  int qk_ok, v_ok, g_ok, z_ok, rot_ok; // rows of q and k / values / gates / decays / tables are made of 16-byte pieces
};

// First token index t in [0, n] with seq_of_token[t] >= s (sequences lie in order in a step): all 32 lanes of
// a warp probe together.
__device__ __forceinline__ int first_token_of(const int32_t* __restrict__ seq_of_token, int n, int s) {
  const int lane = threadIdx.x & 31;
  int lo = 0, len = n;                       // the answer lies in [lo, lo + len]
  while (len > 0) {
    const int step = (len + 31) >> 5;
    const int at = lo + lane * step;
    const bool less = at < lo + len && seq_of_token[at] < s;
    const int below = __popc(__ballot_sync(0xffffffffu, less));
    if (below == 0) break;
    const int end = min(lo + below * step, lo + len);
    lo += (below - 1) * step + 1;
    len = end - lo;
  }
  return lo;
}

__device__ __forceinline__ float gate_value(float g, int mode) {
  const float s = __fdividef(1.f, 1.f + __expf(-g));           // (0 where exp(-g) is infinite)
  return mode == GATE_SILU ? g * s : s;
}
// (the inner exponential's relative error is that of the distance of the decay from 1)
__device__ __forceinline__ float channel_decay(float z) { return expf(-__expf(z)); }

// ln(1 + e^z)
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

__device__ __forceinline__ void async_copy16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(static_cast<unsigned>(__cvta_generic_to_shared(dst))), "l"(src));
}
__device__ __forceinline__ void async_copies_done() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// Two floats as one operand.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
  return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// What one buffer of staged tokens holds, in bytes; every token's part starts on a 16-byte boundary.
struct RawLayout {
  int q, k, v, g, z, cs, sn, bytes;      // offsets of the parts within a buffer; a buffer's size
  int qk_row, v_row, z_row, rot_row;     // bytes of a token in its part (values and gate: v_row)
  int pairs, sums;                       // behind the two buffers: the values as operands, the read-outs; bytes of each
};
__host__ __device__ inline RawLayout raw_layout(int elem, int cols, int rot_pairs, bool channel, bool with_q, bool gated,
                                                int finished_cols) {
  RawLayout r;
  r.qk_row = (kD * elem + 15) / 16 * 16;
  r.v_row = (cols * elem + 15) / 16 * 16;
  r.z_row = channel ? (kD * 4 + 15) / 16 * 16 : 0;
  r.rot_row = (rot_pairs * 4 + 15) / 16 * 16;
  r.q = 0;
  r.k = with_q ? kTok * r.qk_row : 0;
  r.v = r.k + kTok * r.qk_row;
  r.g = r.v + kTok * r.v_row;
  r.z = r.g + (gated ? kTok * r.v_row : 0);
  r.cs = r.z + kTok * r.z_row;
  r.sn = r.cs + kTok * r.rot_row;
  r.bytes = r.sn + kTok * r.rot_row;
  r.pairs = kTok * cols * 8;
  r.sums = kTok * finished_cols * 4;
  return r;
}

// A pair of neighbouring elements (the address is a multiple of the pair's size).
__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }

// mode 0: the whole sequence serially from the slot's state (state written back)
// mode 1: chunk c from zero, no outputs; the chunk's state goes to chunk_state[seq][c]
// mode 3: chunk c from its starting state as pass 2 left it (chunk_state[seq][c - 1]: the state after chunk
//         c - 1; for c = 0 the slot's state, which pass 2 has copied to the entry of the last chunk, since
//         the last chunk's CTA overwrites the slot), outputs written; the last chunk writes the slot
template <typename T, int MODE, int KIND>
__global__ void __launch_bounds__(kMaxThreads, 2)
linear_attention_kernel(const LinArgs<T> a) {
  constexpr bool CHANNEL = KIND == PER_CHANNEL, TOKEN = KIND == PER_TOKEN;
  pdl_launch();
  pdl_wait();
  __shared__ __align__(16) float qs[MODE == 1 ? 1 : kTok][kSm];
  __shared__ __align__(16) float ks[kTok][kSm];
  __shared__ __align__(16) float as[CHANNEL ? kTok : 1][kSm];
  __shared__ __align__(8) float us[CHANNEL && MODE != 1 ? kD : 1], db[CHANNEL ? kD : 1];      // per channel: the head's bonus and decay bias
  __shared__ float bs[kTok];                       // per channel: sum_i q_i u_i k_i of every staged token
  __shared__ float ds[2][TOKEN ? kTok : 1], es[2][TOKEN ? kTok : 1];      // per token: d and the decay of every staged token
  extern __shared__ __align__(16) unsigned char raw[];     // two buffers, the values, the read-outs (RawLayout)
  const int seq = blockIdx.z, head = blockIdx.y % a.heads, c = blockIdx.y / a.heads;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int qk_head = TOKEN ? head / (a.heads / a.qk_heads) : head;
  const int group = lane / kSlots;
  const int block_cols = nwarps * kSlots * kCols;
  const int col0 = blockIdx.x * block_cols;                               // the CTA's first column
  const int local = (warp * kSlots + lane % kSlots) * kCols;
  const int col = col0 + local;
  const bool finish = MODE != 1 && a.y != nullptr, gated = finish && a.gate_mode != GATE_NONE;
  const RawLayout lay = raw_layout(sizeof(T), block_cols, a.rot_pairs, CHANNEL, MODE != 1, gated, finish ? a.dv : 0);
  float* vs = reinterpret_cast<float*>(raw + 2 * lay.bytes);              // [kTok][block_cols] values, each twice
  float* os = vs + lay.pairs / 4;                                         // [kTok][DV] read-outs
  const int seq_begin = first_token_of(a.seq_of_token, a.tokens, seq);
  const int seq_end = first_token_of(a.seq_of_token, a.tokens, seq + 1);
  if (seq_begin >= seq_end) return;
  int t0 = seq_begin, t1 = seq_end;
  if (MODE != 0) {
    t0 = seq_begin + c * a.chunk;
    t1 = min(seq_end, t0 + a.chunk);
    if (t0 >= seq_end) return;
  }
  const bool last_chunk = t1 == seq_end;
  if (MODE == 1 && last_chunk) return;             // nobody starts from the state after the last chunk
  int pos0 = 0;                                    // the position of token t0 (a sequence's positions are consecutive)
  if (a.rot_pairs > 0) {
    pos0 = a.positions[t0];
    if (pos0 < 0 || pos0 + (t1 - t0) > a.max_pos) {
      if (threadIdx.x == 0) atomicOr(a.status, 2);
      pos0 = -1;                                   // every token then takes the tables' first row
    }
  }

  // tokens tb .. tb + nt - 1 on their way into buffer b: a warp takes one token at a time, its lanes the pieces of
  // the token's parts, one part after another
  float z_ahead = 0.f;               // per token: this thread's token's z of the batch on its way
  auto stage = [&](int b, int tb, int nt) {
    constexpr int E = sizeof(T);
    if (TOKEN && threadIdx.x < nt) z_ahead = to_float(a.steps[static_cast<size_t>(tb + threadIdx.x) * a.steps_ld + head]);
    for (int tt = warp; tt < nt; tt += nwarps) {
      unsigned char* buf = raw + b * lay.bytes;
      const size_t t = tb + tt;
      auto part = [&](unsigned char* to, const void* from, int bytes, bool pieces, int elem) {
        if (pieces) {
          for (int e = lane; e < bytes / 16; e += 32) async_copy16(to + e * 16, static_cast<const unsigned char*>(from) + e * 16);
        } else if (elem == 4) {
          for (int e = lane; e < bytes / 4; e += 32) reinterpret_cast<float*>(to)[e] = static_cast<const float*>(from)[e];
        } else {
          for (int e = lane; e < bytes / 2; e += 32) reinterpret_cast<bf16*>(to)[e] = static_cast<const bf16*>(from)[e];
        }
      };
      if (MODE != 1) part(buf + lay.q + tt * lay.qk_row, a.q + t * a.q_ld + qk_head * kD, kD * E, a.qk_ok, E);
      part(buf + lay.k + tt * lay.qk_row, a.k + t * a.k_ld + qk_head * kD, kD * E, a.qk_ok, E);
      const int cols = min(block_cols, a.dv - col0);
      part(buf + lay.v + tt * lay.v_row, a.v + t * a.v_ld + head * a.dv + col0, cols * E, a.v_ok, E);
      if (gated) part(buf + lay.g + tt * lay.v_row, a.gate + t * a.gate_ld + head * a.dv, a.dv * E, a.g_ok, E);
      if (CHANNEL) part(buf + lay.z + tt * lay.z_row, a.decay + (t * a.heads + head) * kD, kD * 4, a.z_ok, 4);
      if (a.rot_pairs > 0) {
        const size_t at = pos0 < 0 ? 0 : static_cast<size_t>(pos0 + tb + tt - t0) * a.rot_pairs;
        part(buf + lay.cs + tt * lay.rot_row, a.cos_t + at, a.rot_pairs * 4, a.rot_ok, 4);
        part(buf + lay.sn + tt * lay.rot_row, a.sin_t + at, a.rot_pairs * 4, a.rot_ok, 4);
      }
    }
  };
  stage(0, t0, min(kTok, t1 - t0));

  const size_t plane = static_cast<size_t>(kD) * a.dv;
  float* slot_state = a.state + static_cast<size_t>(a.state_slot[seq]) * a.slot_stride + head * plane;
  float* chunk_state = MODE == 0 ? nullptr
      : a.chunk_state + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * plane;
  f32x2 S[kRows / 2][kCols];                       // rows 2i and 2i + 1 of the group
  if (MODE == 1) {
#pragma unroll
    for (int i = 0; i < kRows / 2; ++i)
#pragma unroll
      for (int j = 0; j < kCols; ++j) S[i][j] = 0;
  } else {
    const float* from = slot_state;
    if (MODE == 3 && c > 0) from = chunk_state - static_cast<size_t>(a.heads) * plane;
    else if (MODE == 3 && !last_chunk) {
      const int chunks = (seq_end - seq_begin + a.chunk - 1) / a.chunk;
      from = chunk_state + static_cast<size_t>(chunks - 1) * a.heads * plane;
    }
#pragma unroll
    for (int i = 0; i < kRows / 2; ++i) {
      float v[2][kCols];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int row = group * kRows + 2 * i + h;
        const float* p = from + static_cast<size_t>(row) * a.dv + col;
        const bool in = row < kD && col < a.dv;
        if (a.quads_ok) {
          const float4 s = in ? *reinterpret_cast<const float4*>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
          v[h][0] = s.x; v[h][1] = s.y; v[h][2] = s.z; v[h][3] = s.w;
        } else {
#pragma unroll
          for (int j = 0; j < kCols; ++j) v[h][j] = (in && col + j < a.dv) ? p[j] : 0.f;
        }
      }
#pragma unroll
      for (int j = 0; j < kCols; ++j) S[i][j] = pack2(v[0][j], v[1][j]);
    }
  }
  if (kGroups * kRows > kD) {                      // rows beyond D: zero keys and queries, never written again
    for (int i = threadIdx.x; i < kTok * kSm; i += blockDim.x) {
      if (MODE != 1) (&qs[0][0])[i] = 0.f;
      (&ks[0][0])[i] = 0.f;
      if (CHANNEL) (&as[0][0])[i] = 0.f;
    }
  }
  const float decay = KIND == PER_HEAD ? a.decay[head] : 0.f;
  const f32x2 decay2 = pack2(decay, decay);
  const float rate = TOKEN ? expf(a.a_log[head]) : 0.f, step_bias = TOKEN ? a.step_bias[head] : 0.f;
  const float skip = TOKEN ? a.skip[head] : 0.f;
  float all_decays = 1.f;                          // per token, mode 1, thread 0: the product of the decays
  constexpr int kPer = (kD + 31) / 32;             // channels of a lane
  float prod[CHANNEL && MODE == 1 ? kPer : 1];     // per channel, mode 1, warp 0: the products of its channels' decays
  if (CHANNEL) {
    for (int d = threadIdx.x; d < kD; d += blockDim.x) {
      db[d] = a.decay_bias[head * kD + d];
      if (MODE != 1) us[d] = a.bonus[head * kD + d];
    }
    if (MODE == 1) {
#pragma unroll
      for (int j = 0; j < kPer; ++j) prod[j] = 1.f;
    }
  }

  int b = 0;
  for (int tb = t0; tb < t1; tb += kTok, b ^= 1) {
    const int nt = min(kTok, t1 - tb);
    if (TOKEN && threadIdx.x < nt) {           // (the other buffer of these is what the batch before reads)
      const float d = softplus(z_ahead + step_bias);
      ds[b][threadIdx.x] = d;
      es[b][threadIdx.x] = expf(-rate * d);
    }
    async_copies_done();
    __syncthreads();               // this batch has arrived, and the one before has been worked on
    if (tb + kTok < t1) stage(b ^ 1, tb + kTok, min(kTok, t1 - tb - kTok));
    const unsigned char* buf = raw + b * lay.bytes;
    // ---- a warp readies one token at a time, its lanes over the channels (two neighbours each where sizes are even)
    for (int tt = warp; tt < nt; tt += nwarps) {
      const T* qr = reinterpret_cast<const T*>(buf + lay.q + tt * lay.qk_row);
      const T* kr = reinterpret_cast<const T*>(buf + lay.k + tt * lay.qk_row);
      const float* zr = reinterpret_cast<const float*>(buf + lay.z + tt * lay.z_row);
      const float* cs = reinterpret_cast<const float*>(buf + lay.cs + tt * lay.rot_row);
      const float* sn = reinterpret_cast<const float*>(buf + lay.sn + tt * lay.rot_row);
      float bonus = 0.f;
      const float k_scale = TOKEN ? ds[b][tt] : a.k_scale;
      if (kD % 2 == 0 && a.rot_pairs % 2 == 0) {
#pragma unroll
        for (int j = 0; j < (kD + 63) / 64; ++j) {
          const int d = j * 64 + 2 * lane;
          if (d >= kD) continue;
          const int sm = (d / kRows) * kStride + d % kRows;
          float2 kv = load2(kr + d), qv = make_float2(0.f, 0.f);
          if (MODE != 1) qv = load2(qr + d);
          if (d < 2 * a.rot_pairs) {
            const bool first = d < a.rot_pairs;
            const int pair = first ? d : d - a.rot_pairs, other = first ? d + a.rot_pairs : pair;
            const float2 cv = load2(cs + pair);
            float2 sv = load2(sn + pair);
            if (first) sv = make_float2(-sv.x, -sv.y);
            const float2 ko = load2(kr + other);
            kv = make_float2(kv.x * cv.x + ko.x * sv.x, kv.y * cv.y + ko.y * sv.y);
            if (MODE != 1) {
              const float2 qo = load2(qr + other);
              qv = make_float2(qv.x * cv.x + qo.x * sv.x, qv.y * cv.y + qo.y * sv.y);
            }
          }
          kv = make_float2(kv.x * k_scale, kv.y * k_scale);
          *reinterpret_cast<float2*>(&ks[tt][sm]) = kv;
          if (MODE != 1) *reinterpret_cast<float2*>(&qs[tt][sm]) = qv;
          if (CHANNEL) {
            const float2 z = load2(zr + d), bias = load2(db + d);
            *reinterpret_cast<float2*>(&as[tt][sm]) = make_float2(channel_decay(z.x + bias.x), channel_decay(z.y + bias.y));
            if (MODE != 1) {
              const float2 u = load2(us + d);
              bonus = fmaf(qv.x * u.x, kv.x, fmaf(qv.y * u.y, kv.y, bonus));
            }
          }
        }
      } else {
        for (int d = lane; d < kD; d += 32) {
          const int sm = (d / kRows) * kStride + d % kRows;
          float qv = MODE == 1 ? 0.f : to_float(qr[d]), kv = to_float(kr[d]);
          if (d < 2 * a.rot_pairs) {
            const bool first = d < a.rot_pairs;
            const int pair = first ? d : d - a.rot_pairs, other = first ? d + a.rot_pairs : pair;
            const float cv = cs[pair], sv = first ? -sn[pair] : sn[pair];
            kv = kv * cv + to_float(kr[other]) * sv;
            if (MODE != 1) qv = qv * cv + to_float(qr[other]) * sv;
          }
          kv *= k_scale;
          ks[tt][sm] = kv;
          if (MODE != 1) qs[tt][sm] = qv;
          if (CHANNEL) {
            as[tt][sm] = channel_decay(zr[d] + db[d]);
            if (MODE != 1) bonus = fmaf(qv * us[d], kv, bonus);
          }
        }
      }
      if (CHANNEL && MODE != 1) {
        bonus = warp_sum(bonus);
        if (lane == 0) bs[tt] = bonus;
      }
      const T* vr = reinterpret_cast<const T*>(buf + lay.v + tt * lay.v_row);
      for (int i = 2 * lane; i < block_cols; i += 64) {
        const float2 v = load2(vr + i);
        *reinterpret_cast<float4*>(vs + (tt * block_cols + i) * 2) = make_float4(v.x, v.x, v.y, v.y);
      }
    }
    __syncthreads();
    if (CHANNEL && MODE == 1 && blockIdx.x == 0 && warp == 0) {
      for (int tt = 0; tt < nt; ++tt)
#pragma unroll
        for (int j = 0; j < kPer; ++j) {
          const int d = j * 32 + lane;
          if (d < kD) prod[j] *= as[tt][(d / kRows) * kStride + d % kRows];
        }
    }
    if (TOKEN && MODE == 1 && threadIdx.x == 0)
      for (int tt = 0; tt < nt; ++tt) all_decays *= es[b][tt];
    auto token = [&](int tt) {
      const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(&ks[tt][group * kStride]);
      const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(&qs[MODE == 1 ? 0 : tt][group * kStride]);
      const ulonglong2* a4 = reinterpret_cast<const ulonglong2*>(&as[CHANNEL ? tt : 0][group * kStride]);
      const ulonglong2* v4 = reinterpret_cast<const ulonglong2*>(vs + (tt * block_cols + local) * 2);
      const ulonglong2 va = v4[0], vb = v4[1];
      const f32x2 v2[kCols] = {va.x, va.y, vb.x, vb.y};
      f32x2 o2[kCols];
      // (the bonus counts once: in the first half of the first group's pairs)
      const f32x2 bonus = pack2(MODE != 1 && group == 0 ? (CHANNEL ? bs[tt] : (TOKEN ? skip : 0.f)) : 0.f, 0.f);
      const f32x2 own_decay = TOKEN ? pack2(es[b][tt], es[b][tt]) : decay2;
#pragma unroll
      for (int j = 0; j < kCols; ++j) o2[j] = KIND != PER_HEAD && MODE != 1 ? mul2(bonus, v2[j]) : 0;
#pragma unroll
      for (int i = 0; i < kRows / 4; ++i) {
        const ulonglong2 kv = k4[i];
        ulonglong2 qv = make_ulonglong2(0, 0), av = make_ulonglong2(own_decay, own_decay);
        if (MODE != 1) qv = q4[i];
        if (CHANNEL) av = a4[i];
#pragma unroll
        for (int j = 0; j < kCols; ++j) {
          f32x2 &s0 = S[2 * i][j], &s1 = S[2 * i + 1][j];
          if (CHANNEL && MODE != 1) {
            o2[j] = fma2(s0, qv.x, o2[j]);
            o2[j] = fma2(s1, qv.y, o2[j]);
          }
          s0 = fma2(av.x, s0, mul2(kv.x, v2[j]));
          s1 = fma2(av.y, s1, mul2(kv.y, v2[j]));
          if (!CHANNEL && MODE != 1) {
            o2[j] = fma2(s0, qv.x, o2[j]);
            o2[j] = fma2(s1, qv.y, o2[j]);
          }
        }
      }
      if constexpr (MODE != 1) {
        float o[kCols];
#pragma unroll
        for (int j = 0; j < kCols; ++j) {
          float lo, hi;
          unpack2(o2[j], lo, hi);
          o[j] = lo + hi;
        }
        // the groups' partial sums: lanes of two groups exchange the columns the other one keeps
        int keep = 0;
        constexpr int n = kGroups >= 4 ? 1 : (kGroups == 2 ? 2 : kCols);      // columns a lane is left with
        if (kGroups >= 2) {
          const bool up = lane & 16;
          const float r0 = __shfl_xor_sync(0xffffffffu, up ? o[0] : o[2], 16);
          const float r1 = __shfl_xor_sync(0xffffffffu, up ? o[1] : o[3], 16);
          o[0] = (up ? o[2] : o[0]) + r0;
          o[1] = (up ? o[3] : o[1]) + r1;
          keep = up ? 2 : 0;
        }
        if (kGroups >= 4) {
          const bool up = lane & 8;
          const float r0 = __shfl_xor_sync(0xffffffffu, up ? o[0] : o[1], 8);
          o[0] = (up ? o[1] : o[0]) + r0;
          keep += up ? 1 : 0;
        }
        if (kSlots <= 4) o[0] += __shfl_xor_sync(0xffffffffu, o[0], 4);
        if (kSlots <= 2) o[0] += __shfl_xor_sync(0xffffffffu, o[0], 2);
        if (kSlots <= 1) o[0] += __shfl_xor_sync(0xffffffffu, o[0], 1);
        if (kSlots <= 4 && (lane & (8 - kSlots))) return;            // (one lane of those with equal sums writes)
#pragma unroll
        for (int j = 0; j < n; ++j) {
          if (col + keep + j >= a.dv) continue;
          if (finish) os[tt * a.dv + col + keep + j] = o[j];
          else a.out[static_cast<size_t>(tb + tt) * (a.heads * a.dv) + head * a.dv + col + keep + j] = o[j];
        }
      }
    };
#pragma unroll 1
    for (int tt = 0; tt < nt; ++tt) token(tt);
    if (finish) {
      // ---- the staged tokens' heads are complete: unit norm, weight, gate
      __syncthreads();
      for (int tt = warp; tt < nt; tt += nwarps) {
        const float* o = os + tt * a.dv;
        const T* gr = reinterpret_cast<const T*>(buf + lay.g + tt * lay.v_row);
        const size_t t = tb + tt;
        float ss = 0.f;
        for (int d = lane; d < a.dv; d += 32) ss = fmaf(o[d], o[d], ss);
        const float r = rsqrtf(warp_sum(ss) / static_cast<float>(a.dv) + a.eps);
        T* yr = a.y + t * a.y_ld + head * a.dv;
        const float* w = a.norm_w != nullptr ? a.norm_w + head * a.dv : nullptr;
        for (int d = lane; d < a.dv; d += 32) {
          float y = o[d] * r;
          if (w != nullptr) y *= w[d];
          if (gated) y *= gate_value(to_float(gr[d]), a.gate_mode);
          yr[d] = from_float<T>(y);
        }
      }
    }
  }
  if (CHANNEL && MODE == 1 && blockIdx.x == 0 && warp == 0) {
    float* cd = a.chunk_decay + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * kD;
#pragma unroll
    for (int j = 0; j < kPer; ++j)
      if (j * 32 + lane < kD) cd[j * 32 + lane] = prod[j];
  }
  if (TOKEN && MODE == 1 && blockIdx.x == 0 && threadIdx.x == 0)
    a.chunk_decay[(static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head] = all_decays;
  float* to = MODE == 1 ? chunk_state : ((MODE == 0 || last_chunk) ? slot_state : nullptr);
  if (to != nullptr) {
#pragma unroll
    for (int i = 0; i < kRows / 2; ++i) {
      float v[2][kCols];
#pragma unroll
      for (int j = 0; j < kCols; ++j) unpack2(S[i][j], v[0][j], v[1][j]);
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const int row = group * kRows + 2 * i + h;
        if (row >= kD || col >= a.dv) continue;
        float* p = to + static_cast<size_t>(row) * a.dv + col;
        if (a.quads_ok) {
          *reinterpret_cast<float4*>(p) = make_float4(v[h][0], v[h][1], v[h][2], v[h][3]);
        } else {
#pragma unroll
          for (int j = 0; j < kCols; ++j)
            if (col + j < a.dv) p[j] = v[h][j];
        }
      }
    }
  }
}

}  // namespace rl

#if RL_LIN_DIM % 16 == 0
#ifdef RL_LIN_TOKEN
#include "linear_attention_ssd.cuh"
#else
#include "linear_attention_tc.cuh"
#endif
#endif

namespace rl {

// Pass 2: chunk_state[seq][c] <- A_c * (state after chunk c - 1) + chunk_state[seq][c], in order of c; A_c is the
// product of chunk c's decays (every chunk before the last is full; `decays` of them per head).  One thread per
// element of a head's state.
__global__ void linear_attention_chain_kernel(const int32_t* __restrict__ seq_of_token,
                                              const int32_t* __restrict__ state_slot, const float* __restrict__ decay,
                                              const float* __restrict__ chunk_decay, const float* __restrict__ state,
                                              long long slot_stride, float* __restrict__ chunk_state, int tokens,
                                              int heads, int dv, int chunk, int max_chunks, int decays) {
  pdl_launch();
  pdl_wait();
  const int seq = blockIdx.z, head = blockIdx.y;
  const int e = blockIdx.x * blockDim.x + threadIdx.x;
  const size_t plane = static_cast<size_t>(kD) * dv;
  const int t_begin = first_token_of(seq_of_token, tokens, seq);
  const int t_end = first_token_of(seq_of_token, tokens, seq + 1);
  if (e >= plane) return;
  const int chunks = (t_end - t_begin + chunk - 1) / chunk;
  float prev = state[static_cast<size_t>(state_slot[seq]) * slot_stride + head * plane + e];
  float* p = chunk_state + (static_cast<size_t>(seq) * max_chunks * heads + head) * plane + e;
  const size_t step = static_cast<size_t>(heads) * plane;              // from a chunk's entry to the next chunk's
  if (chunks >= 2) p[(chunks - 1) * step] = prev;      // chunk 0's starting state, kept where no chunk's own sum lies
  float dpow = 1.f;                                    // decay^chunk by repeated multiplication, as the recurrence applies it
  const float* cd = nullptr;
  if (chunk_decay != nullptr) {
    cd = chunk_decay + (static_cast<size_t>(seq) * max_chunks * heads + head) * decays + (decays > 1 ? e / dv : 0);
  } else {
    const float dc = decay[head];
    for (int i = 0; i < chunk; ++i) dpow *= dc;
  }
  constexpr int kAhead = 8;           // the chunks' sums are asked for so many at a time, then chained
  for (int c0 = 0; c0 + 1 < chunks; c0 += kAhead) {
    float own[kAhead], dec[kAhead];
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      const bool in = c0 + i + 1 < chunks;
      own[i] = in ? p[(c0 + i) * step] : 0.f;
      dec[i] = (in && cd != nullptr) ? cd[static_cast<size_t>(c0 + i) * heads * decays] : dpow;
    }
#pragma unroll
    for (int i = 0; i < kAhead; ++i) {
      if (c0 + i + 1 < chunks) {
        prev = fmaf(dec[i], prev, own[i]);
        p[(c0 + i) * step] = prev;
      }
    }
  }
}

// y = o / sqrt(mean over the head (o^2) + eps) (* weight) (* act(gate)); a warp per (token, head).
template <typename T>
__global__ void linear_output_kernel(const float* __restrict__ o, const T* __restrict__ gate, int gate_ld,
                                     int gate_mode, const float* __restrict__ w, T* __restrict__ y, int y_ld,
                                     int items, int heads, int dv, float eps) {
  pdl_launch();
  pdl_wait();
  const int lane = threadIdx.x & 31;
  const int item = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (item >= items) return;
  const size_t t = item / heads;
  const int h = item % heads;
  const float* p = o + static_cast<size_t>(item) * dv;
  float ss = 0.f;
  for (int d = lane; d < dv; d += 32) ss = fmaf(p[d], p[d], ss);
  const float r = rsqrtf(warp_sum(ss) / static_cast<float>(dv) + eps);
  for (int d = lane; d < dv; d += 32) {
    const int e = h * dv + d;
    float v = p[d] * r;
    if (w != nullptr) v *= w[e];
    if (gate_mode != GATE_NONE) v *= gate_value(to_float(gate[t * gate_ld + e]), gate_mode);
    y[t * y_ld + e] = from_float<T>(v);
  }
}

inline bool on16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// Threads of a CTA for a head of dv columns.
inline int lin_threads(int dv) {
  const int need = (dv + kCols - 1) / kCols * kGroups;
  return need >= kMaxThreads ? kMaxThreads : (need + 31) / 32 * 32;
}

template <typename T, int MODE, int KIND>
cudaError_t launch_pass(const LinArgs<T>& a, dim3 grid, int th, cudaStream_t stream) {
  const int cols = th / 32 * kSlots * kCols;
  const bool finish = MODE != 1 && a.y != nullptr;
  const RawLayout lay = raw_layout(sizeof(T), cols, a.rot_pairs, KIND == PER_CHANNEL, MODE != 1, finish && a.gate_mode != GATE_NONE,
                                   finish ? a.dv : 0);
  const size_t smem = 2 * static_cast<size_t>(lay.bytes) + lay.pairs + lay.sums;
  static size_t set_for = 0;
  if (smem > set_for) {                  // (the kernel also has static shared memory: beyond 48 KB in all the limit must be raised)
    const cudaError_t e = cudaFuncSetAttribute(linear_attention_kernel<T, MODE, KIND>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
    if (e != cudaSuccess) return e;
    set_for = smem;
  }
  return launch_kernel(linear_attention_kernel<T, MODE, KIND>, grid, dim3(th), smem, stream, a);
}

#if RL_LIN_DIM % 16 == 0 && !defined(RL_LIN_TOKEN)
inline int tc_warps(int dv) { return min(kTcMaxWarps, dv / 16); }

template <typename T, int MODE, int KIND>
cudaError_t launch_tc_pass(const LinArgs<bf16>& a, dim3 grid, int warps, cudaStream_t stream) {
  constexpr bool CHANNEL = KIND == PER_CHANNEL;
  const bool finish = MODE != 1 && a.y != nullptr;
  const TcLayout lay = tc_layout(warps * 16, a.rot_pairs, CHANNEL, MODE != 1, finish && a.gate_mode != GATE_NONE, finish);
  static int set_for = 0;
  if (lay.bytes > set_for) {
    const cudaError_t e = cudaFuncSetAttribute(linear_attention_tc_kernel<MODE, CHANNEL>,
                                               cudaFuncAttributeMaxDynamicSharedMemorySize, lay.bytes);
    if (e != cudaSuccess) return e;
    set_for = lay.bytes;
  }
  return launch_kernel(linear_attention_tc_kernel<MODE, CHANNEL>, grid, dim3(warps * 32), lay.bytes, stream, a);
}
#endif

// One pass of the recurrence in the form that fits: blocks of tokens on the tensor cores, or token by token.
template <typename T, int MODE, int KIND>
cudaError_t launch_either(const LinArgs<T>& a, int rows, int sequences, bool tc, cudaStream_t stream) {
#if RL_LIN_DIM % 16 == 0
  if constexpr (sizeof(T) == 2) {
    if (tc) {
#ifdef RL_LIN_TOKEN
      return launch_ssd_pass<MODE>(a, rows, sequences, stream);
#else
      const int warps = tc_warps(a.dv);
      return launch_tc_pass<T, MODE, KIND>(a, dim3((a.dv + warps * 16 - 1) / (warps * 16), rows, sequences), warps, stream);
#endif
    }
  }
#endif
  const int th = lin_threads(a.dv);
  const int cols = th / 32 * kSlots * kCols;
  return launch_pass<T, MODE, KIND>(a, dim3((a.dv + cols - 1) / cols, rows, sequences), th, stream);
}

template <typename T>
cudaError_t launch_output(const LinArgs<T>& a, cudaStream_t stream) {
  const int items = a.tokens * a.heads, warps = 8;
  return launch_kernel(linear_output_kernel<T>, dim3((items + warps - 1) / warps), dim3(warps * 32), 0, stream,
                       static_cast<const float*>(a.out), a.gate, a.gate_ld, a.gate_mode, a.norm_w, a.y, a.y_ld, items,
                       a.heads, a.dv, a.eps);
}

template <typename T, int KIND>
int launch_linear_attention(const LinArgs<T>& a0, int sequences, bool tc, cudaStream_t stream) {
  // finished heads: by the recurrence itself where one CTA has all columns of a head, else by a kernel behind it
  LinArgs<T> a = a0;
  const int th = lin_threads(a.dv);
  const bool one_block = KIND != PER_TOKEN && a.dv <= (tc ? kTcMaxCols : th / 32 * kSlots * kCols);
  const bool behind = a.y != nullptr && !one_block;
  if (behind) a.y = nullptr;
  cudaError_t e;
  if (a.chunk_state == nullptr || a.max_chunks <= 1) {
    e = launch_either<T, 0, KIND>(a, a.heads, sequences, tc, stream);
  } else {
    e = launch_either<T, 1, KIND>(a, a.heads * a.max_chunks, sequences, tc, stream);
    if (e != cudaSuccess) return static_cast<int>(e);
    const int plane = kD * a.dv;
    e = launch_kernel(linear_attention_chain_kernel, dim3((plane + 255) / 256, a.heads, sequences), dim3(256), 0, stream,
                      a.seq_of_token, a.state_slot, a.decay, static_cast<const float*>(KIND != PER_HEAD ? a.chunk_decay : nullptr),
                      static_cast<const float*>(a.state), a.slot_stride, a.chunk_state, a.tokens, a.heads, a.dv, a.chunk,
                      a.max_chunks, KIND == PER_CHANNEL ? kD : 1);
    if (e != cudaSuccess) return static_cast<int>(e);
    e = launch_either<T, 3, KIND>(a, a.heads * a.max_chunks, sequences, tc, stream);
  }
  if (e == cudaSuccess && behind) e = launch_output(a0, stream);
  return static_cast<int>(e);
}

}  // namespace rl

using namespace rl;

extern "C" {

#ifdef RL_LIN_TOKEN

// The state-space form: q and k of qk_heads heads, z of every token and head in the activation type (row length
// steps_ld), step_bias, a_log and skip float32 [heads].  out [tokens, heads * DV] float32.  longest, chunk_state, chunk
// and max_chunks as below; chunk_decay holds [sequences, max_chunks, heads].
int rl_state_space(int dtype, const void* q, int q_ld, const void* k, int k_ld, int qk_heads, const void* v, int v_ld,
                   const void* steps, int steps_ld, const float* step_bias, const float* a_log, const float* skip,
                   const int32_t* seq_of_token, const int32_t* state_slot, float* state, long long slot_stride, float* out,
                   float* chunk_state, float* chunk_decay, int tokens, int sequences, int heads, int dv, int chunk,
                   int max_chunks, int longest, cudaStream_t stream) {
  if (tokens <= 0 || sequences <= 0) return 0;
  if (out == nullptr || qk_heads <= 0 || heads % qk_heads != 0 || (max_chunks > 1 && chunk_state != nullptr && chunk_decay == nullptr))
    return static_cast<int>(cudaErrorInvalidValue);
#define RL_CASE(T)                                                                                                \
  do {                                                                                                            \
    LinArgs<T> a = {};                                                                                            \
    a.q = static_cast<const T*>(q); a.k = static_cast<const T*>(k); a.v = static_cast<const T*>(v);               \
    a.q_ld = q_ld; a.k_ld = k_ld; a.v_ld = v_ld; a.qk_heads = qk_heads; a.k_scale = 1.f;                          \
    a.steps = static_cast<const T*>(steps); a.steps_ld = steps_ld; a.step_bias = step_bias; a.a_log = a_log;      \
    a.skip = skip; a.seq_of_token = seq_of_token; a.state_slot = state_slot; a.state = state;                     \
    a.slot_stride = slot_stride; a.out = out; a.chunk_state = chunk_state; a.chunk_decay = chunk_decay;           \
    a.tokens = tokens; a.heads = heads; a.dv = dv; a.chunk = chunk; a.max_chunks = max_chunks;                    \
    a.quads_ok = dv % 4 == 0 && slot_stride % 4 == 0 && on16(state) && on16(chunk_state);                         \
    constexpr int E = 16 / sizeof(T);      /* elements of a 16-byte piece */                                      \
    a.qk_ok = kD % E == 0 && q_ld % E == 0 && k_ld % E == 0 && on16(q) && on16(k);                                \
    a.v_ok = dv % E == 0 && v_ld % E == 0 && on16(v);                                                             \
    const bool tc = longest >= kTcMinTokens && sizeof(T) == 2 && kD % 16 == 0 && dv % 16 == 0 && a.qk_ok && a.v_ok; \
    return launch_linear_attention<T, PER_TOKEN>(a, sequences, tc, stream);                                       \
  } while (0)
  if (dtype == 0) RL_CASE(float);
  else RL_CASE(bf16);
#undef RL_CASE
}

#else

// With y the finished heads are asked for, and out [tokens, heads * DV] is scratch that may be used on the way.
// longest: the most tokens any sequence of the step brings (from kTcMinTokens on, and where sizes allow, bfloat16
// steps run in blocks on the tensor cores; 0: never).
// chunk_state null or max_chunks <= 1: every sequence is one serial chain.  Otherwise sequences are cut
// into chunks of `chunk` tokens (max_chunks = the most chunks any sequence of the step has) and
// chunk_state holds [sequences, max_chunks, heads, D, DV] floats, chunk_decay (a decay per channel only)
// [sequences, max_chunks, heads, D].  decay_bias and bonus non-null: a decay per token and key channel.
int rl_linear_attention(int dtype, const void* q, int q_ld, const void* k, int k_ld, const void* v, int v_ld,
                        float k_scale, const float* cos_t, const float* sin_t, const int32_t* positions, int rot_pairs,
                        int max_pos, const int32_t* seq_of_token, const int32_t* state_slot, const float* decay,
                        const float* decay_bias, const float* bonus, float* state, long long slot_stride, float* out,
                        void* y, int y_ld, const void* gate, int gate_ld, int gate_mode, const float* norm_w, float eps,
                        float* chunk_state, float* chunk_decay, int* status, int tokens, int sequences, int heads,
                        int dv, int chunk, int max_chunks, int longest, cudaStream_t stream) {
  if (tokens <= 0 || sequences <= 0) return 0;
  const bool channel = bonus != nullptr;
  if (out == nullptr || (channel && (decay_bias == nullptr || (max_chunks > 1 && chunk_state != nullptr && chunk_decay == nullptr))))
    return static_cast<int>(cudaErrorInvalidValue);
#define RL_CASE(T)                                                                                                \
  do {                                                                                                            \
    LinArgs<T> a = {};                                                                                            \
    a.q = static_cast<const T*>(q); a.k = static_cast<const T*>(k); a.v = static_cast<const T*>(v);               \
    a.q_ld = q_ld; a.k_ld = k_ld; a.v_ld = v_ld; a.k_scale = k_scale; a.cos_t = cos_t; a.sin_t = sin_t;           \
    a.positions = positions; a.rot_pairs = rot_pairs; a.max_pos = max_pos; a.seq_of_token = seq_of_token;         \
    a.state_slot = state_slot; a.decay = decay; a.decay_bias = decay_bias; a.bonus = bonus; a.state = state;      \
    a.slot_stride = slot_stride; a.out = out; a.y = static_cast<T*>(y); a.y_ld = y_ld;                            \
    a.gate = static_cast<const T*>(gate); a.gate_ld = gate_ld; a.gate_mode = gate_mode; a.norm_w = norm_w;        \
    a.eps = eps; a.chunk_state = chunk_state; a.chunk_decay = chunk_decay; a.status = status; a.tokens = tokens;  \
    a.heads = heads; a.dv = dv; a.chunk = chunk; a.max_chunks = max_chunks;                                       \
    a.quads_ok = dv % 4 == 0 && slot_stride % 4 == 0 && on16(state) && on16(chunk_state);                         \
    constexpr int E = 16 / sizeof(T);      /* elements of a 16-byte piece */                                      \
    a.qk_ok = kD % E == 0 && q_ld % E == 0 && k_ld % E == 0 && on16(q) && on16(k);                                \
    a.v_ok = dv % E == 0 && v_ld % E == 0 && on16(v);                                                             \
    a.g_ok = dv % E == 0 && gate_ld % E == 0 && on16(gate);                                                       \
    a.z_ok = kD % 4 == 0 && on16(decay);                                                                          \
    a.rot_ok = rot_pairs % 4 == 0 && on16(cos_t) && on16(sin_t);                                                  \
    const bool tc = longest >= kTcMinTokens && sizeof(T) == 2 && kD % 16 == 0 && dv % 16 == 0 && a.qk_ok &&       \
                    a.v_ok && (a.g_ok || gate_mode == GATE_NONE || y == nullptr) && (a.z_ok || !channel) &&       \
                    (a.rot_ok || rot_pairs == 0);                                                                 \
    if (channel) return launch_linear_attention<T, PER_CHANNEL>(a, sequences, tc, stream);                        \
    return launch_linear_attention<T, PER_HEAD>(a, sequences, tc, stream);                                        \
  } while (0)
  if (dtype == 0) RL_CASE(float);
  else RL_CASE(bf16);
#undef RL_CASE
}

#endif

}  // extern "C"
