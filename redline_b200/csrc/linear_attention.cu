// Linear attention with a decaying state, as a recurrence over a state kept per request.  Per head, S [D, DV]
// in float32:
//
//   one decay per head           S_t = a_h S_(t-1) + k_t v_t^T,            o_t = S_t^T q_t
//   a decay per token and key    o_t = S_(t-1)^T q_t + (sum_i q_i u_i k_i) v_t,
//   channel, with a bonus        S_t = diag(a_t) S_(t-1) + k_t v_t^T,      a_t = exp(-exp(z_t + b))
//
// (the second form's read-out sees the token's own write through the bonus u only).  One kernel serves prompt
// portions and single tokens: a CTA takes one sequence of the step, one head and a block of value columns.
// Columns of S never mix.  A thread keeps two neighbouring columns of a group of rows (up to 32) in
// registers; the G = 2, 4 or 8 groups of a column lie in one warp and their partial read-outs meet by
// shuffles.  The state is read from the request's slot at the start and written back at the end.
//
// q, k and v are read in the activation type and staged a few tokens at a time in shared memory as float32,
// where they may be
//   rotated   entry i of the first 2 * rot_pairs with entry i + rot_pairs, cosines and sines from tables,
//   scaled    k by a constant,
// and the decays are formed from their projections.  The state, the decays, the sums are float32.
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
constexpr int kGroups = kD <= 64 ? 2 : (kD <= 128 ? 4 : 8);            // row groups of a column
constexpr int kRows = ((kD + kGroups - 1) / kGroups + 3) / 4 * 4;      // rows of a group (float4 loads)
constexpr int kStride = kRows + 4;                                     // floats between groups in shared memory (spreads the banks)
constexpr int kSm = kGroups * kStride;                                 // floats of one staged vector
constexpr int kCols = 2;                                               // columns of a thread
constexpr int kSlots = 32 / kGroups;                                   // column pairs of a warp
constexpr int kTok = kD <= 64 ? 16 : 8;                                // tokens staged at a time
constexpr int kMaxThreads = kGroups <= 2 ? 128 : 256;
constexpr int kMaxCols = kMaxThreads / kGroups * kCols;

enum { GATE_NONE = 0, GATE_SIGMOID = 1, GATE_SILU = 2 };

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
  float* out;                    // [tokens, heads * DV], or null with y
  T* y;                          // the finished heads (one CTA per head's columns), or null
  int y_ld;
  const T* gate;
  int gate_ld, gate_mode;
  const float* norm_w;           // [heads * DV] or null
  float eps;
  float* chunk_state;            // [sequences, chunks, heads, D, DV] (chunked passes only)
  float* chunk_decay;            // per channel: [sequences, chunks, heads, D]
  int* status;
  int tokens, heads, dv, chunk, max_chunks;
  int pairs_ok;                  // column pairs of the state start on 8-byte boundaries
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
  const float s = 1.f / (1.f + expf(-g));
  return mode == GATE_SILU ? g * s : s;
}

// mode 0: the whole sequence serially from the slot's state (state written back)
// mode 1: chunk c from zero, no outputs; the chunk's state goes to chunk_state[seq][c]
// mode 3: chunk c from its starting state as pass 2 left it (chunk_state[seq][c - 1]: the state after chunk
//         c - 1; for c = 0 the slot's state, which pass 2 has copied to the entry of the last chunk, since
//         the last chunk's CTA overwrites the slot), outputs written; the last chunk writes the slot
template <typename T, int MODE, bool CHANNEL>
__global__ void __launch_bounds__(kMaxThreads, MODE == 0 ? 1 : 512 / kMaxThreads)
linear_attention_kernel(const LinArgs<T> a) {
  pdl_launch();
  pdl_wait();
  __shared__ __align__(16) float qs[MODE == 1 ? 1 : kTok][kSm];
  __shared__ __align__(16) float ks[kTok][kSm];
  __shared__ __align__(16) float as[CHANNEL ? kTok : 1][kSm];
  __shared__ __align__(8) float vs[kTok][kMaxCols];
  __shared__ float bs[kTok];                       // per channel: sum_i q_i u_i k_i of every staged token
  extern __shared__ float os[];                    // [kTok][DV] read-outs, where the heads are finished here
  const int seq = blockIdx.z, head = blockIdx.y % a.heads, c = blockIdx.y / a.heads;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int group = lane / kSlots;
  const int block_cols = nwarps * kSlots * kCols;
  const int col0 = blockIdx.x * block_cols;                               // the CTA's first column
  const int local = (warp * kSlots + lane % kSlots) * kCols;
  const int col = col0 + local;
  const bool in0 = col < a.dv, in1 = col + 1 < a.dv;
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
  const size_t plane = static_cast<size_t>(kD) * a.dv;
  float* slot_state = a.state + static_cast<size_t>(a.state_slot[seq]) * a.slot_stride + head * plane;
  float* chunk_state = MODE == 0 ? nullptr
      : a.chunk_state + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * plane;

  float S[kRows][kCols];
  if (MODE == 1) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) S[i][0] = S[i][1] = 0.f;
  } else {
    const float* from = slot_state;
    if (MODE == 3 && c > 0) from = chunk_state - static_cast<size_t>(a.heads) * plane;
    else if (MODE == 3 && !last_chunk) {
      const int chunks = (seq_end - seq_begin + a.chunk - 1) / a.chunk;
      from = chunk_state + static_cast<size_t>(chunks - 1) * a.heads * plane;
    }
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int row = group * kRows + i;
      const float* p = from + static_cast<size_t>(row) * a.dv + col;
      if (a.pairs_ok) {
        const float2 s = (in0 && row < kD) ? *reinterpret_cast<const float2*>(p) : make_float2(0.f, 0.f);
        S[i][0] = s.x;
        S[i][1] = s.y;
      } else {
        S[i][0] = (in0 && row < kD) ? p[0] : 0.f;
        S[i][1] = (in1 && row < kD) ? p[1] : 0.f;
      }
    }
  }
  if (kGroups * kRows > kD) {                      // rows beyond D: zero keys and queries, never written again
    for (int i = threadIdx.x; i < kTok * kSm; i += blockDim.x) {
      if (MODE != 1) (&qs[0][0])[i] = 0.f;
      (&ks[0][0])[i] = 0.f;
      if (CHANNEL) (&as[0][0])[i] = 0.f;
    }
  }
  const float decay = CHANNEL ? 0.f : a.decay[head];
  float prod[(kD + 31) / 32];                      // MODE 1, per channel: thread d of warp 0 .. its channels' products
#pragma unroll
  for (int i = 0; i < (kD + 31) / 32; ++i) prod[i] = 1.f;

  for (int tb = t0; tb < t1; tb += kTok) {
    const int nt = min(kTok, t1 - tb);
    __syncthreads();
    // ---- a warp stages one token at a time, its lanes over the channels
    for (int tt = warp; tt < nt; tt += nwarps) {
      const size_t t = tb + tt;
      const T* qr = a.q + t * a.q_ld + head * kD;
      const T* kr = a.k + t * a.k_ld + head * kD;
      const float *cs = nullptr, *sn = nullptr;
      if (a.rot_pairs > 0) {
        int pos = a.positions[t];
        if (pos < 0 || pos >= a.max_pos) {
          if (lane == 0) atomicOr(a.status, 2);
          pos = 0;
        }
        cs = a.cos_t + static_cast<size_t>(pos) * a.rot_pairs;
        sn = a.sin_t + static_cast<size_t>(pos) * a.rot_pairs;
      }
      float bonus = 0.f;
#pragma unroll
      for (int j = 0; j < (kD + 31) / 32; ++j) {
        const int d = j * 32 + lane;
        if (d >= kD) continue;
        const int sm = (d / kRows) * kStride + d % kRows;
        float qv = MODE == 1 ? 0.f : to_float(qr[d]), kv = to_float(kr[d]);
        if (d < 2 * a.rot_pairs) {
          const bool first = d < a.rot_pairs;
          const int pair = first ? d : d - a.rot_pairs, other = first ? d + a.rot_pairs : pair;
          const float cv = cs[pair], sv = first ? -sn[pair] : sn[pair];
          kv = kv * cv + to_float(kr[other]) * sv;
          if (MODE != 1) qv = qv * cv + to_float(qr[other]) * sv;
        }
        kv *= a.k_scale;
        ks[tt][sm] = kv;
        if (MODE != 1) qs[tt][sm] = qv;
        if (CHANNEL) {
          const int ch = head * kD + d;
          as[tt][sm] = expf(-expf(a.decay[t * (a.heads * kD) + ch] + a.decay_bias[ch]));
          if (MODE != 1) bonus = fmaf(qv * a.bonus[ch], kv, bonus);
        }
      }
      if (CHANNEL && MODE != 1) {
        bonus = warp_sum(bonus);
        if (lane == 0) bs[tt] = bonus;
      }
      const T* vr = a.v + t * a.v_ld + head * a.dv + col0;
      for (int i = lane; i < block_cols; i += 32) vs[tt][i] = col0 + i < a.dv ? to_float(vr[i]) : 0.f;
    }
    __syncthreads();
    if (CHANNEL && MODE == 1 && blockIdx.x == 0 && warp == 0) {
      for (int tt = 0; tt < nt; ++tt)
#pragma unroll
        for (int j = 0; j < (kD + 31) / 32; ++j) {
          const int d = j * 32 + lane;
          if (d < kD) prod[j] *= as[tt][(d / kRows) * kStride + d % kRows];
        }
    }
    auto token = [&](int tt) {
      const float4* k4 = reinterpret_cast<const float4*>(&ks[tt][group * kStride]);
      const float4* q4 = reinterpret_cast<const float4*>(&qs[MODE == 1 ? 0 : tt][group * kStride]);
      const float4* a4 = reinterpret_cast<const float4*>(&as[CHANNEL ? tt : 0][group * kStride]);
      const float2 v = *reinterpret_cast<const float2*>(&vs[tt][local]);
      float o00 = 0.f, o01 = 0.f, o10 = 0.f, o11 = 0.f;       // two chains per column
#pragma unroll
      for (int i = 0; i < kRows; i += 4) {
        const float4 kv = k4[i >> 2];
        const float kk[4] = {kv.x, kv.y, kv.z, kv.w};
        float qq[4] = {0.f, 0.f, 0.f, 0.f}, aa[4];
        if (MODE != 1) {
          const float4 qv = q4[i >> 2];
          qq[0] = qv.x; qq[1] = qv.y; qq[2] = qv.z; qq[3] = qv.w;
        }
        if (CHANNEL) {
          const float4 av = a4[i >> 2];
          aa[0] = av.x; aa[1] = av.y; aa[2] = av.z; aa[3] = av.w;
        }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          float &s0 = S[i + j][0], &s1 = S[i + j][1];
          if (CHANNEL) {
            if (MODE != 1) {
              if (j & 1) { o01 = fmaf(s0, qq[j], o01); o11 = fmaf(s1, qq[j], o11); }
              else       { o00 = fmaf(s0, qq[j], o00); o10 = fmaf(s1, qq[j], o10); }
            }
            s0 = fmaf(aa[j], s0, kk[j] * v.x);
            s1 = fmaf(aa[j], s1, kk[j] * v.y);
          } else {
            s0 = fmaf(decay, s0, kk[j] * v.x);
            s1 = fmaf(decay, s1, kk[j] * v.y);
            if (MODE != 1) {
              if (j & 1) { o01 = fmaf(s0, qq[j], o01); o11 = fmaf(s1, qq[j], o11); }
              else       { o00 = fmaf(s0, qq[j], o00); o10 = fmaf(s1, qq[j], o10); }
            }
          }
        }
      }
      if (MODE != 1) {
        float o0 = o00 + o01, o1 = o10 + o11;
#pragma unroll
        for (int off = kSlots; off < 32; off <<= 1) {
          o0 += __shfl_xor_sync(0xffffffffu, o0, off);
          o1 += __shfl_xor_sync(0xffffffffu, o1, off);
        }
        if (CHANNEL) {
          o0 = fmaf(bs[tt], v.x, o0);
          o1 = fmaf(bs[tt], v.y, o1);
        }
        if (group == 0) {
          float* dst = a.y != nullptr ? os + tt * a.dv + col
                                      : a.out + static_cast<size_t>(tb + tt) * (a.heads * a.dv) + head * a.dv + col;
          if (in0) dst[0] = o0;
          if (in1) dst[1] = o1;
        }
      }
    };
    if (nt == kTok) {
#pragma unroll 2
      for (int tt = 0; tt < kTok; ++tt) token(tt);
    } else {
      for (int tt = 0; tt < nt; ++tt) token(tt);
    }
    if (MODE != 1 && a.y != nullptr) {
      // ---- the staged tokens' heads are complete: unit norm, weight, gate
      __syncthreads();
      for (int tt = warp; tt < nt; tt += nwarps) {
        const float* o = os + tt * a.dv;
        float ss = 0.f;
        for (int d = lane; d < a.dv; d += 32) ss = fmaf(o[d], o[d], ss);
        const float r = rsqrtf(warp_sum(ss) / static_cast<float>(a.dv) + a.eps);
        const size_t t = tb + tt;
        for (int d = lane; d < a.dv; d += 32) {
          const int e = head * a.dv + d;
          float y = o[d] * r;
          if (a.norm_w != nullptr) y *= a.norm_w[e];
          if (a.gate_mode != GATE_NONE) y *= gate_value(to_float(a.gate[t * a.gate_ld + e]), a.gate_mode);
          a.y[t * a.y_ld + e] = from_float<T>(y);
        }
      }
    }
  }
  if (CHANNEL && MODE == 1 && blockIdx.x == 0 && warp == 0) {
    float* cd = a.chunk_decay + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * kD;
#pragma unroll
    for (int j = 0; j < (kD + 31) / 32; ++j)
      if (j * 32 + lane < kD) cd[j * 32 + lane] = prod[j];
  }
  float* to = MODE == 1 ? chunk_state : ((MODE == 0 || last_chunk) ? slot_state : nullptr);
  if (to != nullptr) {
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int row = group * kRows + i;
      if (row >= kD) continue;
      float* p = to + static_cast<size_t>(row) * a.dv + col;
      if (a.pairs_ok) {
        if (in0) *reinterpret_cast<float2*>(p) = make_float2(S[i][0], S[i][1]);
      } else {
        if (in0) p[0] = S[i][0];
        if (in1) p[1] = S[i][1];
      }
    }
  }
}

// Pass 2: chunk_state[seq][c] <- A_c * (state after chunk c - 1) + chunk_state[seq][c], in order of c; A_c is the
// product of chunk c's decays (every chunk before the last is full).  One thread per element of a head's state.
__global__ void linear_attention_chain_kernel(const int32_t* __restrict__ seq_of_token,
                                              const int32_t* __restrict__ state_slot, const float* __restrict__ decay,
                                              const float* __restrict__ chunk_decay, const float* __restrict__ state,
                                              long long slot_stride, float* __restrict__ chunk_state, int tokens,
                                              int heads, int dv, int chunk, int max_chunks) {
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
    cd = chunk_decay + (static_cast<size_t>(seq) * max_chunks * heads + head) * kD + e / dv;
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
      dec[i] = (in && cd != nullptr) ? cd[static_cast<size_t>(c0 + i) * heads * kD] : dpow;
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

// Threads of a CTA for a head of dv columns.
inline int lin_threads(int dv) {
  const int need = (dv + kCols - 1) / kCols * kGroups;
  return need >= kMaxThreads ? kMaxThreads : (need + 31) / 32 * 32;
}

template <typename T, bool CHANNEL>
int launch_linear_attention(const LinArgs<T>& a, int sequences, cudaStream_t stream) {
  const int th = lin_threads(a.dv);
  const int cols = th / kGroups * kCols, blocks = (a.dv + cols - 1) / cols;
  const size_t smem = a.y != nullptr ? static_cast<size_t>(kTok) * a.dv * sizeof(float) : 0;
  if (a.y != nullptr && blocks != 1) return static_cast<int>(cudaErrorInvalidValue);
  if (a.chunk_state == nullptr || a.max_chunks <= 1)
    return static_cast<int>(launch_kernel(linear_attention_kernel<T, 0, CHANNEL>, dim3(blocks, a.heads, sequences),
                                          dim3(th), smem, stream, a));
  cudaError_t e = launch_kernel(linear_attention_kernel<T, 1, CHANNEL>, dim3(blocks, a.heads * a.max_chunks, sequences),
                                dim3(th), 0, stream, a);
  if (e != cudaSuccess) return static_cast<int>(e);
  const int plane = kD * a.dv;
  e = launch_kernel(linear_attention_chain_kernel, dim3((plane + 255) / 256, a.heads, sequences), dim3(256), 0, stream,
                    a.seq_of_token, a.state_slot, a.decay, static_cast<const float*>(CHANNEL ? a.chunk_decay : nullptr),
                    static_cast<const float*>(a.state), a.slot_stride, a.chunk_state, a.tokens, a.heads, a.dv, a.chunk,
                    a.max_chunks);
  if (e != cudaSuccess) return static_cast<int>(e);
  return static_cast<int>(launch_kernel(linear_attention_kernel<T, 3, CHANNEL>,
                                        dim3(blocks, a.heads * a.max_chunks, sequences), dim3(th), smem, stream, a));
}

}  // namespace rl

using namespace rl;

extern "C" {

// Whether one CTA covers all columns of a head (the finished heads can then be asked for).
int rl_linear_one_block(int dv) {
  const int th = lin_threads(dv);
  return dv <= th / kGroups * kCols ? 1 : 0;
}

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
                        int dv, int chunk, int max_chunks, cudaStream_t stream) {
  if (tokens <= 0 || sequences <= 0) return 0;
  const bool channel = bonus != nullptr;
  if (channel && (decay_bias == nullptr || (max_chunks > 1 && chunk_state != nullptr && chunk_decay == nullptr)))
    return static_cast<int>(cudaErrorInvalidValue);
#define RL_CASE(T)                                                                                                \
  do {                                                                                                            \
    LinArgs<T> a;                                                                                                 \
    a.q = static_cast<const T*>(q); a.k = static_cast<const T*>(k); a.v = static_cast<const T*>(v);               \
    a.q_ld = q_ld; a.k_ld = k_ld; a.v_ld = v_ld; a.k_scale = k_scale; a.cos_t = cos_t; a.sin_t = sin_t;           \
    a.positions = positions; a.rot_pairs = rot_pairs; a.max_pos = max_pos; a.seq_of_token = seq_of_token;         \
    a.state_slot = state_slot; a.decay = decay; a.decay_bias = decay_bias; a.bonus = bonus; a.state = state;      \
    a.slot_stride = slot_stride; a.out = out; a.y = static_cast<T*>(y); a.y_ld = y_ld;                            \
    a.gate = static_cast<const T*>(gate); a.gate_ld = gate_ld; a.gate_mode = gate_mode; a.norm_w = norm_w;        \
    a.eps = eps; a.chunk_state = chunk_state; a.chunk_decay = chunk_decay; a.status = status; a.tokens = tokens;  \
    a.heads = heads; a.dv = dv; a.chunk = chunk; a.max_chunks = max_chunks;                                       \
    a.pairs_ok = dv % 2 == 0 && slot_stride % 2 == 0 && reinterpret_cast<uintptr_t>(state) % 8 == 0 &&            \
                 reinterpret_cast<uintptr_t>(chunk_state) % 8 == 0;                                               \
    if (channel) return launch_linear_attention<T, true>(a, sequences, stream);                                   \
    return launch_linear_attention<T, false>(a, sequences, stream);                                               \
  } while (0)
  if (dtype == 0) RL_CASE(float);
  else RL_CASE(bf16);
#undef RL_CASE
}

int rl_linear_output(int dtype, const float* o, const void* gate, int gate_ld, int gate_mode, const float* w, void* y,
                     int y_ld, int tokens, int heads, int dv, float eps, cudaStream_t stream) {
  const int items = tokens * heads, warps = 8;
  if (items <= 0) return 0;
  const dim3 grid((items + warps - 1) / warps);
  if (dtype == 0)
    launch_kernel(linear_output_kernel<float>, grid, dim3(warps * 32), 0, stream, o, static_cast<const float*>(gate),
                  gate_ld, gate_mode, w, static_cast<float*>(y), y_ld, items, heads, dv, eps);
  else
    launch_kernel(linear_output_kernel<bf16>, grid, dim3(warps * 32), 0, stream, o, static_cast<const bf16*>(gate),
                  gate_ld, gate_mode, w, static_cast<bf16*>(y), y_ld, items, heads, dv, eps);
  RL_LAUNCH_END();
}

}  // extern "C"
