// The recurrence of linear_attention.cu for bfloat16 portions of several tokens, sixteen tokens at a time on the
// tensor cores.  With c_t the sum of the decays' logarithms of a block's tokens up to and including t (per
// channel, or the same for all channels), S the state before the block and b the sum before t,
//
//   o_t = S^T (q_t exp(b_t)) + sum_s P_ts v_s          P_ts = sum_i q_ti k_si exp(b_ti - c_si)
//   S  <- diag(exp(c_end)) S + sum_s (k_s exp(c_end - c_s)) v_s^T
//
// (a decay per channel: b_t = c_(t-1), s < t, and P_tt = sum q u k; one decay per head: b_t = c_t, s <= t).  Every
// exponent is a sum of negative numbers: nothing overflows and nothing is divided by.  The pairs P are formed on
// the CUDA cores in float32; the rest are products of bfloat16 operands with float32 accumulators in which what
// is not bfloat16 to begin with (state, decayed queries and keys, P) enters as a high and a low part, so that the
// result is off by some 2^-16 of its terms.  A warp keeps the transposed state of 16 value columns as the
// accumulators of its updates; two neighbouring accumulator tiles are the operand of the read-out as they are.
// (mma.sync: a block's operands are 16 rows high and its state lives in registers.)
#pragma once

namespace rl {

constexpr int kBlk = 16;                       // tokens of a block
constexpr int kFS = kD % 32 == 0 ? kD + 16 : kD;       // floats of a row of queries, keys or logarithms (spreads the banks)
constexpr int kQS = kD + 8;                    // elements of a row of decayed queries
constexpr int kKS = kBlk + 2;                  // elements of a row (a channel) of decayed keys; of a row of P
constexpr int kTcMaxWarps = kTcMaxCols / 16;   // 16 value columns each

__device__ __forceinline__ void lin_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pair_bits(float lo, float hi) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// (x, y) as bfloat16 pairs: the high parts and what is left
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pair_bits(x, y);
  lo = pair_bits(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
}
__device__ __forceinline__ void split1(float x, bf16& hi, bf16& lo) {
  hi = __float2bfloat16_rn(x);
  lo = __float2bfloat16_rn(x - __bfloat162float(hi));
}

// 2^x (the logarithms here are to the base 2; results below the smallest normal number are zero)
__device__ __forceinline__ float exp2_of(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}
constexpr float kLog2E = 1.4426950408889634f;
// log2 of exp(-exp(z)).  Bounded where 2^x is zero anyway, so that the sums along a block stay small numbers whose
// differences are exact to rounding (and finite).
__device__ __forceinline__ float log_of_decay(float z) { return fmaxf(-kLog2E * exp2_of(kLog2E * z), -160.f); }

struct TcLayout {                              // bytes from the start of the dynamic shared memory
  int raw_bytes, q, k, v, g, z, cs, sn;        // a raw buffer's size, its parts; rows of qk_row, v_row, ... bytes
  int qk_row, v_row, z_row, rot_row;
  int qf, kf, logs, after, total, chunk, diag, bias, bonus, qd, kd, p, squares, bytes;
};
__host__ __device__ inline TcLayout tc_layout(int cols, int rot_pairs, bool channel, bool with_q, bool gated, bool finish) {
  TcLayout r;
  auto up = [](int n) { return (n + 15) / 16 * 16; };
  r.qk_row = kD * 2;
  r.v_row = up(cols * 2);
  r.z_row = channel ? kD * 4 : 0;
  r.rot_row = up(rot_pairs * 4);
  r.q = 0;
  r.k = with_q ? kBlk * r.qk_row : 0;
  r.v = r.k + kBlk * r.qk_row;
  r.g = r.v + kBlk * r.v_row;
  r.z = r.g + (gated ? kBlk * r.v_row : 0);
  r.cs = r.z + kBlk * r.z_row;
  r.sn = r.cs + kBlk * r.rot_row;
  r.raw_bytes = r.sn + kBlk * r.rot_row;
  int at = 2 * r.raw_bytes;
  auto take = [&](int n) { const int o = at; at += up(n); return o; };
  r.qf = take(with_q ? kBlk * kFS * 4 : 0);
  r.kf = take(kBlk * kFS * 4);
  r.logs = take(channel ? kBlk * kFS * 4 : 0);
  r.after = take(channel && with_q ? kBlk * kFS * 4 : 0);          // their sums up to and including a token
  r.total = take(kD * 4);
  r.chunk = take(kD * 4);
  r.diag = take(kBlk * 4);
  r.bias = take(channel ? kD * 4 : 0);
  r.bonus = take(channel && with_q ? kD * 4 : 0);
  r.qd = take(with_q ? 2 * kBlk * kQS * 2 : 0);          // high parts, then low parts
  r.kd = take(2 * kD * kKS * 2);
  r.p = take(with_q ? 2 * kBlk * kKS * 2 : 0);
  r.squares = take(finish ? kBlk * kTcMaxWarps * 4 : 0);
  r.bytes = at;
  return r;
}

// Modes as in linear_attention_kernel.  A CTA takes one sequence (chunk), one head and 16 value columns per warp.
template <int MODE, bool CHANNEL>
__global__ void __launch_bounds__(kTcMaxWarps * 32, kD <= 128 ? 2 : 1)
linear_attention_tc_kernel(const LinArgs<bf16> a) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) unsigned char sm[];
  const int seq = blockIdx.z, head = blockIdx.y % a.heads, c = blockIdx.y / a.heads;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarps = blockDim.x >> 5;
  const int gid = lane >> 2, tig = lane & 3;
  const int block_cols = nwarps * 16, col0 = blockIdx.x * block_cols;
  const int wcol = col0 + warp * 16;                     // the warp's first column
  const bool live = wcol < a.dv;                         // (dv is a multiple of 16)
  const bool finish = MODE != 1 && a.y != nullptr, gated = finish && a.gate_mode != GATE_NONE;
  const TcLayout lay = tc_layout(block_cols, a.rot_pairs, CHANNEL, MODE != 1, gated, finish);
  float* qf = reinterpret_cast<float*>(sm + lay.qf);
  float* kf = reinterpret_cast<float*>(sm + lay.kf);
  float* after = reinterpret_cast<float*>(sm + lay.after);
  float* logs = reinterpret_cast<float*>(sm + lay.logs);
  float* total = reinterpret_cast<float*>(sm + lay.total);
  float* chunk_log = reinterpret_cast<float*>(sm + lay.chunk);
  bf16* qd = reinterpret_cast<bf16*>(sm + lay.qd);
  bf16* kd = reinterpret_cast<bf16*>(sm + lay.kd);
  bf16* pp = reinterpret_cast<bf16*>(sm + lay.p);
  float* diag = reinterpret_cast<float*>(sm + lay.diag);            // per channel: sum q u k of every token
  float* bias = reinterpret_cast<float*>(sm + lay.bias);
  float* bonus = reinterpret_cast<float*>(sm + lay.bonus);
  float* squares = reinterpret_cast<float*>(sm + lay.squares);      // [tokens][warps]: sums of o^2 over a warp's columns
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
  if (MODE == 1 && last_chunk) return;
  int pos0 = 0;
  if (a.rot_pairs > 0) {
    pos0 = a.positions[t0];
    if (pos0 < 0 || pos0 + (t1 - t0) > a.max_pos) {
      if (threadIdx.x == 0) atomicOr(a.status, 2);
      pos0 = -1;
    }
  }

  // tokens tb .. tb + nt - 1 on their way into buffer b, in pieces of 16 bytes.  A row of values has 2 nwarps pieces,
  // so that every thread has one of them.
  const int v_tok = threadIdx.x / (2 * nwarps), v_piece = threadIdx.x % (2 * nwarps);
  const bool v_in = col0 + v_piece * 8 < a.dv;
  auto stage = [&](int b, int tb, int nt) {
    unsigned char* buf = sm + b * lay.raw_bytes;
    constexpr int kPer = kD / 8;                 // pieces of a row of queries or keys
    for (int i = threadIdx.x; i < kBlk * kPer; i += blockDim.x) {
      const int tt = i / kPer, e = i % kPer;
      if (tt < nt) {
        const size_t t = tb + tt;
        if (MODE != 1) async_copy16(buf + lay.q + tt * lay.qk_row + e * 16, a.q + t * a.q_ld + head * kD + e * 8);
        async_copy16(buf + lay.k + tt * lay.qk_row + e * 16, a.k + t * a.k_ld + head * kD + e * 8);
      }
    }
    if (CHANNEL) {
      constexpr int kPerZ = kD / 4;
      for (int i = threadIdx.x; i < kBlk * kPerZ; i += blockDim.x) {
        const int tt = i / kPerZ, e = i % kPerZ;
        if (tt < nt)
          async_copy16(buf + lay.z + tt * lay.z_row + e * 16, a.decay + (static_cast<size_t>(tb + tt) * a.heads + head) * kD + e * 4);
      }
    }
    if (v_in) {
      const size_t t = tb + v_tok;
      unsigned char* to = buf + v_tok * lay.v_row + v_piece * 16;
      if (v_tok >= nt) {                         // a token that is not there: its value is multiplied by zeros
        *reinterpret_cast<uint4*>(to + lay.v) = make_uint4(0, 0, 0, 0);
      } else {
        async_copy16(to + lay.v, a.v + t * a.v_ld + head * a.dv + col0 + v_piece * 8);
        if (gated) async_copy16(to + lay.g, a.gate + t * a.gate_ld + head * a.dv + v_piece * 8);
      }
    }
    if (a.rot_pairs > 0) {
      const int per = a.rot_pairs / 4;
      for (int tt = warp; tt < nt; tt += nwarps) {
        const size_t at = pos0 < 0 ? 0 : static_cast<size_t>(pos0 + tb + tt - t0) * a.rot_pairs;
        for (int e = lane; e < per; e += 32) {
          async_copy16(buf + lay.cs + tt * lay.rot_row + e * 16, a.cos_t + at + e * 4);
          async_copy16(buf + lay.sn + tt * lay.rot_row + e * 16, a.sin_t + at + e * 4);
        }
      }
    }
  };
  stage(0, t0, min(kBlk, t1 - t0));

  const size_t plane = static_cast<size_t>(kD) * a.dv;
  float* slot_state = a.state + static_cast<size_t>(a.state_slot[seq]) * a.slot_stride + head * plane;
  float* chunk_state = MODE == 0 ? nullptr
      : a.chunk_state + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * plane;
  // S[j]: channels j * 8 + 2 tig and + 1, columns gid and gid + 8 of the warp
  float S[kD / 8][4];
  {
    const float* from = slot_state;
    if (MODE == 3 && c > 0) from = chunk_state - static_cast<size_t>(a.heads) * plane;
    else if (MODE == 3 && !last_chunk) {
      const int chunks = (seq_end - seq_begin + a.chunk - 1) / a.chunk;
      from = chunk_state + static_cast<size_t>(chunks - 1) * a.heads * plane;
    }
#pragma unroll
    for (int j = 0; j < kD / 8; ++j) {
      const float* p = from + static_cast<size_t>(j * 8 + 2 * tig) * a.dv + wcol + gid;
      S[j][0] = MODE != 1 && live ? p[0] : 0.f;
      S[j][1] = MODE != 1 && live ? p[a.dv] : 0.f;
      S[j][2] = MODE != 1 && live ? p[8] : 0.f;
      S[j][3] = MODE != 1 && live ? p[a.dv + 8] : 0.f;
    }
  }
  const float log_decay = CHANNEL ? 0.f : kLog2E * logf(fmaxf(a.decay[head], 1e-30f));
  if (CHANNEL)
    for (int d = threadIdx.x; d < kD; d += blockDim.x) {
      bias[d] = a.decay_bias[head * kD + d];
      if (MODE != 1) bonus[d] = a.bonus[head * kD + d];
      else chunk_log[d] = 0.f;
    }
  float norm_w[2] = {1.f, 1.f};
  if (finish && live && a.norm_w != nullptr) {
    norm_w[0] = a.norm_w[head * a.dv + wcol + gid];
    norm_w[1] = a.norm_w[head * a.dv + wcol + gid + 8];
  }

  int b = 0;
  for (int tb = t0; tb < t1; tb += kBlk, b ^= 1) {
    const int nt = min(kBlk, t1 - tb);
    async_copies_done();
    __syncthreads();
    if (tb + kBlk < t1) stage(b ^ 1, tb + kBlk, min(kBlk, t1 - tb - kBlk));
    const unsigned char* buf = sm + b * lay.raw_bytes;
    // ---- queries and keys as float32 (rotated, scaled), the decays' logarithms; a warp per token
    for (int tt = warp; tt < kBlk; tt += nwarps) {
      const bf16* qr = reinterpret_cast<const bf16*>(buf + lay.q + tt * lay.qk_row);
      const bf16* kr = reinterpret_cast<const bf16*>(buf + lay.k + tt * lay.qk_row);
      const float* zr = reinterpret_cast<const float*>(buf + lay.z + tt * lay.z_row);
      const float* cs = reinterpret_cast<const float*>(buf + lay.cs + tt * lay.rot_row);
      const float* sn = reinterpret_cast<const float*>(buf + lay.sn + tt * lay.rot_row);
      float own = 0.f;
#pragma unroll
      for (int j = 0; j < (kD + 63) / 64; ++j) {
        const int d = j * 64 + 2 * lane;
        if (d >= kD) continue;
        float2 kv = make_float2(0.f, 0.f), qv = kv, lw = kv;
        if (tt < nt) {
          kv = load2(kr + d);
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
          kv = make_float2(kv.x * a.k_scale, kv.y * a.k_scale);
          if (CHANNEL) {
            const float2 z = load2(zr + d), zb = load2(bias + d);
            if (MODE != 1) {
              const float2 u = load2(bonus + d);
              own = fmaf(qv.x * u.x, kv.x, fmaf(qv.y * u.y, kv.y, own));
            }
            lw = make_float2(log_of_decay(z.x + zb.x), log_of_decay(z.y + zb.y));
          }
        }
        *reinterpret_cast<float2*>(kf + tt * kFS + d) = kv;
        if (MODE != 1) *reinterpret_cast<float2*>(qf + tt * kFS + d) = qv;
        if (CHANNEL) *reinterpret_cast<float2*>(logs + tt * kFS + d) = lw;
      }
      if (CHANNEL && MODE != 1) {
        own = warp_sum(own);
        if (lane == 0) diag[tt] = own;
      }
    }
    __syncthreads();
    // ---- per channel along the tokens: decayed queries and keys, the sums of the logarithms
    if (CHANNEL) {
      // (a thread per channel for the keys, another for the queries)
      for (int i = threadIdx.x; i < (MODE == 1 ? kD : 2 * kD); i += blockDim.x) {
        float sum = 0.f;
        if (i < kD) {
          const int d = i;
          float upto[kBlk];
#pragma unroll
          for (int t = 0; t < kBlk; ++t) {
            sum += logs[t * kFS + d];
            upto[t] = sum;
            if (MODE != 1) after[t * kFS + d] = sum;
          }
          total[d] = exp2_of(sum);
          if (MODE == 1) chunk_log[d] += sum;
#pragma unroll
          for (int t = 0; t < kBlk; t += 2) {
            uint32_t hi, lo;
            split2(kf[t * kFS + d] * exp2_of(sum - upto[t]), kf[(t + 1) * kFS + d] * exp2_of(sum - upto[t + 1]), hi, lo);
            *reinterpret_cast<uint32_t*>(kd + d * kKS + t) = hi;
            *reinterpret_cast<uint32_t*>(kd + (kD + d) * kKS + t) = lo;
          }
        } else {
          const int d = i - kD;
#pragma unroll
          for (int t = 0; t < kBlk; ++t) {
            split1(qf[t * kFS + d] * exp2_of(sum), qd[t * kQS + d], qd[(kBlk + t) * kQS + d]);
            sum += logs[t * kFS + d];
          }
        }
      }
    } else {
      for (int i = threadIdx.x; i < (MODE == 1 ? kD : 2 * kD); i += blockDim.x) {
        if (i < kD) {
          const int d = i;
          if (d == 0) total[0] = exp2_of(log_decay * nt);
#pragma unroll
          for (int t = 0; t < kBlk; t += 2) {
            uint32_t hi, lo;       // (a token that is not there has a zero key)
            split2(kf[t * kFS + d] * exp2_of(log_decay * max(nt - 1 - t, 0)),
                   kf[(t + 1) * kFS + d] * exp2_of(log_decay * max(nt - 2 - t, 0)), hi, lo);
            *reinterpret_cast<uint32_t*>(kd + d * kKS + t) = hi;
            *reinterpret_cast<uint32_t*>(kd + (kD + d) * kKS + t) = lo;
          }
        } else {
          const int d = i - kD;
#pragma unroll
          for (int t = 0; t < kBlk; ++t)
            split1(qf[t * kFS + d] * exp2_of(log_decay * (t + 1)), qd[t * kQS + d], qd[(kBlk + t) * kQS + d]);
        }
      }
    }
    __syncthreads();
    // ---- the pairs within the block: four lanes to a pair, a quarter of the channels each
    if (MODE != 1) {
      for (int p0 = warp * 8; p0 < kBlk * kBlk; p0 += nwarps * 8) {
        const int t = p0 >> 4, s = (p0 & 15) + gid;
        float acc = 0.f;
        if (CHANNEL ? s < t : s <= t) {          // (the channels in groups of four, lane after lane)
          const float* qr = qf + t * kFS + tig * 4;
          const float* kr = kf + s * kFS + tig * 4;
          if (!CHANNEL) {
#pragma unroll
            for (int d = 0; d < kD; d += 16) {
              float x[4], y[4];
              load4(qr + d, x);
              load4(kr + d, y);
#pragma unroll
              for (int j = 0; j < 4; ++j) acc = fmaf(x[j], y[j], acc);
            }
            acc *= exp2_of(log_decay * (t - s));
          } else {
            const float* br = after + (t - 1) * kFS + tig * 4;
            const float* ar = after + s * kFS + tig * 4;
#pragma unroll
            for (int d = 0; d < kD; d += 16) {
              float x[4], y[4], e[4], f[4];
              load4(qr + d, x);
              load4(kr + d, y);
              load4(br + d, e);
              load4(ar + d, f);
#pragma unroll
              for (int j = 0; j < 4; ++j) acc = fmaf(x[j] * y[j], exp2_of(e[j] - f[j]), acc);
            }
          }
        }
        acc += __shfl_xor_sync(0xffffffffu, acc, 1);
        acc += __shfl_xor_sync(0xffffffffu, acc, 2);
        if (CHANNEL && s == t) acc = diag[t];
        if (tig == 0) split1(acc, pp[t * kKS + s], pp[(kBlk + t) * kKS + s]);
      }
      __syncthreads();
    }
    // ---- the products
    uint32_t va[4];                              // v^T: the warp's 16 columns x 16 tokens
    {
      const unsigned addr = static_cast<unsigned>(__cvta_generic_to_shared(
          buf + lay.v + ((lane & 7) + (lane & 16 ? 8 : 0)) * lay.v_row + (warp * 16 + (lane & 8 ? 8 : 0)) * 2));
      asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                   : "=r"(va[0]), "=r"(va[1]), "=r"(va[2]), "=r"(va[3]) : "r"(addr));
    }
    auto word = [](const bf16* p) { return *reinterpret_cast<const uint32_t*>(p); };
    if (MODE != 1) {
      float o[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
        const bf16* hi = pp + (n * 8 + gid) * kKS + 2 * tig;
        const bf16* lo = hi + kBlk * kKS;
        lin_mma(o[n], va, word(lo), word(lo + 8));
        lin_mma(o[n], va, word(hi), word(hi + 8));
      }
#pragma unroll
      for (int k = 0; k < kD / 16; ++k) {
        uint32_t sh[4], sl[4];
        split2(S[2 * k][0], S[2 * k][1], sh[0], sl[0]);
        split2(S[2 * k][2], S[2 * k][3], sh[1], sl[1]);
        split2(S[2 * k + 1][0], S[2 * k + 1][1], sh[2], sl[2]);
        split2(S[2 * k + 1][2], S[2 * k + 1][3], sh[3], sl[3]);
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const bf16* hi = qd + (n * 8 + gid) * kQS + k * 16 + 2 * tig;
          const bf16* lo = hi + kBlk * kQS;
          const uint32_t h0 = word(hi), h1 = word(hi + 8);
          lin_mma(o[n], sl, h0, h1);
          lin_mma(o[n], sh, word(lo), word(lo + 8));
          lin_mma(o[n], sh, h0, h1);
        }
      }
      if (!finish) {
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int tt = n * 8 + 2 * tig + (e & 1), col = wcol + gid + (e & 2 ? 8 : 0);
            if (live && tt < nt) a.out[static_cast<size_t>(tb + tt) * (a.heads * a.dv) + head * a.dv + col] = o[n][e];
          }
      } else {
        // unit norm over the head: squares of this warp's columns, then of all warps, token by token
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            float ss = fmaf(o[n][h], o[n][h], o[n][h + 2] * o[n][h + 2]);
            ss += __shfl_xor_sync(0xffffffffu, ss, 4);
            ss += __shfl_xor_sync(0xffffffffu, ss, 8);
            ss += __shfl_xor_sync(0xffffffffu, ss, 16);
            if (gid == 0) squares[(n * 8 + 2 * tig + h) * kTcMaxWarps + warp] = ss;
          }
        __syncthreads();
        const int cols = warp * 16 + gid;
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int h = 0; h < 2; ++h) {
            const int tt = n * 8 + 2 * tig + h;
            float ss = 0.f;
            for (int w = 0; w < nwarps; ++w) ss += squares[tt * kTcMaxWarps + w];
            const float r = rsqrtf(ss / static_cast<float>(a.dv) + a.eps);
            if (tt >= nt) continue;
            bf16* yr = a.y + static_cast<size_t>(tb + tt) * a.y_ld + head * a.dv + cols;
            const bf16* gr = reinterpret_cast<const bf16*>(buf + lay.g + tt * lay.v_row) + cols;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              float y = o[n][h + 2 * e] * r * norm_w[e];
              if (gated) {
                const float g = to_float(gr[8 * e]);
                const float sig = __fdividef(1.f, 1.f + exp2_of(-kLog2E * g));
                y *= a.gate_mode == GATE_SILU ? g * sig : sig;
              }
              yr[8 * e] = __float2bfloat16_rn(y);
            }
          }
      }
    }
#pragma unroll
    for (int j = 0; j < kD / 8; ++j) {
      const float f0 = CHANNEL ? total[j * 8 + 2 * tig] : total[0], f1 = CHANNEL ? total[j * 8 + 2 * tig + 1] : f0;
      S[j][0] *= f0;
      S[j][1] *= f1;
      S[j][2] *= f0;
      S[j][3] *= f1;
      const bf16* hi = kd + (j * 8 + gid) * kKS + 2 * tig;
      const bf16* lo = hi + kD * kKS;
      lin_mma(S[j], va, word(lo), word(lo + 8));
      lin_mma(S[j], va, word(hi), word(hi + 8));
    }
  }
  if (CHANNEL && MODE == 1 && blockIdx.x == 0) {
    __syncthreads();
    float* cd = a.chunk_decay + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * kD;
    for (int d = threadIdx.x; d < kD; d += blockDim.x) cd[d] = exp2f(chunk_log[d]);
  }
  float* to = MODE == 1 ? chunk_state : ((MODE == 0 || last_chunk) ? slot_state : nullptr);
  if (to != nullptr && live) {
#pragma unroll
    for (int j = 0; j < kD / 8; ++j) {
      float* p = to + static_cast<size_t>(j * 8 + 2 * tig) * a.dv + wcol + gid;
      p[0] = S[j][0];
      p[a.dv] = S[j][1];
      p[8] = S[j][2];
      p[a.dv + 8] = S[j][3];
    }
  }
}

}  // namespace rl
