// The state-space recurrence of linear_attention.cu (a decay per token) for bfloat16 portions of several tokens,
// 64 tokens at a time on the tensor cores.  With d_t the step, l_t the sum of the decays' logarithms of a block's
// tokens up to and including t, and S the state before the block,
//
//   o_t = e^(l_t) S^T q_t + sum_(s <= t) M_ts v_s,       M_ts = (q_t . k_s) e^(l_t - l_s) d_s   (+ D where s = t)
//   S  <- e^(l_end) S + sum_s k_s (d_s e^(l_end - l_s) v_s)^T
//
// Every exponent is a sum of negative numbers.  All four products run on mma.sync with float32 accumulators; q, k and v
// are bfloat16 as they are, and what is not (the state, M, the weighted values) enters as a high and a low part, so
// that the result is off by some 2^-16 of its terms.  A CTA takes one sequence (chunk), one head and up to 64 value
// columns; each of its eight warps takes 16 of the block's tokens and half of the columns for the outputs, and every
// eighth tile of 16 rows and half of the columns of the state, which it keeps as accumulators; the state's two parts go
// to shared memory once per block, for the read-out of the next one.
#pragma once

namespace rl {

constexpr int kSL = 64;                        // tokens of a block
constexpr int kSV = 64;                        // value columns of a CTA
constexpr int kSN = kD + 8;                    // elements of a row of queries or keys in shared memory (spreads the banks)
constexpr int kSX = kSV + 8;                   // elements of a row of values; of a row of the state
constexpr int kSH = kSV / 2;                   // columns of a warp
constexpr int kSTiles = (kD / 16 * 2 + 7) / 8; // tiles of the state (16 rows, half of the columns) per warp
constexpr int kSsdThreads = 256;

__device__ __forceinline__ void ssd_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
template <bool TRANS>
__device__ __forceinline__ void ssd_ldmatrix(uint32_t* r, const bf16* p) {
  const unsigned addr = static_cast<unsigned>(__cvta_generic_to_shared(p));
  if (TRANS)
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
  else
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// (x, y) as bfloat16 pairs: the high parts and what is left
__device__ __forceinline__ void ssd_split(float x, float y, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(x - __uint_as_float(hi << 16), y - __uint_as_float(hi & 0xFFFF0000u));
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
// 2^x (results below the smallest normal number are zero)
__device__ __forceinline__ float ssd_exp2(float x) {
  float r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(x));
  return r;
}

struct SsdLayout {                             // bytes from the start of the dynamic shared memory
  int q, k, v, wh, wl, sh, sl, log, step, total, bytes;
};
__host__ __device__ inline SsdLayout ssd_layout(bool with_q) {
  SsdLayout r;
  int at = 0;
  auto take = [&](int n) { const int o = at; at += (n + 15) / 16 * 16; return o; };
  r.q = take(with_q ? kSL * kSN * 2 : 0);
  r.k = take(kSL * kSN * 2);
  r.v = take(kSL * kSX * 2);
  r.wh = take(kSL * kSX * 2);                  // weighted values, high and low parts
  r.wl = take(kSL * kSX * 2);
  r.sh = take(with_q ? kD * kSX * 2 : 0);      // the state's parts
  r.sl = take(with_q ? kD * kSX * 2 : 0);
  r.log = take(kSL * 4);                       // sums of logarithms within each half of the block
  r.step = take(kSL * 4);
  r.total = take(2 * 4);                       // of each half
  r.bytes = at;
  return r;
}

// Modes as in linear_attention_kernel.
template <int MODE>
__global__ void __launch_bounds__(kSsdThreads, kD <= 128 ? 2 : 1)
ssd_kernel(const LinArgs<bf16> a) {
  pdl_launch();
  pdl_wait();
  extern __shared__ __align__(16) unsigned char sm[];
  const int seq = blockIdx.z, head = blockIdx.y % a.heads, c = blockIdx.y / a.heads;
  const int qk_head = head / (a.heads / a.qk_heads);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, gid = lane >> 2, tig = lane & 3;
  const int col0 = blockIdx.x * kSV, cols = min(kSV, a.dv - col0);            // (a multiple of 16)
  const int rows0 = (warp & 3) * 16, half0 = (warp >> 2) * kSH;               // the warp's tokens and columns for the outputs
  const SsdLayout lay = ssd_layout(MODE != 1);
  bf16* qs = reinterpret_cast<bf16*>(sm + lay.q);
  bf16* ks = reinterpret_cast<bf16*>(sm + lay.k);
  bf16* vs = reinterpret_cast<bf16*>(sm + lay.v);
  bf16* wh = reinterpret_cast<bf16*>(sm + lay.wh);
  bf16* wl = reinterpret_cast<bf16*>(sm + lay.wl);
  bf16* sh = reinterpret_cast<bf16*>(sm + lay.sh);
  bf16* sl = reinterpret_cast<bf16*>(sm + lay.sl);
  float* logs = reinterpret_cast<float*>(sm + lay.log);
  float* steps = reinterpret_cast<float*>(sm + lay.step);
  float* total = reinterpret_cast<float*>(sm + lay.total);
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

  // tokens tb .. tb + nt - 1 on their way into shared memory (zeros for tokens that are not there); a thread per token
  // asks for its step's projection
  float z_ahead = 0.f;
  auto stage = [&](int tb, int nt) {
    if (threadIdx.x < nt) z_ahead = to_float(a.steps[static_cast<size_t>(tb + threadIdx.x) * a.steps_ld + head]);
    constexpr int kPer = kD / 8;                   // 16-byte pieces of a row of queries or keys
    for (int i = threadIdx.x; i < kSL * kPer; i += kSsdThreads) {
      const int tt = i / kPer, e = i % kPer;
      bf16 *tk = ks + tt * kSN + e * 8, *tq = qs + tt * kSN + e * 8;
      if (tt < nt) {
        const size_t t = tb + tt;
        async_copy16(tk, a.k + t * a.k_ld + qk_head * kD + e * 8);
        if (MODE != 1) async_copy16(tq, a.q + t * a.q_ld + qk_head * kD + e * 8);
      } else {
        *reinterpret_cast<uint4*>(tk) = make_uint4(0, 0, 0, 0);
        if (MODE != 1) *reinterpret_cast<uint4*>(tq) = make_uint4(0, 0, 0, 0);
      }
    }
    const int per = cols / 8;
    for (int i = threadIdx.x; i < kSL * per; i += kSsdThreads) {
      const int tt = i / per, e = i % per;
      bf16* tv = vs + tt * kSX + e * 8;
      if (tt < nt) async_copy16(tv, a.v + static_cast<size_t>(tb + tt) * a.v_ld + head * a.dv + col0 + e * 8);
      else *reinterpret_cast<uint4*>(tv) = make_uint4(0, 0, 0, 0);
    }
  };
  stage(t0, min(kSL, t1 - t0));

  constexpr float kLog2E = 1.4426950408889634f;
  const float rate = kLog2E * expf(a.a_log[head]), step_bias = a.step_bias[head], skip = a.skip[head];
  const size_t plane = static_cast<size_t>(kD) * a.dv;
  float* slot_state = a.state + static_cast<size_t>(a.state_slot[seq]) * a.slot_stride + head * plane;
  float* chunk_state = MODE == 0 ? nullptr
      : a.chunk_state + ((static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head) * plane;
  // S[i][j]: tile 8 i + warp (two tiles to 16 rows), rows gid and + 8 of it, columns j * 8 + 2 tig and + 1 of its half
  float S[kSTiles][kSH / 8][4];
  const int state_half = (warp & 1) * kSH;         // (8 i + warp and warp have the same half)
  auto row_of = [&](int i) { return (8 * i + warp) / 2 * 16 + gid; };
  auto tile_in = [&](int i) { return (8 * i + warp) / 2 * 16 < kD; };
  {
    const float* from = slot_state;
    if (MODE == 3 && c > 0) from = chunk_state - static_cast<size_t>(a.heads) * plane;
    else if (MODE == 3 && !last_chunk) {
      const int chunks = (seq_end - seq_begin + a.chunk - 1) / a.chunk;
      from = chunk_state + static_cast<size_t>(chunks - 1) * a.heads * plane;
    }
#pragma unroll
    for (int i = 0; i < kSTiles; ++i)
#pragma unroll
      for (int j = 0; j < kSH / 8; ++j) {
        const bool in = MODE != 1 && tile_in(i) && state_half + j * 8 < cols;
        const float* p = from + static_cast<size_t>(row_of(i)) * a.dv + col0 + state_half + j * 8 + 2 * tig;
        float2 x = make_float2(0.f, 0.f), y = x;
        if (in) {
          if (a.quads_ok) {
            x = *reinterpret_cast<const float2*>(p);
            y = *reinterpret_cast<const float2*>(p + 8 * static_cast<size_t>(a.dv));
          } else {
            x = make_float2(p[0], p[1]);
            y = make_float2(p[8 * static_cast<size_t>(a.dv)], p[8 * static_cast<size_t>(a.dv) + 1]);
          }
        }
        S[i][j][0] = x.x; S[i][j][1] = x.y; S[i][j][2] = y.x; S[i][j][3] = y.y;
      }
  }
  float chunk_log = 0.f;

  for (int tb = t0; tb < t1; tb += kSL) {
    const int nt = min(kSL, t1 - tb);
    // ---- steps and the sums of their decays' logarithms (within each half); the state's parts
    if (threadIdx.x < kSL) {
      const float d = threadIdx.x < nt ? softplus(z_ahead + step_bias) : 0.f;
      float l = fmaxf(-rate * d, -160.f);          // (2^l is zero there anyway; the sums stay small numbers)
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, l, o);
        if (lane >= o) l += up;
      }
      logs[threadIdx.x] = l;
      steps[threadIdx.x] = d;
      if (lane == 31) total[warp] = l;
    }
    if (MODE != 1) {
#pragma unroll
      for (int i = 0; i < kSTiles; ++i)
        if (tile_in(i)) {
#pragma unroll
          for (int j = 0; j < kSH / 8; ++j)
            if (state_half + j * 8 < cols) {
              const int at = row_of(i) * kSX + state_half + j * 8 + 2 * tig;
              uint32_t hi, lo;
              ssd_split(S[i][j][0], S[i][j][1], hi, lo);
              *reinterpret_cast<uint32_t*>(sh + at) = hi;
              *reinterpret_cast<uint32_t*>(sl + at) = lo;
              ssd_split(S[i][j][2], S[i][j][3], hi, lo);
              *reinterpret_cast<uint32_t*>(sh + at + 8 * kSX) = hi;
              *reinterpret_cast<uint32_t*>(sl + at + 8 * kSX) = lo;
            }
        }
    }
    async_copies_done();
    __syncthreads();
    const float half = total[0], end = half + total[1];
    auto log_at = [&](int t) { return logs[t] + (t >= 32 ? half : 0.f); };
    // ---- the values times d_s e^(l_end - l_s): four threads to a token
    {
      const int s = threadIdx.x >> 2, c0 = (threadIdx.x & 3) * (kSV / 4);
      const float w = steps[s] * ssd_exp2(end - log_at(s));
#pragma unroll
      for (int e = 0; e < kSV / 4; e += 8)
        if (c0 + e < cols) {
          float v[8];
          load16(vs + s * kSX + c0 + e, v);
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int p = 0; p < 4; ++p) ssd_split(v[2 * p] * w, v[2 * p + 1] * w, hi[p], lo[p]);
          *reinterpret_cast<uint4*>(wh + s * kSX + c0 + e) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
          *reinterpret_cast<uint4*>(wl + s * kSX + c0 + e) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
        }
    }
    if (MODE != 1 && rows0 < nt && half0 < cols) {
      const int r0 = rows0 + gid, r1 = r0 + 8;                   // this thread's two tokens of the block
      float o[kSH / 8][4], g[kSL / 8][4];
#pragma unroll
      for (int j = 0; j < kSH / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
#pragma unroll
      for (int j = 0; j < kSL / 8; ++j) g[j][0] = g[j][1] = g[j][2] = g[j][3] = 0.f;
#pragma unroll 4
      for (int kk = 0; kk < kD / 16; ++kk) {
        uint32_t qa[4];
        ssd_ldmatrix<false>(qa, qs + (rows0 + (lane & 15)) * kSN + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int j = 0; j < kSL / 8; j += 2)
          if (j * 8 < rows0 + 16) {                              // (tokens s <= t only)
            uint32_t b[4];
            ssd_ldmatrix<false>(b, ks + (j * 8 + (lane & 7) + (lane >> 4) * 8) * kSN + kk * 16 + ((lane >> 3) & 1) * 8);
            ssd_mma(g[j], qa, b[0], b[1]);
            ssd_mma(g[j + 1], qa, b[2], b[3]);
          }
#pragma unroll
        for (int j = 0; j < kSH / 8; j += 2)
          if (half0 + j * 8 < cols) {
            uint32_t b[4];
            const int at = (kk * 16 + (lane & 15)) * kSX + half0 + j * 8 + (lane >> 4) * 8;
            ssd_ldmatrix<true>(b, sl + at);
            ssd_mma(o[j], qa, b[0], b[1]);
            ssd_mma(o[j + 1], qa, b[2], b[3]);
            ssd_ldmatrix<true>(b, sh + at);
            ssd_mma(o[j], qa, b[0], b[1]);
            ssd_mma(o[j + 1], qa, b[2], b[3]);
          }
      }
      const float l0 = log_at(r0), l1 = log_at(r1);
      const float e0 = ssd_exp2(l0), e1 = ssd_exp2(l1);
#pragma unroll
      for (int j = 0; j < kSH / 8; ++j) {
        o[j][0] *= e0;
        o[j][1] *= e0;
        o[j][2] *= e1;
        o[j][3] *= e1;
      }
#pragma unroll
      for (int kk = 0; kk < kSL / 16; ++kk) {
        if (kk * 16 > rows0) continue;
        uint32_t mh[4], ml[4];
#pragma unroll
        for (int h = 0; h < 2; ++h) {                            // the 16 columns' two tiles
          const int s = (2 * kk + h) * 8 + 2 * tig;
          const float x0 = log_at(s), x1 = log_at(s + 1), d0 = steps[s], d1 = steps[s + 1];
          auto m = [&](float dot, int t, float lt, int sc, float ls, float d) {
            const float v = sc <= t ? dot * ssd_exp2(lt - ls) * d : 0.f;
            return sc == t ? v + skip : v;
          };
          const float* q = g[2 * kk + h];
          ssd_split(m(q[0], r0, l0, s, x0, d0), m(q[1], r0, l0, s + 1, x1, d1), mh[2 * h], ml[2 * h]);
          ssd_split(m(q[2], r1, l1, s, x0, d0), m(q[3], r1, l1, s + 1, x1, d1), mh[2 * h + 1], ml[2 * h + 1]);
        }
#pragma unroll
        for (int j = 0; j < kSH / 8; j += 2)
          if (half0 + j * 8 < cols) {
            uint32_t b[4];
            ssd_ldmatrix<true>(b, vs + (kk * 16 + (lane & 15)) * kSX + half0 + j * 8 + (lane >> 4) * 8);
            ssd_mma(o[j], ml, b[0], b[1]);
            ssd_mma(o[j + 1], ml, b[2], b[3]);
            ssd_mma(o[j], mh, b[0], b[1]);
            ssd_mma(o[j + 1], mh, b[2], b[3]);
          }
      }
      float* out = a.out + static_cast<size_t>(tb) * (a.heads * a.dv) + head * a.dv + col0 + half0 + 2 * tig;
      const size_t row = static_cast<size_t>(a.heads) * a.dv;
#pragma unroll
      for (int j = 0; j < kSH / 8; ++j)
        if (half0 + j * 8 < cols) {
          if (r0 < nt) *reinterpret_cast<float2*>(out + r0 * row + j * 8) = make_float2(o[j][0], o[j][1]);
          if (r1 < nt) *reinterpret_cast<float2*>(out + r1 * row + j * 8) = make_float2(o[j][2], o[j][3]);
        }
    }
    __syncthreads();                 // the weighted values are there
    if (MODE != 3 || tb + kSL < t1 || last_chunk) {
      const float e = ssd_exp2(end);
#pragma unroll
      for (int i = 0; i < kSTiles; ++i)
        if (tile_in(i)) {
#pragma unroll
          for (int j = 0; j < kSH / 8; ++j) {
            S[i][j][0] *= e;
            S[i][j][1] *= e;
            S[i][j][2] *= e;
            S[i][j][3] *= e;
          }
        }
#pragma unroll
      for (int kk = 0; kk < kSL / 16; ++kk) {
        if (kk * 16 >= nt) continue;
        uint32_t ka[kSTiles][4];
#pragma unroll
        for (int i = 0; i < kSTiles; ++i)
          if (tile_in(i))
            ssd_ldmatrix<true>(ka[i], ks + (kk * 16 + (lane & 7) + (lane >> 4) * 8) * kSN + (8 * i + warp) / 2 * 16 + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int j = 0; j < kSH / 8; j += 2)
          if (state_half + j * 8 < cols) {
            uint32_t bh[4], bl[4];
            const int at = (kk * 16 + (lane & 15)) * kSX + state_half + j * 8 + (lane >> 4) * 8;
            ssd_ldmatrix<true>(bl, wl + at);
            ssd_ldmatrix<true>(bh, wh + at);
#pragma unroll
            for (int i = 0; i < kSTiles; ++i)
              if (tile_in(i)) {
                ssd_mma(S[i][j], ka[i], bl[0], bl[1]);
                ssd_mma(S[i][j + 1], ka[i], bl[2], bl[3]);
                ssd_mma(S[i][j], ka[i], bh[0], bh[1]);
                ssd_mma(S[i][j + 1], ka[i], bh[2], bh[3]);
              }
          }
      }
    }
    if (MODE == 1) chunk_log += end;
    __syncthreads();                 // the block has been worked on
    if (tb + kSL < t1) stage(tb + kSL, min(kSL, t1 - tb - kSL));
  }
  if (MODE == 1 && blockIdx.x == 0 && threadIdx.x == 0)
    a.chunk_decay[(static_cast<size_t>(seq) * a.max_chunks + c) * a.heads + head] = exp2f(chunk_log);
  float* to = MODE == 1 ? chunk_state : ((MODE == 0 || last_chunk) ? slot_state : nullptr);
  if (to == nullptr) return;
#pragma unroll
  for (int i = 0; i < kSTiles; ++i)
    if (tile_in(i)) {
#pragma unroll
      for (int j = 0; j < kSH / 8; ++j)
        if (state_half + j * 8 < cols) {
          float* p = to + static_cast<size_t>(row_of(i)) * a.dv + col0 + state_half + j * 8 + 2 * tig;
          float* p8 = p + 8 * static_cast<size_t>(a.dv);
          if (a.quads_ok) {
            *reinterpret_cast<float2*>(p) = make_float2(S[i][j][0], S[i][j][1]);
            *reinterpret_cast<float2*>(p8) = make_float2(S[i][j][2], S[i][j][3]);
          } else {
            p[0] = S[i][j][0];
            p[1] = S[i][j][1];
            p8[0] = S[i][j][2];
            p8[1] = S[i][j][3];
          }
        }
    }
}

template <int MODE>
cudaError_t launch_ssd_pass(const LinArgs<bf16>& a, int rows, int sequences, cudaStream_t stream) {
  const SsdLayout lay = ssd_layout(MODE != 1);
  static bool set = false;
  if (!set) {
    const cudaError_t e = cudaFuncSetAttribute(ssd_kernel<MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, lay.bytes);
    if (e != cudaSuccess) return e;
    set = true;
  }
  return launch_kernel(ssd_kernel<MODE>, dim3((a.dv + kSV - 1) / kSV, rows, sequences), dim3(kSsdThreads), lay.bytes, stream, a);
}

}  // namespace rl
