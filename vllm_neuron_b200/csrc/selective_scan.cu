// Selective state-space scan with a step size per channel and a full [channel][state] decay matrix (the Mamba-1 form; ssd_scan
// of ssm_scan.cu has one decay per head), over a ragged batch.  Per channel c with N states that start at zero and live in fp32
// per sequence slot:
//     S[n] <- exp(dt A[n]) S[n] + dt x B[n],     y = sum_n S[n] C[n] + D x,     out = y silu(z)
// where dt = softplus(raw dt + bias) per (token, channel), B and C [N] per token are shared by the channels, and z is an output
// gate (its raw projection columns).
//   * CTA = (256 / LPC channels, sequence or segment); LPC lanes share a channel, a thread keeps NPT of its states and the
//     matching decay rates (A log2 e) in registers, states 4 (r + LPC k) + e of lane r.  Tokens are staged 16 at a time through
//     registers one chunk ahead; softplus, dt x and the output gate are computed once per (token, channel) by whichever thread
//     loaded the element.  The decays are one ex2 per (token, channel, state): that is what bounds the kernel (16 per clock and
//     SM), the rest is packed fp32 pairs.  Four tokens per round: their four partial sums are exchanged so that each of four
//     lanes ends up with one token's output (three shuffles instead of eight for LPC = 4).
//   * long portions: when the step carries a segment list, the segments run in parallel.  A segment that starts from S0 gives
//     S_end = exp(A sum dt) S0 + Z_end: the PARTIAL pass leaves Z_end and sum dt of every segment but a sequence's last, an
//     elementwise pass chains them, the FULL pass runs every segment from its true start state.  The recurrence is linear in S:
//     this is the sequential result up to fp32 rounding.
//   * steps whose portions are all short (decoding): a kernel without staging -- every operand goes straight to registers, one
//     dependent round of loads, no barrier; same arithmetic in the same order.
// State layout [slots][C][N].  A sequence whose portion starts at position 0 ignores what its slot held.
#include "hybrid_common.cuh"

namespace b200 {

constexpr int SEL_THREADS = 256;
constexpr int SEL_CHUNK = 16;  // tokens staged per round
constexpr int SEL_STEP_TOKENS = 4;  // longest portion of a step that runs without staging

__device__ __forceinline__ float sel_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(x));
  return y;
}

// MODE 0: grid y = sequence, its whole portion.  MODE 1 / 2: grid y = segment (segs[y] = first token, end token, sequence, 1 = first
// of its sequence | 2 = last): 1 = the partial pass, 2 = the full pass from seg_state[y].
template <typename XT, typename OT, int LPC, int NPT, int MODE>
__global__ void __launch_bounds__(SEL_THREADS)
    selective_scan_kernel(const XT* __restrict__ x, const float* __restrict__ dt_raw, int ld_dt, const float* __restrict__ bc, int ld_bc,
                          int b_col0, int c_col0, const float* __restrict__ z, int ld_z, const float* __restrict__ a_log2,
                          const float* __restrict__ dt_bias, const float* __restrict__ d_skip, float* __restrict__ state,
                          const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot,
                          const int32_t* __restrict__ seq_pos0, OT* __restrict__ out, int C, int N, const int4* __restrict__ segs,
                          float* __restrict__ seg_state, float* __restrict__ seg_dt) {
  griddep_wait();
  constexpr int CH = SEL_THREADS / LPC;                // channels per CTA
  constexpr int NP = LPC * NPT;                        // padded state size
  constexpr int XP = SEL_CHUNK * CH / SEL_THREADS;     // staged (token, channel) elements per thread
  constexpr int BP = SEL_CHUNK * NP / SEL_THREADS;     // staged B (and C) elements per thread
  static_assert(XP >= 1 && BP >= 1 && LPC >= 4 && NPT % 4 == 0, "layout");
  __shared__ __align__(16) float Bs[SEL_CHUNK][NP];
  __shared__ __align__(16) float Cs[SEL_CHUNK][NP];
  __shared__ float2 dd[SEL_CHUNK][CH];                 // (dt, dt x)
  __shared__ float ys[SEL_CHUNK][CH];
  const int tid = threadIdx.x, r = tid % LPC, ch = tid / LPC;
  const int c0 = blockIdx.x * CH, c = c0 + ch;
  int sq = blockIdx.y, t0, t1, flags = 3;
  if (MODE == 0) {
    t0 = seq_start[sq], t1 = seq_start[sq + 1];
  } else {
    const int4 sg = segs[blockIdx.y];
    t0 = sg.x, t1 = sg.y, sq = sg.z, flags = sg.w;
    if (MODE == 1 && (flags & 2)) return;  // nobody continues from a sequence's last segment in this step
  }
  if (t0 >= t1) return;
  const bool live = c < C, vec = (N & 3) == 0;
  float* slot = state + ((int64_t)seq_slot[sq] * C + (live ? c : 0)) * N;
  float* seg = MODE == 0 ? nullptr : seg_state + ((int64_t)blockIdx.y * C + (live ? c : 0)) * N;
  const float* S_in = MODE == 2 ? seg : (MODE == 0 && seq_pos0[sq] > 0 ? slot : nullptr);
  const float* ar = a_log2 + (int64_t)(live ? c : 0) * N;
  float2 S[NPT / 2], A[NPT / 2];
  // states n .. n + 3 of the channel (zero past N and in channels past C)
  auto ld4s = [&](const float* p, int n) -> float4 {
    if (!p || !live) return make_float4(0.f, 0.f, 0.f, 0.f);
    if (vec) return n < N ? *reinterpret_cast<const float4*>(p + n) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(n < N ? p[n] : 0.f, n + 1 < N ? p[n + 1] : 0.f, n + 2 < N ? p[n + 2] : 0.f, n + 3 < N ? p[n + 3] : 0.f);
  };
#pragma unroll
  for (int k = 0; k < NPT / 4; ++k) {
    const float4 s = ld4s(S_in, 4 * (r + LPC * k)), a = ld4s(ar, 4 * (r + LPC * k));
    S[2 * k] = make_float2(s.x, s.y), S[2 * k + 1] = make_float2(s.z, s.w);
    A[2 * k] = make_float2(a.x, a.y), A[2 * k + 1] = make_float2(a.z, a.w);
  }
  // staged elements of this thread: idx = tid + k * 256 -> token idx / CH (or / NP) of the chunk, channel idx % CH (state idx % NP)
  float rx[XP], rdt[XP], rz[XP], rB[BP], rC[BP];
  auto fetch = [&](int tk0) {
    const int nc = t1 - tk0 < SEL_CHUNK ? t1 - tk0 : SEL_CHUNK;
#pragma unroll
    for (int k = 0; k < XP; ++k) {
      const int idx = tid + k * SEL_THREADS, tk = idx / CH, cc = c0 + idx % CH;
      const bool in = tk < nc && cc < C;
      const int64_t t = tk0 + (in ? tk : 0);
      const int col = in ? cc : 0;
      rx[k] = in ? ldf(x, t * C + col) : 0.f;
      rdt[k] = in ? dt_raw[t * ld_dt + col] : 0.f;
      rz[k] = (MODE != 1 && z && in) ? z[t * ld_z + col] : 0.f;
    }
#pragma unroll
    for (int k = 0; k < BP; ++k) {
      const int idx = tid + k * SEL_THREADS, tk = idx / NP, n = idx % NP;
      const bool in = tk < nc && n < N;
      const float* row = bc + (int64_t)(tk0 + (in ? tk : 0)) * ld_bc + (in ? n : 0);
      rB[k] = in ? row[b_col0] : 0.f;
      rC[k] = (MODE != 1 && in) ? row[c_col0] : 0.f;
    }
  };
  float bias[XP], skip[XP];
#pragma unroll
  for (int k = 0; k < XP; ++k) {
    const int cc = c0 + (tid + k * SEL_THREADS) % CH;
    bias[k] = cc < C ? dt_bias[cc] : 0.f;
    skip[k] = cc < C ? d_skip[cc] : 0.f;
  }
  float dsum = 0.f;
  fetch(t0);
  for (int tk0 = t0; tk0 < t1; tk0 += SEL_CHUNK) {
    const int nc = t1 - tk0 < SEL_CHUNK ? t1 - tk0 : SEL_CHUNK;
    __syncthreads();  // the previous chunk has been consumed
    float cx[XP], cz[XP];
#pragma unroll
    for (int k = 0; k < XP; ++k) {
      const int idx = tid + k * SEL_THREADS;
      const float v = rdt[k] + bias[k];
      const float dt = v > 20.f ? v : log1pf(expf(v));
      dd[idx / CH][idx % CH] = make_float2(dt, dt * rx[k]);
      cx[k] = rx[k], cz[k] = rz[k];
    }
#pragma unroll
    for (int k = 0; k < BP; ++k) {
      const int idx = tid + k * SEL_THREADS;
      Bs[idx / NP][idx % NP] = rB[k];
      if (MODE != 1) Cs[idx / NP][idx % NP] = rC[k];
    }
    __syncthreads();
    if (tk0 + SEL_CHUNK < t1) fetch(tk0 + SEL_CHUNK);
    // one token: S <- 2^(dt A) S + (dt x) B; returns this thread's share of S . C
    auto token = [&](int tk) -> float {
      const float2 d = dd[tk][ch];
      if (MODE == 1) dsum += d.x;
      const float2 dt2 = make_float2(d.x, d.x), dx2 = make_float2(d.y, d.y);
      float2 acc = make_float2(0.f, 0.f);
#pragma unroll
      for (int k = 0; k < NPT / 4; ++k) {
        const float4 b4 = *reinterpret_cast<const float4*>(&Bs[tk][4 * (r + LPC * k)]);
        const float2 e0 = fmul2(dt2, A[2 * k]), e1 = fmul2(dt2, A[2 * k + 1]);
        const float2 g0 = make_float2(sel_ex2(e0.x), sel_ex2(e0.y)), g1 = make_float2(sel_ex2(e1.x), sel_ex2(e1.y));
        S[2 * k] = ffma2(g0, S[2 * k], fmul2(dx2, make_float2(b4.x, b4.y)));
        S[2 * k + 1] = ffma2(g1, S[2 * k + 1], fmul2(dx2, make_float2(b4.z, b4.w)));
        if (MODE != 1) {
          const float4 c4 = *reinterpret_cast<const float4*>(&Cs[tk][4 * (r + LPC * k)]);
          acc = ffma2(S[2 * k], make_float2(c4.x, c4.y), acc);
          acc = ffma2(S[2 * k + 1], make_float2(c4.z, c4.w), acc);
        }
      }
      return acc.x + acc.y;
    };
    int tk = 0;
    if (MODE == 1) {
      for (; tk < nc; ++tk) token(tk);
      continue;
    }
    for (; tk + 4 <= nc; tk += 4) {
      const float v0 = token(tk), v1 = token(tk + 1), v2 = token(tk + 2), v3 = token(tk + 3);
      // lane bit 0 takes tokens {2, 3} (else {0, 1}), lane bit 1 the second of the pair
      const bool b0 = (r & 1) != 0, b1 = (r & 2) != 0;
      const float k0 = (b0 ? v2 : v0) + __shfl_xor_sync(0xffffffffu, b0 ? v0 : v2, 1);
      const float k1 = (b0 ? v3 : v1) + __shfl_xor_sync(0xffffffffu, b0 ? v1 : v3, 1);
      float v = (b1 ? k1 : k0) + __shfl_xor_sync(0xffffffffu, b1 ? k0 : k1, 2);
#pragma unroll
      for (int o = 4; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (r < 4) ys[tk + 2 * (r & 1) + (r >> 1)][ch] = v;
    }
    for (; tk < nc; ++tk) {
      float v = token(tk);
      // the same order of additions as above: the result must not depend on where a portion was cut
#pragma unroll
      for (int o = 1; o < LPC; o <<= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if (r == 0) ys[tk][ch] = v;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < XP; ++k) {
      const int idx = tid + k * SEL_THREADS, tkk = idx / CH, cc = c0 + idx % CH;
      if (tkk < nc && cc < C) {
        float y = ys[tkk][idx % CH] + skip[k] * cx[k];
        if (z) y *= silu_f(cz[k]);
        stf(out, (int64_t)(tk0 + tkk) * C + cc, y);
      }
    }
  }
  griddep_launch();
  float* S_out = MODE == 1 ? seg : ((flags & 2) ? slot : nullptr);
  if (S_out && live) {
#pragma unroll
    for (int k = 0; k < NPT / 4; ++k) {
      const int n = 4 * (r + LPC * k);
      if (vec) {
        if (n < N) *reinterpret_cast<float4*>(S_out + n) = make_float4(S[2 * k].x, S[2 * k].y, S[2 * k + 1].x, S[2 * k + 1].y);
      } else {
        if (n < N) S_out[n] = S[2 * k].x;
        if (n + 1 < N) S_out[n + 1] = S[2 * k].y;
        if (n + 2 < N) S_out[n + 2] = S[2 * k + 1].x;
        if (n + 3 < N) S_out[n + 3] = S[2 * k + 1].y;
      }
    }
  }
  if (MODE == 1 && r == 0 && live) seg_dt[(int64_t)blockIdx.y * C + c] = dsum;
}

// Short portions: LPC lanes per channel as above, operands straight from memory; bvec = B and C rows on the 16-byte grid.
template <typename XT, typename OT, int LPC, int NPT>
__global__ void __launch_bounds__(SEL_THREADS)
    selective_step_kernel(const XT* __restrict__ x, const float* __restrict__ dt_raw, int ld_dt, const float* __restrict__ bc, int ld_bc,
                          int b_col0, int c_col0, const float* __restrict__ z, int ld_z, const float* __restrict__ a_log2,
                          const float* __restrict__ dt_bias, const float* __restrict__ d_skip, float* __restrict__ state,
                          const int32_t* __restrict__ seq_start, const int32_t* __restrict__ seq_slot,
                          const int32_t* __restrict__ seq_pos0, OT* __restrict__ out, int C, int N, int bvec) {
  griddep_launch();
  const int idx = blockIdx.x * SEL_THREADS + threadIdx.x, r = idx % LPC, c = idx / LPC, sq = blockIdx.y;
  const bool live = c < C, vec = (N & 3) == 0;
  const int cc = live ? c : 0;
  auto ld4s = [&](const float* p, int n, bool v4) -> float4 {
    if (v4) return n < N ? *reinterpret_cast<const float4*>(p + n) : make_float4(0.f, 0.f, 0.f, 0.f);
    return make_float4(n < N ? p[n] : 0.f, n + 1 < N ? p[n + 1] : 0.f, n + 2 < N ? p[n + 2] : 0.f, n + 3 < N ? p[n + 3] : 0.f);
  };
  // what no kernel of the step writes: decay rates, bias, skip
  float2 S[NPT / 2], A[NPT / 2];
  const float* ar = a_log2 + (int64_t)cc * N;
#pragma unroll
  for (int k = 0; k < NPT / 4; ++k) {
    const float4 a = ld4s(ar, 4 * (r + LPC * k), vec);
    A[2 * k] = make_float2(a.x, a.y), A[2 * k + 1] = make_float2(a.z, a.w);
  }
  const float bias = dt_bias[cc], skip = d_skip[cc];
  griddep_wait();
  const int t0 = seq_start[sq], t1 = seq_start[sq + 1];
  if (t0 >= t1) return;
  float* slot = state + ((int64_t)seq_slot[sq] * C + cc) * N;
  const bool cont = seq_pos0[sq] > 0;
#pragma unroll
  for (int k = 0; k < NPT / 4; ++k) {
    const float4 s = cont ? ld4s(slot, 4 * (r + LPC * k), vec) : make_float4(0.f, 0.f, 0.f, 0.f);
    S[2 * k] = make_float2(s.x, s.y), S[2 * k + 1] = make_float2(s.z, s.w);
  }
  for (int64_t t = t0; t < t1; ++t) {
    const float v = dt_raw[t * ld_dt + cc] + bias, xv = ldf(x, t * C + cc), zv = z ? z[t * ld_z + cc] : 0.f;
    const float dt = v > 20.f ? v : log1pf(expf(v)), dx = dt * xv;
    const float2 dt2 = make_float2(dt, dt), dx2 = make_float2(dx, dx);
    const float* row = bc + t * ld_bc;
    float2 acc = make_float2(0.f, 0.f);
#pragma unroll
    for (int k = 0; k < NPT / 4; ++k) {
      const float4 b4 = ld4s(row + b_col0, 4 * (r + LPC * k), bvec), c4 = ld4s(row + c_col0, 4 * (r + LPC * k), bvec);
      const float2 e0 = fmul2(dt2, A[2 * k]), e1 = fmul2(dt2, A[2 * k + 1]);
      const float2 g0 = make_float2(sel_ex2(e0.x), sel_ex2(e0.y)), g1 = make_float2(sel_ex2(e1.x), sel_ex2(e1.y));
      S[2 * k] = ffma2(g0, S[2 * k], fmul2(dx2, make_float2(b4.x, b4.y)));
      S[2 * k + 1] = ffma2(g1, S[2 * k + 1], fmul2(dx2, make_float2(b4.z, b4.w)));
      acc = ffma2(S[2 * k], make_float2(c4.x, c4.y), acc);
      acc = ffma2(S[2 * k + 1], make_float2(c4.z, c4.w), acc);
    }
    float y = acc.x + acc.y;
#pragma unroll
    for (int o = 1; o < LPC; o <<= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (r == 0 && live) {
      y += skip * xv;
      if (z) y *= silu_f(zv);
      stf(out, t * C + cc, y);
    }
  }
  if (!live) return;
#pragma unroll
  for (int k = 0; k < NPT / 4; ++k) {
    const int n = 4 * (r + LPC * k);
    if (vec) {
      if (n < N) *reinterpret_cast<float4*>(slot + n) = make_float4(S[2 * k].x, S[2 * k].y, S[2 * k + 1].x, S[2 * k + 1].y);
    } else {
      if (n < N) slot[n] = S[2 * k].x;
      if (n + 1 < N) slot[n + 1] = S[2 * k].y;
      if (n + 2 < N) slot[n + 2] = S[2 * k + 1].x;
      if (n + 3 < N) slot[n + 3] = S[2 * k + 1].y;
    }
  }
}

// Chains the segments of every sequence, one thread per state element: segment k's entry of seg_state (Z_end) is replaced by its
// START state; carry <- 2^(A sum_dt[k]) carry + Z_end[k].
__global__ void selective_seg_combine_kernel(const float* __restrict__ state, float* __restrict__ seg_state,
                                             const float* __restrict__ seg_dt, const float* __restrict__ a_log2,
                                             const int32_t* __restrict__ seq_seg0, const int32_t* __restrict__ seq_slot,
                                             const int32_t* __restrict__ seq_pos0, int C, int N, int64_t total) {
  griddep_launch();
  griddep_wait();
  const int64_t per_seq = (int64_t)C * N;
  for (int64_t idx = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; idx < total; idx += (int64_t)gridDim.x * blockDim.x) {
    const int sq = (int)(idx / per_seq);
    const int64_t e = idx - sq * per_seq;
    const int c = (int)(e / N);
    const float a = a_log2[e];
    const int s0 = seq_seg0[sq], s1 = seq_seg0[sq + 1];
    float carry = seq_pos0[sq] > 0 ? state[(int64_t)seq_slot[sq] * per_seq + e] : 0.f;
    // eight segments' loads are issued before the first store
    for (int k0 = s0; k0 < s1; k0 += 8) {
      float zz[8], d[8];
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const int k = k0 + u < s1 ? k0 + u : s1 - 1;
        zz[u] = seg_state[(int64_t)k * per_seq + e];
        d[u] = seg_dt[(int64_t)k * C + c];
      }
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (k0 + u < s1) {
          seg_state[(int64_t)(k0 + u) * per_seq + e] = carry;
          if (k0 + u + 1 < s1) carry = fmaf(sel_ex2(a * d[u]), carry, zz[u]);
        }
      }
    }
  }
}

template <typename XT, typename OT, int LPC, int NPT>
static int launch_selective(const void* x, const float* dt_raw, int ld_dt, const float* bc, int ld_bc, int b_col0, int c_col0,
                            const float* z, int ld_z, const float* a_log2, const float* dt_bias, const float* d_skip, float* state,
                            const int32_t* seq_start, const int32_t* seq_slot, const int32_t* seq_pos0, void* out, int B, int C, int N,
                            const int32_t* segs, int num_segs, const int32_t* seq_seg0, float* seg_state, float* seg_dt,
                            int max_new, cudaStream_t st) {
  if (num_segs == 0 && max_new <= SEL_STEP_TOKENS) {
    const int bvec = (N & 3) == 0 && ld_bc % 4 == 0 && b_col0 % 4 == 0 && c_col0 % 4 == 0 && ((uintptr_t)bc & 15) == 0;
    B200_CUDA_OK(launch_kernel(selective_step_kernel<XT, OT, LPC, NPT>, dim3((unsigned)(((int64_t)C * LPC + SEL_THREADS - 1) / SEL_THREADS), B),
                               dim3(SEL_THREADS), 0, st, (const XT*)x, dt_raw, ld_dt, bc, ld_bc, b_col0, c_col0, z, ld_z, a_log2, dt_bias,
                               d_skip, state, seq_start, seq_slot, seq_pos0, (OT*)out, C, N, bvec));
    return B200_OK;
  }
  const unsigned gx = (C + SEL_THREADS / LPC - 1) / (SEL_THREADS / LPC);
  const int4* sg = reinterpret_cast<const int4*>(segs);
#define SEL_GO(MODE, LAUNCH, NY)                                                                                                 \
  B200_CUDA_OK(LAUNCH(selective_scan_kernel<XT, OT, LPC, NPT, MODE>, dim3(gx, NY), dim3(SEL_THREADS), 0, st, (const XT*)x, dt_raw, \
                      ld_dt, bc, ld_bc, b_col0, c_col0, z, ld_z, a_log2, dt_bias, d_skip, state, seq_start, seq_slot, seq_pos0,  \
                      (OT*)out, C, N, sg, seg_state, seg_dt))
  if (num_segs == 0) {
    SEL_GO(0, launch_kernel_serial, B);
    return B200_OK;
  }
  SEL_GO(1, launch_kernel, num_segs);
  const int64_t total = (int64_t)B * C * N;
  int64_t blocks = (total + 255) / 256;
  blocks = blocks > 148 * 16 ? 148 * 16 : blocks;
  B200_CUDA_OK(launch_kernel(selective_seg_combine_kernel, dim3((unsigned)blocks), dim3(256), 0, st, (const float*)state, seg_state,
                             (const float*)seg_dt, a_log2, seq_seg0, seq_slot, seq_pos0, C, N, total));
  SEL_GO(2, launch_kernel, num_segs);
#undef SEL_GO
  return B200_OK;
}

}  // namespace b200

using namespace b200;

extern "C" {

int b200_selective_scan(const void* x, int x_dtype, const float* dt_raw, int ld_dt, const float* bc, int ld_bc, int b_col0, int c_col0,
                        const float* z, int ld_z, const float* a_log2, const float* dt_bias, const float* d_skip, float* state,
                        const int32_t* seq_start, const int32_t* seq_slot, const int32_t* seq_pos0, void* out, int B, int C, int N,
                        const int32_t* segs, int num_segs, const int32_t* seq_seg0, float* seg_state, float* seg_dt, int max_new,
                        void* stream) {
  B200_REQUIRE(x && dt_raw && bc && a_log2 && dt_bias && d_skip && state && seq_start && seq_slot && seq_pos0 && out,
               "selective_scan: null pointer");
  B200_REQUIRE(C >= 1 && N >= 1, "selective_scan: bad shape");
  B200_REQUIRE(num_segs >= 0 && (num_segs == 0 || (segs && seq_seg0 && seg_state && seg_dt && !((uintptr_t)segs & 15))),
               "selective_scan: %d segments need their buffers", num_segs);
  B200_REQUIRE(!((uintptr_t)state & 15) && !((uintptr_t)a_log2 & 15) && !((uintptr_t)seg_state & 15),
               "selective_scan: state and decay rows must be 16-byte aligned");
  if (N > 256) {
    set_last_error("selective_scan: %d states per channel exceed 256", N);
    return B200_ERR_UNSUPPORTED;
  }
  if (B <= 0) return B200_OK;
  B200_REQUIRE(B <= 65535 && num_segs <= 65535, "selective_scan: %d sequences exceed the grid", B);
  cudaStream_t st = (cudaStream_t)stream;
#define SEL_PICK(LPC, NPT)                                                                                                         \
  return launch_selective<XT, XT, LPC, NPT>(x, dt_raw, ld_dt, bc, ld_bc, b_col0, c_col0, z, ld_z, a_log2, dt_bias, d_skip, state, \
                                            seq_start, seq_slot, seq_pos0, out, B, C, N, segs, num_segs, seq_seg0, seg_state,     \
                                            seg_dt, max_new, st)
  B200_DISPATCH_ELEM(x_dtype, XT, {
    if (N <= 16) SEL_PICK(4, 4);
    if (N <= 32) SEL_PICK(4, 8);
    if (N <= 64) SEL_PICK(4, 16);
    if (N <= 128) SEL_PICK(8, 16);
    SEL_PICK(16, 16);
  });
#undef SEL_PICK
  return B200_OK;
}

}  // extern "C"
