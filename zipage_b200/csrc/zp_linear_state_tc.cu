// Linear attention with a decaying matrix state over prompt portions, 64 tokens at a time (bf16 projections, fp32 state), key sizes
// up to 128.
//
// With L_t the running sums of the log2 decays inside a chunk (per key channel), the recurrence unrolls to
//   O = Q~ S_0 + P V,               Q~_t = q_t 2^(L_t),  P_ts = sum_d q_td k_sd 2^(L_td - L_sd)  (s <= t; D joins the diagonal)
//   S = diag(2^(L_C)) S_0 + diag(2^(L_C - C)) K^T V,  K_s = k_s 2^(C - L_s),  C = L_C to the nearest integer.
// Two kernels:
//   * `linear_prepare_kernel`, parallel over chunks and heads: Q~, K and P, which do not depend on the state, as operands that
//     lie in memory as the tensor cores want them.  P is a sum over channels that each have their own decays, so it is no
//     product of two matrices as it stands; it is one block by block, with every exponent taken against a token between the block's
//     rows and columns and so at most 0: rows 32-63 against columns 0-31, then the same inside the halves (16) and quarters
//     (8).  The 8 x 8 blocks on the diagonal are taken against their fourth token, where exponents reach four tokens' decays:
//     a decay below 2^-24 counts as 2^-24, which is nothing beside 1 in fp32, and keeps them inside the range.  Where no channel
//     of the chunk decays by more than 2^60 in either half, the whole of P is taken against token 31 in one step.  References are whole
//     numbers, so that the pairs of Q~ and K are those of P's operands times powers of two.
//   * `linear_scan_tc_kernel`, one block per (128 value columns, head, sequence), the chunks in order, all products on tcgen05
//     with the value columns as the 128 rows:
//       O^T = S_0^T Q~^T + V^T P^T;   D = V^T K;   S^T = S_0^T diag(2^(L_C)) + D diag(2^(L_C - C))
//     The fp32 state stays in registers; its operand form is written to TMEM.  D does not wait for the state, so the chain from
//     chunk to chunk is one pass over the registers.
// Whatever is fp32 (Q~, K, P, S) enters a product as a pair of bf16 numbers, hi + lo; values are the bf16 rows of the projection.
//
// Scan roles (512 threads): warp 0 = TMA producer, warps 1 and 3 = issuers of O and of D, warp 2 = TMEM owner, warps 4-11 = state (thread <-> TMEM
// lane <-> value column; the two warps of a lane quadrant split the key channels), warps 12-15 = outputs.  Two stages of operands in
// shared memory, two accumulators for O and two operand forms of S in TMEM.  Every wait is bounded; after it the block raises
// the device error word and leaves.
#include "zp_linear_state.cuh"
#include "zp_mma.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

constexpr float LC_LOG2E = 1.4426950408889634f;
constexpr float LC_MIN = -24.f;                  // smallest log2 decay of a token
constexpr int LC_P = 8192;                       // 64 x 64 bf16, swizzled as the operand lies in shared memory
// A chunk of a head in the workspace: K hi, lo | Q~ hi, lo | P hi, lo | factors; DP: key channels padded to 64 or 128
constexpr int lc_op(int DP) { return DP * LC_C * 2; }
constexpr int lc_per(int DP) { return 4 * lc_op(DP) + 2 * LC_P + DP * 8; }

__device__ __forceinline__ float lc_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void lc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack2<__nv_bfloat16>(a - f.x, b - f.y);
}
__device__ __forceinline__ void lc_split(float2 a, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a.x, a.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  ffma2(a, __bfloat1622float2(h), make_float2(-1.f, -1.f));
  lo = pack2<__nv_bfloat16>(a.x, a.y);
}
__device__ __forceinline__ uint32_t lc_scale(uint32_t v, uint32_t f) {      // pairs of bf16; f: powers of two
  const __nv_bfloat162 r = __hmul2(*reinterpret_cast<const __nv_bfloat162*>(&v), *reinterpret_cast<const __nv_bfloat162*>(&f));
  return *reinterpret_cast<const uint32_t*>(&r);
}
__device__ __forceinline__ float2 lc_unpack(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }

// Chunks of sequence b take the slots linear_first_slot(b) .. (a bound that needs no scan over the sequences)
__device__ __forceinline__ int linear_first_slot(const LinearArgs& a, int b) { return (a.cu_seqlens_q[b] - a.cu_seqlens_q[0]) / LC_C + b; }
static int linear_slots(int total_rows, int B) { return total_rows / LC_C + B; }

// fp32 functions on the special-function unit (relative errors of a few 2^-23; the logarithm near 1: absolute)
__device__ __forceinline__ float lc_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float lc_lg2(float x) { float y; asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float lc_sigmoid(float z) { return lc_rcp(1.f + lc_ex2(-LC_LOG2E * z)); }
// log2(1 - k), 0 <= k <= 1; near 1 by the series of the logarithm, where 1 - k has lost digits of k
__device__ __forceinline__ float lc_log2_1m(float k) {
  float p = fmaf(k, 1.f / 6.f, 1.f / 5.f);
  p = fmaf(k, p, 1.f / 4.f);
  p = fmaf(k, p, 1.f / 3.f);
  p = fmaf(k, p, 1.f / 2.f);
  p = fmaf(k, p, 1.f);
  return k < 0.125f ? -LC_LOG2E * k * p : lc_lg2(1.f - k);
}
// log2 of sigmoid(z) = -log2(1 + e^-z)
__device__ __forceinline__ float lc_log2_sigmoid(float z) {
  return fmaf(fminf(z, 0.f), LC_LOG2E, -lc_lg2(1.f + lc_ex2(-LC_LOG2E * fabsf(z))));
}

// ---------------------------------------------------------------------------------------------
// One block per (chunk, head).  A thread owns two key channels of eight tokens.
// ---------------------------------------------------------------------------------------------
constexpr int LP_TG = 8, LP_NG = LC_C / LP_TG;   // tokens of a thread; token groups
constexpr float LC_REACH = 60.f;                 // exponents of either sign that the one-step form of P takes
template <int DP> struct LinPrep {
  static constexpr int THREADS = DP / 2 * LP_NG;
  static constexpr int RB = DP * 2 + 16;         // bytes of an operand row
  static constexpr int ARR = LC_C * RB;          // one array of 64 rows
  static constexpr int TOT = 4 * ARR;            // two arrays, hi and lo, then the groups' sums, then per-token floats
  static constexpr int TOK = TOT + LP_NG * DP * 4;
  static constexpr int TOTAL = TOK + 4 * LC_C * 4;
};

template <int KIND, int DP>
__global__ void __launch_bounds__(LinPrep<DP>::THREADS, 1024 / LinPrep<DP>::THREADS)
linear_prepare_kernel(const LinearArgs a, unsigned char* __restrict__ ws) {
  using T = __nv_bfloat16;
  using G = LinPrep<DP>;
  constexpr int TG = LP_TG, NG = LP_NG, RB = G::RB, OP = lc_op(DP), WARPS = G::THREADS / 32;
  constexpr bool SCALAR = KIND == ZP_LINEAR_SCALAR, FORGET = KIND == ZP_LINEAR_FORGET;
  extern __shared__ __align__(128) unsigned char smem[];
  const int slot = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  int seq = -1;                                  // last sequence whose slots start at or before this one
  for (int b0 = 0; b0 < a.B; b0 += 32) {
    const unsigned m = __ballot_sync(0xffffffffu, b0 + lane < a.B && linear_first_slot(a, b0 + lane) <= slot);
    seq += __popc(m);
    if (m != 0xffffffffu) break;
  }
  const LinearSeq sq = linear_seq(a, max(seq, 0));
  const int t0 = (slot - linear_first_slot(a, max(seq, 0))) * LC_C, n = min(LC_C, sq.count - t0);
  if (n <= 0) return;
  const int64_t row0 = sq.row0 + t0;
  const int cp = tid % (DP / 2), tg = tid / (DP / 2), d = 2 * cp, hk = h / (a.H / a.G);
  const bool in = d < a.dim;
  unsigned char* arr0 = smem;                    // hi, then lo
  unsigned char* arr1 = smem + 2 * G::ARR;
  float* tot = reinterpret_cast<float*>(smem + G::TOT);      // [NG][DP]
  float* tok = reinterpret_cast<float*>(smem + G::TOK);      // SCALAR: sums of log2 decays, steps, factors of queries and of keys [64] each

  // ---- projections -> queries, keys and running sums of the log2 decays of this thread's tokens
  struct Mine {
    uint32_t qr[TG], kr[FORGET ? 1 : TG];
    float2 L[SCALAR ? 1 : TG], kf[FORGET ? TG : 1];          // gates, then sums inside the group; keys that are no projection
  };
  struct Edges { float2 r32, r16, r8, LC; };                 // sums up to token 31 (the reference of the one-step form) and up to the other edges
  auto load = [&](Mine& m) {
    const T* qp = reinterpret_cast<const T*>(a.q) + row0 * a.x_stride + (int64_t)hk * a.dim + d;
    const T* kp = reinterpret_cast<const T*>(a.k) + row0 * a.x_stride + (int64_t)hk * a.dim + d;
    const float* gp = a.gate + row0 * a.gate_stride + (int64_t)h * a.dim + d;
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const int t = tg * TG + u;
      const bool ok = in && t < n;
      m.qr[u] = ok ? *reinterpret_cast<const uint32_t*>(qp + t * a.x_stride) : 0u;
      if constexpr (!FORGET) m.kr[u] = ok ? *reinterpret_cast<const uint32_t*>(kp + t * a.x_stride) : 0u;
      if constexpr (!SCALAR) m.L[u] = ok ? *reinterpret_cast<const float2*>(gp + t * a.gate_stride) : make_float2(0.f, 0.f);
    }
    if constexpr (!SCALAR) {
      const float2 bias = in ? *reinterpret_cast<const float2*>(a.gate_bias + (int64_t)h * a.dim + d) : make_float2(0.f, 0.f);
      float2 low = make_float2(0.f, 0.f), run = low;
      if constexpr (FORGET) {
        if (in) low = *reinterpret_cast<const float2*>(a.lower + (int64_t)h * a.dim + d);
        low = make_float2(1.f - low.x, 1.f - low.y);
      }
#pragma unroll
      for (int u = 0; u < TG; ++u) {
        const bool ok = in && tg * TG + u < n;
        const float zx = m.L[u].x + bias.x, zy = m.L[u].y + bias.y;
        float wx, wy;
        if constexpr (FORGET) {
          m.kf[u] = ok ? make_float2(low.x * lc_sigmoid(-zx), low.y * lc_sigmoid(-zy)) : make_float2(0.f, 0.f);
          wx = lc_log2_1m(m.kf[u].x);
          wy = lc_log2_1m(m.kf[u].y);
        } else {
          wx = ok ? a.rtau * lc_log2_sigmoid(zx) : 0.f;
          wy = ok ? a.rtau * lc_log2_sigmoid(zy) : 0.f;
        }
        run.x += fmaxf(wx, LC_MIN);
        run.y += fmaxf(wy, LC_MIN);
        m.L[u] = run;
      }
    }
  };
  // sums from the chunk's start on
  auto chunk_sums = [&](Mine& m, Edges& e) {
    float2 base = make_float2(0.f, 0.f);
    e.r32 = e.r16 = e.r8 = e.LC = base;
#pragma unroll
    for (int j = 0; j < NG; ++j) {
      if (j == tg) base = e.LC;
      if (j == NG / 2) e.r32 = e.LC;
      if (j == (tg < NG / 2 ? NG / 4 : 3 * NG / 4)) e.r16 = e.LC;
      if (j == (tg | 1)) e.r8 = e.LC;
      const float2 x = *reinterpret_cast<const float2*>(tot + j * DP + d);
      e.LC.x += x.x; e.LC.y += x.y;
    }
    if constexpr (!SCALAR) {
#pragma unroll
      for (int u = 0; u < TG; ++u) { m.L[u].x += base.x; m.L[u].y += base.y; }
    }
  };
  Mine m;
  Edges e;
  bool one_step;
  load(m);
  if constexpr (SCALAR) {
    if (warp == 0) {
      float w[2], dt[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        w[i] = dt[i] = 0.f;
        if (t < n) {
          dt[i] = ls_softplus(a.gate[(row0 + t) * a.gate_stride + h] + a.gate_bias[h]);
          w[i] = fmaxf(-expf(a.A_log[h]) * dt[i] * LC_LOG2E, LC_MIN);
        }
      }
      float F = w[0] + w[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, F, o); if (lane >= o) F += x; }
      const float R = rintf(__shfl_sync(0xffffffffu, F, 15));       // (tokens 30 and 31)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        const float s = i ? F : F - w[1];
        tok[t] = s;
        tok[LC_C + t] = dt[i];
        tok[2 * LC_C + t] = lc_ex2(s - R);
        tok[3 * LC_C + t] = dt[i] * lc_ex2(R - s);
      }
    }
    __syncthreads();
    auto at = [&](int t) { return make_float2(tok[t], tok[t]); };
    e.r32 = at(31); e.r16 = at(tg < NG / 2 ? 15 : 47); e.r8 = at((tg | 1) * TG - 1); e.LC = at(63);
    one_step = -e.r32.x <= LC_REACH && e.r32.x - e.LC.x <= LC_REACH;
  } else {
    *reinterpret_cast<float2*>(tot + tg * DP + d) = m.L[TG - 1];
    __syncthreads();
    chunk_sums(m, e);
    one_step = !__syncthreads_or(fminf(e.r32.x, e.r32.y) < -LC_REACH || fmaxf(e.r32.x - e.LC.x, e.r32.y - e.LC.y) > LC_REACH);
  }
  auto sum = [&](int u) -> float2 {
    if constexpr (SCALAR) return make_float2(tok[tg * TG + u], tok[tg * TG + u]);
    else return m.L[u];
  };
  auto query = [&](int u) -> float2 {
    float2 q = lc_unpack(m.qr[u]);
    if constexpr (FORGET) { q.x *= lc_sigmoid(q.x); q.y *= lc_sigmoid(q.y); }
    else if constexpr (!SCALAR) { q.x *= a.qscale; q.y *= a.qscale; }
    return q;
  };
  auto key = [&](int u) -> float2 {
    if constexpr (FORGET) {
      return m.kf[u];
    } else {
      float2 k = lc_unpack(m.kr[u]);
      if constexpr (SCALAR) { k.x *= tok[LC_C + tg * TG + u]; k.y *= tok[LC_C + tg * TG + u]; }
      return k;
    }
  };
  // ---- Q~ and K in the workspace: two channels a thread, 128 bytes of a row a warp
  unsigned char* dst = ws + ((int64_t)slot * a.H + h) * lc_per(DP);
  unsigned char* mine = dst + (d >> 6) * 8192 + (d & 7) * 2 + tg * (TG * 128);
  auto store = [&](int which, int u, uint32_t hi, uint32_t lo) {   // which: 0 K, 2 Q~
    unsigned char* p = mine + ((((d & 63) >> 3) ^ u) << 4) + (which * OP + u * 128);
    *reinterpret_cast<uint32_t*>(p) = hi;
    *reinterpret_cast<uint32_t*>(p + OP) = lo;
  };
  auto put = [&](unsigned char* arr, int u, uint32_t hi, uint32_t lo) {   // a row of an array in shared memory
    unsigned char* p = arr + tg * (TG * RB) + d * 2 + u * RB;
    *reinterpret_cast<uint32_t*>(p) = hi;
    *reinterpret_cast<uint32_t*>(p + G::ARR) = lo;
  };
  auto put_f = [&](unsigned char* arr, int u, float2 f) {
    uint32_t hi, lo;
    lc_split(f, hi, lo);
    put(arr, u, hi, lo);
  };
  const float2 whole = make_float2(rintf(e.LC.x), rintf(e.LC.y));     // C
  if (tg == 0)                                               // decay of the state, factor of what joins it, channel by channel
    *reinterpret_cast<float4*>(dst + 4 * OP + 2 * LC_P + d * 8) =
        make_float4(lc_ex2(e.LC.x), lc_ex2(e.LC.y), lc_ex2(e.LC.x - whole.x), lc_ex2(e.LC.y - whole.y));
  // 16 rows of A from ra against 16 rows of B from rb, over all channels, the pairs' three larger products
  auto block = [&](const unsigned char* A, int ra, const unsigned char* B, int rb, float (&acc)[2][4]) {
    float x[2][4] = {}, y[2][4] = {};
    const unsigned char* ap = A + (ra + (lane & 15)) * RB + (lane >> 4) * 16;
    const unsigned char* bp = B + (rb + (lane & 7) + (lane >> 4) * 8) * RB + ((lane >> 3) & 1) * 16;
#pragma unroll 4
    for (int kk = 0; kk < DP / 16; ++kk) {
      uint32_t ah[4], al[4], bh[4], bl[4];
      ldmatrix_x4(ah, ap + kk * 32);
      ldmatrix_x4(bh, bp + kk * 32);
      ldmatrix_x4(al, ap + G::ARR + kk * 32);
      ldmatrix_x4(bl, bp + G::ARR + kk * 32);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mma16816<T>(acc[e], ah, bh[2 * e], bh[2 * e + 1]);
        mma16816<T>(x[e], ah, bl[2 * e], bl[2 * e + 1]);
        mma16816<T>(y[e], al, bh[2 * e], bh[2 * e + 1]);
      }
    }
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int i = 0; i < 4; ++i) acc[e][i] += x[e][i] + y[e][i];
  };
  // ---- the image of P, 16 x 16 blocks; it takes the place of arr1's hi part, or arr0's where arr1 is still read
  auto emit = [&](unsigned char* img, int r0, int c0, const float (&x)[2][4]) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      uint32_t hi, lo;
      const int ra = r0 + g, rb = ra + 8, c = (c0 >> 3) + e;
      lc_split(x[e][0], x[e][1], hi, lo);
      *reinterpret_cast<uint32_t*>(img + ra * 128 + ((c ^ (ra & 7)) << 4) + tq * 4) = hi;
      *reinterpret_cast<uint32_t*>(img + LC_P + ra * 128 + ((c ^ (ra & 7)) << 4) + tq * 4) = lo;
      lc_split(x[e][2], x[e][3], hi, lo);
      *reinterpret_cast<uint32_t*>(img + rb * 128 + ((c ^ (rb & 7)) << 4) + tq * 4) = hi;
      *reinterpret_cast<uint32_t*>(img + LC_P + rb * 128 + ((c ^ (rb & 7)) << 4) + tq * 4) = lo;
    }
  };
  float skip = 0.f;
  if constexpr (SCALAR) skip = a.D[h];
  auto triangle = [&](float (&x)[2][4]) {                    // a block on the diagonal: nothing above it
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int r = g + (i >> 1) * 8, c = 8 * e + 2 * tq + (i & 1);
        x[e][i] = c < r ? x[e][i] : c == r ? x[e][i] + skip : 0.f;
      }
  };
  auto zeros = [&](unsigned char* img, int i) {              // block i (0..5) above the diagonal
    const float x[2][4] = {};
    emit(img, i < 3 ? 0 : i < 5 ? 16 : 32, i < 3 ? 16 + 16 * i : i < 5 ? 32 + 16 * (i - 3) : 48, x);
  };
  unsigned char* img = arr0;
  if (one_step) {
    const float2 R = make_float2(rintf(e.r32.x), rintf(e.r32.y));
    const uint32_t up = pack2<T>(lc_ex2(R.x), lc_ex2(R.y)), down = pack2<T>(lc_ex2(whole.x - R.x), lc_ex2(whole.y - R.y));
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const int t = tg * TG + u;
      const float2 q = query(u);
      float2 k, x, y;
      if constexpr (SCALAR) {                                // (the step is part of the keys' factor)
        k = lc_unpack(m.kr[u]);
        x.x = x.y = tok[2 * LC_C + t];
        y.x = y.y = tok[3 * LC_C + t];
      } else {
        k = key(u);
        const float ex = m.L[u].x - R.x, ey = m.L[u].y - R.y;
        x = make_float2(lc_ex2(ex), lc_ex2(ey));
        y = make_float2(lc_ex2(-ex), lc_ex2(-ey));
      }
      uint32_t hi, lo;
      lc_split(fmul2(q, x), hi, lo);
      put(arr0, u, hi, lo);
      store(2, u, lc_scale(hi, up), lc_scale(lo, up));
      lc_split(fmul2(k, y), hi, lo);
      put(arr1, u, hi, lo);
      store(0, u, lc_scale(hi, down), lc_scale(lo, down));
    }
    __syncthreads();
    float p[2][4] = {};
    int r0 = 0, c0 = 0;
    if (WARPS >= 10 ? warp < 10 : true) {                    // ten blocks on and below the diagonal
      static_assert(WARPS == 8 || WARPS == 16, "warps of the block");
      r0 = warp < 1 ? 0 : warp < 3 ? 1 : warp < 6 ? 2 : 3;
      c0 = warp - (r0 * (r0 + 1)) / 2;
      block(arr0, 16 * r0, arr1, 16 * c0, p);
      if (r0 == c0) triangle(p);
    }
    float p2[2][4] = {};
    if (WARPS == 8 && warp < 2) {                            // (eight warps: the last two blocks, (3, 2) and (3, 3))
      block(arr0, 48, arr1, 32 + 16 * warp, p2);
      if (warp == 1) triangle(p2);
    }
    __syncthreads();
    if (WARPS == 8 || warp < 10) emit(img, 16 * r0, 16 * c0, p);
    if (WARPS == 8 && warp < 2) emit(img, 48, 32 + 16 * warp, p2);
    if (WARPS == 8 ? warp >= 2 : warp >= 10) zeros(img, warp - (WARPS == 8 ? 2 : 10));
  } else {
    // (made again: what the one-step form does not need any more would only hold registers there)
    load(m);
    if constexpr (!SCALAR) chunk_sums(m, e);
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const float2 s = sum(u), q = query(u), k = key(u);
      uint32_t hi, lo;
      lc_split(make_float2(k.x * lc_ex2(whole.x - s.x), k.y * lc_ex2(whole.y - s.y)), hi, lo);
      store(0, u, hi, lo);
      lc_split(make_float2(q.x * lc_ex2(s.x), q.y * lc_ex2(s.y)), hi, lo);
      store(2, u, hi, lo);
    }
    // row t of a level: queries where `upper`, keys below, both against `ref`
    auto level = [&](unsigned char* arr, int u, bool upper, float2 ref) {
      const float2 s = sum(u), f = upper ? query(u) : key(u), x = upper ? make_float2(s.x - ref.x, s.y - ref.y) : make_float2(ref.x - s.x, ref.y - s.y);
      put_f(arr, u, make_float2(f.x * lc_ex2(x.x), f.y * lc_ex2(x.y)));
    };
    float p32[2][4] = {}, p16[2][4] = {}, p8[2][4] = {}, pd[2][4] = {};
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const int t = tg * TG + u;
      level(arr0, u, t & 32, e.r32);
      level(arr1, u, t & 16, e.r16);
    }
    __syncthreads();
    if (warp < 4) block(arr0, 32 + 16 * (warp >> 1), arr0, 16 * (warp & 1), p32);
    else if (warp < 6) block(arr1, 16 + 32 * (warp & 1), arr1, 32 * (warp & 1), p16);
    __syncthreads();
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const float2 s = sum(u), ref = sum(3), q = query(u), k = key(u);
      put_f(arr0, u, make_float2(q.x * lc_ex2(s.x - ref.x), q.y * lc_ex2(s.y - ref.y)));
      put_f(arr1, u, make_float2(k.x * lc_ex2(ref.x - s.x), k.y * lc_ex2(ref.y - s.y)));
    }
    __syncthreads();
    const int di = 16 * (warp & 3);
    if (warp < 4) block(arr0, di, arr1, di, pd);
    __syncthreads();
#pragma unroll
    for (int u = 0; u < TG; ++u) level(arr0, u, tg & 1, e.r8);
    __syncthreads();
    if (warp < 4) {
      block(arr0, di, arr0, di, p8);
      triangle(pd);
#pragma unroll
      for (int i = 2; i < 4; ++i) pd[0][i] = p8[0][i];       // rows 8-15 against columns 0-7
    }
    img = arr1;
    if (warp < 4) {
      emit(img, 32 + 16 * (warp >> 1), 16 * (warp & 1), p32);
      emit(img, di, di, pd);
    } else if (warp < 6) {
      emit(img, 16 + 32 * (warp & 1), 32 * (warp & 1), p16);
    }
    if (warp < 6) zeros(img, warp);
  }
  __syncthreads();
  for (int i = tid; i < 2 * LC_P / 16; i += G::THREADS) st16(dst + 4 * OP + i * 16, ld16(img + i * 16));
}

// ---------------------------------------------------------------------------------------------
// One block per (128 value columns, head, sequence).
// ---------------------------------------------------------------------------------------------
constexpr int LS_THREADS = 512;
constexpr int LS_VT = 128;
constexpr int LS_V = 16384;                      // 64 rows x 128 value columns
constexpr uint32_t LS_O = 0, LS_D = 128, LS_S = 256;   // TMEM columns: O (2 x 64), D (128), S (2 x (hi 64, lo 64))

template <int DP> struct __align__(16) LsShared {
  float factors[2][2 * DP];            // for every two channels: two decays, two factors of D
  uint64_t dready[2], dfull, oready[2], ofull[2], empty[2];
  uint32_t tmem_base;
  int abort_flag;
};
template <int DP> constexpr int ls_stage() { return 4 * lc_op(DP) + 2 * LC_P + LS_V; }

__device__ __forceinline__ void ls_bulk(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void ls_prefetch(const void* src, uint32_t bytes) {   // into L2
  asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(src), "r"(bytes) : "memory");
}
// Products whose operands are named by the low words of their descriptors: start address and leading offset; the high word is that of
// every 128-byte swizzled operand here.
constexpr uint32_t LS_DESC_HI = (1024u >> 4) | (1u << 14) | (2u << 29);
__device__ __forceinline__ void ls_umma_ss(uint32_t d_tmem, uint32_t a_lo, uint32_t b_lo, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t.reg .b64 da, db;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "mov.b64 da, {%1, %5};\n\t"
      "mov.b64 db, {%2, %5};\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_lo), "r"(b_lo), "r"(idesc), "r"(acc), "r"(LS_DESC_HI)
      : "memory");
}
__device__ __forceinline__ void ls_umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint32_t b_lo, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t.reg .b64 db;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "mov.b64 db, {%2, %5};\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], db, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "r"(b_lo), "r"(idesc), "r"(acc), "r"(LS_DESC_HI)
      : "memory");
}
__device__ __forceinline__ void ls_ld16(uint32_t taddr, float (&v)[16]) {   // load and wait
  uint32_t r[16];
  asm volatile(
      "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n\t"
      "tcgen05.wait::ld.sync.aligned;"
      : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
        "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
      : "r"(taddr)
      : "memory");
#pragma unroll
  for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
}
__device__ __forceinline__ void ls_st8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
// every lane of a warp waits; the same answer in all of them
__device__ __forceinline__ bool ls_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* error_word, int where) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, error_word, where));
}

// meeting of the four output warps; true when any of them brings false
__device__ __forceinline__ bool ls_meet(bool ok) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, r;\n\t"
      "setp.eq.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred r, 1, 128, p;\n\t"
      "selp.u32 %0, 1, 0, r;\n\t}"
      : "=r"(out) : "r"((uint32_t)ok) : "memory");
  return out != 0;
}

struct LsParams { LinearArgs a; const unsigned char* ws; int* error_word; };

template <int DP>
__global__ void __launch_bounds__(LS_THREADS, 1)
linear_scan_tc_kernel(const __grid_constant__ CUtensorMap tmV, const LsParams p) {
  using T = __nv_bfloat16;
  const LinearArgs& a = p.a;
  const int c0 = blockIdx.x * LS_VT, h = blockIdx.y, b = blockIdx.z;
  const LinearSeq sq = linear_seq(a, b);
  if (sq.count == 0) return;
  const int nc = (sq.count + LC_C - 1) / LC_C;
  constexpr int OP = lc_op(DP), STAGE = ls_stage<DP>();
  extern __shared__ unsigned char smem_raw[];
  unsigned char* stages = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  LsShared<DP>& sh = *reinterpret_cast<LsShared<DP>*>(stages + 2 * STAGE + LS_V);   // a stage: K hi, lo | Q~ hi, lo | P hi, lo | V; then the outputs' tile
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sh.dready[i], 1 + 8);          // K and V there, D read
      mbar_init(&sh.oready[i], 1 + 8 + 4);      // Q~ and P there, S written, O read
      mbar_init(&sh.ofull[i], 1);
      mbar_init(&sh.empty[i], 1 + 8);
    }
    mbar_init(&sh.dfull, 1);
    sh.abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 2) {
    tmem_alloc(&sh.tmem_base, 512);
    tmem_relinquish();
  }
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem = sh.tmem_base;
  volatile int* abortp = &sh.abort_flag;
  int* err = p.error_word;

  if (warp == 0) {
    if (elect_one()) {
      const unsigned char* ws = p.ws + ((int64_t)linear_first_slot(a, b) * a.H + h) * lc_per(DP);
      const int64_t step = (int64_t)a.H * lc_per(DP);
      for (int c = 0; c < nc; ++c) {
        const int s = c & 1;
        if (c + 2 < nc) {                                  // into L2 ahead of its load
          ls_prefetch(ws + (c + 2) * step, lc_per(DP));
          tma_prefetch_l2_5d(&tmV, c0, h, sq.row0 + (c + 2) * LC_C, 0, 0);
          tma_prefetch_l2_5d(&tmV, c0 + 64, h, sq.row0 + (c + 2) * LC_C, 0, 0);
        }
        if (!mbar_wait<true>(&sh.empty[s], ((c >> 1) & 1) ^ 1, abortp, err, 981)) break;
        unsigned char* st = stages + s * STAGE;
        mbar_arrive_expect_tx(&sh.dready[s], 2 * OP + LS_V + DP * 8);
        ls_bulk(st, ws + c * step, 2 * OP, &sh.dready[s]);
        tma_load_5d(st + 4 * OP + 2 * LC_P, &tmV, &sh.dready[s], c0, h, sq.row0 + c * LC_C, 0, 0);
        tma_load_5d(st + 4 * OP + 2 * LC_P + 8192, &tmV, &sh.dready[s], c0 + 64, h, sq.row0 + c * LC_C, 0, 0);
        ls_bulk(sh.factors[s], ws + c * step + 4 * OP + 2 * LC_P, DP * 8, &sh.dready[s]);
        mbar_arrive_expect_tx(&sh.oready[s], 2 * OP + 2 * LC_P);
        ls_bulk(st + 2 * OP, ws + c * step + 2 * OP, 2 * OP + 2 * LC_P, &sh.oready[s]);
      }
    }
  } else if (warp == 1 || warp == 3) {
    if (elect_one()) {
      constexpr uint32_t B_MN = 1u << 16, A_MN = 1u << 15;
      constexpr uint32_t ID_D = idesc_f16(1, 128, DP) | A_MN | B_MN, ID_S = idesc_f16(1, 128, 64), ID_P = ID_S | A_MN;
      // low words of the descriptors of stage 0; everything else is a constant number of 16-byte units further on
      const uint32_t base = smem_u32(stages) >> 4;
      const uint32_t kmn = base | ((8192u >> 4) << 16), vmn = kmn + ((4 * OP + 2 * LC_P) >> 4);      // MN-major: 64-element blocks 8192 bytes apart
      const uint32_t qk = (base + ((2 * OP) >> 4)) | (1u << 16), pk = qk + ((2 * OP) >> 4);
      if (warp == 3) {                                       // D = V^T K
        for (int c = 0; c < nc; ++c) {
          if (!mbar_wait(&sh.dready[c & 1], (c >> 1) & 1, abortp, err, 982)) break;
          fence_after_sync();
          const uint32_t at = (c & 1) * (STAGE >> 4), v = vmn + at, k = kmn + at;
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) {
            ls_umma_ss(tmem + LS_D, v + ks * 128, k + ks * 128, ID_D, ks ? 1u : 0u);
            ls_umma_ss(tmem + LS_D, v + ks * 128, k + (OP >> 4) + ks * 128, ID_D, 1u);
          }
          umma_commit(&sh.dfull);
        }
      } else {                                               // O^T = S^T Q~^T + V^T P^T
        for (int c = 0; c < nc; ++c) {
          const int s = c & 1;
          if (!mbar_wait(&sh.oready[s], (c >> 1) & 1, abortp, err, 983) || !mbar_wait(&sh.dready[s], (c >> 1) & 1, abortp, err, 984)) break;   // (V)
          fence_after_sync();
          const uint32_t at = s * (STAGE >> 4), q = qk + at, pp = pk + at, v = vmn + at;
          const uint32_t o = tmem + LS_O + s * 64, shi = tmem + LS_S + s * 128, slo = shi + 64;
#pragma unroll
          for (int ks = 0; ks < DP / 16; ++ks) {
            const uint32_t qh = q + (ks >> 2) * 512 + 2 * (ks & 3);
            ls_umma_ts(o, shi + ks * 8, qh, ID_S, ks ? 1u : 0u);
            ls_umma_ts(o, slo + ks * 8, qh, ID_S, 1u);
            ls_umma_ts(o, shi + ks * 8, qh + (OP >> 4), ID_S, 1u);
          }
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) {
            ls_umma_ss(o, v + ks * 128, pp + 2 * ks, ID_P, 1u);
            ls_umma_ss(o, v + ks * 128, pp + (LC_P >> 4) + 2 * ks, ID_P, 1u);
          }
          umma_commit(&sh.ofull[s]);
          umma_commit(&sh.empty[s]);
        }
      }
    }
  } else if (warp >= 4 && warp < 12) {
    // ---------------- state ----------------
    constexpr int W = DP / 2;                              // key channels of a thread
    const int q = warp & 3, half = (warp - 4) >> 2, v = c0 + q * 32 + lane;
    const uint32_t lanes = tmem + (static_cast<uint32_t>(q * 32) << 16);
    float* Sg = a.state + (((int64_t)sq.slot * a.H + h) * a.dim + half * W) * a.VP + v;
    const bool mine = v < a.vdim;
    float2 s[W / 2];
#pragma unroll
    for (int i = 0; i < W; ++i) {
      const float x = (mine && !sq.fresh && half * W + i < a.dim) ? Sg[(int64_t)i * a.VP] : 0.f;
      if (i & 1) s[i / 2].y = x; else s[i / 2].x = x;
    }
    auto put = [&](int i, uint32_t buf) {                  // channels i .. i + 15 of this thread as operand, hi and lo
      uint32_t hi[8], lo[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) lc_split(s[i / 2 + j], hi[j], lo[j]);
      const uint32_t at = lanes + LS_S + buf * 128 + (half * W + i) / 2;
      ls_st8(at, hi);
      ls_st8(at + 64, lo);
    };
    auto publish = [&](uint64_t* bar) {
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
#pragma unroll
    for (int i = 0; i < W; i += 16) put(i, 0);
    publish(&sh.oready[0]);
    if (lane == 0) mbar_arrive(&sh.dready[0]);
    bool ok = true;
    for (int c = 0; c < nc; ++c) {
      const int st = c & 1;
      const bool more = c + 1 < nc;
      // (the operand's other buffer is free when the products of the chunk before are done)
      if (!ls_wait(&sh.dready[st], (c >> 1) & 1, abortp, err, 987) || !ls_wait(&sh.dfull, c & 1, abortp, err, 988) ||
          (c > 0 && more && !ls_wait(&sh.ofull[st ^ 1], ((c - 1) >> 1) & 1, abortp, err, 985))) { ok = false; break; }
      fence_after_sync();
#pragma unroll
      for (int i = 0; i < W; i += 16) {
        float y[16];
        ls_ld16(lanes + LS_D + half * W + i, y);
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
          const float4 f = *reinterpret_cast<const float4*>(&sh.factors[st][2 * (half * W + i + j)]);
          const float2 x = s[(i + j) / 2];
          float2 z = fmul2(make_float2(y[j], y[j + 1]), make_float2(f.z, f.w));
          ffma2(z, x, make_float2(f.x, f.y));
          s[(i + j) / 2] = z;
        }
        if (i + 16 == W) {                                 // D and the factors have been read
          fence_before_sync();
          __syncwarp();
          if (lane == 0) { mbar_arrive(&sh.dready[st ^ 1]); mbar_arrive(&sh.empty[st]); }
        }
        if (more) put(i, st ^ 1);
      }
      if (more) publish(&sh.oready[st ^ 1]);
    }
    if (ok && mine) {
#pragma unroll
      for (int i = 0; i < W; ++i)
        if (half * W + i < a.dim) Sg[(int64_t)i * a.VP] = (i & 1) ? s[i / 2].y : s[i / 2].x;
    }
  } else if (warp >= 12) {
    // ---------------- outputs ----------------
    const int q = warp & 3;
    const uint32_t lanes = tmem + (static_cast<uint32_t>(q * 32) << 16);
    T* tile = reinterpret_cast<T*>(stages + 2 * STAGE);    // [64 tokens][128 columns]
    const int rl = lane >> 4, cl = (lane & 15) * 8;        // two rows of 16-byte pieces a warp
    T* out = reinterpret_cast<T*>(a.out) + (int64_t)h * a.vdim + c0 + cl;
    const bool there = c0 + cl < a.vdim;                   // (multiples of 8)
    if (lane == 0) { mbar_arrive(&sh.oready[0]); mbar_arrive(&sh.oready[1]); }
    for (int c = 0; c < nc; ++c) {
      const int s = c & 1, n = min(LC_C, sq.count - c * LC_C);
      const bool ok = ls_wait(&sh.ofull[s], (c >> 1) & 1, abortp, err, 989);
      if (ls_meet(ok)) break;                              // (every warp leaves or none; the tile has been read)
      fence_after_sync();
#pragma unroll 1
      for (int i = 0; i < 64; i += 16) {
        float y[16];
        ls_ld16(lanes + LS_O + s * 64 + i, y);
        if (i == 48) {
          fence_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(&sh.oready[s]);           // (for the chunk after the next)
        }
#pragma unroll
        for (int j = 0; j < 16; ++j) tile[(i + j) * LS_VT + q * 32 + lane] = __float2bfloat16_rn(y[j]);
      }
      ls_meet(true);
      T* o = out + (sq.row0 + (int64_t)c * LC_C) * a.out_stride;
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int t = q * 16 + 2 * i + rl;
        if (t < n && there) st16(o + t * a.out_stride, ld16(tile + t * LS_VT + cl));
      }
    }
  }
  if (*abortp) {                                           // a wait ran out: copies that are still on their way land first
    for (int i = 0; i < 64; ++i) __nanosleep(4000);
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 2) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

bool linear_chunk_supports(const LinearArgs& a) {
  return a.taps == 0 && a.dim <= 128 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.x_stride % 8 == 0 && a.out_stride % 8 == 0 &&
         ((uintptr_t)a.v | (uintptr_t)a.out) % 16 == 0 && ((uintptr_t)a.q | (uintptr_t)a.k) % 4 == 0 &&
         (a.kind == ZP_LINEAR_SCALAR || a.gate_stride % 2 == 0) &&
         (a.kind == ZP_LINEAR_SCALAR || ((uintptr_t)a.gate | (uintptr_t)a.gate_bias | (uintptr_t)a.lower) % 8 == 0);
}
size_t linear_chunk_workspace(int total_rows, int B, int H, int dim) {
  return (size_t)linear_slots(total_rows, B) * H * (dim <= 64 ? lc_per(64) : lc_per(128));
}

template <int KIND, int DP> static int launch_prepare(const LinearArgs& a, cudaStream_t st) {
  constexpr int smem = LinPrep<DP>::TOTAL;
  auto kern = linear_prepare_kernel<KIND, DP>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_linear_state(prepare): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  kern<<<dim3(linear_slots(a.total_rows, a.B), a.H), LinPrep<DP>::THREADS, smem, st>>>(a, (unsigned char*)a.workspace);
  return check_launch("zp_linear_state(prepare)");
}
template <int DP> static int chunk_by_size(const LinearArgs& a, const CUtensorMap& tmV, int* error_word, cudaStream_t st) {
  const int rc = a.kind == ZP_LINEAR_FORGET  ? launch_prepare<ZP_LINEAR_FORGET, DP>(a, st)
                 : a.kind == ZP_LINEAR_POWER ? launch_prepare<ZP_LINEAR_POWER, DP>(a, st)
                                             : launch_prepare<ZP_LINEAR_SCALAR, DP>(a, st);
  if (rc) return rc;
  const LsParams p{a, (const unsigned char*)a.workspace, error_word};
  constexpr int smem = 1024 + 2 * ls_stage<DP>() + LS_V + (int)sizeof(LsShared<DP>);
  static_assert(smem <= 232448, "shared memory of a block");
  auto kern = linear_scan_tc_kernel<DP>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_linear_state(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  kern<<<dim3((a.vdim + LS_VT - 1) / LS_VT, a.H, a.B), LS_THREADS, smem, st>>>(tmV, p);
  return check_launch("zp_linear_state(tcgen05)");
}

// total_rows: rows of q, k and v, of which the portions' are the rows from cu_seqlens_q[0] on
int linear_chunk(const LinearArgs& a, cudaStream_t st) {
  int* error_word = device_error_word();
  if (!error_word) { set_error("zp_linear_state(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  CUtensorMap tmV;
  const uint64_t rs = (uint64_t)a.x_stride;
  const uint64_t dims[5] = {(uint64_t)a.vdim, (uint64_t)a.H, (uint64_t)a.total_rows, 1, 1};
  const uint64_t strides[4] = {(uint64_t)a.vdim, rs, rs * a.total_rows, rs * a.total_rows};
  const uint32_t box[5] = {64, 1, 64, 1, 1};
  if (int rc = make_tensor_map_5d(&tmV, UmmaFmt<__nv_bfloat16>::tm, a.v, dims, strides, box, 2)) return rc;
  return a.dim <= 64 ? chunk_by_size<64>(a, tmV, error_word, st) : chunk_by_size<128>(a, tmV, error_word, st);
}

}  // namespace zp
