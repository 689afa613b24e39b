// Linear attention with a decaying matrix state over prompt portions, 64 tokens at a time (bf16 projections, fp32 state), key sizes
// up to 128.
//
// With L_t the running sums of the log2 decays inside a chunk (per key channel), the recurrence unrolls to
//   O = Q~ S_0 + P V,               Q~_t = q_t 2^(L_t),  P_ts = sum_d q_td k_sd 2^(L_td - L_sd)  (s <= t; D joins the diagonal)
//   S = diag(2^(L_C)) S_0 + K^T V,  K_s = k_s 2^(L_C - L_s).
// Two kernels:
//   * `linear_prepare_kernel`, parallel over chunks and heads: Q~, K and P, which do not depend on the state, as operands that
//     lie in memory as the tensor cores want them.  P is a sum over channels that each have their own decays, so it is no
//     product of two matrices as it stands; it is one block by block, with every exponent taken against a token between the block's
//     rows and columns and so at most 0: rows 32-63 against columns 0-31, then the same inside the halves (16) and quarters
//     (8).  The 8 x 8 blocks on the diagonal are taken against their fourth token, where exponents reach four tokens' decays:
//     a decay below 2^-24 counts as 2^-24, which is nothing beside 1 in fp32, and keeps them inside the range.
//   * `linear_scan_tc_kernel`, one block per (128 value columns, head, sequence), the chunks in order, all products on tcgen05
//     with the value columns as the 128 rows:
//       O^T = S_0^T Q~^T + V^T P^T;   D = V^T K;   S^T = S_0^T diag(2^(L_C)) + D
//     The fp32 state stays in registers; its operand form is written to TMEM.  D does not wait for the state, so the chain from
//     chunk to chunk is one pass over the registers.
// Whatever is fp32 (Q~, K, P, S) enters a product as a pair of bf16 numbers, hi + lo; values are the bf16 rows of the projection.
//
// Scan roles (512 threads): warp 0 = TMA producer, warp 1 = MMA issuer, warp 2 = TMEM owner, warps 4-11 = state (thread <-> TMEM
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
// A chunk of a head in the workspace: K hi, lo | Q~ hi, lo | P hi, lo | 2^(L_C); DP: key channels padded to 64 or 128
constexpr int lc_op(int DP) { return DP * LC_C * 2; }
constexpr int lc_per(int DP) { return 4 * lc_op(DP) + 2 * LC_P + DP * 4; }

__device__ __forceinline__ float lc_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void lc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack2<__nv_bfloat16>(a - f.x, b - f.y);
}
__device__ __forceinline__ float2 lc_unpack(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }

// Chunks of sequence b take the slots linear_first_slot(b) .. (a bound that needs no scan over the sequences)
__device__ __forceinline__ int linear_first_slot(const LinearArgs& a, int b) { return (a.cu_seqlens_q[b] - a.cu_seqlens_q[0]) / LC_C + b; }
static int linear_slots(int total_rows, int B) { return total_rows / LC_C + B; }

// ---------------------------------------------------------------------------------------------
// One block per (chunk, head).  A thread owns two key channels of TG tokens.
// ---------------------------------------------------------------------------------------------
constexpr int LP_THREADS = 256;
template <int DP> struct LinPrep {
  static constexpr int PAIRS = DP / 2, NG = LP_THREADS / PAIRS, TG = LC_C / NG;   // channel pairs; token groups; tokens of a group
  static constexpr int RB = DP * 2 + 16;         // bytes of an operand row
  static constexpr int ARR = LC_C * RB;          // one array of 64 rows
  static constexpr int TOT = 4 * ARR;            // two arrays, hi and lo, then the groups' sums, then per-token floats
  static constexpr int TOK = TOT + NG * DP * 4;
  static constexpr int TOTAL = TOK + 2 * LC_C * 4;
};

template <int KIND, int DP>
__global__ void __launch_bounds__(LP_THREADS, 2) linear_prepare_kernel(const LinearArgs a, unsigned char* __restrict__ ws) {
  using T = __nv_bfloat16;
  using G = LinPrep<DP>;
  constexpr int TG = G::TG, NG = G::NG, RB = G::RB;
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
  const int cp = tid % G::PAIRS, tg = tid / G::PAIRS, d = 2 * cp, hk = h / (a.H / a.G);
  const bool in = d < a.dim;
  unsigned char* arr0 = smem;                    // hi, then lo
  unsigned char* arr1 = smem + 2 * G::ARR;
  float* tot = reinterpret_cast<float*>(smem + G::TOT);      // [NG][DP]
  float* tok = reinterpret_cast<float*>(smem + G::TOK);      // SCALAR: log2 decays [64], steps [64]

  if constexpr (KIND == ZP_LINEAR_SCALAR) {
    if (tid < LC_C) {
      float dt = 0.f, w = 0.f;
      if (tid < n) {
        dt = ls_softplus(a.gate[(row0 + tid) * a.gate_stride + h] + a.gate_bias[h]);
        w = fmaxf(-expf(a.A_log[h]) * dt * LC_LOG2E, LC_MIN);
      }
      tok[tid] = w;
      tok[LC_C + tid] = dt;
    }
  }
  // ---- projections -> queries, keys (fp32) and running sums of the log2 decays of this thread's tokens
  uint32_t qr[TG], kr[KIND == ZP_LINEAR_FORGET ? 1 : TG];
  float2 L[TG];                                  // gates, then sums
  {
    const T* qp = reinterpret_cast<const T*>(a.q) + (int64_t)hk * a.dim + d;
    const T* kp = reinterpret_cast<const T*>(a.k) + (int64_t)hk * a.dim + d;
    const float* zp_ = a.gate + (int64_t)h * a.dim + d;
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const bool ok = in && tg * TG + u < n;
      const int64_t row = row0 + tg * TG + u;
      qr[u] = ok ? *reinterpret_cast<const uint32_t*>(qp + row * a.x_stride) : 0u;
      if constexpr (KIND != ZP_LINEAR_FORGET) kr[u] = ok ? *reinterpret_cast<const uint32_t*>(kp + row * a.x_stride) : 0u;
      if constexpr (KIND != ZP_LINEAR_SCALAR)
        L[u] = ok ? *reinterpret_cast<const float2*>(zp_ + row * a.gate_stride) : make_float2(0.f, 0.f);
    }
  }
  float2 kf[TG];
  float2 run = make_float2(0.f, 0.f);
  if constexpr (KIND == ZP_LINEAR_SCALAR) {
    __syncthreads();
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const float w = tok[tg * TG + u], dt = tok[LC_C + tg * TG + u];
      const float2 k = lc_unpack(kr[u]);
      kf[u] = make_float2(k.x * dt, k.y * dt);
      run.x += w;
      run.y = run.x;
      L[u] = run;
    }
  } else {
    const float2 bias = in ? *reinterpret_cast<const float2*>(a.gate_bias + (int64_t)h * a.dim + d) : make_float2(0.f, 0.f);
    float2 low = make_float2(0.f, 0.f);
    if constexpr (KIND == ZP_LINEAR_FORGET) { if (in) low = *reinterpret_cast<const float2*>(a.lower + (int64_t)h * a.dim + d); }
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const bool ok = in && tg * TG + u < n;
      const float zx = L[u].x + bias.x, zy = L[u].y + bias.y;
      float wx, wy;
      if constexpr (KIND == ZP_LINEAR_FORGET) {
        kf[u] = ok ? make_float2((1.f - low.x) * ls_sigmoid(-zx), (1.f - low.y) * ls_sigmoid(-zy)) : make_float2(0.f, 0.f);
        wx = log1pf(-kf[u].x) * LC_LOG2E;        // a = 1 - k, also where a is near 1
        wy = log1pf(-kf[u].y) * LC_LOG2E;
      } else {
        kf[u] = lc_unpack(kr[u]);
        wx = ok ? -a.rtau * ls_softplus(-zx) * LC_LOG2E : 0.f;
        wy = ok ? -a.rtau * ls_softplus(-zy) * LC_LOG2E : 0.f;
      }
      run.x += fmaxf(wx, LC_MIN);
      run.y += fmaxf(wy, LC_MIN);
      L[u] = run;
    }
  }
  *reinterpret_cast<float2*>(tot + tg * DP + d) = run;
  __syncthreads();
  // sums up to the token groups' edges
  float2 base = make_float2(0.f, 0.f), r32 = base, r16 = base, r8 = base, LC = base;
#pragma unroll
  for (int j = 0; j < NG; ++j) {
    if (j == tg) base = LC;
    if (j == NG / 2) r32 = LC;
    if (j == (tg < NG / 2 ? NG / 4 : 3 * NG / 4)) r16 = LC;
    if (TG == 8 && j == (tg | 1)) r8 = LC;
    const float2 x = *reinterpret_cast<const float2*>(tot + j * DP + d);
    LC.x += x.x; LC.y += x.y;
  }
#pragma unroll
  for (int u = 0; u < TG; ++u) { L[u].x += base.x; L[u].y += base.y; }
  if constexpr (TG == 16) r8 = L[7];

  float2 qf[TG];
#pragma unroll
  for (int u = 0; u < TG; ++u) {
    qf[u] = lc_unpack(qr[u]);
    if constexpr (KIND == ZP_LINEAR_FORGET) {
      qf[u].x *= ls_sigmoid(qf[u].x);
      qf[u].y *= ls_sigmoid(qf[u].y);
    } else if constexpr (KIND == ZP_LINEAR_POWER) {
      qf[u].x *= a.qscale;
      qf[u].y *= a.qscale;
    }
  }
  unsigned char* dst = ws + ((int64_t)slot * a.H + h) * lc_per(DP);
  constexpr int OP = lc_op(DP);
  {  // Q~ and K: two channels a thread, 128 bytes of a row a warp
    const int c = (d & 63) >> 3;
    unsigned char* p = dst + (d >> 6) * 8192 + (d & 7) * 2;
#pragma unroll
    for (int u = 0; u < TG; ++u) {
      const int t = tg * TG + u, off = t * 128 + ((c ^ (t & 7)) << 4);
      uint32_t hi, lo;
      lc_split(kf[u].x * lc_ex2(LC.x - L[u].x), kf[u].y * lc_ex2(LC.y - L[u].y), hi, lo);
      *reinterpret_cast<uint32_t*>(p + off) = hi;
      *reinterpret_cast<uint32_t*>(p + OP + off) = lo;
      lc_split(qf[u].x * lc_ex2(L[u].x), qf[u].y * lc_ex2(L[u].y), hi, lo);
      *reinterpret_cast<uint32_t*>(p + 2 * OP + off) = hi;
      *reinterpret_cast<uint32_t*>(p + 3 * OP + off) = lo;
    }
    if (tg == 0) *reinterpret_cast<float2*>(dst + 4 * OP + 2 * LC_P + d * 4) = make_float2(lc_ex2(LC.x), lc_ex2(LC.y));
  }
  // ---- P: arrays of rows in shared memory, blocks of 16 x 8 by mma.sync
  auto put = [&](unsigned char* arr, int t, float2 f, float2 e) {
    uint32_t hi, lo;
    lc_split(f.x * lc_ex2(e.x), f.y * lc_ex2(e.y), hi, lo);
    *reinterpret_cast<uint32_t*>(arr + t * RB + d * 2) = hi;
    *reinterpret_cast<uint32_t*>(arr + G::ARR + t * RB + d * 2) = lo;
  };
  // row t of a level: queries where `upper`, keys below, both against `ref`
  auto level = [&](unsigned char* arr, int u, bool upper, float2 ref) {
    const float2 e = upper ? make_float2(L[u].x - ref.x, L[u].y - ref.y) : make_float2(ref.x - L[u].x, ref.y - L[u].y);
    put(arr, tg * TG + u, upper ? qf[u] : kf[u], e);
  };
  // 16 rows of A from ra against 8 rows of B from rb, over all channels, the pairs' three larger products
  auto block = [&](const unsigned char* A, int ra, const unsigned char* B, int rb, float (&acc)[4]) {
    float x[4] = {0.f, 0.f, 0.f, 0.f}, y[4] = {0.f, 0.f, 0.f, 0.f};
    const unsigned char* ap = A + (ra + (lane & 15)) * RB + (lane >> 4) * 16;
    const unsigned char* bp = B + (rb + (lane & 7)) * RB + (lane >> 3) * 16;
#pragma unroll
    for (int kk = 0; kk < DP / 32; ++kk) {
      uint32_t bh[4], bl[4];
      ldmatrix_x4(bh, bp + kk * 64);
      ldmatrix_x4(bl, bp + G::ARR + kk * 64);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        uint32_t ah[4], al[4];
        ldmatrix_x4(ah, ap + kk * 64 + e * 32);
        ldmatrix_x4(al, ap + G::ARR + kk * 64 + e * 32);
        mma16816<T>(acc, ah, bh[2 * e], bh[2 * e + 1]);
        mma16816<T>(x, ah, bl[2 * e], bl[2 * e + 1]);
        mma16816<T>(y, al, bh[2 * e], bh[2 * e + 1]);
      }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) acc[i] += x[i] + y[i];
  };
  float p32[4] = {0.f, 0.f, 0.f, 0.f}, p16[4] = {0.f, 0.f, 0.f, 0.f}, p8[4] = {0.f, 0.f, 0.f, 0.f}, pd[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
  for (int u = 0; u < TG; ++u) {
    const int t = tg * TG + u;
    level(arr0, u, t & 32, r32);
    level(arr1, u, t & 16, r16);
  }
  __syncthreads();
  block(arr0, 32 + 16 * (warp >> 2), arr0, 8 * (warp & 3), p32);
  if (warp < 4) block(arr1, 16 + 32 * (warp >> 1), arr1, 32 * (warp >> 1) + 8 * (warp & 1), p16);
  __syncthreads();
#pragma unroll
  for (int u = 0; u < TG; ++u) {
    const float2 ref = L[(u & ~7) + 3];
    put(arr0, tg * TG + u, qf[u], make_float2(L[u].x - ref.x, L[u].y - ref.y));
    put(arr1, tg * TG + u, kf[u], make_float2(ref.x - L[u].x, ref.y - L[u].y));
  }
  __syncthreads();
  const int di = 16 * (warp >> 1), nb = warp & 1;            // diagonal block of 16 rows, its 8 columns
  block(arr0, di, arr1, di + 8 * nb, pd);
  __syncthreads();
#pragma unroll
  for (int u = 0; u < TG; ++u) level(arr0, u, (tg * TG + u) & 8, r8);
  __syncthreads();
  if (nb == 0) block(arr0, di, arr0, di, p8);
  // ---- the image of P
  unsigned char* img = arr1;                                 // hi, lo (the array has been read)
  auto emit = [&](int r0, int c0, float x0, float x1, float x2, float x3) {   // rows r0 + g (+ 8), columns c0 + 2 tq (+ 1)
    uint32_t hi, lo;
    const int ra = r0 + g, rb = ra + 8, c = c0 >> 3;
    lc_split(x0, x1, hi, lo);
    *reinterpret_cast<uint32_t*>(img + ra * 128 + ((c ^ (ra & 7)) << 4) + tq * 4) = hi;
    *reinterpret_cast<uint32_t*>(img + LC_P + ra * 128 + ((c ^ (ra & 7)) << 4) + tq * 4) = lo;
    lc_split(x2, x3, hi, lo);
    *reinterpret_cast<uint32_t*>(img + rb * 128 + ((c ^ (rb & 7)) << 4) + tq * 4) = hi;
    *reinterpret_cast<uint32_t*>(img + LC_P + rb * 128 + ((c ^ (rb & 7)) << 4) + tq * 4) = lo;
  };
  emit(32 + 16 * (warp >> 2), 8 * (warp & 3), p32[0], p32[1], p32[2], p32[3]);
  if (warp < 4) emit(16 + 32 * (warp >> 1), 32 * (warp >> 1) + 8 * (warp & 1), p16[0], p16[1], p16[2], p16[3]);
  {
    float skip = 0.f;
    if constexpr (KIND == ZP_LINEAR_SCALAR) skip = a.D[h];
    const int c = 2 * tq;                                    // column of the 8 x 8 block
    float x[4];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const float lo_ = pd[j], hi_ = pd[2 + j];
      const float on_lo = c + j < g ? lo_ : c + j == g ? lo_ + skip : 0.f, on_hi = c + j < g ? hi_ : c + j == g ? hi_ + skip : 0.f;
      x[j] = nb == 0 ? on_lo : 0.f;
      x[2 + j] = nb == 0 ? p8[2 + j] : on_hi;
    }
    emit(di, di + 8 * nb, x[0], x[1], x[2], x[3]);
  }
  for (int i = warp; i < 12; i += 8) {                       // blocks above the diagonal
    const int r = i < 6 ? 0 : i < 10 ? 16 : 32, c = i < 6 ? 16 + 8 * i : i < 10 ? 32 + 8 * (i - 6) : 48 + 8 * (i - 10);
    emit(r, c, 0.f, 0.f, 0.f, 0.f);
  }
  __syncthreads();
  for (int i = tid; i < 2 * LC_P / 16; i += LP_THREADS) st16(dst + 4 * OP + i * 16, ld16(img + i * 16));
}

// ---------------------------------------------------------------------------------------------
// One block per (128 value columns, head, sequence).
// ---------------------------------------------------------------------------------------------
constexpr int LS_THREADS = 512;
constexpr int LS_VT = 128;
constexpr int LS_V = 16384;                      // 64 rows x 128 value columns
constexpr uint32_t LS_O = 0, LS_D = 128, LS_S = 256;   // TMEM columns: O (2 x 64), D (128), S (2 x (hi 64, lo 64))

template <int DP> struct __align__(16) LsShared {
  float decay[2][DP];
  uint64_t kfull[2], qfull[2], empty[2], sready[2], dfull, dfree, ofull[2], ofree[2];
  uint32_t tmem_base;
  int abort_flag;
};
template <int DP> constexpr int ls_stage() { return 4 * lc_op(DP) + 2 * LC_P + LS_V; }

__device__ __forceinline__ uint64_t ls_desc_mn(uint32_t addr) {   // MN-major, 64-element blocks 8192 bytes apart
  const uint32_t lo = ((addr >> 4) & 0x3FFFu) | ((8192u >> 4) << 16);
  const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
  return (static_cast<uint64_t>(hi) << 32) | lo;
}
__device__ __forceinline__ void ls_bulk(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void ls_umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(acc)
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
  LsShared<DP>& sh = *reinterpret_cast<LsShared<DP>*>(stages + 2 * STAGE);       // a stage: K hi, lo | Q~ hi, lo | P hi, lo | V
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sh.kfull[i], 1); mbar_init(&sh.qfull[i], 1); mbar_init(&sh.empty[i], 9); mbar_init(&sh.sready[i], 8);
      mbar_init(&sh.ofull[i], 1); mbar_init(&sh.ofree[i], 4);
    }
    mbar_init(&sh.dfull, 1);
    mbar_init(&sh.dfree, 8);
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
        if (!mbar_wait<true>(&sh.empty[s], ((c >> 1) & 1) ^ 1, abortp, err, 981)) break;
        unsigned char* st = stages + s * STAGE;
        mbar_arrive_expect_tx(&sh.kfull[s], 2 * OP + LS_V + DP * 4);
        ls_bulk(st, ws + c * step, 2 * OP, &sh.kfull[s]);
        tma_load_5d(st + 4 * OP + 2 * LC_P, &tmV, &sh.kfull[s], c0, h, sq.row0 + c * LC_C, 0, 0);
        tma_load_5d(st + 4 * OP + 2 * LC_P + 8192, &tmV, &sh.kfull[s], c0 + 64, h, sq.row0 + c * LC_C, 0, 0);
        ls_bulk(sh.decay[s], ws + c * step + 4 * OP + 2 * LC_P, DP * 4, &sh.kfull[s]);
        mbar_arrive_expect_tx(&sh.qfull[s], 2 * OP + 2 * LC_P);
        ls_bulk(st + 2 * OP, ws + c * step + 2 * OP, 2 * OP + 2 * LC_P, &sh.qfull[s]);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t B_MN = 1u << 16, A_MN = 1u << 15;
      constexpr uint32_t ID_D = idesc_f16(1, 128, DP) | A_MN | B_MN, ID_S = idesc_f16(1, 128, 64), ID_P = ID_S | A_MN;
      auto issue_d = [&](int c) -> bool {
        if (!mbar_wait(&sh.kfull[c & 1], (c >> 1) & 1, abortp, err, 982)) return false;
        fence_after_sync();
        const uint32_t k = smem_u32(stages + (c & 1) * STAGE), v = k + 4 * OP + 2 * LC_P;
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          const uint64_t vd = ls_desc_mn(v + ks * 2048);
          umma_f16(tmem + LS_D, vd, ls_desc_mn(k + ks * 2048), ID_D, ks ? 1u : 0u);
          umma_f16(tmem + LS_D, vd, ls_desc_mn(k + OP + ks * 2048), ID_D, 1u);
        }
        umma_commit(&sh.dfull);
        return true;
      };
      bool ok = issue_d(0);
      for (int c = 0; ok && c < nc; ++c) {
        const int s = c & 1;
        const uint32_t ph = (c >> 1) & 1;
        if (!mbar_wait(&sh.qfull[s], ph, abortp, err, 983) || !mbar_wait(&sh.ofree[s], ph ^ 1, abortp, err, 984) ||
            !mbar_wait(&sh.sready[s], ph, abortp, err, 985)) break;
        fence_after_sync();
        const uint32_t k = smem_u32(stages + s * STAGE), q = k + 2 * OP, pp = k + 4 * OP, v = pp + 2 * LC_P;
        const uint32_t o = tmem + LS_O + s * 64, shi = tmem + LS_S + s * 128, slo = shi + 64;
#pragma unroll
        for (int ks = 0; ks < DP / 16; ++ks) {
          const uint64_t qh = smem_desc_sw128(q + (ks >> 2) * 8192) + 2u * (ks & 3), ql = smem_desc_sw128(q + OP + (ks >> 2) * 8192) + 2u * (ks & 3);
          ls_umma_ts(o, shi + ks * 8, qh, ID_S, ks ? 1u : 0u);
          ls_umma_ts(o, slo + ks * 8, qh, ID_S, 1u);
          ls_umma_ts(o, shi + ks * 8, ql, ID_S, 1u);
        }
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          const uint64_t vd = ls_desc_mn(v + ks * 2048);
          umma_f16(o, vd, smem_desc_sw128(pp) + 2u * ks, ID_P, 1u);
          umma_f16(o, vd, smem_desc_sw128(pp + LC_P) + 2u * ks, ID_P, 1u);
        }
        umma_commit(&sh.ofull[s]);
        umma_commit(&sh.empty[s]);
        if (c + 1 < nc) ok = mbar_wait(&sh.dfree, c & 1, abortp, err, 986) && issue_d(c + 1);
      }
    }
  } else if (warp >= 4 && warp < 12) {
    // ---------------- state ----------------
    constexpr int W = DP / 2;                              // key channels of a thread
    const int q = warp & 3, half = (warp - 4) >> 2, v = c0 + q * 32 + lane;
    const uint32_t lanes = tmem + (static_cast<uint32_t>(q * 32) << 16);
    float* Sg = a.state + (((int64_t)sq.slot * a.H + h) * a.dim + half * W) * a.VP + v;
    const bool mine = v < a.vdim;
    float s[W];
#pragma unroll
    for (int i = 0; i < W; ++i) s[i] = (mine && !sq.fresh && half * W + i < a.dim) ? Sg[(int64_t)i * a.VP] : 0.f;
    auto put = [&](int i, uint32_t buf) {                  // channels i .. i + 15 of this thread as operand, hi and lo
      uint32_t hi[8], lo[8];
#pragma unroll
      for (int j = 0; j < 8; ++j) lc_split(s[i + 2 * j], s[i + 2 * j + 1], hi[j], lo[j]);
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
    publish(&sh.sready[0]);
    bool ok = true;
    for (int c = 0; c < nc; ++c) {
      const int st = c & 1;
      if (!ls_wait(&sh.kfull[st], (c >> 1) & 1, abortp, err, 987) || !ls_wait(&sh.dfull, c & 1, abortp, err, 988)) { ok = false; break; }
      fence_after_sync();
      const bool more = c + 1 < nc;                        // (the operand's other buffer: read by products before this D's)
#pragma unroll
      for (int i = 0; i < W; i += 16) {
        float y[16];
        ls_ld16(lanes + LS_D + half * W + i, y);
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
          const float4 f = *reinterpret_cast<const float4*>(&sh.decay[st][half * W + i + j]);
          s[i + j] = fmaf(f.x, s[i + j], y[j]);
          s[i + j + 1] = fmaf(f.y, s[i + j + 1], y[j + 1]);
          s[i + j + 2] = fmaf(f.z, s[i + j + 2], y[j + 2]);
          s[i + j + 3] = fmaf(f.w, s[i + j + 3], y[j + 3]);
        }
        if (i + 16 == W) {                                 // D and the decays have been read
          fence_before_sync();
          __syncwarp();
          if (lane == 0) { mbar_arrive(&sh.dfree); mbar_arrive(&sh.empty[st]); }
        }
        if (more) put(i, st ^ 1);
      }
      if (more) publish(&sh.sready[st ^ 1]);
    }
    if (ok && mine) {
#pragma unroll
      for (int i = 0; i < W; ++i)
        if (half * W + i < a.dim) Sg[(int64_t)i * a.VP] = s[i];
    }
  } else if (warp >= 12) {
    // ---------------- outputs ----------------
    const int q = warp & 3, v = c0 + q * 32 + lane;
    const uint32_t lanes = tmem + (static_cast<uint32_t>(q * 32) << 16);
    const bool odd = lane & 1;
    // lanes of a pair share two tokens: the even lane stores both columns of one, the odd lane those of the next
    T* out = reinterpret_cast<T*>(a.out) + (int64_t)h * a.vdim + (v & ~1);
    for (int c = 0; c < nc; ++c) {
      const int s = c & 1, n = min(LC_C, sq.count - c * LC_C);
      if (!ls_wait(&sh.ofull[s], (c >> 1) & 1, abortp, err, 989)) break;
      fence_after_sync();
      const int64_t row0 = sq.row0 + (int64_t)c * LC_C;
#pragma unroll
      for (int i = 0; i < 64; i += 16) {
        float y[16];
        ls_ld16(lanes + LS_O + s * 64 + i, y);
        if (i == 48) {
          fence_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(&sh.ofree[s]);
        }
#pragma unroll
        for (int j = 0; j < 16; j += 2) {
          const float other = __shfl_xor_sync(0xffffffffu, odd ? y[j] : y[j + 1], 1);
          const int t = i + j + (odd ? 1 : 0);
          if (t < n && v < a.vdim)
            *reinterpret_cast<uint32_t*>(out + (row0 + t) * a.out_stride) = odd ? pack2<T>(other, y[j + 1]) : pack2<T>(y[j], other);
        }
      }
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 2) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

bool linear_chunk_supports(const LinearArgs& a) {
  return a.taps == 0 && a.dim <= 128 && a.dim % 8 == 0 && a.vdim % 8 == 0 && a.x_stride % 8 == 0 && a.out_stride % 2 == 0 &&
         (uintptr_t)a.v % 16 == 0 && ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.out) % 4 == 0 &&
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
  kern<<<dim3(linear_slots(a.total_rows, a.B), a.H), LP_THREADS, smem, st>>>(a, (unsigned char*)a.workspace);
  return check_launch("zp_linear_state(prepare)");
}
template <int DP> static int chunk_by_size(const LinearArgs& a, const CUtensorMap& tmV, int* error_word, cudaStream_t st) {
  const int rc = a.kind == ZP_LINEAR_FORGET  ? launch_prepare<ZP_LINEAR_FORGET, DP>(a, st)
                 : a.kind == ZP_LINEAR_POWER ? launch_prepare<ZP_LINEAR_POWER, DP>(a, st)
                                             : launch_prepare<ZP_LINEAR_SCALAR, DP>(a, st);
  if (rc) return rc;
  const LsParams p{a, (const unsigned char*)a.workspace, error_word};
  constexpr int smem = 1024 + 2 * ls_stage<DP>() + (int)sizeof(LsShared<DP>);
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
