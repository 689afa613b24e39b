// Gated delta rule over prompt portions, 64 tokens at a time (bf16 q, k, v; fp32 state), head sizes up to 128.
//
// With L_t the running sum of the log decays inside a chunk, G_t = exp(L_t), the recurrence unrolls to
//   (I + A) U = diag(b) (V - diag(G) K S_0),   A_tj = b_t exp(L_t - L_j) k_t . k_j  (j < t)
//   O = diag(G) Q S_0 + P U,                   P_tj = exp(L_t - L_j) q_t . k_j      (j <= t)
//   S = G_C S_0 + K^T diag(exp(L_C - L)) U
// with every exponent <= 0.  Two kernels:
//   * `delta_prepare_kernel`, parallel over chunks: everything that does not depend on the state, as one 128 x 64
//     operand [M; W], W = (I + A)^-1 diag(b), M = P W, and per-token factors.  Products on mma.sync, the inverse by
//     substitution in fp32 (two 32 x 32 halves and the block that joins them).
//   * `delta_scan_tc_kernel`, one block per (head, sequence), the chunks in order, all products on tcgen05 with 128
//     rows and the accumulators in TMEM:
//       Z = [Q; K] S_0;   R = V - G k-factor Z_K;   Y = [M; W] R;   o = G q-factor Z_Q + Y_O;   D = K^T (factor Y_U);
//       S = G_C S_0 + D  (fp32, in registers)
// Keys and queries enter as the bf16 rows of the convolution; the factors that make them unit vectors are fp32 and
// multiply results.  Whatever else is fp32 (S, R, U, M, W) enters a product as a pair of bf16 numbers, hi + lo.
//
// Scan roles (576 threads, one block per SM): warp 0 = TMA producer and TMEM owner, warp 1 = MMA issuer, warps 2-17 =
// arithmetic (thread <-> TMEM lane; the four warps of a lane quadrant split 128 columns).  A lane is a key dim for the state; of
// a chunk's 128 rows the first 64 are outputs and the others corrections.  Every wait is bounded; after it the block
// raises the device error word and leaves.
#include "zp_delta.cuh"
#include "zp_mma.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

constexpr int DC_IMG = 16384;                    // 128 rows x 64 bf16, swizzled as the operand lies in shared memory
constexpr int DC_FACTORS = 1024;                 // floats: output, correction, update factor of each token; G_C
constexpr int DC_PER = 2 * DC_IMG + DC_FACTORS;  // a chunk of a head: hi, lo, factors
constexpr float DC_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void dc_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack2<__nv_bfloat16>(a - f.x, b - f.y);
}

// Chunks of sequence b take the slots delta_first_slot(b) .. (a bound that needs no scan over the sequences)
__device__ __forceinline__ int delta_first_slot(const DeltaArgs& a, int b) { return (a.cu_q[b] - a.cu_q[0]) / DC_C + b; }
static int delta_slots(int total_rows, int B) { return total_rows / DC_C + B; }

// ---------------------------------------------------------------------------------------------
// One block per (chunk, head).
// ---------------------------------------------------------------------------------------------
constexpr int DP_THREADS = 128;
constexpr int DP_AS = 68;                        // floats per row of A

template <int DP> struct PrepSmem {
  static constexpr int RB = DP * 2 + 16;         // bytes of a key row
  static constexpr int KQ = 2 * DC_C * RB;
  static constexpr int A = KQ > 2 * DC_IMG ? KQ : 2 * DC_IMG;      // keys and queries, then the operand's image
  static constexpr int F = A + DC_C * DP_AS * 4;
  static constexpr int TOTAL = F + 6 * DC_C * 4;
};

template <int DP>
__global__ void __launch_bounds__(DP_THREADS) delta_prepare_kernel(const DeltaArgs a, unsigned char* __restrict__ ws) {
  using T = __nv_bfloat16;
  using L = PrepSmem<DP>;
  extern __shared__ __align__(128) unsigned char smem[];
  const int slot = blockIdx.x, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  int lo_b = 0, hi_b = a.B - 1;                  // last sequence whose slots start at or before this one
  while (lo_b < hi_b) {
    const int mid = (lo_b + hi_b + 1) >> 1;
    if (delta_first_slot(a, mid) <= slot) lo_b = mid; else hi_b = mid - 1;
  }
  const DeltaSeq sq = delta_seq(a, lo_b);
  const int t0 = (slot - delta_first_slot(a, lo_b)) * DC_C, n = min(DC_C, sq.count - t0);
  if (n <= 0) return;
  unsigned char *sQ = smem, *sK = smem + DC_C * L::RB;
  float* sA = reinterpret_cast<float*>(smem + L::A);
  float *sL = reinterpret_cast<float*>(smem + L::F), *sB = sL + 64, *sRk = sL + 128, *sRq = sL + 192, *sLog = sL + 256;
  const int hk = h / (a.H / a.G);
  const int64_t row0 = sq.row0 + t0;
  {
    const T* qb = reinterpret_cast<const T*>(a.x) + (int64_t)hk * a.dim;
    const T* kb = qb + (int64_t)a.G * a.dim;
    constexpr int per = DP / 8;
    for (int i = tid; i < 2 * DC_C * per; i += DP_THREADS) {
      const int half = i / (DC_C * per), r = i / per % DC_C, c = i % per;
      const int ok = (r < n && c * 8 < a.dim) ? 16 : 0;
      cp_async16((half ? sK : sQ) + r * L::RB + c * 16, (half ? kb : qb) + (ok ? (row0 + r) * a.x_stride + c * 8 : 0), ok);
    }
    cp_async_commit();
  }
  if (tid < DC_C) {
    sLog[tid] = tid < n ? delta_log_decay(a, row0 + tid, h) : 0.f;
    sB[tid] = tid < n ? delta_beta(a, row0 + tid, h) : 0.f;
  }
  cp_async_wait<0>();
  __syncthreads();
  if (warp == 0) {                               // L_t, two tokens a lane
    const float f0 = sLog[2 * lane], f1 = sLog[2 * lane + 1];
    float F = f0 + f1;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, F, o); if (lane >= o) F += x; }
    sL[2 * lane] = F - f1;
    sL[2 * lane + 1] = F;
  }
  {                                              // norms: a thread per row of K and of Q
    const unsigned char* r = (tid < DC_C ? sK : sQ) + (tid & 63) * L::RB;
    float ss = 0.f;
#pragma unroll 4
    for (int c = 0; c < DP / 8; ++c) {
      const int4 w = ld16(r + c * 16);
      const __nv_bfloat162* e = reinterpret_cast<const __nv_bfloat162*>(&w);
#pragma unroll
      for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(e[i]); ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss)); }
    }
    const float rn = 1.f / sqrtf(ss + DELTA_UNIT_EPS);
    if (tid < DC_C) sRk[tid] = rn; else sRq[tid & 63] = rn * rsqrtf((float)a.dim);
  }
  float kk[8][4], p[8][4];                       // rows warp * 16 + g (+ 8), columns 8 nb + 2 tq (+ 1)
#pragma unroll
  for (int i = 0; i < 8; ++i) { kk[i][0] = kk[i][1] = kk[i][2] = kk[i][3] = 0.f; p[i][0] = p[i][1] = p[i][2] = p[i][3] = 0.f; }
#pragma unroll 2
  for (int ks = 0; ks < DP / 16; ++ks) {
    uint32_t ka[4], qa[4];
    ldmatrix_x4(ka, sK + (warp * 16 + (lane & 15)) * L::RB + ks * 32 + (lane >> 4) * 16);
    ldmatrix_x4(qa, sQ + (warp * 16 + (lane & 15)) * L::RB + ks * 32 + (lane >> 4) * 16);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np > warp) continue;                   // later keys only
      uint32_t bf[4];
      ldmatrix_x4(bf, sK + (np * 16 + (lane & 7) + (lane >> 4) * 8) * L::RB + ks * 32 + ((lane >> 3) & 1) * 16);
      mma16816<T>(kk[2 * np], ka, bf[0], bf[1]);
      mma16816<T>(kk[2 * np + 1], ka, bf[2], bf[3]);
      mma16816<T>(p[2 * np], qa, bf[0], bf[1]);
      mma16816<T>(p[2 * np + 1], qa, bf[2], bf[3]);
    }
  }
  __syncthreads();                               // sL, norms; the tiles' place is free
  const int ra = warp * 16 + g, rb = ra + 8;
  {
    const float La = sL[ra], Lb = sL[rb], ka = sB[ra] * sRk[ra], kb = sB[rb] * sRk[rb], qa = sRq[ra], qb = sRq[rb];
#pragma unroll
    for (int nb = 0; nb < 8; ++nb) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int col = nb * 8 + 2 * tq + (j & 1), row = j < 2 ? ra : rb;
        const float e = col <= row ? exp2f(((j < 2 ? La : Lb) - sL[col]) * DC_LOG2E) * sRk[col] : 0.f;
        kk[nb][j] = col < row ? kk[nb][j] * e * (j < 2 ? ka : kb) : 0.f;
        p[nb][j] = col <= row ? p[nb][j] * e * (j < 2 ? qa : qb) : 0.f;
      }
      *reinterpret_cast<float2*>(sA + ra * DP_AS + nb * 8 + 2 * tq) = make_float2(kk[nb][0], kk[nb][1]);
      *reinterpret_cast<float2*>(sA + rb * DP_AS + nb * 8 + 2 * tq) = make_float2(kk[nb][2], kk[nb][3]);
    }
  }
  unsigned char* dst = ws + ((int64_t)slot * a.H + h) * DC_PER;
  if (tid < DC_C) {
    float* f = reinterpret_cast<float*>(dst + 2 * DC_IMG);
    const float Lt = sL[tid], LC = sL[DC_C - 1], G = expf(Lt);
    const bool in = tid < n;
    f[tid] = in ? G * sRq[tid] : 0.f;
    f[64 + tid] = in ? G * sRk[tid] : 0.f;
    f[128 + tid] = in ? expf(LC - Lt) * sRk[tid] : 0.f;
    if (tid == 0) f[192] = expf(LC);
  }
  __syncthreads();
  // (I + A)^-1: the two diagonal 32 x 32 blocks, a column per thread, over A's own place
  if (tid < DC_C) {
    const int o = tid & 32, c = tid & 31;
    float x[32];
#pragma unroll
    for (int r = 0; r < 32; ++r) {
      const float* ar = sA + (o + r) * DP_AS + o;
      float s0 = r == c ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
      for (int j = 0; j < r; j += 4) {
        const float4 v = *reinterpret_cast<const float4*>(ar + j);
        s0 = fmaf(-v.x, x[j], s0);
        if (j + 1 < r) s1 = fmaf(-v.y, x[j + 1], s1);
        if (j + 2 < r) s2 = fmaf(-v.z, x[j + 2], s2);
        if (j + 3 < r) s3 = fmaf(-v.w, x[j + 3], s3);
      }
      x[r] = (s0 + s1) + (s2 + s3);
    }
    __syncwarp();                                // (a half's rows are read by its own warp only)
#pragma unroll
    for (int r = 0; r < 32; ++r) sA[(o + r) * DP_AS + o + c] = x[r];
  }
  __syncthreads();
  // the block that joins them, -T22 A21 T11: a row and eight columns per thread; A21 T11 into the upper right block first
  {
    const int i = tid >> 2, j0 = (tid & 3) * 8;
    float acc[8];
    auto product = [&](const float* left, const float* right) {    // rows of DP_AS floats
#pragma unroll
      for (int j = 0; j < 8; ++j) acc[j] = 0.f;
#pragma unroll 8
      for (int k = 0; k < 32; ++k) {
        const float l = left[i * DP_AS + k];
        const float4 u = *reinterpret_cast<const float4*>(right + k * DP_AS + j0), v = *reinterpret_cast<const float4*>(right + k * DP_AS + j0 + 4);
        acc[0] = fmaf(l, u.x, acc[0]); acc[1] = fmaf(l, u.y, acc[1]); acc[2] = fmaf(l, u.z, acc[2]); acc[3] = fmaf(l, u.w, acc[3]);
        acc[4] = fmaf(l, v.x, acc[4]); acc[5] = fmaf(l, v.y, acc[5]); acc[6] = fmaf(l, v.z, acc[6]); acc[7] = fmaf(l, v.w, acc[7]);
      }
    };
    auto put = [&](float* to, float s) {
      *reinterpret_cast<float4*>(to + i * DP_AS + j0) = make_float4(s * acc[0], s * acc[1], s * acc[2], s * acc[3]);
      *reinterpret_cast<float4*>(to + i * DP_AS + j0 + 4) = make_float4(s * acc[4], s * acc[5], s * acc[6], s * acc[7]);
    };
    float *A12 = sA + 32, *A21 = sA + 32 * DP_AS, *A22 = A21 + 32;
    product(A21, sA);
    put(A12, 1.f);
    __syncthreads();
    product(A22, A12);
    __syncthreads();
    put(A21, -1.f);
    __syncthreads();
  }
  // W: rows 64 .. 127 of the image
  for (int i = tid; i < DC_C * 8; i += DP_THREADS) {
    const int r = i >> 3, c = i & 7;
    const bool zero = r < 32 && c >= 4;          // (the upper right block holds other things)
    uint32_t hi[4], lo[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 v = *reinterpret_cast<const float2*>(sA + r * DP_AS + c * 8 + 2 * j);
      dc_split(zero ? 0.f : v.x * sB[c * 8 + 2 * j], zero ? 0.f : v.y * sB[c * 8 + 2 * j + 1], hi[j], lo[j]);
    }
    const int off = (64 + r) * 128 + ((c ^ (r & 7)) << 4);
    st16(smem + off, make_int4((int)hi[0], (int)hi[1], (int)hi[2], (int)hi[3]));
    st16(smem + DC_IMG + off, make_int4((int)lo[0], (int)lo[1], (int)lo[2], (int)lo[3]));
  }
  __syncthreads();
  // M = P W
  float m[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) { m[i][0] = m[i][1] = m[i][2] = m[i][3] = 0.f; }
#pragma unroll
  for (int ks = 0; ks < 4; ++ks) {
    if (ks > warp) continue;
    uint32_t ph[4], pl[4];
    dc_split(p[2 * ks][0], p[2 * ks][1], ph[0], pl[0]);
    dc_split(p[2 * ks][2], p[2 * ks][3], ph[1], pl[1]);
    dc_split(p[2 * ks + 1][0], p[2 * ks + 1][1], ph[2], pl[2]);
    dc_split(p[2 * ks + 1][2], p[2 * ks + 1][3], ph[3], pl[3]);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np > ks) continue;                     // W is lower triangular
      const int r = ks * 16 + (lane & 15), c = np * 2 + (lane >> 4);
      const int off = (64 + r) * 128 + ((c ^ (r & 7)) << 4);
      uint32_t bh[4], bl[4];
      ldmatrix_x4_trans(bh, smem + off);
      ldmatrix_x4_trans(bl, smem + DC_IMG + off);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        mma16816<T>(m[2 * np + e], ph, bh[2 * e], bh[2 * e + 1]);
        mma16816<T>(m[2 * np + e], ph, bl[2 * e], bl[2 * e + 1]);
        mma16816<T>(m[2 * np + e], pl, bh[2 * e], bh[2 * e + 1]);
      }
    }
  }
#pragma unroll
  for (int nb = 0; nb < 8; ++nb) {
    uint32_t hi, lo;
    dc_split(m[nb][0], m[nb][1], hi, lo);
    const int oa = ra * 128 + ((nb ^ (ra & 7)) << 4) + tq * 4, ob = rb * 128 + ((nb ^ (rb & 7)) << 4) + tq * 4;
    *reinterpret_cast<uint32_t*>(smem + oa) = hi;
    *reinterpret_cast<uint32_t*>(smem + DC_IMG + oa) = lo;
    dc_split(m[nb][2], m[nb][3], hi, lo);
    *reinterpret_cast<uint32_t*>(smem + ob) = hi;
    *reinterpret_cast<uint32_t*>(smem + DC_IMG + ob) = lo;
  }
  __syncthreads();
  for (int i = tid; i < 2 * DC_IMG / 16; i += DP_THREADS) st16(dst + i * 16, ld16(smem + i * 16));
}

// ---------------------------------------------------------------------------------------------
// One block per (head, sequence).
// ---------------------------------------------------------------------------------------------
constexpr int DS_THREADS = 576;
constexpr int DS_BLK = 16384;                    // [Q; K] of 64 dims, or 128 state rows x 64 columns
constexpr int DS_HALF = 8192;                    // 64 rows x 64 columns
constexpr uint32_t DS_Z = 0, DS_Y = 128, DS_D = 256;   // TMEM columns

struct __align__(16) DsShared {
  float factors[2][DC_FACTORS / 4];
  float ssq[2][4][64];           // sums of squares per column quarter, by parity
  float norm[128];
  uint64_t full[2], empty[2], ifull, iempty, sready, zfull, rready, yfull, uready, dfull, obar[2];
  uint32_t tmem_base;
  int abort_flag;
};

__device__ __forceinline__ uint64_t ds_desc_mn(uint32_t addr, uint32_t lbo) {   // MN-major, 64-element blocks `lbo` apart
  const uint32_t lo = ((addr >> 4) & 0x3FFFu) | ((lbo >> 4) << 16);
  const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
  return (static_cast<uint64_t>(hi) << 32) | lo;
}
__device__ __forceinline__ void ds_bulk(void* dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(smem_u32(dst)), "l"(src), "r"(bytes), "r"(smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void ds_ld16(uint32_t taddr, float (&v)[16]) {   // load and wait
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
__device__ __forceinline__ float ds_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float ds_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

struct DsParams { DeltaArgs a; const unsigned char* ws; int* error_word; };

__global__ void __launch_bounds__(DS_THREADS, 1)
delta_scan_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const DsParams p) {
  using T = __nv_bfloat16;
  const DeltaArgs& a = p.a;
  const int h = blockIdx.x, b = blockIdx.y;
  const DeltaSeq sq = delta_seq(a, b);
  if (sq.count == 0) return;
  const int nc = (sq.count + DC_C - 1) / DC_C, hk = h / (a.H / a.G);
  extern __shared__ unsigned char smem_raw[];
  unsigned char* stage = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* img = stage + 2 * 2 * DS_BLK;             // hi, lo
  unsigned char* sHi = img + 2 * DC_IMG;                   // state operand, hi and lo: two column blocks each
  unsigned char* sLo = sHi + 2 * DS_BLK;
  unsigned char* uHi = sLo + 2 * DS_BLK;                   // corrections, then updates
  unsigned char* uLo = uHi + 2 * DS_HALF;
  DsShared& sh = *reinterpret_cast<DsShared*>(uLo + 2 * DS_HALF);
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x < 128) sh.norm[threadIdx.x] = (int)threadIdx.x < a.vdim ? a.norm_weight[threadIdx.x] : 0.f;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 17); mbar_init(&sh.obar[i], 4); }
    mbar_init(&sh.ifull, 1); mbar_init(&sh.iempty, 1); mbar_init(&sh.sready, 16); mbar_init(&sh.zfull, 1);
    mbar_init(&sh.rready, 8); mbar_init(&sh.yfull, 1); mbar_init(&sh.uready, 8); mbar_init(&sh.dfull, 1);
    sh.abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
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
      const unsigned char* ws = p.ws + ((int64_t)delta_first_slot(a, b) * a.H + h) * DC_PER;
      const int64_t step = (int64_t)a.H * DC_PER;
      for (int c = 0; c < nc; ++c) {
        const int st = c & 1, row = sq.row0 + c * DC_C;
        if (!mbar_wait<true>(&sh.empty[st], ((c >> 1) & 1) ^ 1, abortp, err, 951)) break;
        unsigned char* dst = stage + st * 2 * DS_BLK;
        mbar_arrive_expect_tx(&sh.full[st], 2 * DS_BLK + DC_FACTORS);
        for (int d = 0; d < 2; ++d) {
          tma_load_5d(dst + d * DS_BLK, &tmQ, &sh.full[st], d * 64, hk, row, 0, 0);
          tma_load_5d(dst + d * DS_BLK + DS_HALF, &tmK, &sh.full[st], d * 64, hk, row, 0, 0);
        }
        ds_bulk(sh.factors[st], ws + c * step + 2 * DC_IMG, DC_FACTORS, &sh.full[st]);
        if (!mbar_wait<true>(&sh.iempty, (c & 1) ^ 1, abortp, err, 952)) break;
        mbar_arrive_expect_tx(&sh.ifull, 2 * DC_IMG);
        ds_bulk(img, ws + c * step, 2 * DC_IMG, &sh.ifull);
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t ID = idesc_f16(1, 128, 128), B_MN = 1u << 16, A_MN = 1u << 15;
      const uint32_t shi = smem_u32(sHi), slo = smem_u32(sLo), uhi = smem_u32(uHi), ulo = smem_u32(uLo), im = smem_u32(img);
      const int ksd = (a.dim + 15) >> 4;         // steps over the key dims
      for (int c = 0; c < nc; ++c) {
        const uint32_t ph = c & 1;
        const int st = c & 1;
        const uint32_t qk = smem_u32(stage + st * 2 * DS_BLK);
        if (!mbar_wait(&sh.full[st], (c >> 1) & 1, abortp, err, 953) || !mbar_wait(&sh.sready, ph, abortp, err, 954)) break;
        fence_after_sync();
        for (int ks = 0; ks < ksd; ++ks) {
          const uint64_t ad = smem_desc_sw128(qk + (ks >> 2) * DS_BLK) + 2u * (ks & 3);
          umma_f16(tmem + DS_Z, ad, ds_desc_mn(shi + ks * 2048, DS_BLK), ID | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + DS_Z, ad, ds_desc_mn(slo + ks * 2048, DS_BLK), ID | B_MN, 1u);
        }
        umma_commit(&sh.zfull);
        if (!mbar_wait(&sh.ifull, ph, abortp, err, 955) || !mbar_wait(&sh.rready, ph, abortp, err, 956)) break;
        fence_after_sync();
        const uint64_t ah = smem_desc_sw128(im), al = smem_desc_sw128(im + DC_IMG);
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          const uint64_t rh = ds_desc_mn(uhi + ks * 2048, DS_HALF), rl = ds_desc_mn(ulo + ks * 2048, DS_HALF);
          umma_f16(tmem + DS_Y, ah + 2u * ks, rh, ID | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + DS_Y, ah + 2u * ks, rl, ID | B_MN, 1u);
          umma_f16(tmem + DS_Y, al + 2u * ks, rh, ID | B_MN, 1u);
        }
        umma_commit(&sh.yfull);
        umma_commit(&sh.iempty);
        if (!mbar_wait(&sh.uready, ph, abortp, err, 957)) break;
        fence_after_sync();
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          const uint64_t kt = ds_desc_mn(qk + DS_HALF + ks * 2048, DS_BLK);
          umma_f16(tmem + DS_D, kt, ds_desc_mn(uhi + ks * 2048, DS_HALF), ID | A_MN | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + DS_D, kt, ds_desc_mn(ulo + ks * 2048, DS_HALF), ID | A_MN | B_MN, 1u);
        }
        umma_commit(&sh.dfull);
        umma_commit(&sh.empty[st]);
      }
    }
  } else {
    const int q = warp & 3, cq = (warp - 2) >> 2;          // lane quadrant; columns cq * 32 .. + 31
    const int r = q * 32 + lane, t = r & 63;               // key dim of the state; token of the chunk
    const bool corr = q >= 2;                              // these rows of Z and Y are corrections, the others outputs
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(q * 32) << 16) + cq * 32;
    const int cols = min(32, a.vdim - cq * 32);            // (multiples of 8; none may be left)
    bool ok = true;
    auto wait = [&](uint64_t* bar, uint32_t parity, int where) -> bool {
      return __all_sync(0xffffffffu, mbar_wait(bar, parity, abortp, err, where));
    };
    auto arrive = [&](uint64_t* bar) {
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    auto fence_async = []() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); };
    // eight columns (chunk i of this thread's 32) of a row as operand, hi and lo, in column blocks of `block` bytes
    auto put = [&](const float* v, unsigned char* hi, unsigned char* lo, int row, int i, int block) {
      uint32_t x[4], y[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) dc_split(v[2 * j], v[2 * j + 1], x[j], y[j]);
      const uint32_t off = (cq >> 1) * block + row * 128 + ((((cq & 1) * 4 + i) ^ (row & 7)) << 4);
      st16(hi + off, make_int4((int)x[0], (int)x[1], (int)x[2], (int)x[3]));
      st16(lo + off, make_int4((int)y[0], (int)y[1], (int)y[2], (int)y[3]));
    };
    auto publish = [&](uint64_t* bar) {          // operand rows written, accumulators read
      fence_async();
      fence_before_sync();
      arrive(bar);
    };
    float s[32];
    float* Sg = a.S + (((int64_t)sq.slot * a.H + h) * a.dim + r) * a.VP + cq * 32;
    const bool mine = r < a.dim;
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float4 x = (mine && !sq.fresh && i < cols) ? *reinterpret_cast<const float4*>(Sg + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[i] = x.x; s[i + 1] = x.y; s[i + 2] = x.z; s[i + 3] = x.w;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) put(s + 8 * i, sHi, sLo, r, i, DS_BLK);
    publish(&sh.sready);

    const T* vrow = reinterpret_cast<const T*>(a.x) + 2 * (int64_t)a.G * a.dim + (int64_t)h * a.vdim + cq * 32;
    const T* grow = reinterpret_cast<const T*>(a.gate) + (int64_t)h * a.vdim + cq * 32;
    T* orow = reinterpret_cast<T*>(a.out) + (int64_t)h * a.vdim + cq * 32;
    const float inv_vdim = 1.f / (float)a.vdim;
    for (int c = 0; c < nc; ++c) {
      const uint32_t ph = c & 1;
      const int st = c & 1, n = min(DC_C, sq.count - c * DC_C);
      const int64_t row = sq.row0 + (int64_t)c * DC_C + t;
      int4 in[4];
      if (corr) {                                          // values of the row
#pragma unroll
        for (int i = 0; i < 4; ++i) in[i] = (t < n && 8 * i < cols) ? ld16(vrow + row * a.x_stride + 8 * i) : make_int4(0, 0, 0, 0);
      }
      if (!wait(&sh.full[st], (c >> 1) & 1, 961)) { ok = false; break; }
      const float f0 = sh.factors[st][corr ? 64 + t : t], f1 = sh.factors[st][128 + t], GC = sh.factors[st][192];
      arrive(&sh.empty[st]);
      if (!wait(&sh.zfull, ph, 962)) { ok = false; break; }
      fence_after_sync();
      float o[32], y[16];
      if (corr) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          ds_ld16(lane_addr + DS_Z + 16 * k, y);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const __nv_bfloat162* e = reinterpret_cast<const __nv_bfloat162*>(&in[2 * k + i]);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const float2 v = __bfloat1622float2(e[j]);
              y[8 * i + 2 * j] = fmaf(-f0, y[8 * i + 2 * j], v.x);
              y[8 * i + 2 * j + 1] = fmaf(-f0, y[8 * i + 2 * j + 1], v.y);
            }
            put(y + 8 * i, uHi, uLo, t, 2 * k + i, DS_HALF);
          }
        }
        publish(&sh.rready);
      } else {
        tmem_ld32(lane_addr + DS_Z, o);
#pragma unroll
        for (int i = 0; i < 32; ++i) o[i] *= f0;
      }
      if (!wait(&sh.yfull, ph, 963)) { ok = false; break; }
      fence_after_sync();
      if (corr) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          ds_ld16(lane_addr + DS_Y + 16 * k, y);
#pragma unroll
          for (int i = 0; i < 16; ++i) y[i] *= f1;
          put(y, uHi, uLo, t, 2 * k, DS_HALF);
          put(y + 8, uHi, uLo, t, 2 * k + 1, DS_HALF);
        }
        publish(&sh.uready);
      } else {
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          ds_ld16(lane_addr + DS_Y + 16 * k, y);
#pragma unroll
          for (int i = 0; i < 16; ++i) {                   // (columns past vdim are zero)
            o[16 * k + i] += y[i];
            ss = fmaf(o[16 * k + i], o[16 * k + i], ss);
          }
        }
        sh.ssq[ph][cq][t] = ss;
        arrive(&sh.obar[q]);
      }
      if (!wait(&sh.dfull, ph, 964)) { ok = false; break; }
      fence_after_sync();
      const bool more = c + 1 < nc;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        ds_ld16(lane_addr + DS_D + 16 * k, y);
#pragma unroll
        for (int i = 0; i < 16; ++i) s[16 * k + i] = fmaf(GC, s[16 * k + i], y[i]);
        if (more) {
          put(s + 16 * k, sHi, sLo, r, 2 * k, DS_BLK);
          put(s + 16 * k + 8, sHi, sLo, r, 2 * k + 1, DS_BLK);
        }
      }
      if (more) publish(&sh.sready);
      if (!corr) {                                         // (in the shadow of the next chunk's first products)
#pragma unroll
        for (int i = 0; i < 4; ++i) in[i] = (t < n && 8 * i < cols) ? ld16(grow + row * a.gate_stride + 8 * i) : make_int4(0, 0, 0, 0);
        if (!wait(&sh.obar[q], ph, 965)) { ok = false; break; }
        const float ss = (sh.ssq[ph][0][t] + sh.ssq[ph][1][t]) + (sh.ssq[ph][2][t] + sh.ssq[ph][3][t]);
        const float rr = a.out_scale * rsqrtf(ss * inv_vdim + a.eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (8 * i >= cols) continue;
          const __nv_bfloat162* e = reinterpret_cast<const __nv_bfloat162*>(&in[i]);
          uint32_t w[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 z = __bfloat1622float2(e[j]);
            const float2 nw = *reinterpret_cast<const float2*>(&sh.norm[cq * 32 + 8 * i + 2 * j]);
            const float x0 = o[8 * i + 2 * j] * rr * nw.x * z.x * ds_rcp(1.f + ds_ex2(-DC_LOG2E * z.x));
            const float x1 = o[8 * i + 2 * j + 1] * rr * nw.y * z.y * ds_rcp(1.f + ds_ex2(-DC_LOG2E * z.y));
            w[j] = pack2<T>(x0, x1);
          }
          if (t < n) st16(orow + row * a.out_stride + 8 * i, make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]));
        }
      }
    }
    if (ok && mine) {
#pragma unroll
      for (int i = 0; i < 32; i += 4)
        if (i < cols) *reinterpret_cast<float4*>(Sg + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

bool delta_chunk_supports(const DeltaArgs& a, int dtype) {
  return dtype == ZP_DTYPE_BF16 && a.taps == 0 && a.dim <= 128 && a.vdim <= 128 && a.dim % 8 == 0 && a.vdim % 8 == 0 &&
         a.x_stride % 8 == 0 && a.gate_stride % 8 == 0 && a.out_stride % 8 == 0 &&
         ((uintptr_t)a.x | (uintptr_t)a.gate | (uintptr_t)a.out) % 16 == 0;
}
size_t delta_chunk_workspace(int total_rows, int B, int H) { return (size_t)delta_slots(total_rows, B) * H * DC_PER; }

template <int DP> static int launch_prepare(const DeltaArgs& a, int slots, unsigned char* ws, cudaStream_t st) {
  constexpr int smem = PrepSmem<DP>::TOTAL;
  cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_gated_delta(prepare): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  delta_prepare_kernel<DP><<<dim3(slots, a.H), DP_THREADS, smem, st>>>(a, ws);
  return check_launch("zp_gated_delta(prepare)");
}

// total_rows: rows of x, of which the portions' are the rows from cu_q[0] on
int delta_chunk(const DeltaArgs& a, int total_rows, void* workspace, cudaStream_t st) {
  DsParams p{a, (const unsigned char*)workspace, device_error_word()};
  if (!p.error_word) { set_error("zp_gated_delta(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  CUtensorMap tm[2];
  for (int i = 0; i < 2; ++i) {
    const uint64_t rs = (uint64_t)a.x_stride;
    const uint64_t dims[5] = {(uint64_t)a.dim, (uint64_t)a.G, (uint64_t)total_rows, 1, 1};
    const uint64_t strides[4] = {(uint64_t)a.dim, rs, rs * total_rows, rs * total_rows};
    const uint32_t box[5] = {64, 1, 64, 1, 1};
    const __nv_bfloat16* base = (const __nv_bfloat16*)a.x + (int64_t)i * a.G * a.dim;
    if (int rc = make_tensor_map_5d(&tm[i], UmmaFmt<__nv_bfloat16>::tm, base, dims, strides, box, 2)) return rc;
  }
  const int slots = delta_slots(total_rows, a.B);
  if (int rc = a.dim <= 64 ? launch_prepare<64>(a, slots, (unsigned char*)workspace, st)
                           : launch_prepare<128>(a, slots, (unsigned char*)workspace, st)) return rc;
  const int smem = 1024 + 4 * DS_BLK + 2 * DC_IMG + 4 * DS_BLK + 4 * DS_HALF + (int)sizeof(DsShared);
  cudaError_t e = cudaFuncSetAttribute(delta_scan_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_gated_delta(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  delta_scan_tc_kernel<<<dim3(a.H, a.B), DS_THREADS, smem, st>>>(tm[0], tm[1], p);
  return check_launch("zp_gated_delta(tcgen05)");
}

}  // namespace zp
