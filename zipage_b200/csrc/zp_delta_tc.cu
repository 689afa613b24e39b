// Gated delta rule over prompt portions, 64 tokens at a time (bf16 q, k, v; fp32 state), key sizes up to 128, value sizes up to 256.
//
// With L_t the running sum of the log decays inside a chunk, G_t = exp(L_t), the recurrence unrolls to
//   (I + A) U = diag(b) (V - diag(G) K S_0),   A_tj = b_t exp(L_t - L_j) k_t . k_j  (j < t)
//   O = diag(G) Q S_0 + P U,                   P_tj = exp(L_t - L_j) q_t . k_j      (j <= t)
//   S = G_C S_0 + K^T diag(exp(L_C - L)) U
// with every exponent <= 0.  Two kernels:
//   * `delta_prepare_kernel`, parallel over chunks: everything that does not depend on the state, as one 128 x 64
//     operand [M; W], W = (I + A)^-1 diag(b), M = P W, and per-token factors.  Products on mma.sync, the inverse by
//     substitution in fp32 for its 16 x 16 diagonal blocks, the rest by products of blocks.
//   * `delta_scan_tc_kernel`, one block per (value tile, head, sequence), the chunks in order, all products on tcgen05 with 128
//     rows and the accumulators in TMEM:
//       Z = [Q; K] S_0;   R = V - G k-factor Z_K;   Y = [M; W] R;   o = G q-factor Z_Q + Y_O;   D = K^T (factor Y_U);
//       S = G_C S_0 + D  (fp32, in registers)
// Keys and queries enter as the bf16 rows of the convolution; the factors that make them unit vectors are fp32 and
// multiply results.  Whatever else is fp32 (S, R, U, M, W) enters a product as a pair of bf16 numbers, hi + lo.
//
// Scan roles (448 threads, two blocks per SM so that one's arithmetic covers the other's products): warp 2 = TMA producer
// and TMEM owner, warp 3 = MMA issuer, warps 4-11 = corrections and state (thread <-> TMEM lane; the two warps of a lane quadrant
// split the block's 64 value columns), warps 0, 1, 12, 13 = outputs, off the path from chunk to chunk.  A lane is a key dim for the state;
// of a chunk's 128 rows the first 64 are outputs and the others corrections.  The blocks of a head push their rows' sums of squares into each other's shared memory (the output norm
// spans all value dims).  Every wait is bounded; after it the block raises the device error word and leaves.
#include "zp_delta.cuh"
#include "zp_mlstm.cuh"    // cluster helpers
#include "zp_mma.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

constexpr int DC_IMG = 16384;                    // 128 rows x 64 bf16, swizzled as the operand lies in shared memory
constexpr int DC_FACTORS = 1024;                 // floats: output, correction, update factor of each token; G_C
constexpr int DC_PER = 2 * DC_IMG + DC_FACTORS;  // a chunk of a head: hi, lo, factors
constexpr float DC_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float dc_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
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
// One block per (chunk, key head), which serves the value heads of that key head in turn.
// ---------------------------------------------------------------------------------------------
constexpr int DP_THREADS = 256;
constexpr int DP_DS = 20;                        // floats per row of a diagonal block

// Shared memory: keys and queries, then the operand's image (M: rows 0-63, W: rows 64-127; hi, lo); A below its diagonal blocks
// (hi, lo); per-token floats.  While W is made, M's place holds A's diagonal blocks (fp32) and their inverses (hi, lo).
template <int DP> struct PrepSmem {
  static constexpr int RB = DP * 2 + 16;         // bytes of a key row
  static constexpr int KQ = 2 * DC_C * RB;
  static constexpr int A = KQ > 2 * DC_IMG ? KQ : 2 * DC_IMG;
  static constexpr int F = A + 2 * 8192;
  static constexpr int TOTAL = F + 5 * DC_C * 4;
};
// 16-byte piece c (0..7) of row r of a swizzled tile of 128-byte rows
__device__ __forceinline__ int dp_piece(int r, int c) { return r * 128 + ((c ^ (r & 7)) << 4); }
// 16 x 16 block (i, j) of a tile as the left operand, as its transpose, and as the right operand (rows = n)
__device__ __forceinline__ void dp_left(uint32_t (&f)[4], const unsigned char* tile, int i, int j, int lane) {
  ldmatrix_x4(f, tile + dp_piece(i * 16 + (lane & 15), 2 * j + (lane >> 4)));
}
__device__ __forceinline__ void dp_left_t(uint32_t (&f)[4], const unsigned char* tile, int i, int j, int lane) {
  ldmatrix_x4_trans(f, tile + dp_piece(i * 16 + (lane >> 4) * 8 + (lane & 7), 2 * j + ((lane >> 3) & 1)));
}
__device__ __forceinline__ void dp_right(uint32_t (&f)[4], const unsigned char* tile, int i, int j, int lane) {
  ldmatrix_x4(f, tile + dp_piece(i * 16 + (lane & 7) + (lane >> 4) * 8, 2 * j + ((lane >> 3) & 1)));
}

template <int DP>
__global__ void __launch_bounds__(DP_THREADS, 3) delta_prepare_kernel(const DeltaArgs a, unsigned char* __restrict__ ws) {
  using T = __nv_bfloat16;
  using L = PrepSmem<DP>;
  extern __shared__ __align__(128) unsigned char smem[];
  const int slot = blockIdx.x, hk = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  int seq = -1;                                  // last sequence whose slots start at or before this one
  for (int b0 = 0; b0 < a.B; b0 += 32) {
    const unsigned m = __ballot_sync(0xffffffffu, b0 + lane < a.B && delta_first_slot(a, b0 + lane) <= slot);
    seq += __popc(m);
    if (m != 0xffffffffu) break;
  }
  const DeltaSeq sq = delta_seq(a, max(seq, 0));
  const int t0 = (slot - delta_first_slot(a, max(seq, 0))) * DC_C, n = min(DC_C, sq.count - t0);
  if (n <= 0) return;
  unsigned char *sQ = smem, *sK = smem + DC_C * L::RB;
  unsigned char *wHi = smem + 8192, *wLo = smem + DC_IMG + 8192;        // W
  unsigned char *tHi = smem + DC_IMG, *tLo = tHi + 2048;                // inverses of the diagonal blocks: 64 rows of 32 bytes
  unsigned char *aHi = smem + L::A, *aLo = aHi + 8192;
  float* diag = reinterpret_cast<float*>(smem);                         // [4][16][DP_DS]
  float *sL = reinterpret_cast<float*>(smem + L::F), *sB = sL + 64, *sRk = sL + 128, *sRq = sL + 192, *sLog = sL + 256;
  const int group = a.H / a.G;
  const int64_t row0 = sq.row0 + t0;
  {
    const T* qb = reinterpret_cast<const T*>(a.x) + (int64_t)hk * a.dim;
    const T* kb = qb + (int64_t)a.G * a.dim;
    constexpr int per = DP / 8;
#pragma unroll 4
    for (int i = tid; i < 2 * DC_C * per; i += DP_THREADS) {
      const int half = i / (DC_C * per), r = i / per % DC_C, c = i % per;
      const int ok = (r < n && c * 8 < a.dim) ? 16 : 0;
      cp_async16((half ? sK : sQ) + r * L::RB + c * 16, (half ? kb : qb) + (ok ? (row0 + r) * a.x_stride + c * 8 : 0), ok);
    }
    cp_async_commit();
  }
  float gate = 0.f;                              // threads 0-63: log decay, 64-127: step of the head to come
  auto gates = [&](int h) {
    const int t = tid & 63;
    if (tid < 2 * DC_C) gate = t < n ? (tid < DC_C ? delta_log_decay(a, row0 + t, h) : delta_beta(a, row0 + t, h)) : 0.f;
  };
  gates(hk * group);
  cp_async_wait<0>();
  __syncthreads();
  {                                              // norms: two threads per row of K and of Q
    const int r = (tid >> 1) & 63;
    const unsigned char* p = (tid < 2 * DC_C ? sK : sQ) + r * L::RB + (tid & 1) * DP;
    float ss = 0.f;
#pragma unroll 4
    for (int c = 0; c < DP / 16; ++c) {
      const int4 w = ld16(p + c * 16);
      const __nv_bfloat162* e = reinterpret_cast<const __nv_bfloat162*>(&w);
#pragma unroll
      for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(e[i]); ss = fmaf(f.x, f.x, fmaf(f.y, f.y, ss)); }
    }
    ss += __shfl_xor_sync(0xffffffffu, ss, 1);
    const float rn = 1.f / sqrtf(ss + DELTA_UNIT_EPS);
    if ((tid & 1) == 0) { if (tid < 2 * DC_C) sRk[r] = rn; else sRq[r] = rn * rsqrtf((float)a.dim); }
  }
  // warps 0-3: K K^T, warps 4-7: Q K^T, rows wr * 16 + g (+ 8), columns 8 nb + 2 tq (+ 1)
  const int wr = warp & 3;
  const bool isq = warp >= 4;
  float s[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i) { s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.f; }
#pragma unroll 2
  for (int ks = 0; ks < DP / 16; ++ks) {
    uint32_t af[4];
    ldmatrix_x4(af, (isq ? sQ : sK) + (wr * 16 + (lane & 15)) * L::RB + ks * 32 + (lane >> 4) * 16);
#pragma unroll
    for (int np = 0; np < 4; ++np) {
      if (np > wr) continue;                     // later keys only
      uint32_t bf[4];
      ldmatrix_x4(bf, sK + (np * 16 + (lane & 7) + (lane >> 4) * 8) * L::RB + ks * 32 + ((lane >> 3) & 1) * 16);
      mma16816<T>(s[2 * np], af, bf[0], bf[1]);
      mma16816<T>(s[2 * np + 1], af, bf[2], bf[3]);
    }
  }
  const int ra = wr * 16 + g, rb = ra + 8;
  for (int hv = 0; hv < group; ++hv) {
    const int h = hk * group + hv;
    if (tid < DC_C) sLog[tid] = gate; else if (tid < 2 * DC_C) sB[tid - DC_C] = gate;
    __syncthreads();                             // (also: norms there, the tiles' place free)
    if (warp == 0) {                             // L_t, two tokens a lane
      const float f0 = sLog[2 * lane], f1 = sLog[2 * lane + 1];
      float F = f0 + f1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, F, o); if (lane >= o) F += x; }
      sL[2 * lane] = F - f1;
      sL[2 * lane + 1] = F;
    }
    if (hv + 1 < group) gates(h + 1);
    __syncthreads();
    float p[8][4];
    {
      const float La = sL[ra] * DC_LOG2E, Lb = sL[rb] * DC_LOG2E;
      const float fa = isq ? sRq[ra] : sB[ra] * sRk[ra], fb = isq ? sRq[rb] : sB[rb] * sRk[rb];
      const int last = isq ? 1 : 0;              // scores take the token itself, A does not
#pragma unroll
      for (int nb = 0; nb < 8; ++nb) {
        p[nb][0] = p[nb][1] = p[nb][2] = p[nb][3] = 0.f;
        if (nb > 2 * wr + 1) continue;
        const int col = nb * 8 + 2 * tq;
        const float2 Lc = *reinterpret_cast<const float2*>(sL + col), rk = *reinterpret_cast<const float2*>(sRk + col);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int c = col + (j & 1), row = j < 2 ? ra : rb;
          const float x = s[nb][j] * (j < 2 ? fa : fb) * ((j & 1) ? rk.y : rk.x);
          p[nb][j] = c < row + last ? x * dc_ex2(fmaf(-DC_LOG2E, (j & 1) ? Lc.y : Lc.x, j < 2 ? La : Lb)) : 0.f;
        }
        if (!isq) {
          if (nb >= 2 * wr) {                    // the diagonal block
            float* d = diag + wr * 16 * DP_DS + (nb - 2 * wr) * 8 + 2 * tq;
            *reinterpret_cast<float2*>(d + g * DP_DS) = make_float2(p[nb][0], p[nb][1]);
            *reinterpret_cast<float2*>(d + (g + 8) * DP_DS) = make_float2(p[nb][2], p[nb][3]);
          } else {
            uint32_t hi, lo;
            dc_split(p[nb][0], p[nb][1], hi, lo);
            *reinterpret_cast<uint32_t*>(aHi + dp_piece(ra, nb) + tq * 4) = hi;
            *reinterpret_cast<uint32_t*>(aLo + dp_piece(ra, nb) + tq * 4) = lo;
            dc_split(p[nb][2], p[nb][3], hi, lo);
            *reinterpret_cast<uint32_t*>(aHi + dp_piece(rb, nb) + tq * 4) = hi;
            *reinterpret_cast<uint32_t*>(aLo + dp_piece(rb, nb) + tq * 4) = lo;
          }
        }
      }
    }
    unsigned char* dst = ws + ((int64_t)slot * a.H + h) * DC_PER;
    if (tid >= DP_THREADS - DC_C) {
      const int t = tid - (DP_THREADS - DC_C);
      float* f = reinterpret_cast<float*>(dst + 2 * DC_IMG);
      const float Lt = sL[t], LC = sL[DC_C - 1], G = expf(Lt);
      const bool in = t < n;
      f[t] = in ? G * sRq[t] : 0.f;
      f[64 + t] = in ? G * sRk[t] : 0.f;
      f[128 + t] = in ? expf(LC - Lt) * sRk[t] : 0.f;
      if (t == 0) f[192] = expf(LC);
    }
    __syncthreads();
    // diagonal blocks of (I + A)^-1 by substitution, a column per thread; W's are theirs times the steps
    if (tid < DC_C) {
      const int o = tid & 48, c = tid & 15;
      const float* A = diag + o * DP_DS;
      float x[16];
#pragma unroll
      for (int r = 0; r < 16; ++r) {
        float s0 = r == c ? 1.f : 0.f, s1 = 0.f, s2 = 0.f, s3 = 0.f;
#pragma unroll
        for (int j = 0; j < r; j += 4) {
          const float4 v = *reinterpret_cast<const float4*>(A + r * DP_DS + j);
          s0 = fmaf(-v.x, x[j], s0);
          if (j + 1 < r) s1 = fmaf(-v.y, x[j + 1], s1);
          if (j + 2 < r) s2 = fmaf(-v.z, x[j + 2], s2);
          if (j + 3 < r) s3 = fmaf(-v.w, x[j + 3], s3);
        }
        x[r] = (s0 + s1) + (s2 + s3);
      }
      const float b = sB[o + c];
#pragma unroll
      for (int r = 0; r < 16; ++r) {
        const T th = __float2bfloat16_rn(x[r]);
        *reinterpret_cast<T*>(tHi + (o + r) * 32 + c * 2) = th;
        *reinterpret_cast<T*>(tLo + (o + r) * 32 + c * 2) = __float2bfloat16_rn(x[r] - __bfloat162float(th));
        const float w = x[r] * b;
        const T wh = __float2bfloat16_rn(w);
        const int at = dp_piece(o + r, (o + c) >> 3) + ((o + c) & 7) * 2;
        *reinterpret_cast<T*>(wHi + at) = wh;
        *reinterpret_cast<T*>(wLo + at) = __float2bfloat16_rn(w - __bfloat162float(wh));
      }
    } else {                                     // blocks above the diagonal are zero
      for (int i = tid - DC_C; i < DC_C * 8; i += DP_THREADS - DC_C) {
        const int r = i >> 3, c = i & 7;
        if (c < 2 * (r >> 4) + 2) continue;
        st16(wHi + dp_piece(r, c), make_int4(0, 0, 0, 0));
        st16(wLo + dp_piece(r, c), make_int4(0, 0, 0, 0));
      }
    }
    __syncthreads();
    // blocks below: W_ij = -T_ii sum_(j <= k < i) A_ik W_kj, one subdiagonal after the other, a warp per block
#pragma unroll
    for (int d = 1; d < 4; ++d) {
      if (warp < 4 - d) {
        const int j = warp, i = warp + d;
        float x[2][4] = {}, xa[2][4] = {}, xb[2][4] = {};      // the sum, transposed: it is the next product's right operand as it lies
#pragma unroll
        for (int k0 = 0; k0 < d; ++k0) {
          const int k = j + k0;
          uint32_t wh[4], wl[4], ah[4], al[4];
          dp_left_t(wh, wHi, k, j, lane);
          dp_left_t(wl, wLo, k, j, lane);
          dp_right(ah, aHi, i, k, lane);
          dp_right(al, aLo, i, k, lane);
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            mma16816<T>(x[e], wh, ah[2 * e], ah[2 * e + 1]);
            mma16816<T>(xa[e], wh, al[2 * e], al[2 * e + 1]);
            mma16816<T>(xb[e], wl, ah[2 * e], ah[2 * e + 1]);
          }
        }
        uint32_t xh[2][2], xl[2][2];             // [column block][half of k]
#pragma unroll
        for (int e = 0; e < 2; ++e) {
#pragma unroll
          for (int u = 0; u < 4; ++u) x[e][u] += xa[e][u] + xb[e][u];
          dc_split(x[e][0], x[e][1], xh[0][e], xl[0][e]);
          dc_split(x[e][2], x[e][3], xh[1][e], xl[1][e]);
        }
        uint32_t th[4], tl[4];
        const int tr = (i * 16 + (lane & 15)) * 32 + (lane >> 4) * 16;
        ldmatrix_x4(th, tHi + tr);
        ldmatrix_x4(tl, tLo + tr);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float y[4] = {}, ya[4] = {}, yb[4] = {};
          mma16816<T>(y, th, xh[e][0], xh[e][1]);
          mma16816<T>(ya, th, xl[e][0], xl[e][1]);
          mma16816<T>(yb, tl, xh[e][0], xh[e][1]);
#pragma unroll
          for (int u = 0; u < 4; ++u) y[u] += ya[u] + yb[u];
          uint32_t hi, lo;
          const int oa = dp_piece(i * 16 + g, 2 * j + e) + tq * 4, ob = dp_piece(i * 16 + g + 8, 2 * j + e) + tq * 4;
          dc_split(-y[0], -y[1], hi, lo);
          *reinterpret_cast<uint32_t*>(wHi + oa) = hi;
          *reinterpret_cast<uint32_t*>(wLo + oa) = lo;
          dc_split(-y[2], -y[3], hi, lo);
          *reinterpret_cast<uint32_t*>(wHi + ob) = hi;
          *reinterpret_cast<uint32_t*>(wLo + ob) = lo;
        }
      }
      __syncthreads();
    }
    if (isq) {                                   // M = P W
      float m[8][4];
#pragma unroll
      for (int i = 0; i < 8; ++i) { m[i][0] = m[i][1] = m[i][2] = m[i][3] = 0.f; }
#pragma unroll
      for (int ks = 0; ks < 4; ++ks) {
        if (ks > wr) continue;
        uint32_t ph[4], pl[4];
        dc_split(p[2 * ks][0], p[2 * ks][1], ph[0], pl[0]);
        dc_split(p[2 * ks][2], p[2 * ks][3], ph[1], pl[1]);
        dc_split(p[2 * ks + 1][0], p[2 * ks + 1][1], ph[2], pl[2]);
        dc_split(p[2 * ks + 1][2], p[2 * ks + 1][3], ph[3], pl[3]);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          if (np > ks) continue;                 // W is lower triangular
          const int off = dp_piece(ks * 16 + (lane & 15), np * 2 + (lane >> 4));
          uint32_t bh[4], bl[4];
          ldmatrix_x4_trans(bh, wHi + off);
          ldmatrix_x4_trans(bl, wLo + off);
          mma16816<T>(m[2 * np], ph, bh[0], bh[1]);
          mma16816<T>(m[2 * np + 1], ph, bh[2], bh[3]);
          mma16816<T>(m[2 * np], ph, bl[0], bl[1]);
          mma16816<T>(m[2 * np + 1], ph, bl[2], bl[3]);
          mma16816<T>(m[2 * np], pl, bh[0], bh[1]);
          mma16816<T>(m[2 * np + 1], pl, bh[2], bh[3]);
        }
      }
#pragma unroll
      for (int nb = 0; nb < 8; ++nb) {
        uint32_t hi, lo;
        dc_split(m[nb][0], m[nb][1], hi, lo);
        *reinterpret_cast<uint32_t*>(smem + dp_piece(ra, nb) + tq * 4) = hi;
        *reinterpret_cast<uint32_t*>(smem + DC_IMG + dp_piece(ra, nb) + tq * 4) = lo;
        dc_split(m[nb][2], m[nb][3], hi, lo);
        *reinterpret_cast<uint32_t*>(smem + dp_piece(rb, nb) + tq * 4) = hi;
        *reinterpret_cast<uint32_t*>(smem + DC_IMG + dp_piece(rb, nb) + tq * 4) = lo;
      }
    }
    __syncthreads();
#pragma unroll
    for (int i = tid; i < 2 * DC_IMG / 16; i += DP_THREADS) st16(dst + i * 16, ld16(smem + i * 16));
    if (hv + 1 < group) __syncthreads();
  }
}

// ---------------------------------------------------------------------------------------------
// One block per (64 value columns, head, sequence); the blocks of a head form a cluster (the output norm).
// ---------------------------------------------------------------------------------------------
constexpr int DS_THREADS = 448;
constexpr int DS_TMA = 2, DS_MMA = 3;            // warps; a warp reaches the TMEM lanes of the quadrant warp % 4
constexpr int DS_VT = 64;                        // value columns of a block
constexpr int DS_MAX_TILES = 4;
constexpr int DS_BLK = 16384;                    // [Q; K] of 64 dims; 128 state rows x 64 columns
constexpr int DS_HALF = 8192;                    // 64 rows x 64 columns
constexpr uint32_t DS_Z = 0, DS_Y = 64, DS_D = 128, DS_COLS = 256;   // TMEM columns

struct __align__(16) DsShared {
  float factors[2][DC_FACTORS / 4];
  float xs[2][2 * DS_MAX_TILES][64];    // sums of squares of every half tile of the head, by parity
  float norm[DS_VT];
  uint64_t full, ffull[2], vfull, ifull, sready, zfull, rready, yfull, uready, dfull, oread, xbar[2];
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
__device__ __forceinline__ void ds_prefetch(const void* src, uint32_t bytes) {   // into L2
  asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(src), "r"(bytes) : "memory");
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
// a float into the shared memory of a block of the cluster (the same place), counted by that block's barrier: no release
// that would wait for the warp's stores to global memory
__device__ __forceinline__ uint32_t ds_map(const void* p, uint32_t rank) {
  uint32_t ra;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(smem_u32(p)), "r"(rank));
  return ra;
}
__device__ __forceinline__ void ds_push(const float* p, const uint64_t* bar, uint32_t rank, float v) {
  asm volatile("st.async.weak.shared::cluster.mbarrier::complete_tx::bytes.b32 [%0], %1, [%2];"
               ::"r"(ds_map(p, rank)), "r"(__float_as_uint(v)), "r"(ds_map(bar, rank)) : "memory");
}
__device__ __forceinline__ bool ds_wait_cluster(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* error_word, int where) {
  for (uint32_t i = 0; i < WAIT_LIMIT; ++i) {
    uint32_t ok;
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "mbarrier.try_wait.parity.acquire.cluster.shared::cta.b64 p, [%1], %2;\n\t"
        "selp.u32 %0, 1, 0, p;\n\t}"
        : "=r"(ok) : "r"(smem_u32(bar)), "r"(parity) : "memory");
    if (ok) return true;
    if (*abort_flag) return false;
  }
  *abort_flag = 1;
  atomicCAS(error_word, 0, where);
  return false;
}

// every lane of a warp waits; the same answer in all of them
__device__ __forceinline__ bool ds_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* error_word, int where) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, error_word, where));
}

struct DsParams { DeltaArgs a; const unsigned char* ws; int* error_word; };

__global__ void __launch_bounds__(DS_THREADS, 2)
delta_scan_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                     const DsParams p) {
  using T = __nv_bfloat16;
  const DeltaArgs& a = p.a;
  const int vt = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tiles = gridDim.x, c0 = vt * DS_VT;
  const DeltaSeq sq = delta_seq(a, b);
  if (sq.count == 0) return;                               // the same decision in every block of the cluster
  const int nc = (sq.count + DC_C - 1) / DC_C, hk = h / (a.H / a.G);
  extern __shared__ unsigned char smem_raw[];
  unsigned char* qk = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* img = qk + 2 * DS_BLK;                    // hi, lo
  unsigned char* sHi = img + 2 * DC_IMG;                   // state operand; between its product and the next state, the corrections,
  unsigned char* sLo = sHi + DS_BLK;                       // then the updates lie in its first half
  unsigned char *uHi = sHi, *uLo = sHi + DS_HALF;
  unsigned char* vbuf = sLo + DS_BLK;
  DsShared& sh = *reinterpret_cast<DsShared*>(vbuf + DS_HALF);
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x < DS_VT) sh.norm[threadIdx.x] = c0 + (int)threadIdx.x < a.vdim ? a.norm_weight[c0 + threadIdx.x] : 0.f;
  if (threadIdx.x == 0) {
    mbar_init(&sh.full, 2); mbar_init(&sh.vfull, 1); mbar_init(&sh.ifull, 1); mbar_init(&sh.sready, 8); mbar_init(&sh.zfull, 1);
    mbar_init(&sh.rready, 4); mbar_init(&sh.yfull, 1); mbar_init(&sh.uready, 4); mbar_init(&sh.dfull, 1);
    mbar_init(&sh.oread, 4);
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.ffull[i], 1); mbar_init(&sh.xbar[i], 1); }
    sh.abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == DS_TMA) {
    tmem_alloc(&sh.tmem_base, DS_COLS);
    tmem_relinquish();
  }
  fence_before_sync();
  __syncthreads();
  if (tiles > 1) cluster_sync();                           // barriers of every block are ready
  fence_after_sync();
  const uint32_t tmem = sh.tmem_base;
  volatile int* abortp = &sh.abort_flag;
  int* err = p.error_word;

  if (warp == DS_TMA) {
    // a buffer is filled again when what reads it is done: Q with Z, the values with R, the operand with Y, K with D
    if (elect_one()) {
      const unsigned char* ws = p.ws + ((int64_t)delta_first_slot(a, b) * a.H + h) * DC_PER;
      const int64_t step = (int64_t)a.H * DC_PER;
      auto load_q = [&](int c) {
        mbar_arrive_expect_tx(&sh.full, 2 * DS_HALF);
        for (int d = 0; d < 2; ++d) tma_load_5d(qk + d * DS_BLK, &tmQ, &sh.full, d * 64, hk, sq.row0 + c * DC_C, 0, 0);
        mbar_arrive_expect_tx(&sh.ffull[c & 1], DC_FACTORS);
        ds_bulk(sh.factors[c & 1], ws + c * step + 2 * DC_IMG, DC_FACTORS, &sh.ffull[c & 1]);
      };
      auto load_k = [&](int c) {
        mbar_arrive_expect_tx(&sh.full, 2 * DS_HALF);
        for (int d = 0; d < 2; ++d) tma_load_5d(qk + d * DS_BLK + DS_HALF, &tmK, &sh.full, d * 64, hk, sq.row0 + c * DC_C, 0, 0);
      };
      auto load_image = [&](int c) {
        mbar_arrive_expect_tx(&sh.ifull, 2 * DC_IMG);
        ds_bulk(img, ws + c * step, 2 * DC_IMG, &sh.ifull);
      };
      auto load_v = [&](int c) {
        mbar_arrive_expect_tx(&sh.vfull, DS_HALF);
        tma_load_5d(vbuf, &tmV, &sh.vfull, c0, h, sq.row0 + c * DC_C, 0, 0);
      };
      load_q(0);
      load_k(0);
      load_v(0);
      load_image(0);
      for (int c = 0; c + 1 < nc; ++c) {
        for (int d = 0; d < 2; ++d) {
          tma_prefetch_l2_5d(&tmQ, d * 64, hk, sq.row0 + (c + 1) * DC_C, 0, 0);
          tma_prefetch_l2_5d(&tmK, d * 64, hk, sq.row0 + (c + 1) * DC_C, 0, 0);
        }
        tma_prefetch_l2_5d(&tmV, c0, h, sq.row0 + (c + 1) * DC_C, 0, 0);
        ds_prefetch(ws + (c + 1) * step, DC_PER);
        if (!mbar_wait<true>(&sh.zfull, c & 1, abortp, err, 951)) break;
        load_q(c + 1);
        if (!mbar_wait<true>(&sh.rready, c & 1, abortp, err, 950)) break;
        load_v(c + 1);
        if (!mbar_wait<true>(&sh.yfull, c & 1, abortp, err, 952)) break;
        load_image(c + 1);
        if (!mbar_wait<true>(&sh.dfull, c & 1, abortp, err, 953)) break;
        load_k(c + 1);
      }
    }
  } else if (warp == DS_MMA) {
    if (elect_one()) {
      constexpr uint32_t ID = idesc_f16(1, 128, DS_VT), B_MN = 1u << 16, A_MN = 1u << 15;
      const uint32_t shi = smem_u32(sHi), slo = smem_u32(sLo), uhi = smem_u32(uHi), ulo = smem_u32(uLo), im = smem_u32(img), q_ = smem_u32(qk);
      const int ksd = (a.dim + 15) >> 4;         // steps over the key dims
      for (int c = 0; c < nc; ++c) {
        const uint32_t ph = c & 1;
        if (!mbar_wait(&sh.full, ph, abortp, err, 954) || !mbar_wait(&sh.oread, ph ^ 1, abortp, err, 959) ||
            !mbar_wait(&sh.sready, ph, abortp, err, 955)) break;
        fence_after_sync();
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          if (ks >= ksd) continue;
          const uint64_t ad = smem_desc_sw128(q_ + (ks >> 2) * DS_BLK) + 2u * (ks & 3);
          umma_f16(tmem + DS_Z, ad, ds_desc_mn(shi + ks * 2048, DS_BLK), ID | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + DS_Z, ad, ds_desc_mn(slo + ks * 2048, DS_BLK), ID | B_MN, 1u);
        }
        umma_commit(&sh.zfull);
        if (!mbar_wait(&sh.ifull, ph, abortp, err, 956) || !mbar_wait(&sh.rready, ph, abortp, err, 957)) break;
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
        if (!mbar_wait(&sh.uready, ph, abortp, err, 958)) break;
        fence_after_sync();
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
          const uint64_t kt = ds_desc_mn(q_ + DS_HALF + ks * 2048, DS_BLK);
          umma_f16(tmem + DS_D, kt, ds_desc_mn(uhi + ks * 2048, DS_HALF), ID | A_MN | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + DS_D, kt, ds_desc_mn(ulo + ks * 2048, DS_HALF), ID | A_MN | B_MN, 1u);
        }
        umma_commit(&sh.dfull);
      }
    }
  } else if (warp >= 4 && warp < 12) {
    // ---------------- corrections and state ----------------
    const int q = warp & 3, cq = (warp - 4) >> 2;          // lane quadrant; columns cq * 32 .. + 31
    const int r = q * 32 + lane, t = r & 63;               // key dim of the state; token of the chunk
    const bool corr = q >= 2;                              // these rows of Z and Y are corrections
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(q * 32) << 16) + cq * 32;
    const int cols = min(32, a.vdim - c0 - cq * 32);       // (multiples of 8; none may be left)
    bool ok = true;
    // eight columns (chunk i of this thread's 32) of a row as operand, hi and lo
    auto put = [&](const float* v, unsigned char* hi, unsigned char* lo, int row, int i) {
      uint32_t x[4], y[4];
#pragma unroll
      for (int j = 0; j < 4; ++j) dc_split(v[2 * j], v[2 * j + 1], x[j], y[j]);
      const uint32_t off = row * 128 + (((cq * 4 + i) ^ (row & 7)) << 4);
      st16(hi + off, make_int4((int)x[0], (int)x[1], (int)x[2], (int)x[3]));
      st16(lo + off, make_int4((int)y[0], (int)y[1], (int)y[2], (int)y[3]));
    };
    auto publish = [&](uint64_t* bar) {          // operand rows written, accumulators read
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    float s[32];
    float* Sg = a.S + (((int64_t)sq.slot * a.H + h) * a.dim + r) * a.VP + c0 + cq * 32;
    const bool mine = r < a.dim;
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float4 x = (mine && !sq.fresh && i < cols) ? *reinterpret_cast<const float4*>(Sg + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      s[i] = x.x; s[i + 1] = x.y; s[i + 2] = x.z; s[i + 3] = x.w;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) put(s + 8 * i, sHi, sLo, r, i);
    publish(&sh.sready);

    for (int c = 0; c < nc; ++c) {
      const uint32_t ph = c & 1;
      if (!ds_wait(&sh.ffull[ph], (c >> 1) & 1, abortp, err, 966)) { ok = false; break; }
      const float* fac = sh.factors[ph];
      float y[16];
      if (corr) {
        if (!ds_wait(&sh.vfull, ph, abortp, err, 970) || !ds_wait(&sh.zfull, ph, abortp, err, 961)) { ok = false; break; }
        fence_after_sync();
        const float f = fac[64 + t];
        const bool there = c * DC_C + t < sq.count;        // (other rows are another sequence's)
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          ds_ld16(lane_addr + DS_Z + 16 * k, y);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            int4 in = ld16(vbuf + t * 128 + (((cq * 4 + 2 * k + i) ^ (t & 7)) << 4));
            if (!there) in = make_int4(0, 0, 0, 0);
            const __nv_bfloat162* e = reinterpret_cast<const __nv_bfloat162*>(&in);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              const float2 v = __bfloat1622float2(e[j]);
              y[8 * i + 2 * j] = fmaf(-f, y[8 * i + 2 * j], v.x);
              y[8 * i + 2 * j + 1] = fmaf(-f, y[8 * i + 2 * j + 1], v.y);
            }
            put(y + 8 * i, uHi, uLo, t, 2 * k + i);
          }
        }
        publish(&sh.rready);
        if (!ds_wait(&sh.yfull, ph, abortp, err, 962)) { ok = false; break; }
        fence_after_sync();
        const float f1 = fac[128 + t];
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          ds_ld16(lane_addr + DS_Y + 16 * k, y);
#pragma unroll
          for (int i = 0; i < 16; ++i) y[i] *= f1;
          put(y, uHi, uLo, t, 2 * k);
          put(y + 8, uHi, uLo, t, 2 * k + 1);
        }
        publish(&sh.uready);
      }
      const float GC = fac[192];
      if (!ds_wait(&sh.dfull, ph, abortp, err, 963)) { ok = false; break; }
      fence_after_sync();
      const bool more = c + 1 < nc;
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        ds_ld16(lane_addr + DS_D + 16 * k, y);
#pragma unroll
        for (int i = 0; i < 16; ++i) s[16 * k + i] = fmaf(GC, s[16 * k + i], y[i]);
        if (more) {
          put(s + 16 * k, sHi, sLo, r, 2 * k);
          put(s + 16 * k + 8, sHi, sLo, r, 2 * k + 1);
        }
      }
      if (more) publish(&sh.sready);
    }
    if (ok && mine) {
#pragma unroll
      for (int i = 0; i < 32; i += 4)
        if (i < cols) *reinterpret_cast<float4*>(Sg + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
    }
  } else {
    // ---------------- outputs ----------------
    const int q = warp & 3, cq = warp >= 12;               // lane quadrant, 0 or 1
    const int t = q * 32 + lane;                           // token of the chunk
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(q * 32) << 16) + cq * 32;
    const int cols = min(32, a.vdim - c0 - cq * 32);
    const int lrow = q * 32 + (lane & ~3), lcol = (lane & 3) * 8;      // first row and column of what this lane loads and stores
    const T* grow = reinterpret_cast<const T*>(a.gate) + (int64_t)h * a.vdim + c0 + cq * 32 + lcol;
    T* orow = reinterpret_cast<T*>(a.out) + (int64_t)h * a.vdim + c0 + cq * 32 + lcol;
    const float inv_vdim = 1.f / (float)a.vdim;
    for (int c = 0; c < nc; ++c) {
      const uint32_t ph = c & 1;
      const int n = min(DC_C, sq.count - c * DC_C);
      const int64_t row0 = sq.row0 + (int64_t)c * DC_C + lrow;
      if (!ds_wait(&sh.ffull[ph], (c >> 1) & 1, abortp, err, 967)) break;
      const float f = sh.factors[ph][t];
      if (!ds_wait(&sh.zfull, ph, abortp, err, 968)) break;
      fence_after_sync();
      float o[32], y[16], ss = 0.f;
      tmem_ld32(lane_addr + DS_Z, o);
      if (!ds_wait(&sh.yfull, ph, abortp, err, 969)) break;
      fence_after_sync();
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        ds_ld16(lane_addr + DS_Y + 16 * k, y);
#pragma unroll
        for (int i = 0; i < 16; ++i) {                     // (columns past vdim are zero)
          o[16 * k + i] = fmaf(f, o[16 * k + i], y[i]);
          ss = fmaf(o[16 * k + i], o[16 * k + i], ss);
        }
      }
      fence_before_sync();
      if (warp == 0 && lane == 0) mbar_arrive_expect_tx(&sh.xbar[ph], 2 * tiles * 64 * 4);
      for (int k = 0; k < tiles; ++k) ds_push(&sh.xs[ph][2 * vt + cq][t], &sh.xbar[ph], k, ss);
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.oread);
      // the output gate, four lanes per row (lane u of a group: chunk u of the group's rows)
      int4 in[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) in[i] = (lrow + i < n && lcol < cols) ? ld16(grow + (row0 + i) * a.gate_stride) : make_int4(0, 0, 0, 0);
      if (!__all_sync(0xffffffffu, ds_wait_cluster(&sh.xbar[ph], (c >> 1) & 1, abortp, err, 965))) break;
      ss = 0.f;                                            // in one order: every block of the head gets the same sum
      for (int k = 0; k < 2 * tiles; ++k) ss += sh.xs[ph][k][t];
      transpose4(in, lane);                                // to this thread's own row
      const float rr = a.out_scale * rsqrtf(ss * inv_vdim + a.eps);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const __nv_bfloat162* e = reinterpret_cast<const __nv_bfloat162*>(&in[i]);
        uint32_t w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 z = __bfloat1622float2(e[j]);
          const float2 nw = *reinterpret_cast<const float2*>(&sh.norm[cq * 32 + 8 * i + 2 * j]);
          const float x0 = o[8 * i + 2 * j] * rr * nw.x * z.x * ds_rcp(1.f + dc_ex2(-DC_LOG2E * z.x));
          const float x1 = o[8 * i + 2 * j + 1] * rr * nw.y * z.y * ds_rcp(1.f + dc_ex2(-DC_LOG2E * z.y));
          w[j] = pack2<T>(x0, x1);
        }
        in[i] = make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]);
      }
      transpose4(in, lane);
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (lrow + i < n && lcol < cols) st16(orow + (row0 + i) * a.out_stride, in[i]);
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == DS_TMA) {
    fence_after_sync();
    tmem_dealloc(tmem, DS_COLS);
  }
  if (tiles > 1) cluster_sync();                           // no block leaves while a peer may still write to it
}

bool delta_chunk_supports(const DeltaArgs& a, int dtype) {
  return dtype == ZP_DTYPE_BF16 && a.taps == 0 && a.dim <= 128 && a.vdim <= DS_VT * DS_MAX_TILES && a.dim % 8 == 0 && a.vdim % 8 == 0 &&
         a.x_stride % 8 == 0 && a.gate_stride % 8 == 0 && a.out_stride % 8 == 0 &&
         ((uintptr_t)a.x | (uintptr_t)a.gate | (uintptr_t)a.out) % 16 == 0;
}
size_t delta_chunk_workspace(int total_rows, int B, int H) { return (size_t)delta_slots(total_rows, B) * H * DC_PER; }

template <int DP> static int launch_prepare(const DeltaArgs& a, int slots, unsigned char* ws, cudaStream_t st) {
  constexpr int smem = PrepSmem<DP>::TOTAL;
  cudaError_t e = cudaFuncSetAttribute(delta_prepare_kernel<DP>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_gated_delta(prepare): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  delta_prepare_kernel<DP><<<dim3(slots, a.G), DP_THREADS, smem, st>>>(a, ws);
  return check_launch("zp_gated_delta(prepare)");
}

// total_rows: rows of x, of which the portions' are the rows from cu_q[0] on
int delta_chunk(const DeltaArgs& a, int total_rows, void* workspace, cudaStream_t st) {
  DsParams p{a, (const unsigned char*)workspace, device_error_word()};
  if (!p.error_word) { set_error("zp_gated_delta(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  CUtensorMap tm[3];                             // queries, keys, values
  for (int i = 0; i < 3; ++i) {
    const uint64_t rs = (uint64_t)a.x_stride, width = i == 2 ? a.vdim : a.dim;
    const uint64_t dims[5] = {width, (uint64_t)(i == 2 ? a.H : a.G), (uint64_t)total_rows, 1, 1};
    const uint64_t strides[4] = {width, rs, rs * total_rows, rs * total_rows};
    const uint32_t box[5] = {64, 1, 64, 1, 1};
    const __nv_bfloat16* base = (const __nv_bfloat16*)a.x + (int64_t)i * a.G * a.dim;
    if (int rc = make_tensor_map_5d(&tm[i], UmmaFmt<__nv_bfloat16>::tm, base, dims, strides, box, 2)) return rc;
  }
  const int slots = delta_slots(total_rows, a.B);
  if (int rc = a.dim <= 64 ? launch_prepare<64>(a, slots, (unsigned char*)workspace, st)
                           : launch_prepare<128>(a, slots, (unsigned char*)workspace, st)) return rc;
  const int smem = 1024 + 4 * DS_BLK + 2 * DC_IMG + DS_HALF + (int)sizeof(DsShared);
  static_assert(2 * (1024 + 4 * DS_BLK + 2 * DC_IMG + DS_HALF + sizeof(DsShared) + 1024) <= 233472, "two blocks share an SM");
  cudaError_t e = cudaFuncSetAttribute(delta_scan_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_gated_delta(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  const int tiles = (a.vdim + DS_VT - 1) / DS_VT;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles, a.H, a.B);
  cfg.blockDim = dim3(DS_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = tiles; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  e = cudaLaunchKernelEx(&cfg, delta_scan_tc_kernel, tm[0], tm[1], tm[2], p);
  if (e != cudaSuccess) { set_error("zp_gated_delta(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  return check_launch("zp_gated_delta(tcgen05)");
}

}  // namespace zp
