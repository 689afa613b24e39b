// Matrix-memory (mLSTM) mixer over prompt portions, 64 tokens at a time on warp-level tensor-core MMAs
// (bf16 projections, fp32 state).
//
// With F_t the running sum of the log forget gates inside a chunk, u_j = i_j - F_j and
// M_t = max(m, max_{j<=t} u_j) (m: the running maximum the chunk starts from), the recurrence unrolls to
//   m_t = M_t + F_t
//   S_t^T q = exp(m - M_t) S^T q + sum_{j<=t} exp(u_j - M_t) (k_j . q) v_j
// and the state after the chunk is exp(m - M_C) S + sum_j exp(u_j - M_C) k_j v_j^T; every exponent is
// <= 0.  n is one more value column whose v is 1.
//
// One block per (64-wide value tile, head, sequence) walks the chunks in order.  Its state tile
// [dim, 64 + 1] stays in fp32 MMA accumulators; only 16-bit operand copies of it pass through shared
// memory.  Whatever is fp32 in the equations enters a product as a pair of bf16 numbers (hi + lo): the state
// in S^T q, the decayed scores, and the decayed values of the state update; q, k and v are bf16
// already.  The blocks of a head form a cluster and exchange per-row sums of squares for the head norm
// through distributed shared memory, so the normalised, gated output leaves the kernel in one pass.
#include <type_traits>

#include "zp_mlstm.cuh"
#include "zp_mma.cuh"

namespace zp {

constexpr int MC_THREADS = 256;
constexpr int MC_C = 64;            // tokens per chunk
constexpr int MC_VT = 64;           // value columns per block
constexpr float MC_LOG2E = 1.4426950408889634f;
constexpr int MC_RB = 144;          // bytes of a 72-column bf16 row (an odd number of 16-byte chunks)

__device__ __forceinline__ float exp2_(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rcp_approx(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack2<__nv_bfloat16>(a - f.x, b - f.y);
}
__device__ __forceinline__ void ldmatrix_x2_trans(uint32_t (&r)[2], const void* smem_row) {
  const uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(smem_row));
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(a));
}

// B fragments of the 8-column blocks [first, first + 5) (or + 4) of 16 rows of a 72-column tile
template <typename F>
__device__ __forceinline__ void for_blocks(const unsigned char* tile, int row0, int half, int lane, F&& fn) {
  const unsigned char* r = tile + (row0 + (lane & 15)) * MC_RB;
  uint32_t b[4];
  ldmatrix_x4_trans(b, r + half * 64 + (lane >> 4) * 16);
  fn(0, b[0], b[1]); fn(1, b[2], b[3]);
  ldmatrix_x4_trans(b, r + half * 64 + 32 + (lane >> 4) * 16);
  fn(2, b[0], b[1]); fn(3, b[2], b[3]);
  if (half) {
    uint32_t c[2];
    ldmatrix_x2_trans(c, r + 128);
    fn(4, c[0], c[1]);
  }
}

// Shared memory, bytes: Q and K tiles, V tile, hi and lo of the state tile, hi and lo of the scores
// (reused by the decayed values), the output gate's tile, per-row floats.  A chunk's tiles are requested as
// soon as the previous chunk has no more use for their place.
template <int DP> struct ChunkSmem {
  static constexpr int RB = DP * 2 + 16;
  static constexpr int Q = 0, K = Q + MC_C * RB, V = K + MC_C * RB, S = V + MC_C * MC_RB, P = S + 2 * DP * MC_RB,
                       G = P + 2 * MC_C * MC_RB, F = G + MC_C * MC_RB, TOTAL = F + 25 * MC_C * 4;
};

template <int DP>
__global__ void __launch_bounds__(MC_THREADS, DP <= 128 ? 2 : 1) mlstm_chunk_kernel(const MlstmArgs a) {
  using T = __nv_bfloat16;
  using L = ChunkSmem<DP>;
  constexpr int MB = DP / 64;                    // 16-row blocks of the state tile per warp
  extern __shared__ __align__(128) unsigned char smem[];
  const int vt = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const MlstmSeq sq = mlstm_seq(a, b);
  if (sq.count == 0) return;                     // the same decision in every block of the cluster
  const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int rg = warp & 3, half = warp >> 2;     // 16-row group, column half of every product
  unsigned char *sQ = smem + L::Q, *sK = smem + L::K, *sV = smem + L::V;
  unsigned char *sSh = smem + L::S, *sSl = sSh + DP * MC_RB;
  unsigned char *sPh = smem + L::P, *sPl = sPh + MC_C * MC_RB;
  float* fl = reinterpret_cast<float*>(smem + L::F);
  float *sDen = fl + 320, *sR = fl + 384;
  float* sScan = fl + 896;                       // [2 parities][M, u, A, E, W][64]: see scan()
  float *sSq = fl + 448;                         // [2 parities][2 halves][64] (read by the cluster)
  float *sMisc = fl + 704;                       // running maximum, decay of the state over the chunk
  float* sAct = fl + 768;                        // log input gates, log forget gates of the chunk
  float* sNorm = fl + 1536;                      // norm weights of the value tile
  unsigned char* sG = smem + L::G;
  const int c0 = vt * MC_VT, vcols = min(MC_VT, a.vdim - c0);
  const int64_t head = (int64_t)sq.slot * a.H + h;
  const T* qb = reinterpret_cast<const T*>(a.q) + (int64_t)h * a.dim;
  const T* kb = reinterpret_cast<const T*>(a.k) + (int64_t)h * a.dim;
  const T* vb = reinterpret_cast<const T*>(a.v) + (int64_t)h * a.vdim + c0;
  const T* gb = reinterpret_cast<const T*>(a.g) + (int64_t)h * a.vdim + c0;
  const bool vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.row_stride % 8 == 0 &&
                   ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.g) % 16 == 0;

  // columns 64..71 of the value tile: the column of ones that carries n, then zeros
  for (int i = tid; i < MC_C * 8; i += MC_THREADS)
    *reinterpret_cast<T*>(sV + (i >> 3) * MC_RB + 128 + (i & 7) * 2) = Elem<T>::from_f32((i & 7) == 0 ? 1.f : 0.f);
  if (tid == 0) sMisc[0] = sq.fresh ? 0.f : a.m[head];

  float s[MB][5][4];                             // the state tile: rows (rg + 4 i) * 16 + g (+ 8)
#pragma unroll
  for (int i = 0; i < MB; ++i)
#pragma unroll
    for (int cb = 0; cb < 5; ++cb)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = (rg + 4 * i) * 16 + g + (j >> 1) * 8, c = half * 32 + cb * 8 + 2 * tq + (j & 1);
        float x = 0.f;
        if (!sq.fresh && r < a.dim) {
          if (cb < 4) { if (c0 + c < a.VP) x = a.S[(head * a.dim + r) * a.VP + c0 + c]; }
          else if (c == 64) x = a.n[head * a.dim + r];
        }
        s[i][cb][j] = x;
      }

  using Wide = std::integral_constant<int, DP>;
  using Narrow = std::integral_constant<int, MC_VT>;
  // tiles of the chunk that starts at token t0 (n tokens; none: only the group is committed)
  auto load_tile = [&](auto width, const T* base, unsigned char* dst, int valid_cols, int t0, int n) {
    constexpr int cols16 = decltype(width)::value / 8, rb = decltype(width)::value == DP ? L::RB : MC_RB;
    const int64_t row0 = sq.row0 + t0;
    if (n > 0) {
      if (vec) {
        _Pragma("unroll")
        for (int i = tid; i < MC_C * cols16; i += MC_THREADS) {
          const int r = i / cols16, c = i % cols16;
          const int ok = (r < n && c * 8 < valid_cols) ? 16 : 0;
          cp_async16(dst + r * rb + c * 16, base + (ok ? (row0 + r) * a.row_stride + c * 8 : 0), ok);
        }
      } else {
        for (int i = tid; i < MC_C * cols16 * 8; i += MC_THREADS) {
          const int r = i / (cols16 * 8), c = i % (cols16 * 8);
          *reinterpret_cast<T*>(dst + r * rb + c * 2) =
              (r < n && c < valid_cols) ? base[(row0 + r) * a.row_stride + c] : Elem<T>::from_f32(0.f);
        }
      }
    }
    cp_async_commit();
  };
  // Gate pre-activation of token t0 + (tid & 63): threads 0-63 input gates, 64-127 forget gates.
  auto gate_raw = [&](int t0, int n) -> float {
    const int t = tid & 63;
    return (tid < 128 && t < n) ? a.gates[(sq.row0 + t0 + t) * a.gates_stride + (tid >> 6) * a.H + h] : 0.f;
  };
  const float gate_bias = tid < 128 ? a.gate_bias[(tid >> 6) * a.H + h] : 0.f;
  auto gate_put = [&](float raw, int n) {
    if (tid < 128) {
      const float x = soft_cap(raw + gate_bias, a.cap);
      sAct[tid] = (tid & 63) < n ? (tid < 64 ? x : log_sigmoid(x)) : (tid < 64 ? -INFINITY : 0.f);
    }
  };
  // one warp: running sums and maxima of the chunk's gates (two tokens per lane)
  const float log2_qscale = log2f(a.qscale);
  auto scan = [&](int par) {
    float *sM = sScan + par * 320, *sU = sM + 64, *sA = sM + 128, *sE = sM + 192, *sW = sM + 256;
    float f[2] = {sAct[64 + 2 * lane], sAct[65 + 2 * lane]}, u[2] = {sAct[2 * lane], sAct[2 * lane + 1]};
    float F = f[0] + f[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, F, o); if (lane >= o) F += x; }
    const float F1 = F, F0 = F - f[1];
    u[0] -= F0; u[1] -= F1;
    float mx = fmaxf(u[0], u[1]);
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, mx, o); if (lane >= o) mx = fmaxf(mx, x); }
    float before = __shfl_up_sync(0xffffffffu, mx, 1);
    const float m = sMisc[0];
    before = lane == 0 ? m : fmaxf(m, before);
    const float M0 = fmaxf(before, u[0]), M1 = fmaxf(M0, u[1]);
    const float MC = __shfl_sync(0xffffffffu, M1, 31), FC = __shfl_sync(0xffffffffu, F1, 31);
    const int t = 2 * lane;
    // (exponents in log2 units, the query scale folded into the row's)
    sM[t] = fmaf(M0, MC_LOG2E, -log2_qscale); sM[t + 1] = fmaf(M1, MC_LOG2E, -log2_qscale);
    sU[t] = u[0] * MC_LOG2E; sU[t + 1] = u[1] * MC_LOG2E;
    sA[t] = expf(m - M0) * a.qscale; sA[t + 1] = expf(m - M1) * a.qscale;
    sE[t] = expf(-(M0 + F0)); sE[t + 1] = expf(-(M1 + F1));
    sW[t] = expf(u[0] - MC); sW[t + 1] = expf(u[1] - MC);
    __syncwarp();
    if (lane == 0) { sMisc[1 + par] = expf(m - MC); sMisc[0] = MC + FC; }
  };

  {
    const int n = min(MC_C, sq.count);
    load_tile(Wide{}, qb, sQ, a.dim, 0, n);
    load_tile(Wide{}, kb, sK, a.dim, 0, n);
    load_tile(Narrow{}, vb, sV, vcols, 0, n);
    gate_put(gate_raw(0, n), n);
    for (int i = tid; i < MC_VT; i += MC_THREADS) sNorm[i] = i < vcols ? a.norm_weight[(int64_t)h * a.vdim + c0 + i] : 0.f;
    __syncthreads();
    if (warp == 0) scan(0);
    __syncthreads();
    const int n1 = min(MC_C, sq.count - MC_C);
    gate_put(gate_raw(MC_C, n1), n1);
  }
  __syncthreads();
  const float inv_vdim = 1.f / (float)a.vdim;
  const int row_a = rg * 16 + g, row_b = row_a + 8;   // this thread's two tokens of the chunk
  for (int t0 = 0, par = 0; t0 < sq.count; t0 += MC_C, par ^= 1) {
    const int n = min(MC_C, sq.count - t0), t1 = t0 + MC_C, n1 = min(MC_C, sq.count - t1);   // n1 <= 0: the last one
    const int t2 = t1 + MC_C, n2 = min(MC_C, sq.count - t2);
    const float raw_next = gate_raw(t2, n2);           // (used two chunks ahead)
    const float *sM = sScan + par * 320, *sU = sM + 64, *sA = sM + 128, *sE = sM + 192, *sW = sM + 256;
    // 16-bit operand copies of the state tile
#pragma unroll
    for (int i = 0; i < MB; ++i)
#pragma unroll
      for (int cb = 0; cb < 5; ++cb) {
        if (cb == 4 && !half) continue;
        const int r = (rg + 4 * i) * 16 + g, off = (half * 32 + cb * 8 + 2 * tq) * 2;
        uint32_t hi, lo;
        split_bf16(s[i][cb][0], s[i][cb][1], hi, lo);
        *reinterpret_cast<uint32_t*>(sSh + r * MC_RB + off) = hi;
        *reinterpret_cast<uint32_t*>(sSl + r * MC_RB + off) = lo;
        split_bf16(s[i][cb][2], s[i][cb][3], hi, lo);
        *reinterpret_cast<uint32_t*>(sSh + (r + 8) * MC_RB + off) = hi;
        *reinterpret_cast<uint32_t*>(sSl + (r + 8) * MC_RB + off) = lo;
      }
    cp_async_wait<0>();
    __syncthreads();
    load_tile(Narrow{}, gb, sG, vcols, t0, n);

    float acc[5][4], p[4][4];
#pragma unroll
    for (int i = 0; i < 5; ++i) { acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f; }
#pragma unroll
    for (int i = 0; i < 4; ++i) { p[i][0] = p[i][1] = p[i][2] = p[i][3] = 0.f; }
    const bool scores = half * 32 <= rg * 16 + 15;     // else every key of this half is later than the rows
#pragma unroll
    for (int kk = 0; kk < DP / 16; ++kk) {
      uint32_t qa[4];
      ldmatrix_x4(qa, sQ + (rg * 16 + (lane & 15)) * L::RB + kk * 32 + (lane >> 4) * 16);
      for_blocks(sSh, kk * 16, half, lane, [&](int i, uint32_t b0, uint32_t b1) { mma16816<T>(acc[i], qa, b0, b1); });
      for_blocks(sSl, kk * 16, half, lane, [&](int i, uint32_t b0, uint32_t b1) { mma16816<T>(acc[i], qa, b0, b1); });
      if (scores) {
#pragma unroll
        for (int np = 0; np < 2; ++np) {
          uint32_t bf[4];
          ldmatrix_x4(bf, sK + (half * 32 + np * 16 + (lane & 7) + (lane >> 4) * 8) * L::RB + kk * 32 + ((lane >> 3) & 1) * 16);
          mma16816<T>(p[2 * np], qa, bf[0], bf[1]);
          mma16816<T>(p[2 * np + 1], qa, bf[2], bf[3]);
        }
      }
    }
    if (scores) {
      const float Ma = sM[row_a], Mb = sM[row_b];
#pragma unroll
      for (int nb = 0; nb < 4; ++nb) {
        const int key = half * 32 + nb * 8 + 2 * tq;
        const float2 u = *reinterpret_cast<const float2*>(sU + key);
        const float p0 = key <= row_a ? p[nb][0] * exp2_(u.x - Ma) : 0.f;
        const float p1 = key + 1 <= row_a ? p[nb][1] * exp2_(u.y - Ma) : 0.f;
        const float p2 = key <= row_b ? p[nb][2] * exp2_(u.x - Mb) : 0.f;
        const float p3 = key + 1 <= row_b ? p[nb][3] * exp2_(u.y - Mb) : 0.f;
        uint32_t hi, lo;
        split_bf16(p0, p1, hi, lo);
        *reinterpret_cast<uint32_t*>(sPh + row_a * MC_RB + key * 2) = hi;
        *reinterpret_cast<uint32_t*>(sPl + row_a * MC_RB + key * 2) = lo;
        split_bf16(p2, p3, hi, lo);
        *reinterpret_cast<uint32_t*>(sPh + row_b * MC_RB + key * 2) = hi;
        *reinterpret_cast<uint32_t*>(sPl + row_b * MC_RB + key * 2) = lo;
      }
    }
    else if (warp == 4) scan(par ^ 1);                 // a warp without scores prepares the next chunk's gates
    {
      const float fa = sA[row_a], fb = sA[row_b];
#pragma unroll
      for (int i = 0; i < 5; ++i) { acc[i][0] *= fa; acc[i][1] *= fa; acc[i][2] *= fb; acc[i][3] *= fb; }
    }
    __syncthreads();
    load_tile(Wide{}, qb, sQ, a.dim, t1, n1);
#pragma unroll
    for (int kk = 0; kk < MC_C / 16; ++kk) {           // keys 16 kk .. 16 kk + 15 of rows up to 16 rg + 15
      if (kk > rg) break;
      uint32_t ph[4], pl[4];
      ldmatrix_x4(ph, sPh + (rg * 16 + (lane & 15)) * MC_RB + kk * 32 + (lane >> 4) * 16);
      ldmatrix_x4(pl, sPl + (rg * 16 + (lane & 15)) * MC_RB + kk * 32 + (lane >> 4) * 16);
      for_blocks(sV, kk * 16, half, lane, [&](int i, uint32_t b0, uint32_t b1) {
        mma16816<T>(acc[i], ph, b0, b1);
        mma16816<T>(acc[i], pl, b0, b1);
      });
    }
    if (half && tq == 0) { sDen[row_a] = acc[4][0]; sDen[row_b] = acc[4][2]; }   // n . q, decayed like the rest
    __syncthreads();
    const float da = rcp_approx(fmaxf(fabsf(sDen[row_a]), sE[row_a]) + MLSTM_DEN_EPS);
    const float db = rcp_approx(fmaxf(fabsf(sDen[row_b]), sE[row_b]) + MLSTM_DEN_EPS);
    float qa2 = 0.f, qb2 = 0.f;
#pragma unroll
    for (int i = 0; i < 4; ++i) {                      // (columns past vdim are zero)
      acc[i][0] *= da; acc[i][1] *= da; acc[i][2] *= db; acc[i][3] *= db;
      qa2 = fmaf(acc[i][0], acc[i][0], fmaf(acc[i][1], acc[i][1], qa2));
      qb2 = fmaf(acc[i][2], acc[i][2], fmaf(acc[i][3], acc[i][3], qb2));
    }
    qa2 += __shfl_xor_sync(0xffffffffu, qa2, 1); qa2 += __shfl_xor_sync(0xffffffffu, qa2, 2);
    qb2 += __shfl_xor_sync(0xffffffffu, qb2, 1); qb2 += __shfl_xor_sync(0xffffffffu, qb2, 2);
    if (tq == 0) { sSq[(par * 2 + half) * 64 + row_a] = qa2; sSq[(par * 2 + half) * 64 + row_b] = qb2; }
    // decayed values (and the decayed column of ones), over the scores' shared memory
    const float w = sW[tid >> 2];
#pragma unroll
    for (int i = 0; i < 9; ++i) {
      const int r = tid >> 2, c = (tid & 3) + 4 * i;
      const float2 v = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sV + r * MC_RB + c * 4));
      uint32_t hi, lo;
      split_bf16(v.x * w, v.y * w, hi, lo);
      *reinterpret_cast<uint32_t*>(sPh + r * MC_RB + c * 4) = hi;
      *reinterpret_cast<uint32_t*>(sPl + r * MC_RB + c * 4) = lo;
    }
    if (cluster_size() > 1) cluster_sync(); else __syncthreads();
    load_tile(Narrow{}, vb, sV, vcols, t1, n1);
    gate_put(raw_next, n2);
    if (tid < MC_C) {
      float ss = 0.f;
      for (uint32_t r = 0; r < cluster_size(); ++r)
        ss += ld_cluster(&sSq[par * 128 + tid], r) + ld_cluster(&sSq[par * 128 + 64 + tid], r);
      sR[tid] = rsqrtf(ss * inv_vdim + a.eps);
    }
    const float decay = sMisc[1 + par];
#pragma unroll
    for (int i = 0; i < MB; ++i) {
      if ((rg + 4 * i) * 16 < a.dim) {
#pragma unroll
        for (int cb = 0; cb < 5; ++cb) { s[i][cb][0] *= decay; s[i][cb][1] *= decay; s[i][cb][2] *= decay; s[i][cb][3] *= decay; }
      }
    }
#pragma unroll
    for (int kk = 0; kk < MC_C / 16; ++kk) {
      if (kk * 16 >= n) break;
      uint32_t ka[MB][4];
#pragma unroll
      for (int i = 0; i < MB; ++i)
        ldmatrix_x4_trans(ka[i], sK + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * L::RB + (rg + 4 * i) * 32 + ((lane >> 3) & 1) * 16);
      auto add = [&](int cb, uint32_t b0, uint32_t b1) {
#pragma unroll
        for (int i = 0; i < MB; ++i) mma16816<T>(s[i][cb], ka[i], b0, b1);
      };
      for_blocks(sPh, kk * 16, half, lane, add);
      for_blocks(sPl, kk * 16, half, lane, add);
    }
    cp_async_wait<2>();                                // the gate tile (two younger groups: the next Q and V)
    __syncthreads();                                   // K free for the next chunk; sR visible
    load_tile(Wide{}, kb, sK, a.dim, t1, n1);
    const float ra = sR[row_a], rb = sR[row_b];
    const int64_t grow = sq.row0 + t0;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int c = c0 + half * 32 + i * 8 + 2 * tq;
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        const int r = y ? row_b : row_a;
        if (r >= n) continue;
        const float rr = y ? rb : ra;
        const int64_t e = (int64_t)h * a.vdim + c;
        const float2 gv = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(sG + r * MC_RB + (half * 32 + i * 8 + 2 * tq) * 2));
        T* op = reinterpret_cast<T*>(a.out) + (grow + r) * a.out_stride + e;
        const float2 nw = *reinterpret_cast<const float2*>(sNorm + half * 32 + i * 8 + 2 * tq);
        const float o[2] = {acc[i][2 * y] * rr * nw.x * rcp_approx(1.f + exp2_(-MC_LOG2E * gv.x)),
                            acc[i][2 * y + 1] * rr * nw.y * rcp_approx(1.f + exp2_(-MC_LOG2E * gv.y))};
        if (vec && a.out_stride % 2 == 0) { if (c < a.vdim) *reinterpret_cast<uint32_t*>(op) = pack2<T>(o[0], o[1]); }
        else {
          if (c < a.vdim) op[0] = Elem<T>::from_f32(o[0]);
          if (c + 1 < a.vdim) op[1] = Elem<T>::from_f32(o[1]);
        }
      }
    }
  }

  if (cluster_size() > 1) cluster_sync();              // peers may still be reading this block's sums
#pragma unroll
  for (int i = 0; i < MB; ++i)
#pragma unroll
    for (int cb = 0; cb < 5; ++cb)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = (rg + 4 * i) * 16 + g + (j >> 1) * 8, c = half * 32 + cb * 8 + 2 * tq + (j & 1);
        if (r >= a.dim) continue;
        if (cb < 4) { if (c0 + c < a.VP) a.S[(head * a.dim + r) * a.VP + c0 + c] = s[i][cb][j]; }
        else if (c == 64 && vt == 0) a.n[head * a.dim + r] = s[i][cb][j];
      }
  if (vt == 0 && tid == 0) a.m[head] = sMisc[0];
}

bool mlstm_chunk_supports(const MlstmArgs& a, int dtype) {
  return dtype == ZP_DTYPE_BF16 && a.dim <= 256 && a.vdim <= 8 * MC_VT;
}

template <int DP>
static int launch_chunk(const MlstmArgs& a, cudaStream_t st) {
  auto kern = mlstm_chunk_kernel<DP>;
  constexpr int smem = ChunkSmem<DP>::TOTAL;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_mlstm(chunk): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  const int tiles = (a.vdim + MC_VT - 1) / MC_VT;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles, a.H, a.B);
  cfg.blockDim = dim3(MC_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = tiles; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  e = cudaLaunchKernelEx(&cfg, kern, a);
  if (e != cudaSuccess) { set_error("zp_mlstm(chunk): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  return check_launch("zp_mlstm(chunk)");
}

int mlstm_chunk(const MlstmArgs& a, cudaStream_t st) {
  if (a.dim <= 64) return launch_chunk<64>(a, st);
  if (a.dim <= 128) return launch_chunk<128>(a, st);
  return launch_chunk<256>(a, st);
}

}  // namespace zp
