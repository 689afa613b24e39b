// Prefill attention with masks (sliding window, chunks), soft cap, sink and output gate on tcgen05 tensor cores:
// bf16, key and value sizes up to 128, paged caches (page size a multiple of 64).
//
// One pass over the visible 128-key tiles:
//   S = Q K^T (M = 128 queries, N = 128 keys, K = 128 dims), accumulated in TMEM,
//   p = exp(score - reference) in fp32, split into two bf16 numbers (hi + lo) in TMEM,
//   O += P_hi V + P_lo V (V is the B operand as it lies in memory: MN-major), accumulated in TMEM,
// and out = O / (row sum + sink's term) * gate.  The reference: a soft cap bounds every score, so it is fixed (the
// cap, or 0; see zp_window_attn_mma.cu) and nothing is ever rescaled; without a cap it is one number per row
// that moves, and O with it, only when a score exceeds it by more than 2^40, which fp32 sums and bf16 pairs
// carry without loss, so nearly always in the first tile only.
//
// Roles (576 threads, one block per SM): warp 0 = TMA producer and TMEM owner, warp 1 = MMA issuer, warps
// 2-17 = softmax (thread <-> TMEM lane <-> query row; the four warps of a lane quadrant split a tile's
// 128 columns).  Shared memory: the Q tile and a ring of five 32 KB K/V stages; TMEM: two S
// accumulators, O, P_hi and P_lo (all 512 columns).  A tile is two 64-key boxes per 64 dims, so its halves
// may lie in different pages; head sizes below 128 are filled with zeros by TMA.  The capped softmax is bound by the
// special-function unit: two exponentials and a reciprocal per score; four reciprocals share one instruction,
// 1/a = bcd / (abcd).
// Every wait is bounded; after it the block raises the device error word and leaves.
#include "zp_tc.cuh"
#include "zp_window_attn.cuh"

namespace zp {

using namespace tc;

constexpr int WT_THREADS = 576;
constexpr int WT_TILE = 32768;     // 128 rows x 128 elements x 2 bytes
constexpr int WT_BLK = 16384;      // one 64-element block of a tile
constexpr int WT_NRING = 5;
constexpr uint32_t WT_O = 256, WT_PHI = 384, WT_PLO = 448;   // TMEM columns after the two S tiles

struct __align__(16) WtShared {
  uint64_t qfull, full[WT_NRING], empty[WT_NRING], sfull[2], sempty[2], pfull, pempty, ofull, sbar;
  float stat[4][128];
  uint32_t tmem_base;
  int abort_flag;
};

// MN-major operand tile, 128-byte swizzle: 64 contiguous elements per K row, 8-row groups `sbo` bytes
// apart along K, the next 64 elements along MN `lbo` bytes away
__device__ __forceinline__ uint64_t desc_mn(uint32_t smem_addr, uint32_t lbo, uint32_t sbo) {
  const uint32_t lo = ((smem_addr >> 4) & 0x3FFFu) | ((lbo >> 4) << 16);
  const uint32_t hi = (sbo >> 4) | (1u << 14) | (2u << 29);
  return (static_cast<uint64_t>(hi) << 32) | lo;
}
__device__ __forceinline__ void umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ void tmem_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ float ex2_(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rcp_(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// four raw products -> exp2(-2c / (1 + exp2(y s)) + off).  The exponent is held at 30: beyond, 1 / (1 + E) is below
// 2^-30 and the weight is 1 to fp32 accuracy, and the product of four stays finite.
__device__ __forceinline__ void weights4(const uint32_t* s, float y, float m2c, float off, float (&p)[4]) {
  float a[4];
#pragma unroll
  for (int i = 0; i < 4; ++i) a[i] = 1.f + ex2_(fminf(__uint_as_float(s[i]) * y, 30.f));
  const float2 ab_cd = fmul2(make_float2(a[0], a[2]), make_float2(a[1], a[3]));
  const float r = rcp_(ab_cd.x * ab_cd.y) * m2c;
  const float2 rr = fmul2(make_float2(ab_cd.y, ab_cd.x), make_float2(r, r));      // m2c / ab, m2c / cd
  const float2 lo = fmul2(make_float2(rr.x, rr.x), make_float2(a[1], a[0]));
  const float2 hi = fmul2(make_float2(rr.y, rr.y), make_float2(a[3], a[2]));
  p[0] = ex2_(lo.x + off); p[1] = ex2_(lo.y + off); p[2] = ex2_(hi.x + off); p[3] = ex2_(hi.y + off);
}

// meeting of the 128 threads of a lane quadrant (barriers 1-4); true when any of them brings true
__device__ __forceinline__ bool wt_meet_any(int q, bool v) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, r;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred r, %2, 128, p;\n\t"
      "selp.u32 %0, 1, 0, r;\n\t}"
      : "=r"(out) : "r"((uint32_t)v), "r"(q + 1) : "memory");
  return out != 0;
}
__device__ __forceinline__ void wt_st32(uint32_t taddr, const uint32_t (&r)[32]) {
  uint32_t x[16], y[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) { x[i] = r[i]; y[i] = r[16 + i]; }
  tmem_st16(taddr, x);
  tmem_st16(taddr + 16, y);
}
constexpr float WT_LAZY = 40.f;    // log2 units

struct WtParams { WinArgs a; int* error_word; };

template <bool CAPPED, bool SLOPED>   // (not both)
__global__ void __launch_bounds__(WT_THREADS, 1)
window_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                         const __grid_constant__ CUtensorMap tmV, const WtParams p) {
  using T = __nv_bfloat16;
  const WinArgs& a = p.a;
  const int b = blockIdx.z, h = blockIdx.y;
  const WinSeq sq = win_seq(a, b);
  const int nqt = (sq.count + 127) >> 7;
  if ((int)blockIdx.x >= nqt) return;
  const int qi0 = (nqt - 1 - blockIdx.x) * 128;      // the tiles with the most keys start first
  const int hk = h / (a.Hq / a.Hkv);
  const int rows = min(128, sq.count - qi0);
  const int p_first = sq.pos0 + qi0, p_last = p_first + rows - 1;
  const WinTiles wt = win_tiles(a, p_first, p_last, 128);
  const int n = wt.n;                                // 128-key tiles

  extern __shared__ unsigned char smem_raw[];
  unsigned char* qbuf = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* ring = qbuf + WT_TILE;
  WtShared& sh = *reinterpret_cast<WtShared*>(ring + WT_NRING * WT_TILE);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&sh.qfull, 1);
    for (int i = 0; i < WT_NRING; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.sfull[i], 1); mbar_init(&sh.sempty[i], 16); }
    mbar_init(&sh.pfull, 16);
    mbar_init(&sh.pempty, 1);
    mbar_init(&sh.ofull, 1);
    mbar_init(&sh.sbar, 16);
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
  const uint32_t tmem_base = sh.tmem_base;
  volatile int* abortp = &sh.abort_flag;
  constexpr uint32_t IDESC_QK = idesc_f16(1, 128, 128);
  constexpr uint32_t IDESC_PV = IDESC_QK | (1u << 16);   // B operand MN-major

  // ring positions: K_j -> 2j, V_j -> 2j + 1
  if (warp == 0) {
    if (lane == 0) {
      prefetch_tensormap(&tmQ);
      prefetch_tensormap(&tmK);
      prefetch_tensormap(&tmV);
      mbar_arrive_expect_tx(&sh.qfull, WT_TILE);
      tma_load_5d(qbuf, &tmQ, &sh.qfull, 0, h, sq.row0 + qi0, 0, 0);
      tma_load_5d(qbuf + WT_BLK, &tmQ, &sh.qfull, 64, h, sq.row0 + qi0, 0, 0);
      bool ok = true;
      for (int j = 0; ok && j < n; ++j) {
        const int key0 = wt.tile(j) * 128;
        const int pg0 = win_page(a, b, key0), pg1 = win_page(a, b, key0 + 64);
        for (int kv = 0; kv < 2; ++kv) {
          const int t = 2 * j + kv, s = t % WT_NRING, k = t / WT_NRING;
          if (!mbar_wait<true>(&sh.empty[s], (k & 1) ^ 1, abortp, p.error_word, 801)) { ok = false; break; }
          const CUtensorMap* tm = kv ? &tmV : &tmK;
          unsigned char* dst = ring + s * WT_TILE;
          mbar_arrive_expect_tx(&sh.full[s], WT_TILE);
#pragma unroll
          for (int d = 0; d < 2; ++d) {
            tma_load_5d(dst + d * WT_BLK, tm, &sh.full[s], d * 64, hk, key0 % a.BS, pg0, 0);
            tma_load_5d(dst + d * WT_BLK + 8192, tm, &sh.full[s], d * 64, hk, (key0 + 64) % a.BS, pg1, 0);
          }
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      bool ok = mbar_wait(&sh.qfull, 0, abortp, p.error_word, 802);
      const uint32_t q_addr = smem_u32(qbuf);
      auto issue_s = [&](int j) -> bool {
        const int t = 2 * j, s = t % WT_NRING, sb = j & 1;
        if (!mbar_wait(&sh.full[s], (t / WT_NRING) & 1, abortp, p.error_word, 803)) return false;
        if (!mbar_wait(&sh.sempty[sb], ((j >> 1) & 1) ^ 1, abortp, p.error_word, 804)) return false;
        fence_after_sync();
        umma_k128(tmem_base + sb * 128, q_addr, WT_BLK, smem_u32(ring + s * WT_TILE), WT_BLK, IDESC_QK);
        umma_commit(&sh.sfull[sb]);
        umma_commit(&sh.empty[s]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; ok && j < n; ++j) {
        if (j + 1 < n) ok = issue_s(j + 1);   // S of the next tile first
        if (!ok) break;
        const int t = 2 * j + 1, s = t % WT_NRING;
        if (!mbar_wait(&sh.full[s], (t / WT_NRING) & 1, abortp, p.error_word, 805)) { ok = false; break; }
        if (!mbar_wait(&sh.pfull, j & 1, abortp, p.error_word, 806)) { ok = false; break; }
        fence_after_sync();
        const uint32_t v_addr = smem_u32(ring + s * WT_TILE);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {      // 16 keys per step: 8 columns of P
          const uint64_t bd = desc_mn(v_addr + ks * 2048, WT_BLK, 1024);
          umma_ts(tmem_base + WT_O, tmem_base + WT_PHI + ks * 8, bd, IDESC_PV, (j | ks) ? 1u : 0u);
          umma_ts(tmem_base + WT_O, tmem_base + WT_PLO + ks * 8, bd, IDESC_PV, 1u);
        }
        umma_commit(&sh.pempty);
        umma_commit(&sh.empty[s]);
      }
      if (ok) umma_commit(&sh.ofull);
    }
  } else {
    const int q = warp & 3;               // TMEM lane quadrant
    const int cq = (warp - 2) >> 2;       // column quarter: keys / dims cq*32 .. +31 of a tile
    const int r = q * 32 + lane;          // query row of the tile
    const int lim = r < rows ? p_first + r : -1;                    // last visible key (-1: none)
    const int lo = r < rows ? win_first(a, p_first + r) : 0x7fffffff;
    const uint32_t lane_base = tmem_base + (static_cast<uint32_t>(q * 32) << 16);
    const float log2e = 1.4426950408889634f;
    const float y = 2.f * log2e * a.scale / a.softcap, m2c = -2.f * a.softcap * log2e;      // (CAPPED)
    const float off = -2.f * m2c <= 200.f ? 0.f : -0.5f * m2c;                              // cap minus reference
    const float sl2 = a.scale * log2e, slope = SLOPED ? win_slope2(a, h) : 0.f;
    bool ok = true;
    uint32_t ra[32];
    float l0 = 0.f, l1 = 0.f, ref = CAPPED ? -0.5f * m2c - off : -INFINITY;
    for (int j = 0; CAPPED ? ok && j < n : j < n; ++j) {
      const int sb = j & 1;
      if constexpr (!CAPPED) {      // (every thread reaches the meetings, whether or not a wait of its ran out)
        const int key0 = wt.tile(j) * 128 + cq * 32;
        const bool whole = (key0 >= lo || key0 + 32 <= a.keep) && key0 + 31 <= lim;
        const float at = SLOPED ? slope * (float)(key0 - (p_first + r)) : 0.f;      // bias of the first column
        float mx = -INFINITY;
        if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&sh.sfull[sb], (j >> 1) & 1, abortp, p.error_word, 807));
        if (ok) {
          fence_after_sync();
          tmem_ld32_issue(lane_base + sb * 128 + cq * 32, ra);
          tmem_ld32_wait(ra);
          fence_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(&sh.sempty[sb]);
          if (!whole) {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (key0 + i > lim || (key0 + i < lo && key0 + i >= a.keep)) ra[i] = 0xff800000u;      // -inf
          }
          if constexpr (SLOPED) {                           // scores in log2 units
#pragma unroll
            for (int i = 0; i < 32; ++i)
              ra[i] = __float_as_uint(fmaf(__uint_as_float(ra[i]), sl2, fmaf(slope, (float)i, at)));
          }
#pragma unroll
          for (int i = 0; i < 32; i += 2) mx = fmax3(mx, __uint_as_float(ra[i]), __uint_as_float(ra[i + 1]));
          if constexpr (!SLOPED) mx *= sl2;
        }
        if (wt_meet_any(q, mx > ref + WT_LAZY)) {           // some row's reference moves
          sh.stat[cq][r] = mx;
          wt_meet_any(q, false);
          const float m = fmaxf(fmaxf(sh.stat[0][r], sh.stat[1][r]), fmaxf(sh.stat[2][r], sh.stat[3][r]));
          float fac = 1.f;
          if (m > ref + WT_LAZY) { fac = ex2_(ref - m); ref = m; }
          l0 *= fac;
          l1 *= fac;
          if (j > 0) {
            if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&sh.pempty, (j & 1) ^ 1, abortp, p.error_word, 812));
            if (ok) {
              fence_after_sync();
              uint32_t o[32];
              tmem_ld32_issue(lane_base + WT_O + cq * 32, o);
              tmem_ld32_wait(o);
#pragma unroll
              for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * fac);
              wt_st32(lane_base + WT_O + cq * 32, o);
              asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            }
          }
          wt_meet_any(q, false);                            // stat may be rewritten
        }
        if (ok) {
          uint32_t hi[16], lw[16];
          if (__any_sync(0xffffffffu, (key0 + 31 >= lo || key0 < a.keep) && key0 <= lim)) {
            const float mref = ref == -INFINITY ? 0.f : ref;   // (a row without keys so far: every weight is exp2(-inf))
#pragma unroll
            for (int i = 0; i < 32; i += 2) {
              const float w0 = ex2_(SLOPED ? __uint_as_float(ra[i]) - mref : fmaf(__uint_as_float(ra[i]), sl2, -mref));
              const float w1 = ex2_(SLOPED ? __uint_as_float(ra[i + 1]) - mref : fmaf(__uint_as_float(ra[i + 1]), sl2, -mref));
              l0 += w0;
              l1 += w1;
              const __nv_bfloat162 x = __floats2bfloat162_rn(w0, w1);
              const float2 f = __bfloat1622float2(x);
              const __nv_bfloat162 z = __floats2bfloat162_rn(w0 - f.x, w1 - f.y);
              hi[i >> 1] = *reinterpret_cast<const uint32_t*>(&x);
              lw[i >> 1] = *reinterpret_cast<const uint32_t*>(&z);
            }
          } else {
#pragma unroll
            for (int i = 0; i < 16; ++i) hi[i] = lw[i] = 0u;
          }
          // rows of the V tile past the sequence become zeros (0 * garbage could be NaN)
          const int first = sq.ctx - wt.tile(j) * 128;
          if (first < 128) {
            const int t = 2 * j + 1, s = t % WT_NRING;
            ok = __all_sync(0xffffffffu, mbar_wait(&sh.full[s], (t / WT_NRING) & 1, abortp, p.error_word, 808));
            unsigned char* vt = ring + s * WT_TILE;
            for (int idx = threadIdx.x - 64; ok && idx < (128 - first) * 16; idx += 512) {
              const int row = first + (idx >> 4), c = idx & 15;
              *reinterpret_cast<int4*>(vt + (c >> 3) * WT_BLK + row * 128 + ((c & 7) << 4)) = make_int4(0, 0, 0, 0);
            }
          }
          if (ok) ok = __all_sync(0xffffffffu, mbar_wait(&sh.pempty, (j & 1) ^ 1, abortp, p.error_word, 809));
          if (ok) {
            fence_after_sync();
            tmem_st16(lane_base + WT_PHI + cq * 16, hi);
            tmem_st16(lane_base + WT_PLO + cq * 16, lw);
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
            if (first < 128) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
          }
        }
        fence_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(&sh.pfull);
      } else {
      if (!mbar_wait(&sh.sfull[sb], (j >> 1) & 1, abortp, p.error_word, 807)) { ok = false; break; }
      fence_after_sync();
      tmem_ld32_issue(lane_base + sb * 128 + cq * 32, ra);
      tmem_ld32_wait(ra);
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.sempty[sb]);
      const int key0 = wt.tile(j) * 128 + cq * 32;
      const bool whole = (key0 >= lo || key0 + 32 <= a.keep) && key0 + 31 <= lim;
      uint32_t hi[16], lw[16];
      if (__any_sync(0xffffffffu, (key0 + 31 >= lo || key0 < a.keep) && key0 <= lim)) {
#pragma unroll
        for (int i = 0; i < 32; i += 4) {
          float w[4];
          weights4(ra + i, y, m2c, off, w);
          if (!whole) {
#pragma unroll
            for (int u = 0; u < 4; ++u)
              if ((key0 + i + u < lo && key0 + i + u >= a.keep) || key0 + i + u > lim) w[u] = 0.f;
          }
          l0 += w[0] + w[1];
          l1 += w[2] + w[3];
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            const __nv_bfloat162 x = __floats2bfloat162_rn(w[2 * u], w[2 * u + 1]);
            const float2 f = __bfloat1622float2(x);
            const __nv_bfloat162 z = __floats2bfloat162_rn(w[2 * u] - f.x, w[2 * u + 1] - f.y);
            hi[(i >> 1) + u] = *reinterpret_cast<const uint32_t*>(&x);
            lw[(i >> 1) + u] = *reinterpret_cast<const uint32_t*>(&z);
          }
        }
      } else {
#pragma unroll
        for (int i = 0; i < 16; ++i) hi[i] = lw[i] = 0u;
      }
      // rows of the V tile past the sequence become zeros (0 * garbage could be NaN)
      const int first = sq.ctx - wt.tile(j) * 128;
      if (first < 128) {
        const int t = 2 * j + 1, s = t % WT_NRING;
        if (!mbar_wait(&sh.full[s], (t / WT_NRING) & 1, abortp, p.error_word, 808)) { ok = false; break; }
        unsigned char* vt = ring + s * WT_TILE;
        for (int idx = threadIdx.x - 64; idx < (128 - first) * 16; idx += 512) {
          const int row = first + (idx >> 4), c = idx & 15;
          *reinterpret_cast<int4*>(vt + (c >> 3) * WT_BLK + row * 128 + ((c & 7) << 4)) = make_int4(0, 0, 0, 0);
        }
      }
      if (!mbar_wait(&sh.pempty, (j & 1) ^ 1, abortp, p.error_word, 809)) { ok = false; break; }
      fence_after_sync();
      tmem_st16(lane_base + WT_PHI + cq * 16, hi);
      tmem_st16(lane_base + WT_PLO + cq * 16, lw);
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      if (first < 128) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.pfull);
      }
    }
    float l = l0 + l1;
    if (ok) {
      sh.stat[cq][r] = l;
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.sbar);
      ok = mbar_wait(&sh.sbar, 0, abortp, p.error_word, 810) && mbar_wait(&sh.ofull, 0, abortp, p.error_word, 811);
    }
    if (ok) {
      l = (sh.stat[0][r] + sh.stat[1][r]) + (sh.stat[2][r] + sh.stat[3][r]);
      if (a.sink) l += ex2_(win_sink2(a, h) - ref);
      fence_after_sync();
      tmem_ld32_issue(lane_base + WT_O + cq * 32, ra);
      tmem_ld32_wait(ra);
      if (r < rows) {
        const int64_t row = sq.row0 + qi0 + r;
        const float inv = l > 0.f ? win_head_factor<T>(a, row, h) / l : 0.f;
        T* o = reinterpret_cast<T*>(a.out) + row * a.out_stride + (int64_t)h * a.DV + cq * 32;
        const T* gate = reinterpret_cast<const T*>(a.gate) + row * a.gate_stride + (int64_t)h * a.DV + cq * 32;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          if (cq * 32 + 8 * c >= a.DV) continue;
          if (a.gate_mode == WIN_GATE_ENTRY) {
            const int4 graw = ld16(gate + 8 * c);
            const T* ge = reinterpret_cast<const T*>(&graw);
#pragma unroll
            for (int i = 0; i < 8; ++i)
              ra[8 * c + i] = __float_as_uint(__uint_as_float(ra[8 * c + i]) * win_sigmoid(__bfloat162float(ge[i])));
          }
          uint32_t w[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 x = __floats2bfloat162_rn(__uint_as_float(ra[8 * c + 2 * i]) * inv,
                                                           __uint_as_float(ra[8 * c + 2 * i + 1]) * inv);
            w[i] = *reinterpret_cast<const uint32_t*>(&x);
          }
          *reinterpret_cast<int4*>(o + 8 * c) = make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]);
        }
      }
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    fence_after_sync();
    tmem_dealloc(tmem_base, 512);
  }
}

// whether the kernel can run this call (total_q: rows of q)
bool window_tc_supports(const WinArgs& a, int total_q, int dtype) {
  return dtype == ZP_DTYPE_BF16 && a.KP <= 128 && a.VP <= 128 && a.D % 8 == 0 && a.DV % 8 == 0 && total_q > 0 &&
         a.softcap * 1.4426950408889634f <= 100.f && !(a.slopes && a.softcap > 0.f) && a.q_stride % 8 == 0 && a.out_stride % 8 == 0 &&
         (a.gate_mode != WIN_GATE_ENTRY || (a.gate_stride % 8 == 0 && (uintptr_t)a.gate % 16 == 0)) &&
         ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.out) % 16 == 0;
}

int window_prefill_tc(const WinArgs& a, int max_q, int total_q, cudaStream_t st) {
  WtParams p{a, device_error_word()};
  if (!p.error_word) { set_error("zp_window_attention(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  CUtensorMap tmQ, tmK, tmV;
  {
    const uint64_t dims[5] = {(uint64_t)a.D, (uint64_t)a.Hq, (uint64_t)total_q, 1, 1};
    const uint64_t strides[4] = {(uint64_t)a.D, (uint64_t)a.q_stride, (uint64_t)a.q_stride, (uint64_t)a.q_stride};
    const uint32_t box[5] = {64, 1, 128, 1, 1};
    if (int rc = make_tensor_map_5d(&tmQ, UmmaFmt<__nv_bfloat16>::tm, a.q, dims, strides, box, 2)) return rc;
  }
  const uint32_t box[5] = {64, 1, 64, 1, 1};
  for (int kv = 0; kv < 2; ++kv) {
    const uint64_t w = kv ? a.VP : a.KP, row = (uint64_t)a.Hkv * w, page = (uint64_t)a.BS * row;
    const uint64_t dims[5] = {w, (uint64_t)a.Hkv, (uint64_t)a.BS, (uint64_t)a.n_pages, 1};
    const uint64_t strides[4] = {w, row, page, page};
    if (int rc = make_tensor_map_5d(kv ? &tmV : &tmK, UmmaFmt<__nv_bfloat16>::tm, kv ? a.v : a.k, dims, strides, box, 2)) return rc;
  }
  const int smem = (1 + WT_NRING) * WT_TILE + (int)sizeof(WtShared) + 1024;
  const auto kern = a.softcap > 0.f ? window_prefill_tc_kernel<true, false> : a.slopes ? window_prefill_tc_kernel<false, true>
                                                                                         : window_prefill_tc_kernel<false, false>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_window_attention(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  kern<<<dim3((max_q + 127) / 128, a.Hq, a.B), WT_THREADS, smem, st>>>(tmQ, tmK, tmV, p);
  return check_launch("zp_window_attention(tcgen05)");
}

}  // namespace zp
