// Causal attention of prompt portions over keys and values computed from latents, on tcgen05 tensor cores
// (bf16): a key is an unrotated part of its head's own and a rotated part that all heads share, so the two are
// fetched from where they lie (the expanded keys, the latent rows) and meet only in the accumulator.
//   S = Qn Kn^T + Qr Kr^T       [128 queries, 128 keys], accumulated in TMEM
//   p = exp2(S scale - m)        fp32, split into bf16 hi + lo in TMEM
//   O += P_hi V + P_lo V         (V is MN-major as it lies), accumulated in TMEM
// m is one reference per row; it moves (and O is rescaled) only when a score exceeds it by more than 2^40,
// which fp32 sums and bf16 pairs carry without loss, so nearly always in the first tile only.
//
// Roles (576 threads, one block per SM): warp 0 = TMA producer and TMEM owner, warp 1 = MMA issuer, warps
// 2-17 = softmax (thread <-> TMEM lane <-> query row; the four warps of a lane quadrant split a tile's 128
// columns and meet on a barrier of their own).  Shared memory: the query tile and a ring of 16 KB blocks (128 rows x
// 64 entries); a tile brings its key blocks, then its value blocks.  Parts whose sizes are not multiples of 64
// are filled with zeros by TMA.  Every wait is bounded.
#include "zp_latent.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

constexpr int LF_THREADS = 576;
constexpr int LF_BLK = 16384;
constexpr int LF_MAXRING = 12;
constexpr float LF_LAZY = 40.f;    // log2 units
constexpr float LF_LOG2E = 1.4426950408889634f;
constexpr uint32_t LF_O = 256, LF_PHI = 384, LF_PLO = 448;   // TMEM columns after the two S tiles

struct __align__(16) LfShared {
  uint64_t qfull, full[LF_MAXRING], empty[LF_MAXRING], sfull[2], sempty[2], pfull, pempty, ofull;
  float stat[4][128];
  uint32_t tmem_base;
  int abort_flag;
};

struct LfParams {
  const int32_t *cu_q, *cu_k;
  __nv_bfloat16* out;
  int H, DV, nbn, nbr, nbv, ring;     // 64-entry blocks of the unrotated, rotated and value parts; blocks of the ring
  int64_t out_stride;
  float scale;
  int* error_word;
};

__device__ __forceinline__ uint64_t lf_desc_mn(uint32_t addr) {   // MN-major, one 64-entry block
  const uint32_t lo = ((addr >> 4) & 0x3FFFu) | ((uint32_t)(LF_BLK >> 4) << 16);
  const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
  return (static_cast<uint64_t>(hi) << 32) | lo;
}
__device__ __forceinline__ void lf_umma_ts(uint32_t d, uint32_t a, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d), "r"(a), "l"(b_desc), "r"(idesc), "r"(acc) : "memory");
}
__device__ __forceinline__ void lf_st16(uint32_t taddr, const uint32_t (&r)[16]) {
  asm volatile(
      "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], "
      "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
      ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]),
        "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]), "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15])
      : "memory");
}
__device__ __forceinline__ void lf_st32(uint32_t taddr, const uint32_t (&r)[32]) {
  uint32_t a[16], b[16];
#pragma unroll
  for (int i = 0; i < 16; ++i) { a[i] = r[i]; b[i] = r[16 + i]; }
  lf_st16(taddr, a);
  lf_st16(taddr + 16, b);
}
__device__ __forceinline__ float lf_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ bool lf_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* error_word, int where) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, error_word, where));
}
// meeting of the 128 threads of a lane quadrant (barriers 1-4); true when any of them brings true
__device__ __forceinline__ bool lf_meet_any(int q, bool v) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, r;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred r, %2, 128, p;\n\t"
      "selp.u32 %0, 1, 0, r;\n\t}"
      : "=r"(out) : "r"((uint32_t)v), "r"(q + 1) : "memory");
  return out != 0;
}

__global__ void __launch_bounds__(LF_THREADS, 1)
latent_prefill_tc_kernel(const __grid_constant__ CUtensorMap tmQn, const __grid_constant__ CUtensorMap tmQr,
                         const __grid_constant__ CUtensorMap tmKn, const __grid_constant__ CUtensorMap tmKr,
                         const __grid_constant__ CUtensorMap tmV, const LfParams p) {
  const int b = blockIdx.z, h = blockIdx.y;
  const int q0 = p.cu_q[b], count = p.cu_q[b + 1] - q0, k0 = p.cu_k[b], ctx = p.cu_k[b + 1] - k0;
  const int pos0 = ctx - count;
  const int nqt = (count + 127) >> 7;
  if ((int)blockIdx.x >= nqt || pos0 < 0) return;
  const int qi0 = (nqt - 1 - blockIdx.x) * 128;      // the tiles with the most keys start first
  const int rows = min(128, count - qi0);
  const int p_first = pos0 + qi0, n = ((p_first + rows - 1) >> 7) + 1;   // 128-key tiles 0 .. n - 1
  const int nbq = p.nbn + p.nbr, per = nbq + p.nbv;

  extern __shared__ unsigned char smem_raw[];
  unsigned char* qbuf = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* ring = qbuf + nbq * LF_BLK;
  LfShared& sh = *reinterpret_cast<LfShared*>(ring + p.ring * LF_BLK);
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&sh.qfull, 1);
    for (int i = 0; i < p.ring; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.sfull[i], 1); mbar_init(&sh.sempty[i], 16); }
    mbar_init(&sh.pfull, 16);
    mbar_init(&sh.pempty, 1);
    mbar_init(&sh.ofull, 1);
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

  if (warp == 0) {
    if (elect_one()) {
      mbar_arrive_expect_tx(&sh.qfull, (uint32_t)(nbq * LF_BLK));
      for (int i = 0; i < p.nbn; ++i) tma_load_5d(qbuf + i * LF_BLK, &tmQn, &sh.qfull, i * 64, h, q0 + qi0, 0, 0);
      for (int i = 0; i < p.nbr; ++i) tma_load_5d(qbuf + (p.nbn + i) * LF_BLK, &tmQr, &sh.qfull, i * 64, h, q0 + qi0, 0, 0);
      bool ok = true;
      int slot = 0, round = 0;
      for (int j = 0; ok && j < n; ++j) {
        const int key = k0 + j * 128;
        for (int i = 0; i < per; ++i) {
          if (!mbar_wait<true>(&sh.empty[slot], (round & 1) ^ 1, abortp, p.error_word, 921)) { ok = false; break; }
          mbar_arrive_expect_tx(&sh.full[slot], LF_BLK);
          unsigned char* dst = ring + slot * LF_BLK;
          if (i < p.nbn) tma_load_5d(dst, &tmKn, &sh.full[slot], i * 64, h, key, 0, 0);
          else if (i < nbq) tma_load_5d(dst, &tmKr, &sh.full[slot], (i - p.nbn) * 64, 0, key, 0, 0);
          else tma_load_5d(dst, &tmV, &sh.full[slot], (i - nbq) * 64, h, key, 0, 0);
          if (++slot == p.ring) { slot = 0; ++round; }
        }
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t ID_S = idesc_f16(1, 128, 128);
      constexpr uint32_t ID_O = idesc_f16(1, 128, 64) | (1u << 16);   // V MN-major, one 64-entry block at a time
      bool ok = mbar_wait(&sh.qfull, 0, abortp, p.error_word, 922);
      const uint32_t q_addr = smem_u32(qbuf), r_addr = smem_u32(ring);
      auto issue_s = [&](int j) -> bool {
        const int sb = j & 1;
        if (!mbar_wait(&sh.sempty[sb], ((j >> 1) & 1) ^ 1, abortp, p.error_word, 923)) return false;
        for (int i = 0; i < nbq; ++i) {
          const int t = j * per + i, s = t % p.ring;
          if (!mbar_wait(&sh.full[s], (t / p.ring) & 1, abortp, p.error_word, 924)) return false;
          fence_after_sync();
          const uint64_t ad = smem_desc_sw128(q_addr + i * LF_BLK), bd = smem_desc_sw128(r_addr + s * LF_BLK);
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) umma_f16(tmem + sb * 128, ad + 2u * ks, bd + 2u * ks, ID_S, (i | ks) ? 1u : 0u);
          umma_commit(&sh.empty[s]);
        }
        umma_commit(&sh.sfull[sb]);
        return true;
      };
      if (ok) ok = issue_s(0);
      for (int j = 0; ok && j < n; ++j) {
        if (j + 1 < n) ok = issue_s(j + 1);   // S of the next tile first
        if (!ok) break;
        if (!mbar_wait(&sh.pfull, j & 1, abortp, p.error_word, 925)) { ok = false; break; }
        for (int i = 0; ok && i < p.nbv; ++i) {
          const int t = j * per + nbq + i, s = t % p.ring;
          if (!mbar_wait(&sh.full[s], (t / p.ring) & 1, abortp, p.error_word, 926)) { ok = false; break; }
          fence_after_sync();
          const uint32_t v_addr = r_addr + s * LF_BLK;
#pragma unroll
          for (int ks = 0; ks < 8; ++ks) {      // 16 keys per step: 8 columns of P
            const uint64_t bd = lf_desc_mn(v_addr + ks * 2048);
            lf_umma_ts(tmem + LF_O + i * 64, tmem + LF_PHI + ks * 8, bd, ID_O, (j | ks) ? 1u : 0u);
            lf_umma_ts(tmem + LF_O + i * 64, tmem + LF_PLO + ks * 8, bd, ID_O, 1u);
          }
          umma_commit(&sh.empty[s]);
        }
        umma_commit(&sh.pempty);
      }
      if (ok) umma_commit(&sh.ofull);
    }
  } else {
    const int q = warp & 3;               // TMEM lane quadrant
    const int cq = (warp - 2) >> 2;       // column quarter: keys / value entries cq*32 .. +31
    const int r = q * 32 + lane;          // query row of the tile
    const int lim = r < rows ? p_first + r : -1;                    // last visible key (-1: none)
    const uint32_t lane_base = tmem + (static_cast<uint32_t>(q * 32) << 16);
    const float sl2 = p.scale * LF_LOG2E;
    bool ok = true;
    uint32_t ra[32];
    float l0 = 0.f, l1 = 0.f, ref = -INFINITY;
    for (int j = 0; j < n; ++j) {
      const int sb = j & 1, key0 = j * 128 + cq * 32;
      const bool whole = key0 + 31 <= lim;
      float mx = -INFINITY;
      if (ok) ok = lf_wait(&sh.sfull[sb], (j >> 1) & 1, abortp, p.error_word, 927);
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
            if (key0 + i > lim) ra[i] = 0xff800000u;      // -inf
        }
#pragma unroll
        for (int i = 0; i < 32; i += 2) mx = fmax3(mx, __uint_as_float(ra[i]), __uint_as_float(ra[i + 1]));
        mx *= sl2;
      }
      if (lf_meet_any(q, mx > ref + LF_LAZY)) {           // some row's reference moves
        sh.stat[cq][r] = mx;
        lf_meet_any(q, false);
        const float m = fmaxf(fmaxf(sh.stat[0][r], sh.stat[1][r]), fmaxf(sh.stat[2][r], sh.stat[3][r]));
        float fac = 1.f;
        if (m > ref + LF_LAZY) { fac = lf_ex2(ref - m); ref = m; }
        l0 *= fac;
        l1 *= fac;
        if (j > 0) {
          if (ok) ok = lf_wait(&sh.pempty, (j & 1) ^ 1, abortp, p.error_word, 928);
          if (ok && cq * 32 < p.nbv * 64) {
            fence_after_sync();
            uint32_t o[32];
            tmem_ld32_issue(lane_base + LF_O + cq * 32, o);
            tmem_ld32_wait(o);
#pragma unroll
            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * fac);
            lf_st32(lane_base + LF_O + cq * 32, o);
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
          }
        }
        lf_meet_any(q, false);                            // stat may be rewritten
      }
      if (ok) {
        uint32_t hi[16], lw[16];
        if (__any_sync(0xffffffffu, key0 <= lim)) {
          const float mref = ref == -INFINITY ? 0.f : ref;   // (a row without queries: every weight is exp2(-inf))
#pragma unroll
          for (int i = 0; i < 32; i += 2) {
            const float w0 = lf_ex2(fmaf(__uint_as_float(ra[i]), sl2, -mref)), w1 = lf_ex2(fmaf(__uint_as_float(ra[i + 1]), sl2, -mref));
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
        // rows of the V blocks past the sequence become zeros (0 * another sequence's values could be NaN)
        const int first = ctx - j * 128;
        if (first < 128) {
          for (int i = 0; ok && i < p.nbv; ++i) {
            const int t = j * per + nbq + i, s = t % p.ring;
            ok = lf_wait(&sh.full[s], (t / p.ring) & 1, abortp, p.error_word, 929);
            for (int idx = threadIdx.x - 64; ok && idx < (128 - first) * 8; idx += 512)
              *reinterpret_cast<int4*>(ring + s * LF_BLK + (first + (idx >> 3)) * 128 + ((idx & 7) << 4)) = make_int4(0, 0, 0, 0);
          }
        }
        if (ok) ok = lf_wait(&sh.pempty, (j & 1) ^ 1, abortp, p.error_word, 930);
        if (ok) {
          fence_after_sync();
          lf_st16(lane_base + LF_PHI + cq * 16, hi);
          lf_st16(lane_base + LF_PLO + cq * 16, lw);
          asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
          if (first < 128) asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        }
      }
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.pfull);
    }
    sh.stat[cq][r] = l0 + l1;
    lf_meet_any(q, false);
    if (ok) ok = lf_wait(&sh.ofull, 0, abortp, p.error_word, 931);
    if (ok && cq * 32 < p.nbv * 64) {
      const float l = (sh.stat[0][r] + sh.stat[1][r]) + (sh.stat[2][r] + sh.stat[3][r]);
      fence_after_sync();
      tmem_ld32_issue(lane_base + LF_O + cq * 32, ra);
      tmem_ld32_wait(ra);
      if (r < rows) {
        const float inv = l > 0.f ? 1.f / l : 0.f;
        __nv_bfloat16* o = p.out + (int64_t)(q0 + qi0 + r) * p.out_stride + (int64_t)h * p.DV + cq * 32;
#pragma unroll
        for (int c = 0; c < 4; ++c) {
          uint32_t w[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const __nv_bfloat162 x = __floats2bfloat162_rn(__uint_as_float(ra[8 * c + 2 * i]) * inv,
                                                           __uint_as_float(ra[8 * c + 2 * i + 1]) * inv);
            w[i] = *reinterpret_cast<const uint32_t*>(&x);
          }
          if (cq * 32 + 8 * c < p.DV) *reinterpret_cast<int4*>(o + 8 * c) = make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]);
        }
      }
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
}

}  // namespace zp

extern "C" int zp_latent_prefill_supported(int dim, int rot, int vdim, int kv_rank, int KP, int dtype) {
  const int nbq = (dim + 63) / 64 + (rot + 63) / 64;
  return dtype == ZP_DTYPE_BF16 && dim > 0 && vdim > 0 && vdim <= 128 && nbq <= 4 && dim % 8 == 0 && rot % 8 == 0 && vdim % 8 == 0 &&
         kv_rank % 8 == 0 && KP % 8 == 0;
}

extern "C" int zp_latent_prefill(const void* q, int64_t q_stride, const void* kv, const void* latent, const int32_t* cu_seqlens_q,
                                 const int32_t* cu_seqlens_k, void* out, int64_t out_stride, int B, int max_seqlen_q, int total_q,
                                 int total_k, int H, int dim, int rot, int vdim, int kv_rank, int KP, float scale, int dtype,
                                 void* stream) {
  using namespace zp;
  using namespace zp::tc;
  if (B == 0 || max_seqlen_q == 0) return ZP_OK;
  ZP_REQUIRE(q && kv && (latent || rot == 0) && cu_seqlens_q && cu_seqlens_k && out, "zp_latent_prefill: null pointer");
  ZP_REQUIRE(H > 0 && H <= 65535 && B <= 65535 && total_q > 0 && total_k > 0 && KP >= kv_rank + rot, "zp_latent_prefill: bad sizes");
  if (!zp_latent_prefill_supported(dim, rot, vdim, kv_rank, KP, dtype) || q_stride % 8 || out_stride % 8 ||
      ((uintptr_t)q | (uintptr_t)kv | (uintptr_t)latent | (uintptr_t)out) % 16) {
    set_error("zp_latent_prefill: needs bf16, head sizes that are multiples of 8 (values at most 128) and 16-byte aligned rows");
    return ZP_ERR_UNSUPPORTED;
  }
  LfParams p;
  p.cu_q = cu_seqlens_q; p.cu_k = cu_seqlens_k; p.out = (__nv_bfloat16*)out; p.H = H; p.DV = vdim;
  p.nbn = (dim + 63) / 64; p.nbr = (rot + 63) / 64; p.nbv = (vdim + 63) / 64;
  p.out_stride = out_stride; p.scale = scale;
  p.error_word = device_error_word();
  if (!p.error_word) { set_error("zp_latent_prefill: no device error word"); return ZP_ERR_CUDA; }
  const int nbq = p.nbn + p.nbr;
  const int fixed = 1024 + nbq * LF_BLK + (int)sizeof(LfShared);
  p.ring = (232448 - fixed) / LF_BLK;
  if (p.ring > LF_MAXRING) p.ring = LF_MAXRING;
  const int smem = fixed + p.ring * LF_BLK;
  const auto fmt = UmmaFmt<__nv_bfloat16>::tm;
  const __nv_bfloat16* qb = (const __nv_bfloat16*)q;
  const __nv_bfloat16* kb = (const __nv_bfloat16*)kv;
  const uint64_t kv_stride = (uint64_t)H * (dim + vdim), hd = dim + rot, qs = q_stride;
  const uint64_t uq = total_q, uk = total_k, uh = H;
  const uint32_t box[5] = {64, 1, 128, 1, 1};
  CUtensorMap tmQn, tmQr, tmKn, tmKr, tmV;
  const uint64_t sq[4] = {hd, qs, qs * uq, qs * uq}, sk[4] = {(uint64_t)dim, kv_stride, kv_stride * uk, kv_stride * uk},
                 sv[4] = {(uint64_t)vdim, kv_stride, kv_stride * uk, kv_stride * uk},
                 sl[4] = {(uint64_t)KP, (uint64_t)KP, (uint64_t)KP * uk, (uint64_t)KP * uk};
  const uint64_t dqn[5] = {(uint64_t)dim, uh, uq, 1, 1}, dqr[5] = {(uint64_t)rot, uh, uq, 1, 1}, dkn[5] = {(uint64_t)dim, uh, uk, 1, 1},
                 dkr[5] = {(uint64_t)rot, 1, uk, 1, 1}, dv[5] = {(uint64_t)vdim, uh, uk, 1, 1};
  if (int rc = make_tensor_map_5d(&tmQn, fmt, qb, dqn, sq, box, 2)) return rc;
  if (int rc = make_tensor_map_5d(&tmKn, fmt, kb, dkn, sk, box, 2)) return rc;
  if (int rc = make_tensor_map_5d(&tmV, fmt, kb + (int64_t)H * dim, dv, sv, box, 2)) return rc;
  tmQr = tmQn;
  tmKr = tmKn;
  if (rot) {
    if (int rc = make_tensor_map_5d(&tmQr, fmt, qb + dim, dqr, sq, box, 2)) return rc;
    if (int rc = make_tensor_map_5d(&tmKr, fmt, (const __nv_bfloat16*)latent + kv_rank, dkr, sl, box, 2)) return rc;
  }
  cudaError_t e = cudaFuncSetAttribute(latent_prefill_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_latent_prefill: %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  latent_prefill_tc_kernel<<<dim3((max_seqlen_q + 127) / 128, H, B), LF_THREADS, smem, (cudaStream_t)stream>>>(tmQn, tmQr, tmKn, tmKr, tmV, p);
  return check_launch("zp_latent_prefill");
}
