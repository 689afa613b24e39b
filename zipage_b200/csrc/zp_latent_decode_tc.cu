// Attention of queries that meet cached latents directly, on tcgen05 tensor cores (bf16): the keys are whole
// cache rows [latent | rotated part], the values the first R entries of the same rows, so a row is fetched
// once for scores and values and for every query head.
//
// The (row, head) pairs of a sequence's queries are the columns of the products; a block takes NC columns and
// one span of keys, 64 keys (one TMA box of a page) at a time:
//   S^T [keys, columns]    = C Q^T          A = the tile as it lies (K-major), accumulated in TMEM
//   p = exp2(S scale - m)                   fp32; written to shared memory as bf16 pairs hi | lo
//   O^T [latent, columns] += C^T [hi | lo]  A = the same tile, MN-major; hi and lo have columns of their own
// m is one reference per column.  It moves (and O is rescaled) only when a score exceeds it by more than 2^40,
// which fp32 sums and bf16 pairs carry without loss, so nearly always once per span.
// M = 128 also for 64-key tiles: the upper lanes of S^T come from whatever follows in shared memory and are not read.
//
// Roles (384 threads, one block per SM): warp 0 = TMA producer and TMEM owner, warp 1 issues the score products, warp
// 2 the value products, warps 4-11 = softmax in lane quadrants 0-1 (thread <-> key, two warps split the columns),
// rescaling and output in all four (lane <-> latent entry).
// Shared memory: the queries, stages of 128-entry chunks (64 rows each), two P tiles.  Every wait is bounded.
#include "zp_latent.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

constexpr int LD_THREADS = 384;
constexpr int LD_SUB = 8192;           // 64 keys x 64 entries
constexpr int LD_CHUNK = 16384;        // 64 keys x 128 entries
constexpr int LD_MAXC = 5, LD_MAXS = 8;
constexpr float LD_LAZY = 40.f;        // log2 units
constexpr float LD_LOG2E = 1.4426950408889634f;

struct __align__(16) LdShared {
  uint64_t qfull, full[LD_MAXS][LD_MAXC], empty[LD_MAXS][LD_MAXC], sfull[2], sempty[2], pfull[2], pempty[2], obar;
  float ref[32], fac[32], tmax[2][32], lsum[2][32];
  int lim[32];
  uint32_t tmem_base;
  int abort_flag;
};

__device__ __forceinline__ uint64_t ld_desc_mn(uint32_t addr, uint32_t lbo) {   // MN-major, 64-entry blocks lbo apart
  const uint32_t lo = ((addr >> 4) & 0x3FFFu) | ((lbo >> 4) << 16);
  const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
  return (static_cast<uint64_t>(hi) << 32) | lo;
}
template <int N> struct LdTmem;
template <> struct LdTmem<16> {
  static __device__ __forceinline__ void ld(uint32_t a, float (&v)[16]) {
    uint32_t r[16];
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];\n\t"
        "tcgen05.wait::ld.sync.aligned;"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]),
          "=r"(r[9]), "=r"(r[10]), "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(a) : "memory");
#pragma unroll
    for (int i = 0; i < 16; ++i) v[i] = __uint_as_float(r[i]);
  }
  static __device__ __forceinline__ void st(uint32_t a, const float (&v)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16};"
        ::"r"(a), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7]), "f"(v[8]), "f"(v[9]),
          "f"(v[10]), "f"(v[11]), "f"(v[12]), "f"(v[13]), "f"(v[14]), "f"(v[15])
        : "memory");
  }
};
template <> struct LdTmem<8> {
  static __device__ __forceinline__ void ld(uint32_t a, float (&v)[8]) {
    uint32_t r[8];
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0, %1, %2, %3, %4, %5, %6, %7}, [%8];\n\t"
        "tcgen05.wait::ld.sync.aligned;"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
        : "r"(a) : "memory");
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = __uint_as_float(r[i]);
  }
  static __device__ __forceinline__ void st(uint32_t a, const float (&v)[8]) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};"
                 ::"r"(a), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7])
                 : "memory");
  }
};
__device__ __forceinline__ float ld_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
// a wait whose outcome is the same in all lanes (what follows may be warp-wide)
__device__ __forceinline__ bool ld_wait(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* error_word, int where) {
  return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, error_word, where));
}
// meeting of the 256 threads of warps 4-11; true when any of them brings true
__device__ __forceinline__ bool ld_meet_any(bool v) {
  uint32_t out;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred q, 1, 256, p;\n\t"
      "selp.u32 %0, 1, 0, q;\n\t}"
      : "=r"(out) : "r"((uint32_t)v) : "memory");
  return out != 0;
}

struct LdParams {
  LatentArgs a;
  int nb, nc, nv, stages;     // 64-entry blocks of a row; 128-entry chunks; chunks that hold values; stages
  int pairs;                  // a row is whole blocks, and a chunk (the queries) is one load
  int* error_word;
};

template <int NC>
__global__ void __launch_bounds__(LD_THREADS, 1)
latent_decode_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmC, const LdParams p) {
  constexpr int CW = NC / 2;                        // columns of a softmax warp
  constexpr uint32_t O_COL = 2 * NC;                // TMEM: two S^T tiles, then O^T
  const LatentArgs& a = p.a;
  const int b = blockIdx.z, ct = blockIdx.y, split = blockIdx.x;
  const LatSeq sq = lat_seq(a, b);
  const int col0 = ct * NC, ncol = min(NC, sq.count * a.H - col0);
  if (ncol <= 0) return;
  // keys of this block: tiles t0 .. t0 + n - 1
  const int p_first = sq.pos0 + col0 / a.H, p_last = sq.pos0 + (col0 + ncol - 1) / a.H;
  const int total = (p_last >> 6) + 1;
  const int t0 = (int)((int64_t)total * split / a.nsplit), n = (int)((int64_t)total * (split + 1) / a.nsplit) - t0;
  const int64_t flat0 = (int64_t)sq.row0 * a.H + col0;           // (row, head) pair of column 0

  extern __shared__ unsigned char smem_raw[];
  unsigned char* qbuf = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* stage0 = qbuf + p.nb * NC * 128;
  unsigned char* pbuf = stage0 + p.stages * p.nc * LD_CHUNK;     // two tiles of 64 keys x 128 bytes
  LdShared& sh = *reinterpret_cast<LdShared*>(pbuf + 2 * LD_SUB);
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&sh.qfull, 1);
    for (int s = 0; s < p.stages; ++s)
      for (int c = 0; c < p.nc; ++c) { mbar_init(&sh.full[s][c], 1); mbar_init(&sh.empty[s][c], 1); }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sh.sfull[i], 1); mbar_init(&sh.sempty[i], 4); mbar_init(&sh.pfull[i], 8); mbar_init(&sh.pempty[i], 1);
    }
    mbar_init(&sh.obar, 1);
    sh.abort_flag = 0;
    fence_mbar_init();
  }
  if (threadIdx.x < NC) {
    sh.ref[threadIdx.x] = -INFINITY;
    sh.lim[threadIdx.x] = (int)threadIdx.x < ncol ? sq.pos0 + (col0 + (int)threadIdx.x) / a.H : -1;
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
    if (n > 0 && elect_one()) {
      prefetch_tensormap(&tmQ);
      prefetch_tensormap(&tmC);
      mbar_arrive_expect_tx(&sh.qfull, (uint32_t)(p.nb * NC * 128));
      if (p.pairs) tma_load_5d(qbuf, &tmQ, &sh.qfull, 0, (int)flat0, 0, 0, 0);
      else
        for (int k = 0; k < p.nb; ++k) tma_load_5d(qbuf + k * NC * 128, &tmQ, &sh.qfull, k * 64, (int)flat0, 0, 0, 0);
      bool ok = true;
      int s = 0, parity = 1;
      unsigned char* dst = stage0;
      for (int j = 0; ok && j < n; ++j) {
        const int key0 = (t0 + j) * 64, page = lat_page(a, b, key0), off = key0 % a.BS;
        for (int c = 0; c < p.nc; ++c, dst += LD_CHUNK) {
          if (!mbar_wait<true>(&sh.empty[s][c], parity, abortp, p.error_word, 901)) { ok = false; break; }
          if (p.pairs) {          // both halves of the chunk at once (one past the row's end is filled with zeros)
            mbar_arrive_expect_tx(&sh.full[s][c], LD_CHUNK);
            tma_load_5d(dst, &tmC, &sh.full[s][c], 0, off, 2 * c, page, 0);
          } else {
            const int subs = min(2, p.nb - 2 * c);
            mbar_arrive_expect_tx(&sh.full[s][c], (uint32_t)(subs * LD_SUB));
            for (int u = 0; u < subs; ++u) tma_load_5d(dst + u * LD_SUB, &tmC, &sh.full[s][c], (2 * c + u) * 64, off, 0, page, 0);
          }
        }
        if (++s == p.stages) { s = 0; parity ^= 1; dst = stage0; }
      }
    }
  } else if (warp == 1) {
    if (n > 0 && elect_one()) {               // scores
      constexpr uint32_t ID_S = idesc_f16(1, 128, NC);
      bool ok = mbar_wait(&sh.qfull, 0, abortp, p.error_word, 902);
      const uint64_t q_desc = smem_desc_sw128(smem_u32(qbuf));
      uint64_t c_desc = smem_desc_sw128(smem_u32(stage0));
      int s = 0, parity = 0;
      for (int j = 0; ok && j < n; ++j) {
        const uint32_t d = tmem + (j & 1) * NC;
        if (!mbar_wait(&sh.sempty[j & 1], ((j >> 1) & 1) ^ 1, abortp, p.error_word, 903)) break;
        uint64_t bd = q_desc;
        for (int c = 0; c < p.nc; ++c, c_desc += LD_CHUNK >> 4, bd += 2 * NC * 8) {
          if (!mbar_wait(&sh.full[s][c], parity, abortp, p.error_word, 904)) { ok = false; break; }
          fence_after_sync();
          umma_f16(d, c_desc, bd, ID_S, c ? 1u : 0u);
#pragma unroll
          for (int ks = 1; ks < 4; ++ks) umma_f16(d, c_desc + 2u * ks, bd + 2u * ks, ID_S, 1u);
          if (2 * c + 1 < p.nb) {
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) umma_f16(d, c_desc + (LD_SUB >> 4) + 2u * ks, bd + NC * 8 + 2u * ks, ID_S, 1u);
          }
          if (c >= p.nv) umma_commit(&sh.empty[s][c]);
        }
        if (!ok) break;
        umma_commit(&sh.sfull[j & 1]);
        if (++s == p.stages) { s = 0; parity ^= 1; c_desc = smem_desc_sw128(smem_u32(stage0)); }
      }
    }
  } else if (warp == 2) {
    if (n > 0 && elect_one()) {               // values
      constexpr uint32_t ID_O = idesc_f16(1, 128, 2 * NC) | (1u << 15) | (1u << 16);   // both operands MN-major
      const uint64_t p_desc = ld_desc_mn(smem_u32(pbuf), LD_SUB);
      uint64_t c_desc = ld_desc_mn(smem_u32(stage0), LD_SUB);
      bool ok = true;
      int s = 0;
      for (int j = 0; j < n; ++j) {
        if (!mbar_wait(&sh.pfull[j & 1], (j >> 1) & 1, abortp, p.error_word, 905)) { ok = false; break; }
        fence_after_sync();
        const uint64_t pd = p_desc + (j & 1) * (LD_SUB >> 4);
        uint64_t ad = c_desc;
        for (int m = 0; m < p.nv; ++m, ad += LD_CHUNK >> 4) {
          const uint32_t d = tmem + O_COL + m * 2 * NC;
          umma_f16(d, ad, pd, ID_O, j ? 1u : 0u);
#pragma unroll
          for (int ks = 1; ks < 4; ++ks) umma_f16(d, ad + (2048 >> 4) * ks, pd + (2048 >> 4) * ks, ID_O, 1u);
          umma_commit(&sh.empty[s][m]);
        }
        umma_commit(&sh.pempty[j & 1]);
        c_desc += (uint32_t)(p.nc * (LD_CHUNK >> 4));
        if (++s == p.stages) { s = 0; c_desc = ld_desc_mn(smem_u32(stage0), LD_SUB); }
      }
      if (ok) umma_commit(&sh.obar);
    }
  } else if (warp >= 4) {
    const int q = warp & 3, ch = (warp - 4) >> 2;        // lane quadrant, half of the columns
    const int key = q * 32 + lane;                       // key of the tile (quadrants 0 and 1)
    const uint32_t lane_base = tmem + (static_cast<uint32_t>(q * 32) << 16);
    const float sl2 = a.scale * LD_LOG2E;
    const int tid = threadIdx.x - 128;
    bool ok = true;
    float l[CW], ref[CW];
#pragma unroll
    for (int i = 0; i < CW; ++i) { l[i] = 0.f; ref[i] = -INFINITY; }
    for (int j = 0; j < n; ++j) {
      const int key0 = (t0 + j) * 64, sb = j & 1;
      float x[CW];
      bool over = false;
      const bool whole = key0 + 63 <= p_first && ncol == NC;
      if (q < 2) {
        ok = ld_wait(&sh.sfull[sb], (j >> 1) & 1, abortp, p.error_word, 907);
        if (ok) {
          fence_after_sync();
          LdTmem<CW>::ld(lane_base + sb * NC + ch * CW, x);
          fence_before_sync();
          __syncwarp();
          if (lane == 0) mbar_arrive(&sh.sempty[sb]);
#pragma unroll
          for (int i = 0; i < CW; ++i) {
            x[i] *= sl2;
            if (!whole && key0 + key > sh.lim[ch * CW + i]) x[i] = -INFINITY;
            over |= x[i] > ref[i] + LD_LAZY;
          }
        }
      }
      if (ld_meet_any(over)) {                           // some column's reference moves
        if (q < 2) {
#pragma unroll
          for (int i = 0; i < CW; ++i) {
            const float m = warp_max(x[i]);
            if (lane == 0) sh.tmax[q][ch * CW + i] = m;
          }
        }
        ld_meet_any(false);
        if (tid < NC) {
          const float old = sh.ref[tid], m = fmaxf(sh.tmax[0][tid], sh.tmax[1][tid]);
          const bool move = m > old + LD_LAZY;
          sh.fac[tid] = move ? ld_ex2(old - m) : 1.f;
          if (move) sh.ref[tid] = m;
        }
        ld_meet_any(false);
        if (q < 2) {
#pragma unroll
          for (int i = 0; i < CW; ++i) { l[i] *= sh.fac[ch * CW + i]; ref[i] = sh.ref[ch * CW + i]; }
        }
        if (j > 0) {
          // every product into O so far has completed once the previous tile's P is free again
          if (ok) ok = ld_wait(&sh.pempty[(j - 1) & 1], ((j - 1) >> 1) & 1, abortp, p.error_word, 908);
          if (ok) {
            fence_after_sync();
            for (int m = 0; m < p.nv; ++m)
              for (int part = 0; part < 2; ++part) {     // hi, lo
                const uint32_t at = lane_base + O_COL + m * 2 * NC + part * NC + ch * CW;
                float o[CW];
                LdTmem<CW>::ld(at, o);
#pragma unroll
                for (int i = 0; i < CW; ++i) o[i] *= sh.fac[ch * CW + i];
                LdTmem<CW>::st(at, o);
              }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
          }
        }
        ld_meet_any(false);                              // fac and tmax may be rewritten
      }
      if (q < 2 && ok) {
        if (j >= 2) ok = ld_wait(&sh.pempty[sb], ((j >> 1) & 1) ^ 1, abortp, p.error_word, 909);
        if (ok) {
          unsigned char* row = pbuf + sb * LD_SUB + key * 128;
          uint32_t hi[CW / 2], lo[CW / 2];
#pragma unroll
          for (int i = 0; i < CW; i += 2) {
            float w[2];
#pragma unroll
            for (int u = 0; u < 2; ++u) {
              w[u] = x[i + u] == -INFINITY ? 0.f : ld_ex2(x[i + u] - ref[i + u]);
              l[i + u] += w[u];
            }
            const __nv_bfloat162 h = __floats2bfloat162_rn(w[0], w[1]);
            const float2 f = __bfloat1622float2(h);
            const __nv_bfloat162 g = __floats2bfloat162_rn(w[0] - f.x, w[1] - f.y);
            hi[i / 2] = *reinterpret_cast<const uint32_t*>(&h);
            lo[i / 2] = *reinterpret_cast<const uint32_t*>(&g);
          }
          constexpr int PC = CW / 8;                     // 16-byte pieces of a half's hi (and lo) columns
#pragma unroll
          for (int i = 0; i < PC; ++i) {
            st16(row + (((ch * PC + i) ^ (key & 7)) << 4), make_int4(hi[4 * i], hi[4 * i + 1], hi[4 * i + 2], hi[4 * i + 3]));
            st16(row + (((2 * PC + ch * PC + i) ^ (key & 7)) << 4), make_int4(lo[4 * i], lo[4 * i + 1], lo[4 * i + 2], lo[4 * i + 3]));
          }
        }
        // rows of the tile past the sequence become zeros (0 * garbage could be NaN)
        const int first = sq.ctx - key0;
        if (ok && first < 64) {
          const int s = j % p.stages;
          for (int c = 0; ok && c < p.nv; ++c) {
            ok = ld_wait(&sh.full[s][c], (j / p.stages) & 1, abortp, p.error_word, 910);
            unsigned char* t = stage0 + (s * p.nc + c) * LD_CHUNK;
            if (key >= first) {
              for (int i = 0; i < 8; ++i) st16(t + ch * LD_SUB + key * 128 + (i << 4), make_int4(0, 0, 0, 0));
            }
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      }
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.pfull[sb]);
    }
    // row sums
    if (q < 2) {
#pragma unroll
      for (int i = 0; i < CW; ++i) {
        const float s = warp_sum(l[i]);
        if (lane == 0) sh.lsum[q][ch * CW + i] = s;
      }
    }
    if (ok && n > 0) ok = ld_wait(&sh.obar, 0, abortp, p.error_word, 911);
    ld_meet_any(false);
    // O^T to rows in shared memory (the stages are free), then whole rows to global memory
    if (ok) {
      fence_after_sync();
      const bool whole = a.nsplit == 1;
      float inv[CW];
#pragma unroll
      for (int i = 0; i < CW; ++i) {
        const float s = sh.lsum[0][ch * CW + i] + sh.lsum[1][ch * CW + i];
        inv[i] = whole ? (s > 0.f ? 1.f / s : 0.f) : 1.f;
      }
      for (int m = 0; m < p.nv; ++m) {
        float o[CW], o2[CW];
        if (n > 0) {
          const uint32_t at = lane_base + O_COL + m * 2 * NC + ch * CW;
          LdTmem<CW>::ld(at, o);
          LdTmem<CW>::ld(at + NC, o2);
        }
        const int d = m * 128 + q * 32 + lane;
        if (d < a.R) {
#pragma unroll
          for (int i = 0; i < CW; ++i) {
            const float v = n > 0 ? (o[i] + o2[i]) * inv[i] : 0.f;
            const int at = (ch * CW + i) * a.R + d;
            if (whole) reinterpret_cast<__nv_bfloat16*>(stage0)[at] = __float2bfloat16_rn(v);
            else reinterpret_cast<float*>(stage0)[at] = v;
          }
        }
      }
    }
    ld_meet_any(false);
    if (ok) {
      const int row = a.R * (a.nsplit == 1 ? 2 : 4);      // bytes
      char* dst = a.nsplit == 1 ? reinterpret_cast<char*>(a.out) + flat0 * row
                                : reinterpret_cast<char*>(a.part) + (flat0 * a.nsplit + split) * row;
      const int64_t step = (int64_t)row * a.nsplit;       // between the columns' rows
      if (row % 16 == 0) {
        const int per = row / 16;
        for (int i = tid; i < ncol * per; i += 256) st16(dst + (i / per) * step + (i % per) * 16, ld16(stage0 + i * 16));
      } else {
        const int per = row / 2;
        for (int i = tid; i < ncol * per; i += 256)
          *reinterpret_cast<uint16_t*>(dst + (i / per) * step + (i % per) * 2) = *reinterpret_cast<const uint16_t*>(stage0 + i * 2);
      }
      if (a.nsplit > 1 && tid < ncol) {
        float* ml = a.part + (int64_t)a.pairs * a.nsplit * a.R + ((flat0 + tid) * a.nsplit + split) * 2;
        ml[0] = sh.ref[tid];
        ml[1] = sh.lsum[0][tid] + sh.lsum[1][tid];
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

// out [pair, R] from the spans' unnormalised sums, references and row sums; one block per pair, four entries a thread
__global__ void __launch_bounds__(128) latent_combine_kernel(const LatentArgs a) {
  // rows that no sequence of this call names (another call's, or padding) keep what they hold
  __shared__ float w[32];
  const int b = blockIdx.y, i = blockIdx.x;
  const LatSeq sq = lat_seq(a, b);
  if (i >= sq.count * a.H) return;
  const int64_t pair = (int64_t)sq.row0 * a.H + i;
  if (threadIdx.x < 32) {                   // (at most 32 spans)
    const float* ml = a.part + (int64_t)a.pairs * a.nsplit * a.R + pair * a.nsplit * 2;
    const bool in = (int)threadIdx.x < a.nsplit;
    const float2 v = in ? make_float2(ml[2 * threadIdx.x], ml[2 * threadIdx.x + 1]) : make_float2(-INFINITY, 0.f);
    const float m = warp_max(v.x), f = v.x == -INFINITY ? 0.f : ld_ex2(v.x - m), l = warp_sum(f * v.y);
    w[threadIdx.x] = l > 0.f ? f / l : 0.f;
  }
  __syncthreads();
  const float* part = a.part + pair * a.nsplit * a.R;
  __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(a.out) + pair * a.R;
  if (a.R % 4 == 0) {
    for (int d = threadIdx.x * 4; d < a.R; d += 512) {
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
      for (int s = 0; s < a.nsplit; ++s) {
        const float4 v = *reinterpret_cast<const float4*>(part + (int64_t)s * a.R + d);
        const float f = w[s];
        if (f > 0.f) { o.x = fmaf(f, v.x, o.x); o.y = fmaf(f, v.y, o.y); o.z = fmaf(f, v.z, o.z); o.w = fmaf(f, v.w, o.w); }
      }
      const __nv_bfloat162 r[2] = {__floats2bfloat162_rn(o.x, o.y), __floats2bfloat162_rn(o.z, o.w)};
      *reinterpret_cast<uint2*>(out + d) = *reinterpret_cast<const uint2*>(r);
    }
  } else {
    for (int d = threadIdx.x; d < a.R; d += 128) {
      float o = 0.f;
      for (int s = 0; s < a.nsplit; ++s)
        if (w[s] > 0.f) o = fmaf(w[s], part[(int64_t)s * a.R + d], o);
      out[d] = __float2bfloat16_rn(o);
    }
  }
}

static int ld_smem(int nb, int nc, int NC, int stages) {
  return 1024 + nb * NC * 128 + stages * nc * LD_CHUNK + 2 * LD_SUB + (int)sizeof(LdShared);
}

bool latent_decode_tc_supports(const LatentArgs& a, int dtype) {
  return dtype == ZP_DTYPE_BF16 && a.KP % 16 == 0 && a.KP <= 640 && a.R <= 512 && a.R > 0 && a.R <= a.KP &&
         ((uintptr_t)a.q | (uintptr_t)a.cache | (uintptr_t)a.out) % 16 == 0;
}

// columns of a block for sequences of at most max_q rows
static int ld_columns(const LatentArgs& a, int max_q) { return (int64_t)max_q * a.H > 16 ? 32 : 16; }

int latent_decode_splits(int B, int max_q, int H, int span) {
  const int NC = (int64_t)max_q * H > 16 ? 32 : 16;
  const int64_t blocks = (int64_t)B * (((int64_t)max_q * H + NC - 1) / NC);
  const int tiles = (span + 63) / 64;
  int best = 1;
  double cost = 1e30;
  for (int s = 1; s <= 32 && s <= tiles; ++s) {     // waves of blocks times a block's tiles (and its start, about 3 tiles)
    const double c = (double)((blocks * s + 147) / 148) * ((double)tiles / s + 3.0 + (s > 1 ? 1.0 : 0.0));
    if (c < cost * 0.98) { cost = c; best = s; }
  }
  return best;
}

template <int NC> static int ld_launch(const LatentArgs& a, int max_q, int total_rows, cudaStream_t st) {
  LdParams p;
  p.a = a;
  p.nb = (a.KP + 63) / 64;
  p.pairs = a.KP % 64 == 0;
  p.nc = (p.nb + 1) / 2;
  p.nv = (a.R + 127) / 128;
  p.error_word = device_error_word();
  if (!p.error_word) { set_error("zp_latent_attention(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  p.stages = LD_MAXS;
  while (p.stages > 1 && ld_smem(p.nb, p.nc, NC, p.stages) > 232448) --p.stages;
  const int smem = ld_smem(p.nb, p.nc, NC, p.stages);
  if (smem > 232448 || p.stages < 2) { set_error("zp_latent_attention(tcgen05): rows of %d entries do not fit", a.KP); return ZP_ERR_UNSUPPORTED; }
  CUtensorMap tmQ, tmC;
  const uint64_t pairs = (uint64_t)total_rows * a.H;
  {
    const uint64_t dims[5] = {p.pairs ? 64u : (uint64_t)a.KP, pairs, p.pairs ? (uint64_t)p.nb : 1u, 1, 1};
    const uint64_t strides[4] = {(uint64_t)a.KP, p.pairs ? 64u : pairs * a.KP, pairs * a.KP, pairs * a.KP};
    const uint32_t box[5] = {64, NC, p.pairs ? (uint32_t)p.nb : 1u, 1, 1};
    if (int rc = make_tensor_map_5d(&tmQ, UmmaFmt<__nv_bfloat16>::tm, a.q, dims, strides, box, 2)) return rc;
  }
  {
    const uint64_t page = (uint64_t)a.BS * a.KP;
    // whole 64-entry blocks: [block][key][entry] boxes of two blocks; else one block's box, cut at the row's end
    const uint64_t dims[5] = {p.pairs ? 64u : (uint64_t)a.KP, (uint64_t)a.BS, p.pairs ? (uint64_t)p.nb : 1u, (uint64_t)a.n_pages, 1};
    const uint64_t strides[4] = {(uint64_t)a.KP, p.pairs ? 64u : (uint64_t)a.KP, page, page * a.n_pages};
    const uint32_t box[5] = {64, 64, p.pairs ? 2u : 1u, 1, 1};
    if (int rc = make_tensor_map_5d(&tmC, UmmaFmt<__nv_bfloat16>::tm, a.cache, dims, strides, box, 2)) return rc;
  }
  cudaError_t e = cudaFuncSetAttribute(latent_decode_tc_kernel<NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_latent_attention(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  const int tiles = (int)(((int64_t)max_q * a.H + NC - 1) / NC);
  latent_decode_tc_kernel<NC><<<dim3(a.nsplit, tiles, a.B), LD_THREADS, smem, st>>>(tmQ, tmC, p);
  if (a.nsplit > 1) latent_combine_kernel<<<dim3((unsigned)(max_q * a.H), a.B), 128, 0, st>>>(a);
  return check_launch("zp_latent_attention(tcgen05)");
}

int latent_decode_tc(const LatentArgs& a, int max_q, int total_rows, cudaStream_t st) {
  return ld_columns(a, max_q) == 16 ? ld_launch<16>(a, max_q, total_rows, st) : ld_launch<32>(a, max_q, total_rows, st);
}

}  // namespace zp
