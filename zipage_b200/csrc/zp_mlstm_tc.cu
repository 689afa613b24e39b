// Matrix-memory (mLSTM) mixer over prompt portions on tcgen05 tensor cores: bf16 projections, key size 128,
// value size a multiple of 128 (up to 1024), fp32 state; 128 tokens at a time.
//
// Same unrolled recurrence as zp_mlstm_chunk.cu (F_t running sum of the log forget gates in the chunk,
// u_j = i_j - F_j, M_t = max(m, max_{j<=t} u_j)); one block per (128-wide value tile, head, sequence) walks
// the chunks in order.  Per chunk, all accumulators in TMEM:
//   SC = Q K^T                              [128 tokens, 128 tokens]
//   OX = Q S                                [128 tokens, 128 values]   S as bf16 hi + lo in shared memory
//   P  = SC * exp(u_j - M_t), j <= t        fp32, split into bf16 hi + lo, back to TMEM as the A operand
//   OI = P V
//   D  = K^T (w V), w_j = exp(u_j - M_C)    over SC; w V as bf16 hi + lo, over S's shared memory
//   o  = (exp(m - M_t) OX + OI) / normaliser;  S = exp(m - M_C) S + D   (fp32, in registers)
// n, n . q and the row sums of P are fp32 on the CUDA cores.  K, and the state and value tiles, are MN-major
// operands: they lie in shared memory as TMA (or the threads) wrote them.
//
// Roles (576 threads, one block per SM): warp 0 = TMA producer, gates of the next chunk, TMEM owner; warp 1 = MMA
// issuer; warps 2-17 = arithmetic (thread <-> TMEM lane; four warps of a lane quadrant split 128 columns).
// A lane is a token for P and the output, a key dim for the state.  The blocks of a head form a cluster and
// push their rows' sums of squares into each other's shared memory (the head norm spans all value dims).
// Every wait is bounded; after it the block raises the device error word and leaves.
#include "zp_mlstm.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

constexpr int MT_THREADS = 576;
constexpr int MT_TILE = 32768;      // 128 rows x 128 bf16
constexpr int MT_BLK = 16384;       // one 64-column block of a tile
constexpr int MT_NRING = 4;
constexpr int MT_MAX_TILES = 8;
constexpr uint32_t MT_SC = 0, MT_PHI = 128, MT_PLO = 192, MT_OX = 256, MT_OI = 384;   // TMEM columns
constexpr float MT_LOG2E = 1.4426950408889634f;

struct __align__(16) MtShared {
  uint64_t full[MT_NRING], empty[MT_NRING], gfull[2], gempty[2], sready, scfull, oxfull, pfull, wready, dfull, sbar, xbar[2];
  float scan[2][5][128];            // M, u (log2 units), A, E, W of a chunk, by parity
  float decay[2];
  float n[128];
  float npart[16][128];
  float stat[2][4][128];            // per column quarter: row sums and n . q
  float ssq[4][128];
  float xs[2][MT_MAX_TILES][128];   // sums of squares of every value tile, by parity
  float norm[128];
  uint32_t tmem_base;
  int abort_flag;
};

__device__ __forceinline__ uint64_t mt_desc_mn(uint32_t smem_addr) {   // MN-major tile of 64-column blocks
  const uint32_t lo = ((smem_addr >> 4) & 0x3FFFu) | ((uint32_t)(MT_BLK >> 4) << 16);
  const uint32_t hi = (1024u >> 4) | (1u << 14) | (2u << 29);
  return (static_cast<uint64_t>(hi) << 32) | lo;
}
__device__ __forceinline__ void mt_umma_ts(uint32_t d_tmem, uint32_t a_tmem, uint64_t b_desc, uint32_t idesc, uint32_t acc) {
  asm volatile(
      "{\n\t.reg .pred p;\n\t"
      "setp.ne.b32 p, %4, 0;\n\t"
      "tcgen05.mma.cta_group::1.kind::f16 [%0], [%1], %2, %3, p;\n\t}"
      ::"r"(d_tmem), "r"(a_tmem), "l"(b_desc), "r"(idesc), "r"(acc)
      : "memory");
}
__device__ __forceinline__ void mt_ld16(uint32_t taddr, float (&v)[16]) {   // load and wait
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
__device__ __forceinline__ void mt_st8(uint32_t taddr, const uint32_t (&r)[8]) {
  asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};"
               ::"r"(taddr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7])
               : "memory");
}
__device__ __forceinline__ float mt_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float mt_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void mt_split(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  const float2 f = __bfloat1622float2(h);
  const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 mt_pair(uint32_t w) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&w)); }
// 16-byte chunk c (0..15) of row r of a 128-column tile: two swizzled 64-column blocks
__device__ __forceinline__ uint32_t mt_chunk(int r, int c) {
  return (uint32_t)((c >> 3) * MT_BLK + r * 128 + (((c & 7) ^ (r & 7)) << 4));
}
// push a float / arrive on a barrier in another block of the cluster
__device__ __forceinline__ uint32_t mt_map(const void* p, uint32_t rank) {
  uint32_t ra;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(smem_u32(p)), "r"(rank));
  return ra;
}
__device__ __forceinline__ void mt_push(const float* p, uint32_t rank, float v) {
  asm volatile("st.shared::cluster.f32 [%0], %1;" ::"r"(mt_map(p, rank)), "f"(v) : "memory");
}
__device__ __forceinline__ void mt_arrive_peer(const uint64_t* bar, uint32_t rank) {
  asm volatile("mbarrier.arrive.release.cluster.shared::cluster.b64 _, [%0];" ::"r"(mt_map(bar, rank)) : "memory");
}
__device__ __forceinline__ bool mt_wait_cluster(uint64_t* bar, uint32_t parity, volatile int* abort_flag, int* error_word, int where) {
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

struct MtParams { MlstmArgs a; int* error_word; };

__global__ void __launch_bounds__(MT_THREADS, 1)
mlstm_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK,
                const __grid_constant__ CUtensorMap tmV, const MtParams p) {
  using T = __nv_bfloat16;
  const MlstmArgs& a = p.a;
  const int vt = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const MlstmSeq sq = mlstm_seq(a, b);
  if (sq.count == 0) return;                       // the same decision in every block of the cluster
  const int nc = (sq.count + 127) >> 7, tiles = gridDim.x, c0 = vt * 128;
  const int64_t head = (int64_t)sq.slot * a.H + h;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  unsigned char* sHi = ring + MT_NRING * MT_TILE;  // state operand, then decayed values
  unsigned char* sLo = sHi + MT_TILE;
  MtShared& sh = *reinterpret_cast<MtShared*>(sLo + MT_TILE);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  float m = sq.fresh ? 0.f : a.m[head];            // (read before the cluster meets: written by one block at the end)
  if (threadIdx.x < 128) {
    sh.n[threadIdx.x] = sq.fresh ? 0.f : a.n[head * 128 + threadIdx.x];
    sh.norm[threadIdx.x] = a.norm_weight[(int64_t)h * a.vdim + c0 + threadIdx.x];
  }
  if (threadIdx.x == 0) {
    for (int i = 0; i < MT_NRING; ++i) { mbar_init(&sh.full[i], 1); mbar_init(&sh.empty[i], 17); }
    for (int i = 0; i < 2; ++i) {
      mbar_init(&sh.gfull[i], 1); mbar_init(&sh.gempty[i], 16);
      mbar_init(&sh.xbar[i], tiles > 1 ? 4 * (tiles - 1) : 1);
    }
    mbar_init(&sh.sready, 16); mbar_init(&sh.scfull, 1); mbar_init(&sh.oxfull, 1); mbar_init(&sh.pfull, 16);
    mbar_init(&sh.wready, 16); mbar_init(&sh.dfull, 1); mbar_init(&sh.sbar, 16);
    sh.abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(&sh.tmem_base, 512);
    tmem_relinquish();
  }
  fence_before_sync();
  __syncthreads();
  if (tiles > 1) cluster_sync();                   // barriers of every block are ready
  fence_after_sync();
  const uint32_t tmem = sh.tmem_base;
  volatile int* abortp = &sh.abort_flag;
  int* err = p.error_word;

  // ring positions of chunk c: Q 3c, K 3c + 1, V 3c + 2
  auto slot = [](int t) { return t % MT_NRING; };
  auto phase = [](int t) { return (uint32_t)((t / MT_NRING) & 1); };
  if (warp == 0) {
    // ---------------- TMA producer; gates one chunk ahead ----------------
    const float log2_qscale = log2f(a.qscale);
    auto gates = [&](int c) -> bool {
      const int par = c & 1, n = min(128, sq.count - c * 128);
      int good = 1;
      if (lane == 0) good = mbar_wait<true>(&sh.gempty[par], ((c >> 1) & 1) ^ 1, abortp, err, 901);
      if (!__shfl_sync(0xffffffffu, good, 0)) return false;
      float f[4], u[4], F = 0.f, mx = -INFINITY;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = 4 * lane + j;
        const int64_t row = sq.row0 + c * 128 + t;
        f[j] = t < n ? log_forget_gate(a, row, h) : 0.f;
        u[j] = t < n ? log_input_gate(a, row, h) : -INFINITY;
        F += f[j];
      }
      float incl = F;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, incl, o); if (lane >= o) incl += x; }
      float run = incl - F;
#pragma unroll
      for (int j = 0; j < 4; ++j) { run += f[j]; f[j] = run; u[j] -= run; mx = fmaxf(mx, u[j]); }   // f: F_t from here on
      float cm = mx;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) { const float x = __shfl_up_sync(0xffffffffu, cm, o); if (lane >= o) cm = fmaxf(cm, x); }
      float before = __shfl_up_sync(0xffffffffu, cm, 1);
      float M = lane == 0 ? m : fmaxf(m, before);
      const float MC = fmaxf(m, __shfl_sync(0xffffffffu, cm, 31)), FC = __shfl_sync(0xffffffffu, incl, 31);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int t = 4 * lane + j;
        M = fmaxf(M, u[j]);
        sh.scan[par][0][t] = fmaf(M, MT_LOG2E, -log2_qscale);     // exponents in log2 units, the query scale folded in
        sh.scan[par][1][t] = u[j] * MT_LOG2E;
        sh.scan[par][2][t] = expf(m - M) * a.qscale;
        sh.scan[par][3][t] = expf(-(M + f[j]));
        sh.scan[par][4][t] = expf(u[j] - MC);
      }
      if (lane == 0) sh.decay[par] = expf(m - MC);
      m = MC + FC;
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.gfull[par]);
      return true;
    };
    if (lane == 0) { prefetch_tensormap(&tmQ); prefetch_tensormap(&tmK); prefetch_tensormap(&tmV); }
    bool ok = gates(0);
    for (int c = 0; ok && c < nc; ++c) {
      int good = 1;
      if (lane == 0) {
        const int row = sq.row0 + c * 128;
        for (int i = 0; i < 3; ++i) {
          const int t = 3 * c + i, s = slot(t);
          if (!mbar_wait<true>(&sh.empty[s], phase(t) ^ 1, abortp, err, 902)) { good = 0; break; }
          const CUtensorMap* tm = i == 0 ? &tmQ : i == 1 ? &tmK : &tmV;
          const int x = i == 2 ? h * a.vdim + c0 : h * 128;
          mbar_arrive_expect_tx(&sh.full[s], MT_TILE);
          tma_load_5d(ring + s * MT_TILE, tm, &sh.full[s], x, row, 0, 0, 0);
          tma_load_5d(ring + s * MT_TILE + MT_BLK, tm, &sh.full[s], x + 64, row, 0, 0, 0);
        }
      }
      ok = __shfl_sync(0xffffffffu, good, 0) != 0;
      if (ok && c + 1 < nc) ok = gates(c + 1);
    }
    if (ok && vt == 0 && lane == 0) a.m[head] = m;
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      constexpr uint32_t ID = idesc_f16(1, 128, 128), B_MN = 1u << 16, A_MN = 1u << 15;
      const uint32_t hi = smem_u32(sHi), lo = smem_u32(sLo);
      for (int c = 0; c < nc; ++c) {
        const uint32_t ph = c & 1;
        const int tq = 3 * c, tk = tq + 1, tv = tq + 2;
        const uint32_t qa = smem_u32(ring + slot(tq) * MT_TILE), ka = smem_u32(ring + slot(tk) * MT_TILE),
                       va = smem_u32(ring + slot(tv) * MT_TILE);
        if (!mbar_wait(&sh.full[slot(tq)], phase(tq), abortp, err, 911) || !mbar_wait(&sh.full[slot(tk)], phase(tk), abortp, err, 912) ||
            !mbar_wait(&sh.sready, ph, abortp, err, 913)) break;
        fence_after_sync();
        umma_k128(tmem + MT_SC, qa, MT_BLK, ka, MT_BLK, ID);
        umma_commit(&sh.scfull);
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint64_t ad = smem_desc_sw128(qa + (ks >> 2) * MT_BLK) + 2u * (ks & 3);
          umma_f16(tmem + MT_OX, ad, mt_desc_mn(hi + ks * 2048), ID | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + MT_OX, ad, mt_desc_mn(lo + ks * 2048), ID | B_MN, 1u);
        }
        umma_commit(&sh.oxfull);
        umma_commit(&sh.empty[slot(tq)]);
        if (!mbar_wait(&sh.full[slot(tv)], phase(tv), abortp, err, 914) || !mbar_wait(&sh.pfull, ph, abortp, err, 915)) break;
        fence_after_sync();
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint64_t bd = mt_desc_mn(va + ks * 2048);
          mt_umma_ts(tmem + MT_OI, tmem + MT_PHI + ks * 8, bd, ID | B_MN, ks ? 1u : 0u);
          mt_umma_ts(tmem + MT_OI, tmem + MT_PLO + ks * 8, bd, ID | B_MN, 1u);
        }
        umma_commit(&sh.empty[slot(tv)]);
        if (!mbar_wait(&sh.wready, ph, abortp, err, 916)) break;
        fence_after_sync();
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
          const uint64_t ad = mt_desc_mn(ka + ks * 2048);
          umma_f16(tmem + MT_SC, ad, mt_desc_mn(hi + ks * 2048), ID | A_MN | B_MN, ks ? 1u : 0u);
          umma_f16(tmem + MT_SC, ad, mt_desc_mn(lo + ks * 2048), ID | A_MN | B_MN, 1u);
        }
        umma_commit(&sh.dfull);
        umma_commit(&sh.empty[slot(tk)]);
      }
    }
  } else {
    // ---------------- arithmetic ----------------
    const int cw = warp - 2, q = warp & 3, cq = cw >> 2;   // lane quadrant; columns cq * 32 .. + 31
    const int r = q * 32 + lane;                   // token of the chunk, or key dim of the state
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(q * 32) << 16);
    bool ok = true;
    uint32_t sph = 0;
    auto csync = [&](int where) -> bool {          // the sixteen arithmetic warps (a bounded wait, unlike bar.sync)
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.sbar);
      const bool good = mbar_wait(&sh.sbar, sph & 1, abortp, err, where);
      ++sph;
      return good;
    };
    auto arrive = [&](uint64_t* bar) {
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    auto fence_async = []() { asm volatile("fence.proxy.async.shared::cta;" ::: "memory"); };
    float s[32];                                   // state: row r (key dim), columns c0 + cq * 32 + i
    float* Sg = a.S + (head * 128 + r) * (int64_t)a.VP + c0 + cq * 32;
#pragma unroll
    for (int i = 0; i < 32; i += 4) {
      const float4 x = sq.fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(Sg + i);
      s[i] = x.x; s[i + 1] = x.y; s[i + 2] = x.z; s[i + 3] = x.w;
    }
    auto put_state = [&]() {                       // the state as operand: row r of the hi and lo tiles
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        uint32_t hi[4], lo[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) mt_split(s[8 * i + 2 * j], s[8 * i + 2 * j + 1], hi[j], lo[j]);
        const uint32_t off = mt_chunk(r, cq * 4 + i);
        st16(sHi + off, make_int4((int)hi[0], (int)hi[1], (int)hi[2], (int)hi[3]));
        st16(sLo + off, make_int4((int)lo[0], (int)lo[1], (int)lo[2], (int)lo[3]));
      }
      fence_async();
      fence_before_sync();
      arrive(&sh.sready);
    };
    put_state();

    for (int c = 0; c < nc; ++c) {
      const int par = c & 1, n = min(128, sq.count - c * 128);
      const uint32_t ph = c & 1;
      const int tq = 3 * c, tk = tq + 1, tv = tq + 2;
      const unsigned char *Qs = ring + slot(tq) * MT_TILE, *Ks = ring + slot(tk) * MT_TILE, *Vs = ring + slot(tv) * MT_TILE;
      if (!mbar_wait(&sh.gfull[par], (c >> 1) & 1, abortp, err, 921)) { ok = false; break; }
      if (n < 128) {                               // rows past the sequence belong to others: zero as keys and values
        if (!mbar_wait(&sh.full[slot(tk)], phase(tk), abortp, err, 922) || !mbar_wait(&sh.full[slot(tv)], phase(tv), abortp, err, 923)) {
          ok = false; break;
        }
        for (int i = threadIdx.x - 64; i < (128 - n) * 16; i += 512) {
          const uint32_t off = mt_chunk(n + (i >> 4), i & 15);
          st16(const_cast<unsigned char*>(Ks) + off, make_int4(0, 0, 0, 0));
          st16(const_cast<unsigned char*>(Vs) + off, make_int4(0, 0, 0, 0));
        }
        fence_async();
        if (!csync(924)) { ok = false; break; }
      }
      // n . q over this thread's 32 key dims
      if (!mbar_wait(&sh.full[slot(tq)], phase(tq), abortp, err, 925)) { ok = false; break; }
      float nq = 0.f;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int4 w = ld16(Qs + mt_chunk(r, cq * 4 + i));
        const float* nn = sh.n + cq * 32 + 8 * i;
        const int ww[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 f = mt_pair((uint32_t)ww[j]);
          nq = fmaf(f.x, nn[2 * j], fmaf(f.y, nn[2 * j + 1], nq));
        }
      }
      arrive(&sh.empty[slot(tq)]);
      // P
      if (!mbar_wait(&sh.scfull, ph, abortp, err, 926)) { ok = false; break; }
      fence_after_sync();
      const float M = sh.scan[par][0][r];
      float rs = 0.f;
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        uint32_t hi[8], lo[8];
        if (cq <= q) {                             // (later columns are later tokens for every row of the warp)
          float x[16];
          mt_ld16(lane_addr + MT_SC + cq * 32 + 16 * y, x);
#pragma unroll
          for (int i = 0; i < 16; i += 2) {
            const int key = cq * 32 + 16 * y + i;
            const float2 u = *reinterpret_cast<const float2*>(&sh.scan[par][1][key]);
            const float p0 = key <= r ? x[i] * mt_ex2(u.x - M) : 0.f;
            const float p1 = key + 1 <= r ? x[i + 1] * mt_ex2(u.y - M) : 0.f;
            rs += p0 + p1;
            mt_split(p0, p1, hi[i >> 1], lo[i >> 1]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 8; ++i) hi[i] = lo[i] = 0u;
        }
        mt_st8(lane_addr + MT_PHI + cq * 16 + 8 * y, hi);
        mt_st8(lane_addr + MT_PLO + cq * 16 + 8 * y, lo);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      fence_before_sync();
      arrive(&sh.pfull);
      sh.stat[0][cq][r] = rs;
      sh.stat[1][cq][r] = nq;
      // decayed values over the state operand (its product is done)
      if (!mbar_wait(&sh.oxfull, ph, abortp, err, 927) || !mbar_wait(&sh.full[slot(tv)], phase(tv), abortp, err, 928)) { ok = false; break; }
      {
        const float w = sh.scan[par][4][r];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          const uint32_t off = mt_chunk(r, cq * 4 + i);
          const int4 v = ld16(Vs + off);
          const int vv[4] = {v.x, v.y, v.z, v.w};
          uint32_t hi[4], lo[4];
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float2 f = mt_pair((uint32_t)vv[j]);
            mt_split(f.x * w, f.y * w, hi[j], lo[j]);
          }
          st16(sHi + off, make_int4((int)hi[0], (int)hi[1], (int)hi[2], (int)hi[3]));
          st16(sLo + off, make_int4((int)lo[0], (int)lo[1], (int)lo[2], (int)lo[3]));
        }
        fence_async();
        arrive(&sh.wready);
        arrive(&sh.empty[slot(tv)]);
      }
      // n: this warp's eight tokens, four key dims per lane
      if (!mbar_wait(&sh.full[slot(tk)], phase(tk), abortp, err, 929)) { ok = false; break; }
      {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int t = cw * 8 + i;
          const float w = sh.scan[par][4][t];
          const uint2 kk = *reinterpret_cast<const uint2*>(Ks + mt_chunk(t, lane >> 1) + (lane & 1) * 8);
          const float2 k0 = mt_pair(kk.x), k1 = mt_pair(kk.y);
          acc.x = fmaf(w, k0.x, acc.x); acc.y = fmaf(w, k0.y, acc.y);
          acc.z = fmaf(w, k1.x, acc.z); acc.w = fmaf(w, k1.y, acc.w);
        }
        *reinterpret_cast<float4*>(&sh.npart[cw][4 * lane]) = acc;
        arrive(&sh.empty[slot(tk)]);
      }
      if (!csync(930)) { ok = false; break; }
      const float decay = sh.decay[par], A = sh.scan[par][2][r];
      if (threadIdx.x - 64 < 128) {
        const int d = threadIdx.x - 64;
        float x = decay * sh.n[d];
#pragma unroll
        for (int i = 0; i < 16; ++i) x += sh.npart[i][d];
        sh.n[d] = x;                               // (read again after the next meeting)
      }
      float den;
      {
        const float nqs = (sh.stat[1][0][r] + sh.stat[1][1][r]) + (sh.stat[1][2][r] + sh.stat[1][3][r]);
        const float rss = (sh.stat[0][0][r] + sh.stat[0][1][r]) + (sh.stat[0][2][r] + sh.stat[0][3][r]);
        den = mt_rcp(fmaxf(fabsf(fmaf(A, nqs, rss)), sh.scan[par][3][r]) + MLSTM_DEN_EPS);
      }
      arrive(&sh.gempty[par]);
      // outputs and state
      if (!mbar_wait(&sh.dfull, ph, abortp, err, 931)) { ok = false; break; }
      fence_after_sync();
      float o[32];
#pragma unroll
      for (int y = 0; y < 2; ++y) {
        float x[16];
        mt_ld16(lane_addr + MT_OX + cq * 32 + 16 * y, x);
#pragma unroll
        for (int i = 0; i < 16; ++i) o[16 * y + i] = A * x[i];
        mt_ld16(lane_addr + MT_OI + cq * 32 + 16 * y, x);
#pragma unroll
        for (int i = 0; i < 16; ++i) o[16 * y + i] += x[i];
        mt_ld16(lane_addr + MT_SC + cq * 32 + 16 * y, x);
#pragma unroll
        for (int i = 0; i < 16; ++i) s[16 * y + i] = fmaf(decay, s[16 * y + i], x[i]);
      }
      if (c + 1 < nc) put_state();
      float ss = 0.f;
#pragma unroll
      for (int i = 0; i < 32; ++i) { o[i] *= den; ss = fmaf(o[i], o[i], ss); }
      sh.ssq[cq][r] = ss;
      // the output gate, four lanes per row (lane t of a group: chunk t of the group's rows)
      int4 gt[4];
      const int lrow = q * 32 + (lane & ~3);
      const int64_t lrow0 = sq.row0 + (int64_t)c * 128 + lrow, lcol = (int64_t)h * a.vdim + c0 + cq * 32 + (lane & 3) * 8;
#pragma unroll
      for (int i = 0; i < 4; ++i)
        gt[i] = lrow + i < n ? ld16(reinterpret_cast<const T*>(a.g) + (lrow0 + i) * a.row_stride + lcol) : make_int4(0, 0, 0, 0);
      if (!csync(932)) { ok = false; break; }
      ss = (sh.ssq[0][r] + sh.ssq[1][r]) + (sh.ssq[2][r] + sh.ssq[3][r]);
      if (tiles > 1) {
        if (cq == 0) {
          for (int k = 0; k < tiles; ++k)
            if (k != vt) mt_push(&sh.xs[par][vt][r], k, ss);
          __syncwarp();
          if (lane == 0)
            for (int k = 0; k < tiles; ++k)
              if (k != vt) mt_arrive_peer(&sh.xbar[par], k);
        }
        if (!mt_wait_cluster(&sh.xbar[par], (c >> 1) & 1, abortp, err, 933)) { ok = false; break; }
        float all = 0.f;                           // in tile order: every block of the head gets the same sum
        for (int k = 0; k < tiles; ++k) all += k == vt ? ss : sh.xs[par][k][r];
        ss = all;
      }
      const float rr = rsqrtf(ss / (float)a.vdim + a.eps);
      transpose4(gt, lane);                     // to this thread's own row
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int gg[4] = {gt[i].x, gt[i].y, gt[i].z, gt[i].w};
        uint32_t w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float2 gv = mt_pair((uint32_t)gg[j]);
          const float2 nw = *reinterpret_cast<const float2*>(&sh.norm[cq * 32 + 8 * i + 2 * j]);
          const float x = o[8 * i + 2 * j] * rr * nw.x * mt_rcp(1.f + mt_ex2(-MT_LOG2E * gv.x));
          const float z = o[8 * i + 2 * j + 1] * rr * nw.y * mt_rcp(1.f + mt_ex2(-MT_LOG2E * gv.y));
          const __nv_bfloat162 pr = __floats2bfloat162_rn(x, z);
          w[j] = *reinterpret_cast<const uint32_t*>(&pr);
        }
        gt[i] = make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]);
      }
      transpose4(gt, lane);
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (lrow + i < n) st16(reinterpret_cast<T*>(a.out) + (lrow0 + i) * a.out_stride + lcol, gt[i]);
    }
    if (ok) {
#pragma unroll
      for (int i = 0; i < 32; i += 4) *reinterpret_cast<float4*>(Sg + i) = make_float4(s[i], s[i + 1], s[i + 2], s[i + 3]);
      if (vt == 0 && threadIdx.x - 64 < 128) a.n[head * 128 + threadIdx.x - 64] = sh.n[threadIdx.x - 64];
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    fence_after_sync();
    tmem_dealloc(tmem, 512);
  }
  if (tiles > 1) cluster_sync();                   // no block leaves while a peer may still write to it
}

// whether the kernel can run this call (total_rows: rows of q, k, v, g; 0 = not told)
bool mlstm_tc_supports(const MlstmArgs& a, int total_rows, int dtype) {
  return dtype == ZP_DTYPE_BF16 && total_rows > 0 && a.dim == 128 && a.vdim % 128 == 0 && a.vdim <= 128 * MT_MAX_TILES &&
         a.VP == a.vdim && a.row_stride % 8 == 0 && a.out_stride % 8 == 0 && a.qscale > 0.f &&
         ((uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.g | (uintptr_t)a.out) % 16 == 0;
}

int mlstm_tc(const MlstmArgs& a, int total_rows, cudaStream_t st) {
  MtParams p{a, device_error_word()};
  if (!p.error_word) { set_error("zp_mlstm(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  CUtensorMap tm[3];
  const void* base[3] = {a.q, a.k, a.v};
  for (int i = 0; i < 3; ++i) {
    const uint64_t cols = (uint64_t)a.H * (i == 2 ? a.vdim : a.dim), rs = (uint64_t)a.row_stride;
    const uint64_t dims[5] = {cols, (uint64_t)total_rows, 1, 1, 1};
    const uint64_t strides[4] = {rs, rs * total_rows, rs * total_rows, rs * total_rows};
    const uint32_t box[5] = {64, 128, 1, 1, 1};
    if (int rc = make_tensor_map_5d(&tm[i], UmmaFmt<__nv_bfloat16>::tm, base[i], dims, strides, box, 2)) return rc;
  }
  const int smem = (MT_NRING + 2) * MT_TILE + (int)sizeof(MtShared) + 1024;
  cudaError_t e = cudaFuncSetAttribute(mlstm_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_mlstm(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  const int tiles = a.vdim / 128;
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles, a.H, a.B);
  cfg.blockDim = dim3(MT_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = tiles; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  e = cudaLaunchKernelEx(&cfg, mlstm_tc_kernel, tm[0], tm[1], tm[2], p);
  if (e != cudaSuccess) { set_error("zp_mlstm(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  return check_launch("zp_mlstm(tcgen05)");
}

}  // namespace zp
