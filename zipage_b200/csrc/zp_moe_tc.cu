// Per-expert matrix products on tcgen05 tensor cores (bf16): out[p, n] = act(x[r(p)] . w[e, n]) for the places p of
// every expert, 128 places x BN outputs a tile, 64 entries of the contraction a stage.
//
// The grid is persistent: every block walks the tiles blockIdx.x, + gridDim.x, ... of the list (expert, 128
// places, BN outputs), whose length it derives from the experts' offsets on the device, so the launch is the
// same whatever the routing chose (graphs).
//
// Roles: warp 0 = TMA producer; warp 1 = MMA issuer, accumulating in TMEM, two tiles in turn; warps 2-5 = epilogue
// (thread <-> TMEM lane <-> place): activation, rounding, store.  Every wait is bounded.  How the rows arrive:
//   GT_FEW     four-row gathers, one per lane, of which only those with places are issued (a decode step brings a few rows
//              per expert, and the rest of the 128-row operand is whatever the stage held: rows do not mix);
//   GT_TILE    one 128-row load (rows that already lie in the order of the places);
//   GT_GATHER  four more warps copy the rows' 16-byte pieces with cp.async (a gather load fetches rows at a
//              small part of a tile load's rate), publishing a stage two stages later, when its copies have landed.
#include <type_traits>

#include "zp_moe.cuh"
#include "zp_tc.cuh"

namespace zp {

using namespace tc;

enum { GT_FEW = 0, GT_TILE = 1, GT_GATHER = 2 };
constexpr int GT_LAG = 2;                 // stages between the issue of a stage's copies and its publication
constexpr int GT_A = 16384;               // 128 rows x 64 entries
constexpr int GT_MAXS = 8, GT_MAXE = 1024;

struct __align__(16) GtShared {
  uint64_t full[GT_MAXS], empty[GT_MAXS], afull[2], aempty[2];
  uint32_t tmem_base;
  int abort_flag;
  int mtiles[GT_MAXE + 1];                // tiles of 128 places before each expert
};

struct GtParams {
  GroupedArgs a;
  int ntn, kb, stages;                    // output tiles, stages of the contraction, stages in shared memory
  int* error_word;
};

// four rows of a two-dimensional map (box: one row of 64 entries) into 512 consecutive bytes
__device__ __forceinline__ void gt_gather4(void* dst, const CUtensorMap* m, uint64_t* bar, int x, int4 r) {
  asm volatile(
      "cp.async.bulk.tensor.2d.shared::cluster.global.tile::gather4.mbarrier::complete_tx::bytes "
      "[%0], [%1, {%3, %4, %5, %6, %7}], [%2];"
      ::"r"(smem_u32(dst)), "l"(reinterpret_cast<uint64_t>(m)), "r"(smem_u32(bar)), "r"(x), "r"(r.x), "r"(r.y), "r"(r.z), "r"(r.w)
      : "memory");
}

struct GtTile { int e, first, count, n0; };
template <int BN> __device__ __forceinline__ GtTile gt_tile(const GtParams& p, const GtShared& sh, int t) {
  const int mi = t / p.ntn;
  int lo = 0, hi = p.a.E - 1;             // last expert whose tiles start at or before mi
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (sh.mtiles[mid] <= mi) lo = mid; else hi = mid - 1;
  }
  GtTile r;
  r.e = lo;
  r.first = p.a.offsets[lo] + (mi - sh.mtiles[lo]) * 128;
  r.count = min(128, p.a.offsets[lo + 1] - r.first);
  r.n0 = (t - mi * p.ntn) * BN;
  return r;
}

__device__ __forceinline__ void gt_copy16(uint32_t dst, const void* src, int bytes) {   // the rest of 16 bytes becomes zero
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(bytes) : "memory");
}
// the copies of the stage issued GT_LAG stages ago (or, LEFT = 0, all) have landed: tell the tensor cores
template <int LEFT> __device__ __forceinline__ void gt_publish(uint64_t* bar, int lane) {
  asm volatile("cp.async.wait_group %0;" ::"n"(LEFT) : "memory");
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  __syncwarp();
  if (lane == 0) mbar_arrive(bar);
}

template <int MODE> constexpr int gt_threads() { return MODE == GT_GATHER ? 320 : 192; }

template <int BN, int ACT, int MODE>
__global__ void __launch_bounds__(gt_threads<MODE>(), 1)
grouped_gemm_tc_kernel(const __grid_constant__ CUtensorMap tmX, const __grid_constant__ CUtensorMap tmW, const GtParams p) {
  constexpr int STAGE = GT_A + BN * 128;
  extern __shared__ unsigned char smem_raw[];
  unsigned char* ring = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  GtShared& sh = *reinterpret_cast<GtShared*>(ring + p.stages * STAGE);
  const int warp = warp_index(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int s = 0; s < p.stages; ++s) { mbar_init(&sh.full[s], MODE == GT_GATHER ? 5 : 1); mbar_init(&sh.empty[s], 1); }
    for (int i = 0; i < 2; ++i) { mbar_init(&sh.afull[i], 1); mbar_init(&sh.aempty[i], 4); }
    sh.abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0) {
    tmem_alloc(&sh.tmem_base, 2 * BN);
    tmem_relinquish();
  } else if (warp == 1) {
    int base = 0;
    for (int e0 = 0; e0 < p.a.E; e0 += 32) {
      const int e = e0 + lane, c = e < p.a.E ? (p.a.offsets[e + 1] - p.a.offsets[e] + 127) >> 7 : 0;
      int s = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int t = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += t;
      }
      if (e < p.a.E) sh.mtiles[e] = base + s - c;
      base += __shfl_sync(0xffffffffu, s, 31);
    }
    if (lane == 0) sh.mtiles[p.a.E] = base;
  }
  fence_before_sync();
  __syncthreads();
  fence_after_sync();
  const uint32_t tmem = sh.tmem_base;
  volatile int* abortp = &sh.abort_flag;
  const int total = sh.mtiles[p.a.E] * p.ntn;

  if (warp == 0) {
    if constexpr (MODE == GT_FEW) {
      bool ok = true;
      int slot = 0, round = 0;
      for (int t = blockIdx.x; ok && t < total; t += gridDim.x) {
        const GtTile tl = gt_tile<BN>(p, sh, t);
        const int groups = (tl.count + 3) >> 2;
        int4 r;
        {
          int v[4];
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            const int at = tl.first + min(4 * lane + i, tl.count - 1);
            v[i] = p.a.rows ? min(max(p.a.rows[at], 0), p.a.src_rows - 1) : at;
          }
          r = make_int4(v[0], v[1], v[2], v[3]);
        }
        for (int k = 0; k < p.kb; ++k) {
          ok = __all_sync(0xffffffffu, mbar_wait(&sh.empty[slot], (round & 1) ^ 1, abortp, p.error_word, 941));
          if (!ok) break;
          unsigned char* dst = ring + slot * STAGE;
          if (elect_one()) {
            mbar_arrive_expect_tx(&sh.full[slot], (uint32_t)(groups * 512 + BN * 128));
            tma_load_5d(dst + GT_A, &tmW, &sh.full[slot], k * 64, tl.n0, tl.e, 0, 0);
          }
          __syncwarp();
          if (lane < groups) gt_gather4(dst + lane * 512, &tmX, &sh.full[slot], k * 64, r);
          if (++slot == p.stages) { slot = 0; ++round; }
        }
      }
    } else if (elect_one()) {
      bool ok = true;
      int slot = 0, round = 0;
      for (int t = blockIdx.x; ok && t < total; t += gridDim.x) {
        const GtTile tl = gt_tile<BN>(p, sh, t);
        for (int k = 0; k < p.kb; ++k) {
          if (!mbar_wait(&sh.empty[slot], (round & 1) ^ 1, abortp, p.error_word, 941)) { ok = false; break; }
          unsigned char* dst = ring + slot * STAGE;
          mbar_arrive_expect_tx(&sh.full[slot], (uint32_t)((MODE == GT_TILE ? GT_A : 0) + BN * 128));
          if (MODE == GT_TILE) tma_load_5d(dst, &tmX, &sh.full[slot], k * 64, tl.first, 0, 0, 0);
          tma_load_5d(dst + GT_A, &tmW, &sh.full[slot], k * 64, tl.n0, tl.e, 0, 0);
          if (++slot == p.stages) { slot = 0; ++round; }
        }
      }
    }
  } else if (warp == 1) {
    if (elect_one()) {
      constexpr uint32_t ID = idesc_f16(1, 128, BN);
      bool ok = true;
      int slot = 0, round = 0, i = 0;
      for (int t = blockIdx.x; ok && t < total; t += gridDim.x, ++i) {
        const int acc = i & 1;
        if (!mbar_wait(&sh.aempty[acc], ((i >> 1) & 1) ^ 1, abortp, p.error_word, 942)) break;
        fence_after_sync();
        for (int k = 0; k < p.kb; ++k) {
          if (!mbar_wait(&sh.full[slot], round & 1, abortp, p.error_word, 943)) { ok = false; break; }
          fence_after_sync();
          const uint32_t at = smem_u32(ring + slot * STAGE);
          const uint64_t ad = smem_desc_sw128(at), bd = smem_desc_sw128(at + GT_A);
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) umma_f16(tmem + acc * BN, ad + 2u * ks, bd + 2u * ks, ID, (k | ks) ? 1u : 0u);
          umma_commit(&sh.empty[slot]);
          if (++slot == p.stages) { slot = 0; ++round; }
        }
        if (ok) umma_commit(&sh.afull[acc]);
      }
    }
  } else if (warp >= 6) {                      // (GT_GATHER) eight lanes a row, four rows an instruction
    const __nv_bfloat16* x = reinterpret_cast<const __nv_bfloat16*>(p.a.x);
    const int r0 = (warp - 6) * 32 + (lane >> 3), piece = lane & 7;
    bool ok = true;
    int slot = 0, round = 0, late = 0, pending = 0;          // late: the slot to publish next
    for (int t = blockIdx.x; ok && t < total; t += gridDim.x) {
      const GtTile tl = gt_tile<BN>(p, sh, t);
      const __nv_bfloat16* src[8];
#pragma unroll
      for (int i = 0; i < 8; ++i) {
        const int at = tl.first + min(r0 + 4 * i, tl.count - 1);
        src[i] = x + (int64_t)min(max(p.a.rows[at], 0), p.a.src_rows - 1) * p.a.x_stride + piece * 8;
      }
      for (int k = 0; k < p.kb; ++k) {
        ok = __all_sync(0xffffffffu, mbar_wait(&sh.empty[slot], (round & 1) ^ 1, abortp, p.error_word, 945));
        if (!ok) break;
        const uint32_t dst = smem_u32(ring + slot * STAGE);
        const int bytes = k * 64 + piece * 8 < p.a.K ? 16 : 0;
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int r = r0 + 4 * i;
          gt_copy16(dst + r * 128 + ((piece ^ (r & 7)) << 4), bytes ? src[i] + k * 64 : x, bytes);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (++pending > GT_LAG) {
          gt_publish<GT_LAG>(&sh.full[late], lane);
          --pending;
          if (++late == p.stages) late = 0;
        }
        if (++slot == p.stages) { slot = 0; ++round; }
      }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    for (; ok && pending > 0; --pending) {
      gt_publish<0>(&sh.full[late], lane);
      if (++late == p.stages) late = 0;
    }
  } else {
    const int q = warp & 3, row = q * 32 + lane;
    const uint32_t lane_base = tmem + (static_cast<uint32_t>(q * 32) << 16);
    const bool vec = p.a.Nout % 8 == 0;
    constexpr bool GATED = ACT == ZP_ACT_SILU_MUL;
    __nv_bfloat16* out = reinterpret_cast<__nv_bfloat16*>(p.a.out);
    bool ok = true;
    int i = 0;
    for (int t = blockIdx.x; t < total; t += gridDim.x, ++i) {
      const GtTile tl = gt_tile<BN>(p, sh, t);
      const int acc = i & 1;
      ok = __all_sync(0xffffffffu, mbar_wait(&sh.afull[acc], (i >> 1) & 1, abortp, p.error_word, 944));
      if (!ok) break;
      fence_after_sync();
      if (q * 32 < tl.count) {
        __nv_bfloat16* o = GATED ? out + (int64_t)(tl.first + row) * (p.a.Nout >> 1) + (tl.n0 >> 1)
                                 : out + (int64_t)(tl.first + row) * p.a.Nout + tl.n0;
        const float scale = GATED && p.a.row_scale && row < tl.count ? p.a.row_scale[tl.first + row] : 1.f;
        const int cols = min(BN, p.a.Nout - tl.n0);
        for (int c0 = 0; c0 < cols; c0 += 32) {
          float v[32];
          tmem_ld32(lane_base + acc * BN + c0, v);
          if constexpr (GATED) {             // 16 gates, then the 16 entries of `up` that they meet
            if (row < tl.count) {
#pragma unroll
              for (int c = 0; c < 16; c += 8) {
                uint32_t w[4];
#pragma unroll
                for (int u = 0; u < 8; u += 2) {
                  const float g0 = v[c + u] * scale, g1 = v[c + u + 1] * scale;
                  const float y0 = __fdividef(g0, 1.f + __expf(fminf(-g0, 80.f))) * (v[16 + c + u] * scale);
                  const float y1 = __fdividef(g1, 1.f + __expf(fminf(-g1, 80.f))) * (v[17 + c + u] * scale);
                  const __nv_bfloat162 x = __floats2bfloat162_rn(y0, y1);
                  w[u >> 1] = *reinterpret_cast<const uint32_t*>(&x);
                }
                st16(o + (c0 >> 1) + c, make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]));
              }
            }
            continue;
          }
          if (ACT == ZP_ACT_RELU_SQUARED) {
#pragma unroll
            for (int u = 0; u < 32; ++u) { const float z = fmaxf(v[u], 0.f); v[u] = z * z; }
          }
          if (row < tl.count) {
#pragma unroll
            for (int c = 0; c < 32; c += 8) {
              if (vec) {
                uint32_t w[4];
#pragma unroll
                for (int u = 0; u < 4; ++u) {
                  const __nv_bfloat162 x = __floats2bfloat162_rn(v[c + 2 * u], v[c + 2 * u + 1]);
                  w[u] = *reinterpret_cast<const uint32_t*>(&x);
                }
                if (c0 + c < cols) st16(o + c0 + c, make_int4((int)w[0], (int)w[1], (int)w[2], (int)w[3]));
              } else {
#pragma unroll
                for (int u = 0; u < 8; ++u)
                  if (c0 + c + u < cols) o[c0 + c + u] = __float2bfloat16_rn(v[c + u]);
              }
            }
          }
        }
      }
      fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&sh.aempty[acc]);
    }
  }
  fence_before_sync();
  __syncthreads();
  if (warp == 0) {
    fence_after_sync();
    tmem_dealloc(tmem, 2 * BN);
  }
}

bool grouped_tc_supports(const GroupedArgs& a, int dtype) {
  return dtype == ZP_DTYPE_BF16 && a.K % 8 == 0 && a.x_stride % 8 == 0 && a.E <= GT_MAXE &&
         ((uintptr_t)a.x | (uintptr_t)a.w | (uintptr_t)a.out) % 16 == 0;
}

template <int BN, int ACT, int MODE> static int gt_launch(const GroupedArgs& a, cudaStream_t st) {
  constexpr int STAGE = GT_A + BN * 128;
  GtParams p;
  p.a = a;
  p.ntn = (a.Nout + BN - 1) / BN;
  p.kb = (a.K + 63) / 64;
  p.stages = (232448 - 1024 - (int)sizeof(GtShared)) / STAGE;
  if (p.stages > GT_MAXS) p.stages = GT_MAXS;
  p.error_word = device_error_word();
  if (!p.error_word) { set_error("zp_grouped_gemm(tcgen05): no device error word"); return ZP_ERR_CUDA; }
  const int smem = 1024 + p.stages * STAGE + (int)sizeof(GtShared);
  CUtensorMap tmX, tmW;
  if (MODE == GT_TILE) {
    const uint64_t all = (uint64_t)a.src_rows * a.x_stride;
    const uint64_t dims[5] = {(uint64_t)a.K, (uint64_t)a.src_rows, 1, 1, 1}, strides[4] = {(uint64_t)a.x_stride, all, all, all};
    const uint32_t box[5] = {64, 128, 1, 1, 1};
    if (int rc = make_tensor_map_5d(&tmX, UmmaFmt<__nv_bfloat16>::tm, a.x, dims, strides, box, 2)) return rc;
  } else {
    if (int rc = make_tensor_map_rows(&tmX, UmmaFmt<__nv_bfloat16>::tm, a.x, (uint64_t)a.K, (uint64_t)a.src_rows, (uint64_t)a.x_stride, 2)) return rc;
  }
  {
    const uint64_t per = (uint64_t)a.Nout * a.K;
    const uint64_t dims[5] = {(uint64_t)a.K, (uint64_t)a.Nout, (uint64_t)a.E, 1, 1};
    const uint64_t strides[4] = {(uint64_t)a.K, per, per * a.E, per * a.E};
    const uint32_t box[5] = {64, BN, 1, 1, 1};
    if (int rc = make_tensor_map_5d(&tmW, UmmaFmt<__nv_bfloat16>::tm, a.w, dims, strides, box, 2)) return rc;
  }
  const auto kern = grouped_gemm_tc_kernel<BN, ACT, MODE>;
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  if (e != cudaSuccess) { set_error("zp_grouped_gemm(tcgen05): %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  const int64_t most = ((int64_t)a.places / 128 + (a.places < a.E ? a.places : a.E)) * p.ntn;   // tiles, at most
  kern<<<(int)(most < 148 ? (most < 1 ? 1 : most) : 148), gt_threads<MODE>(), smem, st>>>(tmX, tmW, p);
  return check_launch("zp_grouped_gemm(tcgen05)");
}

template <int BN, int ACT> static int gt_pick(const GroupedArgs& a, bool many, cudaStream_t st) {
  if (!many) return gt_launch<BN, ACT, GT_FEW>(a, st);
  return a.rows ? gt_launch<BN, ACT, GT_GATHER>(a, st) : gt_launch<BN, ACT, GT_TILE>(a, st);
}

int grouped_gemm_tc(const GroupedArgs& a, cudaStream_t st) {
  // few places per expert: the weights stream through, and narrower tiles spread them better over the SMs
  const bool many = a.places >= 32 * (int64_t)a.E, wide = many && a.Nout > 128;
  auto by_act = [&](auto act) {
    constexpr int ACT = decltype(act)::value;
    return wide ? gt_pick<256, ACT>(a, many, st) : gt_pick<128, ACT>(a, many, st);
  };
  if (a.act == ZP_ACT_SILU_MUL) return by_act(std::integral_constant<int, ZP_ACT_SILU_MUL>{});
  if (a.act == ZP_ACT_RELU_SQUARED) return by_act(std::integral_constant<int, ZP_ACT_RELU_SQUARED>{});
  return by_act(std::integral_constant<int, ZP_ACT_NONE>{});
}

}  // namespace zp
