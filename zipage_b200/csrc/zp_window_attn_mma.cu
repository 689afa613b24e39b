// Sliding-window, soft-capped attention for 16-bit paged caches of any head sizes (keys and values
// padded to multiples of 16, up to 256) on warp-level tensor-core MMAs: a prefill kernel (flash tiling, 64
// queries x 64 keys) and a split-KV decode kernel.
//
// Scores, soft cap and softmax weights are fp32.  The weights enter the second product as a pair of
// 16-bit numbers (hi + lo, ~16 significant bits), so that no step of the softmax is rounded to the
// tensor dtype.
//
// The soft cap bounds every score to [-c, c].  With a moderate cap (2 c log2(e) <= 100) and a bf16
// operand (fp32's exponent range) the prefill kernel exponentiates against the bound c itself: no
// running maximum, no rescaling of the accumulators, and, with E = exp(2 s / c),
//   c tanh(s / c) - c = -2 c / (1 + E),
// so a weight costs two exponentials and one reciprocal.  Caps up to c log2(e) = 100 do the same against 0: weights
// within 2^-100 .. 2^100.
#include "zp_mma.cuh"
#include "zp_window_attn.cuh"

namespace zp {

constexpr int WM_THREADS = 128;
constexpr int WM_TQ = 64, WM_TK = 64;
constexpr float WM_LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

// score in log2 units after scale and cap, the distance's bias not yet taken off (c = cap * log2 e, y = 2 scale log2 e / cap)
struct CapConst { float lin, y, c, cap, ref; };
__device__ __forceinline__ CapConst cap_const(const WinArgs& a) {
  CapConst k;
  k.lin = a.scale * WM_LOG2E; k.cap = a.softcap;
  k.y = a.softcap > 0.f ? 2.f * WM_LOG2E * a.scale / a.softcap : 0.f;
  k.c = a.softcap * WM_LOG2E;
  k.ref = 2.f * k.c <= 100.f ? k.c : 0.f;
  return k;
}
__device__ __forceinline__ float capped(float s, const CapConst& k, float scale) {
  if (k.cap <= 0.f) return s * k.lin;
  // 1 - 2 / (1 + e^2x) has an absolute error of a few 2^-23: fine in units of an ordinary cap
  if (k.cap <= 100.f) return fmaf(-2.f * k.c, rcp(1.f + ex2(s * k.y)), k.c);
  return k.c * tanhf(s * scale / k.cap);
}

// the two 16-bit halves of a pair of fp32 weights
template <typename T> __device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo);
template <> __device__ __forceinline__ void split2<__nv_bfloat16>(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __bfloat1622float2(h);
  lo = pack2<__nv_bfloat16>(a - f.x, b - f.y);
}
template <> __device__ __forceinline__ void split2<__half>(float a, float b, uint32_t& hi, uint32_t& lo) {
  const __half2 h = __floats2half2_rn(a, b);
  hi = *reinterpret_cast<const uint32_t*>(&h);
  const float2 f = __half22float2(h);
  lo = pack2<__half>(a - f.x, b - f.y);
}

// byte stride of a row of `elems` 16-bit elements in shared memory: an odd number of 16-byte
// chunks, which makes the eight rows of an ldmatrix land in different banks
__host__ __device__ __forceinline__ int row_bytes(int elems) { return elems * 2 + 16; }

// (EXACT kernels: KP = VP = 16 NV16, so every size below is a compile-time constant)
// 64 rows of one head of the K (V) page that holds key0, rows past n_valid filled with zeros
__device__ __forceinline__ void load_page_rows(unsigned char* dst, const char* cache, int64_t slot0, int Hkv, int hk,
                                               int elems, int n_valid) {
  const int per = elems / 8, rb = row_bytes(elems);
  const char* base = cache + ((slot0 * Hkv + hk) * elems) * 2;
  const int64_t stride = (int64_t)Hkv * elems * 2;
  for (int i = threadIdx.x; i < WM_TK * per; i += WM_THREADS) {
    const int r = i / per, c = i - r * per;
    const int ok = r < n_valid ? 16 : 0;
    cp_async16(dst + r * rb + c * 16, base + (ok ? r : 0) * stride + c * 16, ok);
  }
}

template <typename T, int NV16, bool BOUNDED, bool EXACT>
__global__ void __launch_bounds__(WM_THREADS) window_prefill_mma_kernel(const WinArgs a) {
  extern __shared__ __align__(128) unsigned char smem[];   // Q | 2 x (K | V)
  const int b = blockIdx.z, h = blockIdx.y;
  const WinSeq sq = win_seq(a, b);
  const int qi0 = blockIdx.x * WM_TQ;
  if (qi0 >= sq.count) return;
  const int hk = h / (a.Hq / a.Hkv);
  const int KP = EXACT ? NV16 * 16 : a.KP, VP = EXACT ? NV16 * 16 : a.VP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int rbk = row_bytes(KP), rbv = row_bytes(VP);
  unsigned char* sQ = smem;
  unsigned char* sKV = smem + WM_TQ * rbk;
  const int stage_bytes = WM_TK * (rbk + rbv);
  const int rows = min(WM_TQ, sq.count - qi0);
  const int p_first = sq.pos0 + qi0, p_last = p_first + rows - 1;   // positions of the tile's rows
  const WinTiles wt = win_tiles(a, p_first, p_last, WM_TK);

  auto load_tile = [&](int t, int stage) {
    const int key0 = t * WM_TK;
    const int64_t slot0 = (int64_t)win_page(a, b, key0) * a.BS + key0 % a.BS;
    unsigned char* ks = sKV + stage * stage_bytes;
    const int n_valid = min(WM_TK, sq.ctx - key0);
    load_page_rows(ks, reinterpret_cast<const char*>(a.k), slot0, a.Hkv, hk, KP, n_valid);
    load_page_rows(ks + WM_TK * rbk, reinterpret_cast<const char*>(a.v), slot0, a.Hkv, hk, VP, n_valid);
  };
  load_tile(wt.tile(0), 0);
  cp_async_commit();
  {  // the query tile, its padding columns and missing rows zero
    const T* qp = reinterpret_cast<const T*>(a.q) + (int64_t)(sq.row0 + qi0) * a.q_stride + (int64_t)h * a.D;
    if (a.D % 8 == 0 && a.q_stride % 8 == 0 && (uintptr_t)a.q % 16 == 0) {
      const int per = KP / 8;
      for (int i = tid; i < WM_TQ * per; i += WM_THREADS) {
        const int r = i / per, c = i - r * per;
        int4 v = make_int4(0, 0, 0, 0);
        if (r < rows && c * 8 < a.D) v = ld16(qp + r * a.q_stride + c * 8);
        st16(sQ + r * rbk + c * 16, v);
      }
    } else {
      for (int i = tid; i < WM_TQ * KP; i += WM_THREADS) {
        const int r = i / KP, c = i - r * KP;
        *reinterpret_cast<T*>(sQ + r * rbk + c * 2) = (r < rows && c < a.D) ? qp[r * a.q_stride + c] : Elem<T>::from_f32(0.f);
      }
    }
  }
  const CapConst cc = cap_const(a);
  const int row0 = warp * 16 + g;                 // this thread's two query rows of the tile
  const int pos0 = p_first + row0, pos1 = pos0 + 8;
  const int lo0 = win_first(a, pos0), lo1 = win_first(a, pos1);
  const int wp0 = p_first + warp * 16, wp1 = wp0 + 15;   // positions of the warp's first and last row
  const int nv16 = VP / 16, nk16 = KP / 16;
  float o[2 * NV16][4];
#pragma unroll
  for (int i = 0; i < 2 * NV16; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;

  const float slope = win_slope2(a, h);
  for (int ti = 0; ti < wt.n; ++ti) {
    if (ti + 1 < wt.n) load_tile(wt.tile(ti + 1), (ti + 1) & 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const unsigned char* ks = sKV + (ti & 1) * stage_bytes;
    const unsigned char* vs = ks + WM_TK * rbk;
    const int key0 = wt.tile(ti) * WM_TK;
    auto hidden = [&](int key, int pos, int lo) { return key > pos || (key < lo && key >= a.keep); };
    if (key0 <= wp1 && (key0 + WM_TK > win_first(a, wp0) || key0 < a.keep)) {   // else the warp's rows see none of these keys
      float s[8][4];
#pragma unroll
      for (int nb = 0; nb < 8; ++nb) { s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.f; }
#pragma unroll 2
      for (int kk = 0; kk < nk16; ++kk) {
        uint32_t qa[4];
        ldmatrix_x4(qa, sQ + (warp * 16 + (lane & 15)) * rbk + kk * 32 + (lane >> 4) * 16);
#pragma unroll
        for (int np = 0; np < 4; ++np) {
          uint32_t bf[4];
          ldmatrix_x4(bf, ks + (np * 16 + (lane & 7) + (lane >> 4) * 8) * rbk + kk * 32 + ((lane >> 3) & 1) * 16);
          mma16816<T>(s[2 * np], qa, bf[0], bf[1]);
          mma16816<T>(s[2 * np + 1], qa, bf[2], bf[3]);
        }
      }
      const bool whole = key0 + WM_TK - 1 <= wp0 && (key0 >= win_first(a, wp1) || key0 + WM_TK <= a.keep);   // no masking in this tile
      if constexpr (BOUNDED) {
#pragma unroll
        for (int nb = 0; nb < 8; ++nb) {
#pragma unroll
          for (int j = 0; j < 4; ++j) s[nb][j] = ex2(fmaf(-2.f * cc.c, rcp(1.f + ex2(s[nb][j] * cc.y)), cc.c - cc.ref));
          if (!whole) {
            const int key = key0 + nb * 8 + 2 * tq;
            if (hidden(key, pos0, lo0)) s[nb][0] = 0.f;
            if (hidden(key + 1, pos0, lo0)) s[nb][1] = 0.f;
            if (hidden(key, pos1, lo1)) s[nb][2] = 0.f;
            if (hidden(key + 1, pos1, lo1)) s[nb][3] = 0.f;
          }
          l0 += s[nb][0] + s[nb][1];
          l1 += s[nb][2] + s[nb][3];
        }
      } else {
        float mx0 = m0, mx1 = m1;
#pragma unroll
        for (int nb = 0; nb < 8; ++nb) {
          const int key = key0 + nb * 8 + 2 * tq;
#pragma unroll
          for (int j = 0; j < 4; ++j)
            s[nb][j] = fmaf(-slope, (float)((j < 2 ? pos0 : pos1) - key - (j & 1)), capped(s[nb][j], cc, a.scale));
          if (!whole) {
            if (hidden(key, pos0, lo0)) s[nb][0] = -INFINITY;
            if (hidden(key + 1, pos0, lo0)) s[nb][1] = -INFINITY;
            if (hidden(key, pos1, lo1)) s[nb][2] = -INFINITY;
            if (hidden(key + 1, pos1, lo1)) s[nb][3] = -INFINITY;
          }
          mx0 = fmaxf(mx0, fmaxf(s[nb][0], s[nb][1]));
          mx1 = fmaxf(mx1, fmaxf(s[nb][2], s[nb][3]));
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float c0 = mx0 == -INFINITY ? 1.f : ex2(m0 - mx0);
        const float c1 = mx1 == -INFINITY ? 1.f : ex2(m1 - mx1);
        const float e0 = mx0 == -INFINITY ? 0.f : mx0, e1 = mx1 == -INFINITY ? 0.f : mx1;
        m0 = mx0; m1 = mx1;
        l0 *= c0; l1 *= c1;
#pragma unroll
        for (int nb = 0; nb < 8; ++nb) {
          s[nb][0] = ex2(s[nb][0] - e0); s[nb][1] = ex2(s[nb][1] - e0);
          s[nb][2] = ex2(s[nb][2] - e1); s[nb][3] = ex2(s[nb][3] - e1);
          l0 += s[nb][0] + s[nb][1];
          l1 += s[nb][2] + s[nb][3];
        }
#pragma unroll
        for (int i = 0; i < 2 * NV16; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
      }
#pragma unroll
      for (int kk = 0; kk < 4; ++kk) {
        uint32_t hi[4], lo[4];
        split2<T>(s[2 * kk][0], s[2 * kk][1], hi[0], lo[0]);
        split2<T>(s[2 * kk][2], s[2 * kk][3], hi[1], lo[1]);
        split2<T>(s[2 * kk + 1][0], s[2 * kk + 1][1], hi[2], lo[2]);
        split2<T>(s[2 * kk + 1][2], s[2 * kk + 1][3], hi[3], lo[3]);
#pragma unroll
        for (int np = 0; np < NV16; ++np) {
          if (np < nv16) {
            uint32_t bf[4];
            ldmatrix_x4_trans(bf, vs + (kk * 16 + (lane & 15)) * rbv + np * 32 + (lane >> 4) * 16);
            mma16816<T>(o[2 * np], hi, bf[0], bf[1]);
            mma16816<T>(o[2 * np], lo, bf[0], bf[1]);
            mma16816<T>(o[2 * np + 1], hi, bf[2], bf[3]);
            mma16816<T>(o[2 * np + 1], lo, bf[2], bf[3]);
          }
        }
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  const int64_t grow = sq.row0 + qi0;
  if (a.sink) {
    const float s2 = win_sink2(a, h), r0 = BOUNDED ? cc.ref : m0, r1 = BOUNDED ? cc.ref : m1;
    l0 += ex2(s2 - r0); l1 += ex2(s2 - r1);
  }
  const float i0 = l0 > 0.f && row0 < rows ? win_head_factor<T>(a, grow + row0, h) / l0 : 0.f;
  const float i1 = l1 > 0.f && row0 + 8 < rows ? win_head_factor<T>(a, grow + row0 + 8, h) / l1 : 0.f;
  T* ob = reinterpret_cast<T*>(a.out) + (int64_t)(sq.row0 + qi0) * a.out_stride + (int64_t)h * a.DV;
  const bool pairs = a.DV % 2 == 0 && a.out_stride % 2 == 0;
#pragma unroll
  for (int i = 0; i < 2 * NV16; ++i) {
    const int d = i * 8 + 2 * tq;
    if (d >= a.DV) continue;
    if (a.gate_mode == WIN_GATE_ENTRY) {
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int r = row0 + (j >> 1) * 8;
        if (r < rows && d + (j & 1) < a.DV) o[i][j] *= win_entry_factor<T>(a, grow + r, h, d + (j & 1));
      }
    }
    if (pairs) {
      if (row0 < rows) *reinterpret_cast<uint32_t*>(ob + row0 * a.out_stride + d) = pack2<T>(o[i][0] * i0, o[i][1] * i0);
      if (row0 + 8 < rows) *reinterpret_cast<uint32_t*>(ob + (row0 + 8) * a.out_stride + d) = pack2<T>(o[i][2] * i1, o[i][3] * i1);
    } else {
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        if (d + j >= a.DV) continue;
        if (row0 < rows) ob[row0 * a.out_stride + d + j] = Elem<T>::from_f32(o[i][j] * i0);
        if (row0 + 8 < rows) ob[(row0 + 8) * a.out_stride + d + j] = Elem<T>::from_f32(o[i][2 + j] * i1);
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------
// Decode: one block per (sequence, kv head, split of the visible keys).  The G query heads of the
// group are the 16-row A operand; each of the four warps takes 16 keys of a 64-key tile; warps, then
// splits, are merged with the (max, sum, weighted output) rule.
// ---------------------------------------------------------------------------------------------
template <typename T, int NV16, bool EXACT>
__global__ void __launch_bounds__(WM_THREADS) window_decode_mma_kernel(const WinArgs a) {
  extern __shared__ __align__(128) unsigned char smem[];   // Q (16 rows) | 2 x (K | V); reused by the merge
  const int b = blockIdx.x, hk = blockIdx.y, split = blockIdx.z;
  const WinSeq sq = win_seq(a, b);
  if (sq.count == 0) return;
  const int G = a.Hq / a.Hkv;
  const int KP = EXACT ? NV16 * 16 : a.KP, VP = EXACT ? NV16 * 16 : a.VP;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, tq = lane & 3;
  const int rbk = row_bytes(KP), rbv = row_bytes(VP);
  unsigned char* sQ = smem;
  unsigned char* sKV = smem + 16 * rbk;
  const int stage_bytes = WM_TK * (rbk + rbv);
  const int pos = sq.ctx - 1, lo = win_first(a, pos);
  const WinTiles wt = win_tiles(a, pos, pos, WM_TK);
  const int per = (wt.n + a.nsplit - 1) / a.nsplit;
  const int t0 = split * per, t1 = min(t0 + per, wt.n);   // tiles [t0, t1) of the list

  auto load_tile = [&](int t, int stage) {
    const int key0 = t * WM_TK;
    const int64_t slot0 = (int64_t)win_page(a, b, key0) * a.BS + key0 % a.BS;
    unsigned char* ks = sKV + stage * stage_bytes;
    const int n_valid = min(WM_TK, sq.ctx - key0);
    load_page_rows(ks, reinterpret_cast<const char*>(a.k), slot0, a.Hkv, hk, KP, n_valid);
    load_page_rows(ks + WM_TK * rbk, reinterpret_cast<const char*>(a.v), slot0, a.Hkv, hk, VP, n_valid);
  };
  if (t0 < t1) load_tile(wt.tile(t0), 0);
  cp_async_commit();
  {
    const T* qp = reinterpret_cast<const T*>(a.q) + (int64_t)sq.row0 * a.q_stride + (int64_t)hk * G * a.D;
    for (int i = tid; i < 16 * KP; i += WM_THREADS) {
      const int r = i / KP, c = i - r * KP;
      *reinterpret_cast<T*>(sQ + r * rbk + c * 2) = (r < G && c < a.D) ? qp[r * a.D + c] : Elem<T>::from_f32(0.f);
    }
  }
  const CapConst cc = cap_const(a);
  const int nv16 = VP / 16, nk16 = KP / 16;
  float o[2 * NV16][4];
#pragma unroll
  for (int i = 0; i < 2 * NV16; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
  float m0 = -INFINITY, m1 = -INFINITY, l0 = 0.f, l1 = 0.f;   // rows g and g + 8
  const float slope0 = g < G ? win_slope2(a, hk * G + g) : 0.f, slope1 = g + 8 < G ? win_slope2(a, hk * G + g + 8) : 0.f;

  for (int t = t0; t < t1; ++t) {
    if (t + 1 < t1) load_tile(wt.tile(t + 1), (t + 1 - t0) & 1);
    cp_async_commit();
    cp_async_wait<1>();
    __syncthreads();
    const unsigned char* ks = sKV + ((t - t0) & 1) * stage_bytes;
    const unsigned char* vs = ks + WM_TK * rbk;
    const int kw = warp * 16;
    float s[2][4];
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) { s[nb][0] = s[nb][1] = s[nb][2] = s[nb][3] = 0.f; }
#pragma unroll 2
    for (int kk = 0; kk < nk16; ++kk) {
      uint32_t qa[4], bf[4];
      ldmatrix_x4(qa, sQ + (lane & 15) * rbk + kk * 32 + (lane >> 4) * 16);
      ldmatrix_x4(bf, ks + (kw + (lane & 7) + (lane >> 4) * 8) * rbk + kk * 32 + ((lane >> 3) & 1) * 16);
      mma16816<T>(s[0], qa, bf[0], bf[1]);
      mma16816<T>(s[1], qa, bf[2], bf[3]);
    }
    float mx0 = m0, mx1 = m1;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      const int key = wt.tile(t) * WM_TK + kw + nb * 8 + 2 * tq;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int kj = key + (j & 1);
        const float sc = fmaf(-((j < 2) ? slope0 : slope1), (float)(pos - kj), capped(s[nb][j], cc, a.scale));
        s[nb][j] = (kj <= pos && (kj >= lo || kj < a.keep)) ? sc : -INFINITY;
      }
      mx0 = fmaxf(mx0, fmaxf(s[nb][0], s[nb][1]));
      mx1 = fmaxf(mx1, fmaxf(s[nb][2], s[nb][3]));
    }
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
    mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
    mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
    const float c0 = mx0 == -INFINITY ? 1.f : ex2(m0 - mx0);
    const float c1 = mx1 == -INFINITY ? 1.f : ex2(m1 - mx1);
    const float e0 = mx0 == -INFINITY ? 0.f : mx0, e1 = mx1 == -INFINITY ? 0.f : mx1;
    m0 = mx0; m1 = mx1;
    l0 *= c0; l1 *= c1;
#pragma unroll
    for (int nb = 0; nb < 2; ++nb) {
      s[nb][0] = ex2(s[nb][0] - e0); s[nb][1] = ex2(s[nb][1] - e0);
      s[nb][2] = ex2(s[nb][2] - e1); s[nb][3] = ex2(s[nb][3] - e1);
      l0 += s[nb][0] + s[nb][1];
      l1 += s[nb][2] + s[nb][3];
    }
    uint32_t hi[4], lw[4];
    split2<T>(s[0][0], s[0][1], hi[0], lw[0]);
    split2<T>(s[0][2], s[0][3], hi[1], lw[1]);
    split2<T>(s[1][0], s[1][1], hi[2], lw[2]);
    split2<T>(s[1][2], s[1][3], hi[3], lw[3]);
#pragma unroll
    for (int i = 0; i < 2 * NV16; ++i) { o[i][0] *= c0; o[i][1] *= c0; o[i][2] *= c1; o[i][3] *= c1; }
#pragma unroll
    for (int np = 0; np < NV16; ++np) {
      if (np < nv16) {
        uint32_t bf[4];
        ldmatrix_x4_trans(bf, vs + (kw + (lane & 15)) * rbv + np * 32 + (lane >> 4) * 16);
        mma16816<T>(o[2 * np], hi, bf[0], bf[1]);
        mma16816<T>(o[2 * np], lw, bf[0], bf[1]);
        mma16816<T>(o[2 * np + 1], hi, bf[2], bf[3]);
        mma16816<T>(o[2 * np + 1], lw, bf[2], bf[3]);
      }
    }
    __syncthreads();
  }
  cp_async_wait<0>();
  l0 += __shfl_xor_sync(0xffffffffu, l0, 1); l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
  l1 += __shfl_xor_sync(0xffffffffu, l1, 1); l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
  __syncthreads();
  const int W = VP + 2;
  float* mbuf = reinterpret_cast<float*>(smem);   // [4 warps][16 rows][VP + 2]: O, m, l
  {
    float* w0 = mbuf + (warp * 16 + g) * W;
    float* w1 = w0 + 8 * W;
#pragma unroll
    for (int i = 0; i < 2 * NV16; ++i)
      if (i < 2 * nv16) {
        w0[i * 8 + 2 * tq] = o[i][0]; w0[i * 8 + 2 * tq + 1] = o[i][1];
        w1[i * 8 + 2 * tq] = o[i][2]; w1[i * 8 + 2 * tq + 1] = o[i][3];
      }
    if (tq == 0) { w0[VP] = m0; w0[VP + 1] = l0; w1[VP] = m1; w1[VP + 1] = l1; }
  }
  __syncthreads();
  for (int i = tid; i < G * a.DV; i += WM_THREADS) {
    const int row = i / a.DV, d = i - row * a.DV;
    float M = -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) M = fmaxf(M, mbuf[(w * 16 + row) * W + VP]);
    float num = 0.f, den = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      const float* rr = mbuf + (w * 16 + row) * W;
      const float wgt = rr[VP] == -INFINITY ? 0.f : ex2(rr[VP] - M);
      num = fmaf(wgt, rr[d], num);
      den = fmaf(wgt, rr[VP + 1], den);
    }
    const int hq = hk * G + row;
    if (a.nsplit == 1) {
      if (a.sink) den += ex2(win_sink2(a, hq) - M);
      const float f = win_head_factor<T>(a, sq.row0, hq) * win_entry_factor<T>(a, sq.row0, hq, d);
      reinterpret_cast<T*>(a.out)[(int64_t)sq.row0 * a.out_stride + (int64_t)hq * a.DV + d] =
          Elem<T>::from_f32(den > 0.f ? num / den * f : 0.f);
    } else {
      float* pp = a.part + (((int64_t)b * a.Hq + hq) * a.nsplit + split) * W;
      pp[d] = num;
      if (d == 0) { pp[VP] = M; pp[VP + 1] = den; }
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(128) window_decode_merge_kernel(const WinArgs a) {
  const int b = blockIdx.x, hq = blockIdx.y, W = a.VP + 2;
  const WinSeq sq = win_seq(a, b);
  if (sq.count == 0) return;
  const float* base = a.part + ((int64_t)b * a.Hq + hq) * a.nsplit * W;
  float M = -INFINITY;
  for (int s = 0; s < a.nsplit; ++s) M = fmaxf(M, base[s * W + a.VP]);
  for (int d = threadIdx.x; d < a.DV; d += blockDim.x) {
    float num = 0.f, den = 0.f;
    for (int s = 0; s < a.nsplit; ++s) {
      const float* rr = base + s * W;
      if (rr[a.VP] == -INFINITY) continue;   // a split without keys
      const float w = ex2(rr[a.VP] - M);
      num = fmaf(w, rr[d], num);
      den = fmaf(w, rr[a.VP + 1], den);
    }
    if (a.sink) den += ex2(win_sink2(a, hq) - M);
    const float f = win_head_factor<T>(a, sq.row0, hq) * win_entry_factor<T>(a, sq.row0, hq, d);
    reinterpret_cast<T*>(a.out)[(int64_t)sq.row0 * a.out_stride + (int64_t)hq * a.DV + d] =
        Elem<T>::from_f32(den > 0.f ? num / den * f : 0.f);
  }
}

static int prefill_smem(const WinArgs& a) {
  return WM_TQ * row_bytes(a.KP) + 2 * WM_TK * (row_bytes(a.KP) + row_bytes(a.VP));
}
static int decode_smem(const WinArgs& a) {
  const int tiles = 16 * row_bytes(a.KP) + 2 * WM_TK * (row_bytes(a.KP) + row_bytes(a.VP));
  const int merge = 4 * 16 * (a.VP + 2) * (int)sizeof(float);
  return tiles > merge ? tiles : merge;
}

bool window_mma_supports(const WinArgs& a) { return a.KP <= 256 && a.VP <= 256 && a.Hq / a.Hkv <= 16; }

int window_decode_splits(int B, int Hkv, int span) {
  const int target = 148 * 4, tiles = (span + WM_TK - 1) / WM_TK;
  int s = (target + B * Hkv - 1) / (B * Hkv);
  if (s > (tiles + 1) / 2) s = (tiles + 1) / 2;   // at least two tiles each
  if (s > 32) s = 32;
  return s < 1 ? 1 : s;
}

template <typename K> static int set_smem(K kern, int bytes, const char* what) {
  cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
  if (e != cudaSuccess) { set_error("%s: %s", what, cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  return ZP_OK;
}

template <typename T, int NV16, bool BOUNDED>
static int launch_prefill(const WinArgs& a, int max_q, cudaStream_t st) {
  constexpr bool CAN = NV16 <= 8;      // (larger tiles have no registers left for it)
  const bool exact = CAN && a.KP == NV16 * 16 && a.VP == NV16 * 16;
  auto kern = exact ? window_prefill_mma_kernel<T, NV16, BOUNDED, CAN> : window_prefill_mma_kernel<T, NV16, BOUNDED, false>;
  const int smem = prefill_smem(a);
  if (int rc = set_smem(kern, smem, "zp_window_attention(prefill)")) return rc;
  kern<<<dim3((max_q + WM_TQ - 1) / WM_TQ, a.Hq, a.B), WM_THREADS, smem, st>>>(a);
  return check_launch("zp_window_attention(prefill)");
}
template <typename T, bool BOUNDED>
static int prefill_by_size(const WinArgs& a, int max_q, cudaStream_t st) {
  if (a.VP <= 64) return launch_prefill<T, 4, BOUNDED>(a, max_q, st);
  if (a.VP <= 128) return launch_prefill<T, 8, BOUNDED>(a, max_q, st);
  return launch_prefill<T, 16, BOUNDED>(a, max_q, st);
}
int window_prefill_mma(const WinArgs& a, int max_q, int dtype, cudaStream_t st) {
  const bool bounded = a.softcap > 0.f && a.softcap * WM_LOG2E <= 100.f && !a.slopes;
  if (dtype == ZP_DTYPE_F16) return prefill_by_size<__half, false>(a, max_q, st);   // (2^-100 does not fit fp16)
  if (bounded) return prefill_by_size<__nv_bfloat16, true>(a, max_q, st);
  return prefill_by_size<__nv_bfloat16, false>(a, max_q, st);
}

template <typename T, int NV16>
static int launch_decode(const WinArgs& a, cudaStream_t st) {
  const bool exact = a.KP == NV16 * 16 && a.VP == NV16 * 16;
  auto kern = exact ? window_decode_mma_kernel<T, NV16, true> : window_decode_mma_kernel<T, NV16, false>;
  const int smem = decode_smem(a);
  if (int rc = set_smem(kern, smem, "zp_window_attention(decode)")) return rc;
  kern<<<dim3(a.B, a.Hkv, a.nsplit), WM_THREADS, smem, st>>>(a);
  if (int rc = check_launch("zp_window_attention(decode)")) return rc;
  if (a.nsplit == 1) return ZP_OK;
  window_decode_merge_kernel<T><<<dim3(a.B, a.Hq), 128, 0, st>>>(a);
  return check_launch("zp_window_attention(merge)");
}
template <typename T> static int decode_by_size(const WinArgs& a, cudaStream_t st) {
  if (a.VP <= 64) return launch_decode<T, 4>(a, st);
  if (a.VP <= 128) return launch_decode<T, 8>(a, st);
  return launch_decode<T, 16>(a, st);
}
int window_decode_mma(const WinArgs& a, int dtype, cudaStream_t st) {
  if (dtype == ZP_DTYPE_BF16) return decode_by_size<__nv_bfloat16>(a, st);
  return decode_by_size<__half>(a, st);
}

}  // namespace zp
