// Short causal convolution over time, per channel, with an optional bias and silu: portions of prompts.  A thread owns V adjacent
// channels and walks a run of tokens in batches, the next batch's loads in flight.  (Decoded tokens: zp_conv.cuh.)
#include "zp_tc.cuh"       // packed fp32 pairs

namespace zp {

struct ConvArgs {
  const void* x; const float* w; const float* bias; void* ring; void* out;
  const int32_t *cu_q, *context_lens, *slots;
  int64_t x_stride, out_stride;
  int C, taps, n_slots;
};
__device__ __forceinline__ float cv_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float cv_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
constexpr int CV_THREADS = 256, CV_MAX_TAPS = 8;
constexpr int cv_batch(int taps) { return 8 / taps * taps; }      // (whole turns of the circle of inputs)
constexpr int cv_run(int taps) { return 4 * cv_batch(taps); }     // tokens of a thread

template <typename T, int V> struct __align__(V == 1 ? sizeof(T) : 8) ChanVec { T e[V]; };        // V * sizeof(T) = 8, or one entry
template <typename T, int V> __device__ __forceinline__ ChanVec<T, V> cv_load(const T* p) {
  ChanVec<T, V> r;
  if constexpr (V == 1) r.e[0] = *p;
  else *reinterpret_cast<uint2*>(&r) = *reinterpret_cast<const uint2*>(p);
  return r;
}
template <typename T, int V> __device__ __forceinline__ void cv_floats(const ChanVec<T, V>& r, float (&f)[V]) {
#pragma unroll
  for (int i = 0; i < V; ++i) f[i] = Elem<T>::to_f32(r.e[i]);
}
template <typename T, int V> __device__ __forceinline__ void cv_store(T* p, const float (&f)[V]) {
  ChanVec<T, V> r;
#pragma unroll
  for (int i = 0; i < V; ++i) r.e[i] = Elem<T>::from_f32(f[i]);
  if constexpr (V == 1) *p = r.e[0];
  else *reinterpret_cast<uint2*>(p) = *reinterpret_cast<const uint2*>(&r);
}

template <typename T, int V, int TAPS, bool BIAS>
__global__ void __launch_bounds__(CV_THREADS, TAPS <= 4 ? 3 : 2) short_conv_kernel(const ConvArgs a) {
  constexpr int BATCH = cv_batch(TAPS), RUN = cv_run(TAPS);
  const int b = blockIdx.z, c = (blockIdx.x * CV_THREADS + threadIdx.x) * V;
  const int row0 = a.cu_q[b], count = a.cu_q[b + 1] - row0, ctx = a.context_lens[b], slot = a.slots[b];
  const int t0 = blockIdx.y * RUN, t1 = min(count, t0 + RUN);
  if (c >= a.C || t0 >= count || ctx < count || slot < 0 || slot >= a.n_slots) return;
  const T* __restrict__ x = reinterpret_cast<const T*>(a.x) + (int64_t)row0 * a.x_stride + c;
  const T* __restrict__ ring = reinterpret_cast<const T*>(a.ring) + (int64_t)slot * TAPS * a.C + c;
  T* __restrict__ out = reinterpret_cast<T*>(a.out) + (int64_t)row0 * a.out_stride + c;
  const int pos0 = ctx - count;
  ChanVec<T, V> next[BATCH];
  auto fetch = [&](int t) {
#pragma unroll
    for (int u = 0; u < BATCH; ++u)
      if (t + u < t1) next[u] = cv_load<T, V>(x + (int64_t)(t + u) * a.x_stride);
  };
  fetch(t0);
  float w[TAPS][V], f[TAPS][V], bias[V];     // f: inputs of the current token, in a circle
#pragma unroll
  for (int i = 0; i < V; ++i) bias[i] = BIAS ? a.bias[c + i] : 0.f;
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {       // those ahead of the run
    const int t = t0 + j - (TAPS - 1);
#pragma unroll
    for (int i = 0; i < V; ++i) f[j][i] = 0.f;
    if (t >= 0) cv_floats(cv_load<T, V>(x + (int64_t)t * a.x_stride), f[j]);
    else if (pos0 + t >= 0) cv_floats(cv_load<T, V>(ring + (int64_t)((pos0 + t) % TAPS) * a.C), f[j]);
  }
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
    const float* p = a.w + (int64_t)j * a.C + c;
    if constexpr (V == 4) {
      const float4 q = *reinterpret_cast<const float4*>(p);
      w[j][0] = q.x; w[j][1] = q.y; w[j][2] = q.z; w[j][3] = q.w;
    } else {
#pragma unroll
      for (int i = 0; i < V; ++i) w[j][i] = p[i];
    }
  }
#pragma unroll 1
  for (int tb = t0; tb < t1; tb += BATCH) {
    ChanVec<T, V> cur[BATCH];
#pragma unroll
    for (int u = 0; u < BATCH; ++u) cur[u] = next[u];
    fetch(tb + BATCH);
#pragma unroll
    for (int u = 0; u < BATCH; ++u) {
      if (tb + u >= t1) break;
      cv_floats(cur[u], f[(u + TAPS - 1) % TAPS]);
      float y[V];
      if constexpr (V == 4 && sizeof(T) == 2) {
        float2 lo = make_float2(bias[0], bias[1]), hi = make_float2(bias[2], bias[3]);      // pairs of channels
#pragma unroll
        for (int j = 0; j < TAPS; ++j) {
          const float* g = f[(u + j) % TAPS];
          tc::ffma2(lo, make_float2(w[j][0], w[j][1]), make_float2(g[0], g[1]));
          tc::ffma2(hi, make_float2(w[j][2], w[j][3]), make_float2(g[2], g[3]));
        }
        // four sigmoids from one reciprocal, 1 / a = bcd / (abcd); beyond an exponent of 30 the value is 0 to bf16 accuracy
        const float z[4] = {lo.x, lo.y, hi.x, hi.y};
        float e[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) e[i] = 1.f + cv_ex2(fminf(-1.4426950408889634f * z[i], 30.f));
        const float ab = e[0] * e[1], cd = e[2] * e[3], r = cv_rcp(ab * cd), rab = r * cd, rcd = r * ab;
        y[0] = z[0] * (rab * e[1]); y[1] = z[1] * (rab * e[0]); y[2] = z[2] * (rcd * e[3]); y[3] = z[3] * (rcd * e[2]);
      } else {
#pragma unroll
        for (int i = 0; i < V; ++i) {
          float acc = bias[i];
#pragma unroll
          for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j][i], f[(u + j) % TAPS][i], acc);
          y[i] = acc / (1.f + expf(-acc));
        }
      }
      cv_store<T, V>(out + (int64_t)(tb + u) * a.out_stride, y);
    }
  }
}

// the portion's last inputs -> ring (after the convolution has read what the ring held)
template <typename T> __global__ void __launch_bounds__(256) conv_keep_kernel(const ConvArgs a) {
  const int b = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
  const int row0 = a.cu_q[b], count = a.cu_q[b + 1] - row0, ctx = a.context_lens[b], slot = a.slots[b];
  if (c >= a.C || ctx < count || slot < 0 || slot >= a.n_slots) return;
  T* ring = reinterpret_cast<T*>(a.ring) + (int64_t)slot * a.taps * a.C + c;
  for (int j = 0; j < min(a.taps, count); ++j)
    ring[(int64_t)((ctx - 1 - j) % a.taps) * a.C] = reinterpret_cast<const T*>(a.x)[(int64_t)(row0 + count - 1 - j) * a.x_stride + c];
}

template <typename T, int V, bool BIAS> static int conv_by_taps(const ConvArgs& a, dim3 grid, cudaStream_t st) {
  switch (a.taps) {
#define ZP_CONV(n) case n: short_conv_kernel<T, V, n, BIAS><<<grid, CV_THREADS, 0, st>>>(a); break
    ZP_CONV(1); ZP_CONV(2); ZP_CONV(3); ZP_CONV(4); ZP_CONV(5); ZP_CONV(6); ZP_CONV(7); ZP_CONV(8);
#undef ZP_CONV
    default: return ZP_ERR_UNSUPPORTED;
  }
  return check_launch("zp_short_conv");
}

}  // namespace zp

extern "C" int zp_short_conv(const void* x, int64_t x_stride, const float* weight, const float* bias, void* ring, const int32_t* cu_seqlens_q,
                             const int32_t* context_lens, const int32_t* slots, void* out, int64_t out_stride, int B,
                             int max_seqlen_q, int channels, int taps, int n_slots, int dtype, void* stream) {
  if (B == 0 || max_seqlen_q == 0) return ZP_OK;
  ZP_REQUIRE(x && weight && ring && cu_seqlens_q && context_lens && slots && out, "zp_short_conv: null pointer");
  ZP_REQUIRE(channels > 0 && taps > 0 && taps <= zp::CV_MAX_TAPS && n_slots > 0 && B <= 65535 && x_stride >= channels && out_stride >= channels,
             "zp_short_conv: bad sizes (%d taps, at most %d)", taps, zp::CV_MAX_TAPS);
  zp::ConvArgs a{x, weight, bias, ring, out, cu_seqlens_q, context_lens, slots, x_stride, out_stride, channels, taps, n_slots};
  cudaStream_t st = (cudaStream_t)stream;
  int rc = ZP_OK;
  ZP_DISPATCH_DTYPE(dtype, T, {
    constexpr int V = 8 / sizeof(T);
    const bool vec = channels % V == 0 && x_stride % V == 0 && out_stride % V == 0 && ((uintptr_t)x | (uintptr_t)ring | (uintptr_t)out) % 8 == 0 &&
                     (V != 4 || (uintptr_t)weight % 16 == 0);
    const int per = zp::CV_THREADS * (vec ? V : 1), run = zp::cv_run(taps), runs = (max_seqlen_q + run - 1) / run;
    ZP_REQUIRE(runs <= 65535, "zp_short_conv: portions of %d tokens", max_seqlen_q);
    const dim3 grid((channels + per - 1) / per, runs, B);
    if (bias) rc = vec ? zp::conv_by_taps<T, V, true>(a, grid, st) : zp::conv_by_taps<T, 1, true>(a, grid, st);
    else rc = vec ? zp::conv_by_taps<T, V, false>(a, grid, st) : zp::conv_by_taps<T, 1, false>(a, grid, st);
    if (rc == ZP_OK) {
      zp::conv_keep_kernel<T><<<dim3((channels + 255) / 256, B), 256, 0, st>>>(a);
      rc = zp::check_launch("zp_short_conv(keep)");
    }
  });
  return rc;
}
