// Queries and keys of a projection on their way to attention: optional RMS norm per head, rotary positions on the
// first `dims` entries of each head (interleaved or half-split pairs), queries in place, keys and values into padded
// paged caches.  The values may be the keys themselves, as projected.
//
// One block per token: its cosines and sines are made once (fp64 turns, reduced before the sine) and shared by all heads; a
// warp takes a head at a time, holding the row in shared memory because pairs lie in different lanes.
#include "zp_common.cuh"

namespace zp {

constexpr int RO_THREADS = 256, RO_WARPS = RO_THREADS / 32;

struct RotateArgs {
  void* q; const void* k; const void* v;   // [tokens, heads * D | DV], one row stride
  int64_t row_stride;
  const int64_t* positions;
  const double* turns;                     // [dims / 2]
  const float *q_weight, *k_weight;        // [D] or NULL
  void* k_cache; void* v_cache;
  const int32_t* slots;
  int64_t n_slots;
  int Hq, Hkv, D, DV, KP, VP, dims, interleaved;
  float mul, eps;
};

template <typename T, int V> __device__ __forceinline__ void ro_load(const T* p, float (&f)[V]) {
  if constexpr (V == 1) f[0] = Elem<T>::to_f32(p[0]);
  else {
    constexpr int N = V * sizeof(T) / 8;
    uint2 raw[N];
#pragma unroll
    for (int i = 0; i < N; ++i) raw[i] = reinterpret_cast<const uint2*>(p)[i];
    const T* e = reinterpret_cast<const T*>(raw);
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = Elem<T>::to_f32(e[i]);
  }
}
template <typename T, int V> __device__ __forceinline__ void ro_store(T* p, const float (&f)[V]) {
  if constexpr (V == 1) p[0] = Elem<T>::from_f32(f[0]);
  else {
    constexpr int N = V * sizeof(T) / 8;
    uint2 raw[N];
    T* e = reinterpret_cast<T*>(raw);
#pragma unroll
    for (int i = 0; i < V; ++i) e[i] = Elem<T>::from_f32(f[i]);
#pragma unroll
    for (int i = 0; i < N; ++i) reinterpret_cast<uint2*>(p)[i] = raw[i];
  }
}

template <typename T, int V>   // V: entries per access
__global__ void __launch_bounds__(RO_THREADS) rotate_store_kernel(const RotateArgs a) {
  extern __shared__ __align__(16) float ro_sm[];   // cos [dims / 2], sin [dims / 2], one row per warp
  const int64_t n = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = a.dims >> 1;
  float *cs = ro_sm, *sn = cs + half;
  float* row = ro_sm + ((2 * half + 3) & ~3) + warp * ((a.D + 3) & ~3);
  const double p = (double)a.positions[n];
  for (int i = threadIdx.x; i < half; i += RO_THREADS) {
    const double t = p * a.turns[i];
    float s, c;
    sincospif(2.f * (float)(t - rint(t)), &s, &c);
    cs[i] = c * a.mul;
    sn[i] = s * a.mul;
  }
  __syncthreads();
  const int64_t slot = a.slots[n];
  const bool stored = slot >= 0 && slot < a.n_slots;
  const int total = a.Hq + 2 * a.Hkv;
  for (int item = warp; item < total; item += RO_WARPS) {
    if (item >= a.Hq + a.Hkv) {                      // a value row: copied
      if (!stored) continue;
      const int h = item - a.Hq - a.Hkv;
      const T* src = reinterpret_cast<const T*>(a.v) + n * a.row_stride + (int64_t)h * a.DV;
      T* dst = reinterpret_cast<T*>(a.v_cache) + (slot * a.Hkv + h) * a.VP;
      for (int d = lane * V; d < a.DV; d += 32 * V) {
        float f[V];
        ro_load<T, V>(src + d, f);
        ro_store<T, V>(dst + d, f);
      }
      continue;
    }
    const bool is_q = item < a.Hq;
    const int h = is_q ? item : item - a.Hq;
    if (!is_q && !stored) continue;
    const T* src = reinterpret_cast<const T*>(is_q ? a.q : a.k) + n * a.row_stride + (int64_t)h * a.D;
    T* dst = is_q ? reinterpret_cast<T*>(a.q) + n * a.row_stride + (int64_t)h * a.D
                  : reinterpret_cast<T*>(a.k_cache) + (slot * a.Hkv + h) * a.KP;
    const float* w = is_q ? a.q_weight : a.k_weight;
    float ss = 0.f;
    for (int d = lane * V; d < a.D; d += 32 * V) {
      float f[V];
      ro_load<T, V>(src + d, f);
#pragma unroll
      for (int i = 0; i < V; ++i) {
        ss = fmaf(f[i], f[i], ss);
        row[d + i] = w ? f[i] * w[d + i] : f[i];
      }
    }
    const float r = w ? 1.f / sqrtf(warp_sum(ss) / (float)a.D + a.eps) : 1.f;
    __syncwarp();
    for (int d = lane * V; d < a.D; d += 32 * V) {
      float f[V];
#pragma unroll
      for (int i = 0; i < V; ++i) {
        const int e = d + i;
        float x = row[e];
        if (e < a.dims) {
          const bool second = a.interleaved ? e & 1 : e >= half;
          const int at = a.interleaved ? e >> 1 : (second ? e - half : e);
          const float y = row[a.interleaved ? e ^ 1 : (second ? at : e + half)];
          x = second ? fmaf(x, cs[at], y * sn[at]) : fmaf(x, cs[at], -y * sn[at]);
        }
        f[i] = x * r;
      }
      ro_store<T, V>(dst + d, f);
    }
    __syncwarp();
  }
}

}  // namespace zp

extern "C" int zp_rotate_store(void* q, const void* k, const void* v, int64_t row_stride, const int64_t* positions,
                               const double* turns, int dims, int interleaved, float mul, const float* q_weight,
                               const float* k_weight, float eps, void* k_cache, void* v_cache, const int32_t* slot_mapping,
                               int n_tokens, int Hq, int Hkv, int D, int DV, int KP, int VP, int64_t n_slots, int dtype,
                               void* stream) {
  if (n_tokens == 0) return ZP_OK;
  ZP_REQUIRE(q && k && v && positions && (turns || dims == 0) && k_cache && v_cache && slot_mapping, "zp_rotate_store: null pointer");
  ZP_REQUIRE(Hq > 0 && Hkv > 0 && D > 0 && D <= 1024 && DV > 0 && KP >= D && VP >= DV && dims >= 0 && dims <= D && dims % 2 == 0,
             "zp_rotate_store: bad sizes (heads of %d with %d rotated entries)", D, dims);
  zp::RotateArgs a{q, k, v, row_stride, positions, turns, q_weight, k_weight, k_cache, v_cache, slot_mapping, n_slots,
                   Hq, Hkv, D, DV, KP, VP, dims, interleaved, mul, eps};
  const bool vec = D % 4 == 0 && DV % 4 == 0 && KP % 4 == 0 && VP % 4 == 0 && row_stride % 4 == 0 &&
                   ((uintptr_t)q | (uintptr_t)k | (uintptr_t)v | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16 == 0;
  const size_t smem = sizeof(float) * (((dims + 3) & ~3) + zp::RO_WARPS * ((D + 3) & ~3));
  ZP_DISPATCH_DTYPE(dtype, T, {
    if (vec) zp::rotate_store_kernel<T, 4><<<n_tokens, zp::RO_THREADS, smem, (cudaStream_t)stream>>>(a);
    else zp::rotate_store_kernel<T, 1><<<n_tokens, zp::RO_THREADS, smem, (cudaStream_t)stream>>>(a);
  });
  return zp::check_launch("zp_rotate_store");
}
