// Queries and keys of a projection on their way to attention: optional RMS norm per head, rotary positions on the
// first `dims` entries of each head (interleaved or half-split pairs), queries in place, keys and values into padded
// paged caches.  The values may be the keys themselves, as projected.
//
// One block per token: its cosines and sines are made once (fp64 turns, reduced before the sine) and shared by all heads.
// 16-bit rows of whole 16-byte pieces: a half warp (or, above 128 entries, a warp) takes a head, eight entries a lane, several
// heads in flight, and pairs that lie in different lanes meet by shuffles.  Other rows: a warp takes a head at a time
// and holds the row in shared memory.
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

// LANES: lanes of a head; NI: heads of a group of lanes in flight
template <typename T, int LANES, int NI>
__global__ void __launch_bounds__(RO_THREADS) rotate_store_vec_kernel(const RotateArgs a) {
  extern __shared__ __align__(16) float ro_sm[];   // cos [dims / 2], sin [dims / 2]
  constexpr int GROUPS = RO_THREADS / LANES;
  const int64_t n = blockIdx.x;
  const int grp = threadIdx.x / LANES, l = threadIdx.x & (LANES - 1), half = a.dims >> 1, e0 = 8 * l;
  float *cs = ro_sm, *sn = cs + half;
  const int64_t slot = a.slots[n];
  const bool stored = slot >= 0 && slot < a.n_slots;
  const int total = a.Hq + 2 * a.Hkv;
  auto row_of = [&](int item) -> const T* {
    if (item < a.Hq) return reinterpret_cast<const T*>(a.q) + n * a.row_stride + (int64_t)item * a.D;
    item -= a.Hq;
    if (item < a.Hkv) return reinterpret_cast<const T*>(a.k) + n * a.row_stride + (int64_t)item * a.D;
    return reinterpret_cast<const T*>(a.v) + n * a.row_stride + (int64_t)(item - a.Hkv) * a.DV;
  };
  auto width_of = [&](int item) { return item < a.Hq + a.Hkv ? a.D : a.DV; };
  int4 raw[NI];
  auto fetch = [&](int first) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int item = first + i * GROUPS;
      raw[i] = item < total && e0 < width_of(item) ? ld16(row_of(item) + e0) : make_int4(0, 0, 0, 0);
    }
  };
  fetch(grp);
  const double p = (double)a.positions[n];
  for (int i = threadIdx.x; i < half; i += RO_THREADS) {
    const double t = p * a.turns[i];
    float s, c;
    sincospif(2.f * (float)(t - rint(t)), &s, &c);
    cs[i] = c * a.mul;
    sn[i] = s * a.mul;
  }
  __syncthreads();
  // where this lane's pairs are: in the lane itself, or eight entries of another lane
  const bool turns_here = e0 < a.dims, second = !a.interleaved && e0 >= half;
  const int lane0 = (threadIdx.x & 31) - l, mate = lane0 + (a.interleaved || !turns_here ? l : (second ? l - (half >> 3) : l + (half >> 3)));
  for (int base = grp; base - grp < total; base += NI * GROUPS) {      // (the same number of rounds in every lane)
    if (base != grp) fetch(base);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int item = base + i * GROUPS;
      const bool is_q = item < a.Hq, is_k = !is_q && item < a.Hq + a.Hkv, live = item < total && e0 < width_of(item);
      float f[8];
      const T* e = reinterpret_cast<const T*>(&raw[i]);
#pragma unroll
      for (int u = 0; u < 8; ++u) f[u] = Elem<T>::to_f32(e[u]);
      const float* w = is_q ? a.q_weight : is_k ? a.k_weight : nullptr;
      float ss = 0.f;
#pragma unroll
      for (int u = 0; u < 8; ++u) ss = fmaf(f[u], f[u], ss);
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      float r = 1.f;
      if (w && live) {
        r = 1.f / sqrtf(ss / (float)a.D + a.eps);
        const float4 w0 = *reinterpret_cast<const float4*>(w + e0), w1 = *reinterpret_cast<const float4*>(w + e0 + 4);
        f[0] *= w0.x; f[1] *= w0.y; f[2] *= w0.z; f[3] *= w0.w; f[4] *= w1.x; f[5] *= w1.y; f[6] *= w1.z; f[7] *= w1.w;
      }
      float y[8];
      if (a.interleaved) {
        if (turns_here && (is_q || is_k)) {
#pragma unroll
          for (int u = 0; u < 8; u += 2) {
            if (e0 + u >= a.dims) continue;
            const float c = cs[(e0 + u) >> 1], s = sn[(e0 + u) >> 1], x0 = f[u], x1 = f[u + 1];
            f[u] = fmaf(x0, c, -x1 * s);
            f[u + 1] = fmaf(x1, c, x0 * s);
          }
        }
      } else {
#pragma unroll
        for (int u = 0; u < 8; ++u) y[u] = __shfl_sync(0xffffffffu, f[u], mate);
        if (turns_here && (is_q || is_k)) {
          const int at = second ? e0 - half : e0;
#pragma unroll
          for (int u = 0; u < 8; ++u) f[u] = fmaf(f[u], cs[at + u], (second ? y[u] : -y[u]) * sn[at + u]);
        }
      }
      if (live && (is_q || stored)) {
        int4 o;
        T* oe = reinterpret_cast<T*>(&o);
#pragma unroll
        for (int u = 0; u < 8; ++u) oe[u] = Elem<T>::from_f32(f[u] * r);
        T* dst = is_q ? const_cast<T*>(row_of(item))
                      : is_k ? reinterpret_cast<T*>(a.k_cache) + (slot * a.Hkv + item - a.Hq) * a.KP
                             : reinterpret_cast<T*>(a.v_cache) + (slot * a.Hkv + item - a.Hq - a.Hkv) * a.VP;
        st16(dst + e0, o);
      }
    }
  }
}

template <typename T> static int launch_rotate(const RotateArgs& a, int n_tokens, cudaStream_t st) {
  const uintptr_t al = (uintptr_t)a.q | (uintptr_t)a.k | (uintptr_t)a.v | (uintptr_t)a.k_cache | (uintptr_t)a.v_cache |
                       (uintptr_t)a.q_weight | (uintptr_t)a.k_weight;
  const int widest = a.D > a.DV ? a.D : a.DV;
  if (sizeof(T) == 2 && a.D % 8 == 0 && a.DV % 8 == 0 && a.KP % 8 == 0 && a.VP % 8 == 0 && a.row_stride % 8 == 0 && widest <= 256 &&
      (a.interleaved || a.dims % 16 == 0) && al % 16 == 0) {
    const size_t smem = sizeof(float) * a.dims;
    if (widest <= 128) rotate_store_vec_kernel<T, 16, 3><<<n_tokens, RO_THREADS, smem, st>>>(a);
    else rotate_store_vec_kernel<T, 32, 3><<<n_tokens, RO_THREADS, smem, st>>>(a);
  } else {
    const bool vec = a.D % 4 == 0 && a.DV % 4 == 0 && a.KP % 4 == 0 && a.VP % 4 == 0 && a.row_stride % 4 == 0 && al % 16 == 0;
    const size_t smem = sizeof(float) * (((a.dims + 3) & ~3) + RO_WARPS * ((a.D + 3) & ~3));
    if (vec) rotate_store_kernel<T, 4><<<n_tokens, RO_THREADS, smem, st>>>(a);
    else rotate_store_kernel<T, 1><<<n_tokens, RO_THREADS, smem, st>>>(a);
  }
  return check_launch("zp_rotate_store");
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
  ZP_DISPATCH_DTYPE(dtype, T, { return zp::launch_rotate<T>(a, n_tokens, (cudaStream_t)stream); });
  return ZP_OK;
}
