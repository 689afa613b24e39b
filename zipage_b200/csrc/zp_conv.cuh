// The causal convolution of one decoded token, per channel, with its earlier inputs in a ring: shared by the recurrent kernels that
// have it as part of their launch.
#pragma once
#include "zp_common.cuh"

namespace zp {

// Where a sequence's inputs are: weight [taps, C], bias [C] (or NULL), ring [taps, C] of its slot; row: p % taps of the token's
// position p; seen: how many earlier inputs there are.
template <typename T> struct ConvSource {
  const float *w, *bias;
  T* ring;
  int C, taps, row, seen;
};
// The inputs of one channel's convolution at a token, all loads in flight together (more than four taps: the rest in
// `conv_finish`).
template <typename T> struct ConvIn { T now, back[3]; float w[4], bias; };
template <typename T>
__device__ __forceinline__ void conv_start(ConvIn<T>& v, const ConvSource<T>& a, T now, int c) {
  v.now = now;
  v.w[0] = a.w[(int64_t)(a.taps - 1) * a.C + c];
  v.bias = a.bias ? a.bias[c] : 0.f;
#pragma unroll
  for (int j = 1; j < 4; ++j) {
    v.back[j - 1] = Elem<T>::from_f32(0.f);
    v.w[j] = 0.f;
    if (j <= a.seen) {
      const int r = a.row - j;
      v.back[j - 1] = a.ring[(int64_t)(r < 0 ? r + a.taps : r) * a.C + c];
      v.w[j] = a.w[(int64_t)(a.taps - 1 - j) * a.C + c];
    }
  }
}
template <typename T>
__device__ __forceinline__ float conv_finish(const ConvIn<T>& v, const ConvSource<T>& a, int c) {
  float acc = fmaf(Elem<T>::to_f32(v.now), v.w[0], v.bias);
#pragma unroll
  for (int j = 1; j < 4; ++j) acc = fmaf(Elem<T>::to_f32(v.back[j - 1]), v.w[j], acc);
  for (int j = 4; j <= a.seen; ++j) {
    const int r = a.row - j;
    acc = fmaf(Elem<T>::to_f32(a.ring[(int64_t)(r < 0 ? r + a.taps : r) * a.C + c]), a.w[(int64_t)(a.taps - 1 - j) * a.C + c], acc);
  }
  return acc / (1.f + expf(-acc));
}
template <typename T>
__device__ __forceinline__ void conv_keep(const ConvIn<T>& v, const ConvSource<T>& a, int c) { a.ring[(int64_t)a.row * a.C + c] = v.now; }

}  // namespace zp
