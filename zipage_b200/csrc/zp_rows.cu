// Row ops of decoders that keep the residual stream in fp32 between 16-bit matrix products:
//   * token embedding, scaled, plus a sinusoidal position vector (and its copy as T),
//   * RMSNorm of an fp32 row to T with the weight stored as an offset (out = x * r * (w + offset)),
//     or, without a weight, the plain conversion of the row,
//   * tanh-form GELU.
// All are streams over HBM with fp32 maths and one rounding to T at the end.
#include "zp_common.cuh"

namespace zp {

// four consecutive values rounded to T and stored as one vector
template <typename T> __device__ __forceinline__ void st4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void st4<float>(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
template <> __device__ __forceinline__ void st4<__nv_bfloat16>(__nv_bfloat16* p, float a, float b, float c, float d) {
  __nv_bfloat162 v[2] = {__floats2bfloat162_rn(a, b), __floats2bfloat162_rn(c, d)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(v);
}
template <> __device__ __forceinline__ void st4<__half>(__half* p, float a, float b, float c, float d) {
  __half2 v[2] = {__floats2half2_rn(a, b), __floats2half2_rn(c, d)};
  *reinterpret_cast<uint2*>(p) = *reinterpret_cast<uint2*>(v);
}

// ---------------------------------------------------------------------------------------------
// x[n, 2i] = E[tok, 2i] * scale + sin(p w_i),  x[n, 2i + 1] = E[tok, 2i + 1] * scale + cos(p w_i).
// `turns[i]` = w_i / (2 pi) in fp64: p * turns is reduced to a fraction of a turn before the
// conversion to fp32, so the angle keeps its accuracy at any position.
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
embed_position_kernel(const int64_t* __restrict__ tokens, const int64_t* __restrict__ positions,
                      const T* __restrict__ table, const double* __restrict__ turns, float scale,
                      float* __restrict__ x, T* __restrict__ x_t, int H, int64_t vocab) {
  const int64_t n = blockIdx.x;
  const int64_t tok = min(max(tokens[n], (int64_t)0), vocab - 1);   // (the host rejects ids outside the table)
  const double p = (double)positions[n];
  for (int i = threadIdx.x; 2 * i < H; i += blockDim.x) {
    float s = 0.f, c = 0.f;
    if (turns) {
      const double t = p * turns[i];
      sincospif(2.f * (float)(t - rint(t)), &s, &c);
    }
    const float a = fmaf(Elem<T>::to_f32(table[tok * H + 2 * i]), scale, s);
    x[n * H + 2 * i] = a;
    if (x_t) x_t[n * H + 2 * i] = Elem<T>::from_f32(a);
    if (2 * i + 1 < H) {
      const float b = fmaf(Elem<T>::to_f32(table[tok * H + 2 * i + 1]), scale, c);
      x[n * H + 2 * i + 1] = b;
      if (x_t) x_t[n * H + 2 * i + 1] = Elem<T>::from_f32(b);
    }
  }
}

// ---------------------------------------------------------------------------------------------
// out = T(x * rsqrt(mean(x^2) + eps) * (w + offset)); weight == NULL: out = T(x).
// One block per row; VPT float4 per thread stay in registers between the two passes (VPT = 0:
// any row length, the row is read twice).
// ---------------------------------------------------------------------------------------------
template <typename T, int VPT>
__global__ void __launch_bounds__(256)
rms_norm_f32_kernel(const float* __restrict__ x, const float* __restrict__ weight, float offset,
                    T* __restrict__ out, int H, float eps) {
  __shared__ float red[32];
  const float* xr = x + (int64_t)blockIdx.x * H;
  T* orow = out + (int64_t)blockIdx.x * H;
  if constexpr (VPT > 0) {
    const int nvec = H / 4;
    float4 v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) {
        v[i] = reinterpret_cast<const float4*>(xr)[c];
        ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
        ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
      }
    }
    float r = 1.f;
    if (weight) r = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) {
        float4 w = make_float4(1.f, 1.f, 1.f, 1.f);
        if (weight) {
          w = reinterpret_cast<const float4*>(weight)[c];
          w.x += offset; w.y += offset; w.z += offset; w.w += offset;
        }
        st4<T>(orow + 4 * c, v[i].x * r * w.x, v[i].y * r * w.y, v[i].z * r * w.z, v[i].w * r * w.w);
      }
    }
  } else {
    float r = 1.f;
    if (weight) {
      float ss = 0.f;
      for (int c = threadIdx.x; c < H; c += blockDim.x) ss = fmaf(xr[c], xr[c], ss);
      r = 1.f / sqrtf(block_sum(ss, red) / (float)H + eps);
    }
    for (int c = threadIdx.x; c < H; c += blockDim.x)
      orow[c] = Elem<T>::from_f32(xr[c] * r * (weight ? weight[c] + offset : 1.f));
  }
}

// ---------------------------------------------------------------------------------------------
// out = T(0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3))))
// ---------------------------------------------------------------------------------------------
template <typename T>
__device__ __forceinline__ float gelu_tanh_f32(float z) {
  const float a = 0.7978845608028654f * fmaf(0.044715f * z, z * z, z);
  if constexpr (sizeof(T) == 4) return 0.5f * z * (1.f + tanhf(a));
  // 0.5 (1 + tanh a) = 1 / (1 + exp(-2a)); the fast forms' last bits disappear in the rounding to T
  else return __fdividef(z, 1.f + __expf(fminf(-2.f * a, 80.f)));
}

template <typename T>
__global__ void __launch_bounds__(256)
gelu_tanh_kernel(const T* __restrict__ x, T* __restrict__ out, int64_t n, int64_t nvec) {
  constexpr int EPV = 16 / sizeof(T);
  const int64_t stride = (int64_t)gridDim.x * blockDim.x;
  const int64_t i0 = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  for (int64_t v0 = i0; v0 < nvec; v0 += 2 * stride) {
    int4 raw[2];
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (v0 + u * stride < nvec) raw[u] = ld16(x + (v0 + u * stride) * EPV);
#pragma unroll
    for (int u = 0; u < 2; ++u)
      if (v0 + u * stride < nvec) {
        const T* e = reinterpret_cast<const T*>(&raw[u]);
        T* o = out + (v0 + u * stride) * EPV;
        float f[EPV];
#pragma unroll
        for (int j = 0; j < EPV; ++j) f[j] = gelu_tanh_f32<T>(Elem<T>::to_f32(e[j]));
#pragma unroll
        for (int j = 0; j < EPV; j += 4) st4<T>(o + j, f[j], f[j + 1], f[j + 2], f[j + 3]);
      }
  }
  for (int64_t i = nvec * EPV + i0; i < n; i += stride) out[i] = Elem<T>::from_f32(gelu_tanh_f32<T>(Elem<T>::to_f32(x[i])));
}

}  // namespace zp

extern "C" int zp_embed_position(const int64_t* tokens, const int64_t* positions, const void* table,
                                 const double* turns, float scale, float* x, void* x_t, int n_tokens,
                                 int hidden, int64_t vocab, int dtype, void* stream) {
  if (n_tokens == 0) return ZP_OK;
  ZP_REQUIRE(tokens && positions && table && x, "zp_embed_position: null pointer");
  ZP_REQUIRE(hidden > 0 && vocab > 0, "zp_embed_position: bad sizes");
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::embed_position_kernel<T><<<n_tokens, 256, 0, (cudaStream_t)stream>>>(
        tokens, positions, (const T*)table, turns, scale, x, (T*)x_t, hidden, vocab);
  });
  return zp::check_launch("zp_embed_position");
}

extern "C" int zp_rms_norm_f32(const float* x, const float* weight, float weight_offset, void* out,
                               int n_rows, int hidden, float eps, int dtype, void* stream) {
  if (n_rows == 0) return ZP_OK;
  ZP_REQUIRE(x && out, "zp_rms_norm_f32: null pointer");
  ZP_REQUIRE(hidden > 0, "zp_rms_norm_f32: bad row length");
  const bool vec = hidden % 4 == 0 && hidden <= 8192 && ((uintptr_t)x | (uintptr_t)weight | (uintptr_t)out) % 16 == 0;
  cudaStream_t st = (cudaStream_t)stream;
  ZP_DISPATCH_DTYPE(dtype, T, {
    T* o = (T*)out;
    if (!vec) zp::rms_norm_f32_kernel<T, 0><<<n_rows, 256, 0, st>>>(x, weight, weight_offset, o, hidden, eps);
    else if (hidden <= 1024) zp::rms_norm_f32_kernel<T, 1><<<n_rows, 256, 0, st>>>(x, weight, weight_offset, o, hidden, eps);
    else if (hidden <= 2048) zp::rms_norm_f32_kernel<T, 2><<<n_rows, 256, 0, st>>>(x, weight, weight_offset, o, hidden, eps);
    else if (hidden <= 4096) zp::rms_norm_f32_kernel<T, 4><<<n_rows, 256, 0, st>>>(x, weight, weight_offset, o, hidden, eps);
    else zp::rms_norm_f32_kernel<T, 8><<<n_rows, 256, 0, st>>>(x, weight, weight_offset, o, hidden, eps);
  });
  return zp::check_launch("zp_rms_norm_f32");
}

extern "C" int zp_gelu_tanh(const void* x, void* out, int64_t n, int dtype, void* stream) {
  if (n == 0) return ZP_OK;
  ZP_REQUIRE(x && out, "zp_gelu_tanh: null pointer");
  const int epv = (int)(16 / zp::dtype_size(dtype));
  const int64_t nvec = ((uintptr_t)x | (uintptr_t)out) % 16 == 0 ? n / epv : 0;
  const int64_t want = ((nvec ? nvec : n) + 255) / 256;
  const int grid = (int)(want < 148 * 16 ? want : 148 * 16);
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::gelu_tanh_kernel<T><<<grid, 256, 0, (cudaStream_t)stream>>>((const T*)x, (T*)out, n, nvec);
  });
  return zp::check_launch("zp_gelu_tanh");
}
