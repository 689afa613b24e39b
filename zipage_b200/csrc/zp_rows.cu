// Row ops of decoders that keep the residual stream in fp32 between 16-bit matrix products:
//   * token embedding, scaled, plus a sinusoidal or a learned position vector (and its copy as T),
//   * RMSNorm of an fp32 row to T with the weight stored as an offset (out = x * r * (w + offset)),
//     or, without a weight, the plain conversion of the row,
//   * the boundary between two layers whose mixer and feed-forward read the same x: both results (with
//     their layer scales, the experts' weights and a gate; the mixer's also as the mean of two that are normed first) join x, and
//     the next layer's norms follow from the row while it is in registers,
//   * activations: tanh-form GELU, its gated form, squared ReLU; the soft cap of the logits.
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

// four consecutive values of T as fp32
template <typename T> __device__ __forceinline__ float4 ldf4(const T* p) {
  const uint2 raw = *reinterpret_cast<const uint2*>(p);
  const T* e = reinterpret_cast<const T*>(&raw);
  return make_float4(Elem<T>::to_f32(e[0]), Elem<T>::to_f32(e[1]), Elem<T>::to_f32(e[2]), Elem<T>::to_f32(e[3]));
}
template <> __device__ __forceinline__ float4 ldf4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }

// ---------------------------------------------------------------------------------------------
// x[n, 2i] = E[tok, 2i] * scale + sin(p w_i),  x[n, 2i + 1] = E[tok, 2i + 1] * scale + cos(p w_i).
// `turns[i]` = w_i / (2 pi) in fp64: p * turns is reduced to a fraction of a turn before the
// conversion to fp32, so the angle keeps its accuracy at any position.  `learned`: row p of that table is added instead.
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
embed_position_kernel(const int64_t* __restrict__ tokens, const int64_t* __restrict__ positions,
                      const T* __restrict__ table, const double* __restrict__ turns, float scale,
                      const T* __restrict__ learned, int64_t n_learned, float* __restrict__ x, T* __restrict__ x_t, int H, int64_t vocab) {
  const int64_t n = blockIdx.x;
  const int64_t tok = min(max(tokens[n], (int64_t)0), vocab - 1);   // (the host rejects ids outside the table)
  const double p = (double)positions[n];
  const int64_t at = min(max(positions[n], (int64_t)0), n_learned - 1);
  for (int i = threadIdx.x; 2 * i < H; i += blockDim.x) {
    float s = 0.f, c = 0.f;
    if (turns) {
      const double t = p * turns[i];
      sincospif(2.f * (float)(t - rint(t)), &s, &c);
    }
    if (learned) {
      s = Elem<T>::to_f32(learned[at * H + 2 * i]);
      c = 2 * i + 1 < H ? Elem<T>::to_f32(learned[at * H + 2 * i + 1]) : 0.f;
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

// ---------------------------------------------------------------------------------------------
// x += ls_a * a + ls_b * (sigmoid(gate) * b + sum_k w_k y[pos_k]) + pair_scale * (rms(m1) * mw1 + rms(m2) * mw2);  out_i = T(norm of x with w_i, bias_i), the layer
// norm or (rms) the one that takes no mean off.
// Every part may be missing.  One block per row; VPT float4 per thread stay in registers (VPT = 0: any
// row length, each thread reads back the entries of x that it wrote).
// ---------------------------------------------------------------------------------------------
struct JoinArgs {
  float* x;
  const void *a, *b, *y;
  const float *ls_a, *ls_b, *gate, *wts;
  const int32_t* pos;
  const float *w1, *bias1, *w2, *bias2;
  void *out1, *out2;
  const void *m1, *m2;        // both or none
  const float *mw1, *mw2;
  int64_t gate_stride, y_rows;
  int top, H, rms;
  float eps, pair_scale;
};

template <typename T, int V> struct JoinVec;      // V consecutive entries of a row
template <typename T> struct JoinVec<T, 4> {
  static __device__ __forceinline__ float4 ld(const void* p, int64_t i) { return ldf4<T>(reinterpret_cast<const T*>(p) + i); }
  static __device__ __forceinline__ float4 ldf(const float* p, int64_t i) { return *reinterpret_cast<const float4*>(p + i); }
  static __device__ __forceinline__ void stf(float* p, int64_t i, float4 v) { *reinterpret_cast<float4*>(p + i) = v; }
  static __device__ __forceinline__ void st(void* p, int64_t i, float4 v) { st4<T>(reinterpret_cast<T*>(p) + i, v.x, v.y, v.z, v.w); }
};
template <typename T> struct JoinVec<T, 1> {      // only .x is used
  static __device__ __forceinline__ float4 ld(const void* p, int64_t i) { return make_float4(Elem<T>::to_f32(reinterpret_cast<const T*>(p)[i]), 0.f, 0.f, 0.f); }
  static __device__ __forceinline__ float4 ldf(const float* p, int64_t i) { return make_float4(p[i], 0.f, 0.f, 0.f); }
  static __device__ __forceinline__ void stf(float* p, int64_t i, float4 v) { p[i] = v.x; }
  static __device__ __forceinline__ void st(void* p, int64_t i, float4 v) { reinterpret_cast<T*>(p)[i] = Elem<T>::from_f32(v.x); }
};
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}
__device__ __forceinline__ float4 splat4(float s) { return make_float4(s, s, s, s); }

// What joins x at entry c of a row: `add` gathers it, so that the loads of all of a thread's entries can be in
// flight before the first of them is stored.
template <typename T, int V, bool PAIR>
__device__ __forceinline__ float4 join_add(const JoinArgs& p, int64_t row, int c, const float* swts, const int32_t* spos, float g, float2 rp) {
  using L = JoinVec<T, V>;
  float4 add = splat4(0.f);
  if constexpr (PAIR) {
    const float4 u = L::ld(p.m1, row * p.H + c), v = L::ld(p.m2, row * p.H + c), s = L::ldf(p.mw1, c), t = L::ldf(p.mw2, c);
    add = make_float4(u.x * rp.x * s.x + v.x * rp.y * t.x, u.y * rp.x * s.y + v.y * rp.y * t.y, u.z * rp.x * s.z + v.z * rp.y * t.z,
                      u.w * rp.x * s.w + v.w * rp.y * t.w);
  }
  if (p.a) {
    float4 a = L::ld(p.a, row * p.H + c);
    if (p.ls_a) { const float4 s = L::ldf(p.ls_a, c); a = make_float4(a.x * s.x, a.y * s.y, a.z * s.z, a.w * s.w); }
    add = PAIR ? make_float4(add.x + a.x, add.y + a.y, add.z + a.z, add.w + a.w) : a;
  }
  if (p.b || p.y) {
    float4 f = splat4(0.f);
#pragma unroll 4
    for (int k = 0; k < p.top; ++k) f = fma4(splat4(swts[k]), L::ld(p.y, (int64_t)spos[k] * p.H + c), f);
    if (p.b) f = fma4(splat4(g), L::ld(p.b, row * p.H + c), f);
    add = fma4(p.ls_b ? L::ldf(p.ls_b, c) : splat4(1.f), f, add);
  }
  return add;
}
template <typename T, int V>
__device__ __forceinline__ void join_norm(const JoinArgs& p, int64_t row, int c, float4 d, float r) {
  using L = JoinVec<T, V>;
  d = make_float4(d.x * r, d.y * r, d.z * r, d.w * r);
  if (p.out1) L::st(p.out1, row * p.H + c, fma4(d, p.w1 ? L::ldf(p.w1, c) : splat4(1.f), p.bias1 ? L::ldf(p.bias1, c) : splat4(0.f)));
  if (p.out2) L::st(p.out2, row * p.H + c, fma4(d, p.w2 ? L::ldf(p.w2, c) : splat4(1.f), p.bias2 ? L::ldf(p.bias2, c) : splat4(0.f)));
}

constexpr int JOIN_TOP = 64;
template <typename T, int VPT, bool PAIR>
__global__ void __launch_bounds__(256) join_norms_kernel(const JoinArgs p) {
  __shared__ float red[32];
  __shared__ float swts[JOIN_TOP];
  __shared__ int32_t spos[JOIN_TOP];
  const int64_t row = blockIdx.x;
  if (p.top) {
    for (int k = threadIdx.x; k < p.top; k += blockDim.x) {
      swts[k] = p.wts ? p.wts[row * p.top + k] : 1.f;
      spos[k] = (int32_t)min(max((int64_t)p.pos[row * p.top + k], (int64_t)0), p.y_rows - 1);
    }
    __syncthreads();
  }
  const float g = p.gate ? 1.f / (1.f + expf(-p.gate[row * p.gate_stride])) : 1.f;
  const bool norm = p.out1 || p.out2, any = PAIR || p.a || p.b || p.y;
  float2 rp = make_float2(0.f, 0.f);        // pair_scale over the root mean squares of the pair's rows
  if constexpr (PAIR) {
    constexpr int V = VPT > 0 ? 4 : 1;
    using L = JoinVec<T, V>;
    float s1 = 0.f, s2 = 0.f;
    for (int c = threadIdx.x * V; c < p.H; c += blockDim.x * V) {
      const float4 u = L::ld(p.m1, row * p.H + c), v = L::ld(p.m2, row * p.H + c);
      s1 = fmaf(u.x, u.x, s1); s1 = fmaf(u.y, u.y, s1); s1 = fmaf(u.z, u.z, s1); s1 = fmaf(u.w, u.w, s1);
      s2 = fmaf(v.x, v.x, s2); s2 = fmaf(v.y, v.y, s2); s2 = fmaf(v.z, v.z, s2); s2 = fmaf(v.w, v.w, s2);
    }
    rp.x = p.pair_scale / sqrtf(block_sum(s1, red) / (float)p.H + p.eps);
    rp.y = p.pair_scale / sqrtf(block_sum(s2, red) / (float)p.H + p.eps);
  }
  if constexpr (VPT > 0) {
    const int nvec = p.H / 4;
    using L = JoinVec<T, 4>;
    float4 v[VPT];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) {
        const float4 x = L::ldf(p.x, row * p.H + 4 * c);
        if (!any) { v[i] = x; continue; }
        const float4 d = join_add<T, 4, PAIR>(p, row, 4 * c, swts, spos, g, rp);
        v[i] = make_float4(x.x + d.x, x.y + d.y, x.z + d.z, x.w + d.w);
      }
    }
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) {
        if (any) L::stf(p.x, row * p.H + 4 * c, v[i]);
        s += (v[i].x + v[i].y) + (v[i].z + v[i].w);
      }
    }
    if (!norm) return;
    const float mean = p.rms ? 0.f : block_sum(s, red) / (float)p.H;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) {
        v[i] = make_float4(v[i].x - mean, v[i].y - mean, v[i].z - mean, v[i].w - mean);
        ss = fmaf(v[i].x, v[i].x, ss); ss = fmaf(v[i].y, v[i].y, ss);
        ss = fmaf(v[i].z, v[i].z, ss); ss = fmaf(v[i].w, v[i].w, ss);
      }
    }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.H + p.eps);
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
      const int c = threadIdx.x + i * 256;
      if (c < nvec) join_norm<T, 4>(p, row, 4 * c, v[i], r);
    }
  } else {
    float s = 0.f;
    for (int c = threadIdx.x; c < p.H; c += blockDim.x) {
      float v = p.x[row * p.H + c];
      if (any) p.x[row * p.H + c] = v += join_add<T, 1, PAIR>(p, row, c, swts, spos, g, rp).x;
      s += v;
    }
    if (!norm) return;
    const float mean = p.rms ? 0.f : block_sum(s, red) / (float)p.H;
    float ss = 0.f;
    for (int c = threadIdx.x; c < p.H; c += blockDim.x) { const float d = p.x[row * p.H + c] - mean; ss = fmaf(d, d, ss); }
    const float r = 1.f / sqrtf(block_sum(ss, red) / (float)p.H + p.eps);
    for (int c = threadIdx.x; c < p.H; c += blockDim.x) join_norm<T, 1>(p, row, c, make_float4(p.x[row * p.H + c] - mean, 0.f, 0.f, 0.f), r);
  }
}

template <typename T, bool PAIR> static void launch_join(const JoinArgs& p, int n_rows, bool vec, cudaStream_t st) {
  if (!vec) join_norms_kernel<T, 0, PAIR><<<n_rows, 256, 0, st>>>(p);
  else if (p.H <= 1024) join_norms_kernel<T, 1, PAIR><<<n_rows, 256, 0, st>>>(p);
  else if (p.H <= 2048) join_norms_kernel<T, 2, PAIR><<<n_rows, 256, 0, st>>>(p);
  else if (p.H <= 4096) join_norms_kernel<T, 4, PAIR><<<n_rows, 256, 0, st>>>(p);
  else join_norms_kernel<T, 8, PAIR><<<n_rows, 256, 0, st>>>(p);
}

// ---------------------------------------------------------------------------------------------
// gate | up [n, 2 F] -> T(gelu_tanh(gate) * up) [n, F];  x -> T(max(x, 0)^2);  z -> cap tanh(z / cap)
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256)
gelu_tanh_and_mul_kernel(const T* __restrict__ x, T* __restrict__ out, int64_t n, int F, int vec) {
  const int64_t stride = (int64_t)gridDim.x * blockDim.x, i0 = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (vec) {
    const int per = F / 4;
    for (int64_t i = i0; i < n * per; i += stride) {
      const int64_t row = i / per;
      const int c = (int)(i - row * per) * 4;
      const float4 g = ldf4<T>(x + row * 2 * F + c), u = ldf4<T>(x + row * 2 * F + F + c);
      st4<T>(out + row * F + c, gelu_tanh_f32<T>(g.x) * u.x, gelu_tanh_f32<T>(g.y) * u.y, gelu_tanh_f32<T>(g.z) * u.z,
             gelu_tanh_f32<T>(g.w) * u.w);
    }
  } else {
    for (int64_t i = i0; i < n * F; i += stride) {
      const int64_t row = i / F;
      const int c = (int)(i - row * F);
      out[i] = Elem<T>::from_f32(gelu_tanh_f32<T>(Elem<T>::to_f32(x[row * 2 * F + c])) * Elem<T>::to_f32(x[row * 2 * F + F + c]));
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) relu_squared_kernel(const T* __restrict__ x, T* __restrict__ out, int64_t n, int64_t nvec) {
  const int64_t stride = (int64_t)gridDim.x * blockDim.x, i0 = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  for (int64_t i = i0; i < nvec; i += stride) {
    float4 v = ldf4<T>(x + 4 * i);
    v = make_float4(fmaxf(v.x, 0.f), fmaxf(v.y, 0.f), fmaxf(v.z, 0.f), fmaxf(v.w, 0.f));
    st4<T>(out + 4 * i, v.x * v.x, v.y * v.y, v.z * v.z, v.w * v.w);
  }
  for (int64_t i = 4 * nvec + i0; i < n; i += stride) { const float v = fmaxf(Elem<T>::to_f32(x[i]), 0.f); out[i] = Elem<T>::from_f32(v * v); }
}

__global__ void __launch_bounds__(256) soft_cap_kernel(float* __restrict__ z, int64_t n, float cap) {
  const int64_t stride = (int64_t)gridDim.x * blockDim.x;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += stride) z[i] = cap * tanhf(z[i] / cap);
}

// blocks of a grid-stride launch over n items
static int stream_grid(int64_t n) {
  const int64_t want = (n + 255) / 256;
  return (int)(want < 148 * 16 ? (want < 1 ? 1 : want) : 148 * 16);
}

}  // namespace zp

extern "C" int zp_embed_position(const int64_t* tokens, const int64_t* positions, const void* table,
                                 const double* turns, float scale, const void* learned, int64_t n_learned, float* x, void* x_t, int n_tokens,
                                 int hidden, int64_t vocab, int dtype, void* stream) {
  if (n_tokens == 0) return ZP_OK;
  ZP_REQUIRE(tokens && positions && table && x, "zp_embed_position: null pointer");
  ZP_REQUIRE(hidden > 0 && vocab > 0 && (!learned || (n_learned > 0 && !turns)), "zp_embed_position: bad sizes, or two kinds of positions");
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::embed_position_kernel<T><<<n_tokens, 256, 0, (cudaStream_t)stream>>>(
        tokens, positions, (const T*)table, turns, scale, (const T*)learned, n_learned, x, (T*)x_t, hidden, vocab);
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

extern "C" int zp_join_norms(float* x, const void* a, const float* ls_a, const void* b, const float* ls_b,
                             const float* gate, int64_t gate_stride, const void* y, int64_t y_rows,
                             const int32_t* pos, const float* wts, int top, const void* m1, const float* mw1, const void* m2,
                             const float* mw2, float pair_scale, const float* w1, const float* bias1,
                             void* out1, const float* w2, const float* bias2, void* out2, int n_rows, int hidden,
                             float eps, int rms, int dtype, void* stream) {
  if (n_rows == 0) return ZP_OK;
  ZP_REQUIRE(x, "zp_join_norms: null pointer");
  ZP_REQUIRE(hidden > 0 && top >= 0 && top <= zp::JOIN_TOP, "zp_join_norms: bad sizes (%d experts a token, at most %d)", top, zp::JOIN_TOP);
  ZP_REQUIRE(top == 0 || (y && pos && y_rows > 0), "zp_join_norms: expert rows without places");
  ZP_REQUIRE(!m1 == !m2 && (!m1 || (mw1 && mw2)), "zp_join_norms: a pair takes two rows and two weights");
  zp::JoinArgs p;
  p.m1 = m1; p.m2 = m2; p.mw1 = mw1; p.mw2 = mw2; p.pair_scale = pair_scale;
  p.x = x; p.a = a; p.b = b; p.y = top ? y : nullptr; p.ls_a = ls_a; p.ls_b = ls_b; p.gate = gate; p.wts = wts; p.pos = pos;
  p.w1 = w1; p.bias1 = bias1; p.w2 = w2; p.bias2 = bias2; p.out1 = out1; p.out2 = out2; p.gate_stride = gate_stride;
  p.y_rows = y_rows; p.top = top; p.H = hidden; p.eps = eps; p.rms = rms;
  const uintptr_t al = (uintptr_t)x | (uintptr_t)a | (uintptr_t)b | (uintptr_t)p.y | (uintptr_t)m1 | (uintptr_t)m2 | (uintptr_t)mw1 | (uintptr_t)mw2 | (uintptr_t)ls_a | (uintptr_t)ls_b | (uintptr_t)w1 |
                       (uintptr_t)bias1 | (uintptr_t)out1 | (uintptr_t)w2 | (uintptr_t)bias2 | (uintptr_t)out2;
  const bool vec = hidden % 4 == 0 && hidden <= 8192 && al % 16 == 0;
  cudaStream_t st = (cudaStream_t)stream;
  ZP_DISPATCH_DTYPE(dtype, T, {
    if (m1) zp::launch_join<T, true>(p, n_rows, vec, st);
    else zp::launch_join<T, false>(p, n_rows, vec, st);
  });
  return zp::check_launch("zp_join_norms");
}

extern "C" int zp_gelu_tanh_and_mul(const void* x, void* out, int n_rows, int width, int dtype, void* stream) {
  if (n_rows == 0) return ZP_OK;
  ZP_REQUIRE(x && out && width > 0, "zp_gelu_tanh_and_mul: null pointer or bad size");
  const int vec = width % 4 == 0 && ((uintptr_t)x | (uintptr_t)out) % 16 == 0;
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::gelu_tanh_and_mul_kernel<T><<<zp::stream_grid((int64_t)n_rows * width / (vec ? 4 : 1)), 256, 0, (cudaStream_t)stream>>>(
        (const T*)x, (T*)out, n_rows, width, vec);
  });
  return zp::check_launch("zp_gelu_tanh_and_mul");
}

extern "C" int zp_relu_squared(const void* x, void* out, int64_t n, int dtype, void* stream) {
  if (n == 0) return ZP_OK;
  ZP_REQUIRE(x && out, "zp_relu_squared: null pointer");
  const int64_t nvec = ((uintptr_t)x | (uintptr_t)out) % 16 == 0 ? n / 4 : 0;
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::relu_squared_kernel<T><<<zp::stream_grid(nvec ? nvec : n), 256, 0, (cudaStream_t)stream>>>((const T*)x, (T*)out, n, nvec);
  });
  return zp::check_launch("zp_relu_squared");
}

extern "C" int zp_soft_cap(float* z, int64_t n, float cap, void* stream) {
  if (n == 0) return ZP_OK;
  ZP_REQUIRE(z && cap > 0.f, "zp_soft_cap: null pointer or a cap that is not positive");
  zp::soft_cap_kernel<<<zp::stream_grid(n), 256, 0, (cudaStream_t)stream>>>(z, n, cap);
  return zp::check_launch("zp_soft_cap");
}
