// Linear attention with a decaying matrix state, token by token: the decode kernel (from projections to outputs in one launch),
// also used for prompts in fp32, and the norm with gates that follows it.
//
// HBM-bound: a decoded token reads and writes the head's whole fp32 state once.  One block per (value tile, head,
// sequence); its part of the state stays in registers (up to 16 rows of four columns a thread), all of its loads in flight
// while keys, queries and decays are made.
#include "zp_conv.cuh"
#include "zp_linear_state.cuh"
#include "zp_mma.cuh"       // packed 16-bit pairs

namespace zp {

constexpr int LR_THREADS = 256;

template <typename T, int KIND, int RPT>   // RPT: state rows per thread
__global__ void __launch_bounds__(LR_THREADS, RPT == 16 ? 2 : RPT == 8 ? 3 : 4) linear_recurrent_kernel(const LinearArgs a, int VT) {
  extern __shared__ __align__(16) float sm[];
  const int vt = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const LinearSeq sq = linear_seq(a, b);
  if (sq.count == 0) return;
  const int group = a.H / a.G, hk = h / group, C = a.H * a.vdim + 2 * a.G * a.dim;
  const int c0 = vt * VT, ncg = VT / 4, nrg = LR_THREADS / ncg;   // (powers of two; ncg <= 32)
  float4* sqk = reinterpret_cast<float4*>(sm);   // [dim] q, k, a
  float* sv = sm + 4 * a.dim;                    // [VT] v
  float* part = sv + VT;                         // [8 warps][VT]
  const int cg = tid & (ncg - 1), rg = tid / ncg, col = c0 + 4 * cg;
  const bool mine = col < a.VP, out_col = tid < VT && c0 + tid < a.vdim;      // (VT <= 128)
  float* S = a.state + ((int64_t)sq.slot * a.H + h) * a.dim * a.VP + col;
  float4 s[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = rg + i * nrg;
    s[i] = (mine && r < a.dim && !sq.fresh) ? *reinterpret_cast<const float4*>(S + (int64_t)r * a.VP) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const T *xq = reinterpret_cast<const T*>(a.q), *xk = reinterpret_cast<const T*>(a.k), *xv = reinterpret_cast<const T*>(a.v);
  const bool keeper = h % group == 0 && vt == 0;      // of the keys' and queries' inputs
  ConvSource<T> cv{a.conv_weight, a.conv_bias, reinterpret_cast<T*>(a.ring) + (int64_t)sq.slot * a.taps * C, C, a.taps, 0, 0};

  for (int t = 0; t < sq.count; ++t) {
    const int64_t row = sq.row0 + t;
    const int p = sq.ctx - sq.count + t;
    if (a.taps) { cv.row = p % a.taps; cv.seen = min(p, a.taps - 1); }
    const float* z = a.gate + row * a.gate_stride;
    float dt = 0.f, as = 0.f;
    if constexpr (KIND == ZP_LINEAR_SCALAR) {
      dt = ls_softplus(z[h] + a.gate_bias[h]);
      as = expf(-expf(a.A_log[h]) * dt);
    }
    if (tid < 128) {             // queries, keys and decays; the other half brings the values
#pragma unroll 1
      for (int d = tid; d < a.dim; d += 128) {
        const int c = hk * a.dim + d;
        float q, k, f;
        if constexpr (KIND == ZP_LINEAR_SCALAR) {
          if (a.taps) {
            const int ck = a.H * a.vdim + c, cq = ck + a.G * a.dim;
            ConvIn<T> vq, vk;
            conv_start(vq, cv, xq[row * a.x_stride + c], cq);
            conv_start(vk, cv, xk[row * a.x_stride + c], ck);
            q = conv_finish(vq, cv, cq);
            k = conv_finish(vk, cv, ck);
            if (keeper) { conv_keep(vq, cv, cq); conv_keep(vk, cv, ck); }
          } else {
            q = Elem<T>::to_f32(xq[row * a.x_stride + c]);
            k = Elem<T>::to_f32(xk[row * a.x_stride + c]);
          }
          k *= dt;
          f = as;
        } else {
          const float zz = z[c] + a.gate_bias[c];
          q = Elem<T>::to_f32(xq[row * a.x_stride + c]);
          if constexpr (KIND == ZP_LINEAR_FORGET) {
            const float l = a.lower[c];
            f = fmaf(1.f - l, ls_sigmoid(zz), l);
            k = (1.f - l) * ls_sigmoid(-zz);
            q = q * ls_sigmoid(q);
          } else {
            f = expf(-a.rtau * ls_softplus(-zz));
            k = Elem<T>::to_f32(xk[row * a.x_stride + c]);
            q *= a.qscale;
          }
        }
        sqk[d] = make_float4(q, k, f, 0.f);
      }
    } else if (tid - 128 < VT) {
      const int c = tid - 128, ch = h * a.vdim + c0 + c;
      float v = 0.f;
      if (c0 + c < a.vdim) {
        if (KIND == ZP_LINEAR_SCALAR && a.taps) {
          ConvIn<T> vv;
          conv_start(vv, cv, xv[row * a.x_stride + ch], ch);
          v = conv_finish(vv, cv, ch);
          conv_keep(vv, cv, ch);
        } else {
          v = Elem<T>::to_f32(xv[row * a.x_stride + ch]);
        }
      }
      sv[c] = v;
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    const float4 v = *reinterpret_cast<const float4*>(sv + 4 * cg);
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * nrg;
      if (r < a.dim) {
        const float4 x = sqk[r];
        s[i].x = fmaf(x.y, v.x, x.z * s[i].x); s[i].y = fmaf(x.y, v.y, x.z * s[i].y);
        s[i].z = fmaf(x.y, v.z, x.z * s[i].z); s[i].w = fmaf(x.y, v.w, x.z * s[i].w);
        o.x = fmaf(s[i].x, x.x, o.x); o.y = fmaf(s[i].y, x.x, o.y); o.z = fmaf(s[i].z, x.x, o.z); o.w = fmaf(s[i].w, x.x, o.w);
        if (t + 1 == sq.count && mine) *reinterpret_cast<float4*>(S + (int64_t)r * a.VP) = s[i];
      }
    }
    for (int w = 16; w >= ncg; w >>= 1) {     // the row groups of a warp
      o.x += __shfl_xor_sync(0xffffffffu, o.x, w); o.y += __shfl_xor_sync(0xffffffffu, o.y, w);
      o.z += __shfl_xor_sync(0xffffffffu, o.z, w); o.w += __shfl_xor_sync(0xffffffffu, o.w, w);
    }
    if (lane < ncg) *reinterpret_cast<float4*>(part + warp * VT + 4 * cg) = o;
    __syncthreads();
    if (out_col) {
      float y = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) y += part[w * VT + tid];
      if constexpr (KIND == ZP_LINEAR_SCALAR) y = fmaf(a.D[h], sv[tid], y);
      reinterpret_cast<T*>(a.out)[row * a.out_stride + (int64_t)h * a.vdim + c0 + tid] = Elem<T>::from_f32(y);
    }
    if (t + 1 < sq.count) __syncthreads();   // q, k, v and the sums are rewritten by the next token
  }
}

template <typename T, int KIND, int RPT>
static int launch_recurrent(const LinearArgs& a, int VT, cudaStream_t st) {
  const size_t smem = sizeof(float) * (4 * (size_t)a.dim + 9 * (size_t)VT);
  auto kern = linear_recurrent_kernel<T, KIND, RPT>;
  if (smem > 49152) {
    cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) { set_error("zp_linear_state: %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  }
  kern<<<dim3((a.VP + VT - 1) / VT, a.H, a.B), LR_THREADS, smem, st>>>(a, VT);
  return check_launch("zp_linear_state");
}

template <typename T, int KIND> static int linear_recurrent(const LinearArgs& a, cudaStream_t st) {
  auto rpt = [&](int w) { const int nrg = LR_THREADS / (w / 4); return (a.dim + nrg - 1) / nrg; };
  auto tiles = [&](int w) { return (a.VP + w - 1) / w; };
  // value columns of a block: as many as keep the state in registers, fewer when the batch leaves SMs without a block
  int VT = 128;
  while (VT > 4 && (VT / 2 >= a.VP || rpt(VT) > 16)) VT /= 2;
  while (VT > 16 && (int64_t)a.B * a.H * tiles(VT) < 148 * 2) VT /= 2;
  if (rpt(VT) > 16) { set_error("zp_linear_state: a key size of %d does not fit a block's registers", a.dim); return ZP_ERR_UNSUPPORTED; }
  if (rpt(VT) <= 4) return launch_recurrent<T, KIND, 4>(a, VT, st);
  if (rpt(VT) <= 8) return launch_recurrent<T, KIND, 8>(a, VT, st);
  return launch_recurrent<T, KIND, 16>(a, VT, st);
}

// ---------------------------------------------------------------------------------------------
// out = T(rms of every part of (silu(pre) x) * weight * silu(post)).  A part per warp, or per block when it is long; VPL
// 16-byte pieces per thread stay in registers (VPL = 0: any width, the part is read twice).
// ---------------------------------------------------------------------------------------------
struct GroupNormArgs {
  const void *x, *pre, *post;
  const float* w;
  void* out;
  int64_t x_stride, pre_stride, post_stride, out_stride, n;   // n: rows * parts
  int parts, width, per_part;
  float eps;
};
__device__ __forceinline__ float gn_ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float gn_rcp(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
template <typename T> __device__ __forceinline__ float gn_gate(float z) {
  if constexpr (sizeof(T) == 4) return z / (1.f + expf(-z));
  else return z * gn_rcp(1.f + gn_ex2(-1.4426950408889634f * z));      // (the fast forms' last bits disappear in the rounding to T)
}
// a 16-byte piece as fp32 and back
template <typename T> __device__ __forceinline__ void gn_unpack(const int4& raw, float (&v)[16 / sizeof(T)]) {
  if constexpr (sizeof(T) == 4) {
    v[0] = __int_as_float(raw.x); v[1] = __int_as_float(raw.y); v[2] = __int_as_float(raw.z); v[3] = __int_as_float(raw.w);
  } else {
    const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
    for (int j = 0; j < 8; ++j) v[j] = Elem<T>::to_f32(e[j]);
  }
}
template <typename T> __device__ __forceinline__ int4 gn_pack(const float (&v)[16 / sizeof(T)]) {
  if constexpr (sizeof(T) == 4) return make_int4(__float_as_int(v[0]), __float_as_int(v[1]), __float_as_int(v[2]), __float_as_int(v[3]));
  else return make_int4((int)pack2<T>(v[0], v[1]), (int)pack2<T>(v[2], v[3]), (int)pack2<T>(v[4], v[5]), (int)pack2<T>(v[6], v[7]));
}

template <typename T, int VPL, int TPP, int IT>   // TPP: threads of a part (32 or 256); IT: parts that a warp or block takes at a time
__global__ void __launch_bounds__(256) group_norm_gate_kernel(const GroupNormArgs a) {
  __shared__ float red[32];
  constexpr int EPV = 16 / sizeof(T);
  const uint32_t first = (TPP == 32 ? blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x) * IT, count = (uint32_t)a.n;   // (below 2^31)
  if (first >= count) return;                    // (a whole warp or block)
  const int lane = TPP == 32 ? threadIdx.x & 31 : threadIdx.x;
  struct Part { int64_t row; int c0; };
  const uint32_t row0 = first / (uint32_t)a.parts, part0 = first - row0 * a.parts;
  auto at = [&](int t) {                         // the t-th of this warp's or block's parts
    uint32_t row = row0, part = part0 + t;
    while (part >= (uint32_t)a.parts) { part -= a.parts; ++row; }
    return Part{(int64_t)row, (int)part * a.width};
  };
  const T *x = reinterpret_cast<const T*>(a.x), *pre = reinterpret_cast<const T*>(a.pre), *post = reinterpret_cast<const T*>(a.post);
  T* out = reinterpret_cast<T*>(a.out);
  if constexpr (VPL > 0) {
    const int nvec = a.width / EPV;
    int4 raw[IT][VPL], g[IT][VPL];
#pragma unroll
    for (int t = 0; t < IT; ++t) {
      const Part p = at(min((uint32_t)t, count - 1 - first));
#pragma unroll
      for (int i = 0; i < VPL; ++i)
        if (lane + i * TPP < nvec) {
          const int c = p.c0 + (lane + i * TPP) * EPV;
          raw[t][i] = ld16(x + p.row * a.x_stride + c);
          if (pre) g[t][i] = ld16(pre + p.row * a.pre_stride + c);
          else if (post) g[t][i] = ld16(post + p.row * a.post_stride + c);
        }
    }
#pragma unroll
    for (int t = 0; t < IT; ++t) {
      if (first + t >= count) break;
      const Part p = at(t);
      float v[VPL][EPV], ss = 0.f;
#pragma unroll
      for (int i = 0; i < VPL; ++i)
        if (lane + i * TPP < nvec) {
          gn_unpack<T>(raw[t][i], v[i]);
          if (pre) {
            float z[EPV];
            gn_unpack<T>(g[t][i], z);
#pragma unroll
            for (int j = 0; j < EPV; ++j) v[i][j] *= gn_gate<T>(z[j]);
          }
#pragma unroll
          for (int j = 0; j < EPV; ++j) ss = fmaf(v[i][j], v[i][j], ss);
        }
      ss = TPP == 32 ? warp_sum(ss) : block_sum(ss, red);
      const float r = 1.f / sqrtf(ss / (float)a.width + a.eps);
      const float* w = a.w + (a.per_part ? p.c0 : 0);
#pragma unroll
      for (int i = 0; i < VPL; ++i)
        if (lane + i * TPP < nvec) {
          const int c = (lane + i * TPP) * EPV;
          if (pre && post) g[t][i] = ld16(post + p.row * a.post_stride + p.c0 + c);
#pragma unroll
          for (int j = 0; j < EPV; j += 4) {
            const float4 wv = *reinterpret_cast<const float4*>(w + c + j);
            v[i][j] *= r * wv.x; v[i][j + 1] *= r * wv.y; v[i][j + 2] *= r * wv.z; v[i][j + 3] *= r * wv.w;
          }
          if (post) {
            float z[EPV];
            gn_unpack<T>(g[t][i], z);
#pragma unroll
            for (int j = 0; j < EPV; ++j) v[i][j] *= gn_gate<T>(z[j]);
          }
          st16(out + p.row * a.out_stride + p.c0 + c, gn_pack<T>(v[i]));
        }
    }
  } else {
    const Part p = at(0);
    const float* w = a.w + (a.per_part ? p.c0 : 0);
    auto entry = [&](int c) {
      const float y = Elem<T>::to_f32(x[p.row * a.x_stride + p.c0 + c]);
      return pre ? y * gn_gate<T>(Elem<T>::to_f32(pre[p.row * a.pre_stride + p.c0 + c])) : y;
    };
    float ss = 0.f;
    for (int c = lane; c < a.width; c += TPP) { const float y = entry(c); ss = fmaf(y, y, ss); }
    ss = TPP == 32 ? warp_sum(ss) : block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)a.width + a.eps);
    for (int c = lane; c < a.width; c += TPP) {
      float y = entry(c) * r * w[c];
      if (post) y *= gn_gate<T>(Elem<T>::to_f32(post[p.row * a.post_stride + p.c0 + c]));
      out[p.row * a.out_stride + p.c0 + c] = Elem<T>::from_f32(y);
    }
  }
}

template <typename T, int VPL, int TPP, int IT> static void group_norm_items(const GroupNormArgs& a, cudaStream_t st) {
  const int64_t per = (TPP == 32 ? 8 : 1) * IT;
  group_norm_gate_kernel<T, VPL, TPP, IT><<<(unsigned)((a.n + per - 1) / per), 256, 0, st>>>(a);
}
template <typename T> static void launch_group_norm(const GroupNormArgs& a, bool vec, cudaStream_t st) {
  const int nv = a.width / (int)(16 / sizeof(T));
  const bool many = a.n >= 148 * 8 * 8 * 4;      // (few parts: spread over the SMs instead)
  if (!vec) {
    if (a.width <= 1024) group_norm_items<T, 0, 32, 1>(a, st);
    else group_norm_items<T, 0, 256, 1>(a, st);
  } else if (nv <= 32) {
    if (many) group_norm_items<T, 1, 32, 4>(a, st); else group_norm_items<T, 1, 32, 1>(a, st);
  } else if (nv <= 64) {
    if (many) group_norm_items<T, 2, 32, 2>(a, st); else group_norm_items<T, 2, 32, 1>(a, st);
  } else if (nv <= 256) {
    if (many) group_norm_items<T, 1, 256, 2>(a, st); else group_norm_items<T, 1, 256, 1>(a, st);
  } else if (nv <= 512) group_norm_items<T, 2, 256, 1>(a, st);
  else if (nv <= 1024) group_norm_items<T, 4, 256, 1>(a, st);
  else group_norm_items<T, 0, 256, 1>(a, st);
}

}  // namespace zp

extern "C" size_t zp_linear_state_workspace_bytes(int total_rows, int B, int H, int dim) {
  return total_rows > 0 && B > 0 && H > 0 && dim > 0 ? zp::linear_chunk_workspace(total_rows, B, H, dim) : 0;
}

extern "C" int zp_linear_state(const zp_linear_state_params* params, int impl, int dtype, void* stream) {
  ZP_REQUIRE(params, "zp_linear_state: null pointer");
  const zp_linear_state_params& a = *params;
  if (a.B == 0) return ZP_OK;
  const bool forget = a.kind == ZP_LINEAR_FORGET, scalar = a.kind == ZP_LINEAR_SCALAR;
  ZP_REQUIRE(forget || scalar || a.kind == ZP_LINEAR_POWER, "zp_linear_state: unknown kind %d", a.kind);
  ZP_REQUIRE(a.q && (a.k || forget) && a.v && a.gate && a.gate_bias && a.context_lens && a.slots && a.state && a.out,
             "zp_linear_state: null pointer");
  ZP_REQUIRE((!forget || a.lower) && (!scalar || (a.A_log && a.D)), "zp_linear_state: null pointer");
  ZP_REQUIRE(a.taps >= 0 && (a.taps == 0 || (scalar && a.conv_weight && a.ring && !a.cu_seqlens_q)),
             "zp_linear_state: the convolution is part of the launch for single rows of scalar decays only");
  ZP_REQUIRE(a.G > 0 && a.H % a.G == 0 && (scalar || a.G == a.H) && a.H <= 65535 && a.B <= 65535 && a.dim > 0 && a.dim <= 4096 && a.vdim > 0 &&
             a.VP >= a.vdim && a.VP % 4 == 0 && a.n_slots > 0, "zp_linear_state: bad sizes");
  ZP_REQUIRE((uintptr_t)a.state % 16 == 0, "zp_linear_state: the state must be 16-byte aligned");
  cudaStream_t st = (cudaStream_t)stream;
  const bool tc = a.cu_seqlens_q && a.total_rows > 0 && dtype == ZP_DTYPE_BF16 && zp::linear_chunk_supports(a);
  if (impl == ZP_IMPL_TCGEN05 && !tc) {
    zp::set_error("zp_linear_state: the tcgen05 kernels need bf16 portions, head sizes that are multiples of 8, keys up to 128 and 16-byte aligned rows");
    return ZP_ERR_UNSUPPORTED;
  }
  if (tc && (impl == ZP_IMPL_TCGEN05 || (impl == ZP_IMPL_AUTO && a.total_rows >= 8 * a.B))) {
    const size_t need = zp::linear_chunk_workspace(a.total_rows, a.B, a.H, a.dim);
    ZP_REQUIRE(a.workspace && a.workspace_bytes >= need && (uintptr_t)a.workspace % 16 == 0, "zp_linear_state: workspace of %zu bytes, %zu needed",
               a.workspace_bytes, need);
    return zp::linear_chunk(a, st);
  }
  ZP_DISPATCH_DTYPE(dtype, T, {
    if (forget) return zp::linear_recurrent<T, ZP_LINEAR_FORGET>(a, st);
    if (scalar) return zp::linear_recurrent<T, ZP_LINEAR_SCALAR>(a, st);
    return zp::linear_recurrent<T, ZP_LINEAR_POWER>(a, st);
  });
  return ZP_OK;
}

extern "C" int zp_group_norm_gate(const void* x, int64_t x_stride, const void* pre_gate, int64_t pre_stride, const void* post_gate,
                                  int64_t post_stride, const float* weight, int weight_per_part, void* out, int64_t out_stride, int n_rows,
                                  int parts, int width, float eps, int dtype, void* stream) {
  if (n_rows == 0) return ZP_OK;
  ZP_REQUIRE(x && weight && out, "zp_group_norm_gate: null pointer");
  ZP_REQUIRE(parts > 0 && width > 0 && (int64_t)n_rows * parts < (1ll << 31) && x_stride >= (int64_t)parts * width && out_stride >= (int64_t)parts * width,
             "zp_group_norm_gate: bad sizes");
  const int epv = (int)(16 / zp::dtype_size(dtype));
  const bool vec = width % epv == 0 && x_stride % epv == 0 && out_stride % epv == 0 && (!pre_gate || pre_stride % epv == 0) &&
                   (!post_gate || post_stride % epv == 0) &&
                   ((uintptr_t)x | (uintptr_t)pre_gate | (uintptr_t)post_gate | (uintptr_t)weight | (uintptr_t)out) % 16 == 0;
  zp::GroupNormArgs a{x, pre_gate, post_gate, weight, out, x_stride, pre_stride, post_stride, out_stride, (int64_t)n_rows * parts, parts, width,
                      weight_per_part, eps};
  ZP_DISPATCH_DTYPE(dtype, T, { zp::launch_group_norm<T>(a, vec, (cudaStream_t)stream); });
  return zp::check_launch("zp_group_norm_gate");
}
