// Linear attention with a decaying matrix state, token by token: the decode kernel (from projections to outputs in one launch),
// also used for prompts in fp32, and the norm with gates that follows it.
//
// HBM-bound: a decoded token reads and writes the head's whole fp32 state once.  One block per (value tile, head,
// sequence); its part of the state stays in registers (up to 16 rows of four columns a thread), all of its loads in flight
// while keys, queries and decays are made.
#include "zp_conv.cuh"
#include "zp_linear_state.cuh"

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
template <typename T> __device__ __forceinline__ float gn_gate(float z) {
  if constexpr (sizeof(T) == 4) return z / (1.f + expf(-z));
  else return __fdividef(z, 1.f + __expf(-z));      // (the fast forms' last bits disappear in the rounding to T)
}

template <typename T, int VPL, int TPP>   // TPP: threads of a part (32 or 256)
__global__ void __launch_bounds__(256) group_norm_gate_kernel(const GroupNormArgs a) {
  __shared__ float red[32];
  constexpr int EPV = 16 / sizeof(T);
  const int64_t item = TPP == 32 ? (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5) : blockIdx.x;
  if (item >= a.n) return;                       // (a whole warp or block)
  const int lane = TPP == 32 ? threadIdx.x & 31 : threadIdx.x;
  const int64_t row = item / a.parts;
  const int part = (int)(item - row * a.parts), c0 = part * a.width;
  const T* x = reinterpret_cast<const T*>(a.x) + row * a.x_stride + c0;
  const T* pre = a.pre ? reinterpret_cast<const T*>(a.pre) + row * a.pre_stride + c0 : nullptr;
  const T* post = a.post ? reinterpret_cast<const T*>(a.post) + row * a.post_stride + c0 : nullptr;
  const float* w = a.w + (a.per_part ? c0 : 0);
  T* out = reinterpret_cast<T*>(a.out) + row * a.out_stride + c0;
  float ss = 0.f;
  if constexpr (VPL > 0) {
    const int nvec = a.width / EPV;
    int4 raw[VPL], g[VPL];
    float v[VPL][EPV];
#pragma unroll
    for (int i = 0; i < VPL; ++i)
      if (lane + i * TPP < nvec) {
        raw[i] = ld16(x + (lane + i * TPP) * EPV);
        if (pre) g[i] = ld16(pre + (lane + i * TPP) * EPV);
        else if (post) g[i] = ld16(post + (lane + i * TPP) * EPV);
      }
#pragma unroll
    for (int i = 0; i < VPL; ++i)
      if (lane + i * TPP < nvec) {
        const T *e = reinterpret_cast<const T*>(&raw[i]), *f = reinterpret_cast<const T*>(&g[i]);
#pragma unroll
        for (int j = 0; j < EPV; ++j) {
          v[i][j] = Elem<T>::to_f32(e[j]);
          if (pre) v[i][j] *= gn_gate<T>(Elem<T>::to_f32(f[j]));
          ss = fmaf(v[i][j], v[i][j], ss);
        }
      }
    ss = TPP == 32 ? warp_sum(ss) : block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)a.width + a.eps);
#pragma unroll
    for (int i = 0; i < VPL; ++i)
      if (lane + i * TPP < nvec) {
        const int c = (lane + i * TPP) * EPV;
        if (pre && post) g[i] = ld16(post + c);
        const T* f = reinterpret_cast<const T*>(&g[i]);
        int4 res;
        T* o = reinterpret_cast<T*>(&res);
#pragma unroll
        for (int j = 0; j < EPV; j += 4) {
          const float4 wv = *reinterpret_cast<const float4*>(w + c + j);
          const float ww[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            float y = v[i][j + u] * r * ww[u];
            if (post) y *= gn_gate<T>(Elem<T>::to_f32(f[j + u]));
            o[j + u] = Elem<T>::from_f32(y);
          }
        }
        st16(out + c, res);
      }
  } else {
    for (int c = lane; c < a.width; c += TPP) {
      float y = Elem<T>::to_f32(x[c]);
      if (pre) y *= gn_gate<T>(Elem<T>::to_f32(pre[c]));
      ss = fmaf(y, y, ss);
    }
    ss = TPP == 32 ? warp_sum(ss) : block_sum(ss, red);
    const float r = 1.f / sqrtf(ss / (float)a.width + a.eps);
    for (int c = lane; c < a.width; c += TPP) {
      float y = Elem<T>::to_f32(x[c]);
      if (pre) y *= gn_gate<T>(Elem<T>::to_f32(pre[c]));
      y *= r * w[c];
      if (post) y *= gn_gate<T>(Elem<T>::to_f32(post[c]));
      out[c] = Elem<T>::from_f32(y);
    }
  }
}

template <typename T> static void launch_group_norm(const GroupNormArgs& a, bool vec, cudaStream_t st) {
  constexpr int EPV = 16 / sizeof(T);
  const unsigned warps = (unsigned)((a.n + 7) / 8), blocks = (unsigned)a.n;
  const int nv = a.width / EPV;
  if (!vec) {
    if (a.width <= 1024) group_norm_gate_kernel<T, 0, 32><<<warps, 256, 0, st>>>(a);
    else group_norm_gate_kernel<T, 0, 256><<<blocks, 256, 0, st>>>(a);
  } else if (nv <= 32) group_norm_gate_kernel<T, 1, 32><<<warps, 256, 0, st>>>(a);
  else if (nv <= 64) group_norm_gate_kernel<T, 2, 32><<<warps, 256, 0, st>>>(a);
  else if (nv <= 256) group_norm_gate_kernel<T, 1, 256><<<blocks, 256, 0, st>>>(a);
  else if (nv <= 512) group_norm_gate_kernel<T, 2, 256><<<blocks, 256, 0, st>>>(a);
  else if (nv <= 1024) group_norm_gate_kernel<T, 4, 256><<<blocks, 256, 0, st>>>(a);
  else group_norm_gate_kernel<T, 0, 256><<<blocks, 256, 0, st>>>(a);
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
