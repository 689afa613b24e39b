// Gated delta rule, token by token: the decode kernel (from projections to gated output in one launch), also used for
// prompts in fp32.
//
// HBM-bound: a decoded token reads and writes the head's whole fp32 state once.  One block per (value tile, head,
// sequence); its part of the state stays in registers (up to 16 rows of four columns a thread), so the read that the
// correction needs (S^T k) and the update are one pass over memory: with S^T k and S^T q of the old state,
//   u = b (v - g S^T k),   o = g S^T q + (k . q) u,   S <- g S + k u^T.
// The blocks of a head form a cluster when there are several: the output norm spans all value dims.
#include "zp_conv.cuh"
#include "zp_delta.cuh"
#include "zp_mlstm.cuh"    // cluster helpers

namespace zp {

constexpr int DR_THREADS = 256;

template <typename T, int RPT>   // RPT: state rows per thread
__global__ void __launch_bounds__(DR_THREADS, RPT == 16 ? 2 : RPT == 8 ? 3 : 4) delta_recurrent_kernel(const DeltaArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[3][8], red2[8];
  __shared__ float xsum[2];      // this block's sum of squares, by token parity
  const int vt = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const DeltaSeq sq = delta_seq(a, b);
  if (sq.count == 0) return;     // the same decision in every block of the cluster
  const int group = a.H / a.G, hk = h / group, C = 2 * a.G * a.dim + a.H * a.vdim;
  const int c0 = vt * a.VT, ncg = a.VT / 4, nrg = DR_THREADS / ncg;   // (powers of two; ncg <= 32)
  float* sq_ = sm;               // [dim] q
  float* sk = sq_ + a.dim;       // [dim] k
  float* sv = sm + ((2 * a.dim + 3) & ~3);   // [VT] v
  float* su = sv + a.VT;         // [VT] the update's row
  float* part = su + a.VT;       // [2][8 warps][VT]
  const int cg = tid & (ncg - 1), rg = tid / ncg, col = c0 + 4 * cg;
  const bool mine = col < a.VP, out_col = tid < a.VT && c0 + tid < a.vdim;      // (VT <= 128)
  float* S = a.S + ((int64_t)sq.slot * a.H + h) * a.dim * a.VP + col;
  float4 s[RPT];
#pragma unroll
  for (int i = 0; i < RPT; ++i) {
    const int r = rg + i * nrg;
    s[i] = (mine && r < a.dim && !sq.fresh) ? *reinterpret_cast<const float4*>(S + (int64_t)r * a.VP) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const T* x = reinterpret_cast<const T*>(a.x);
  ConvSource<T> cv{a.conv_w, nullptr, reinterpret_cast<T*>(a.ring) + (int64_t)sq.slot * a.taps * C, C, a.taps, 0, 0};
  const float qscale = rsqrtf((float)a.dim), nw = out_col ? a.norm_weight[c0 + tid] : 0.f;
  const bool keeper = h % group == 0 && vt == 0;      // of the keys' and queries' inputs

  for (int t = 0; t < sq.count; ++t) {
    const int64_t row = sq.row0 + t;
    const int p = sq.ctx - sq.count + t;
    const T* xr = x + row * a.x_stride;
    const float z = out_col ? Elem<T>::to_f32(reinterpret_cast<const T*>(a.gate)[row * a.gate_stride + (int64_t)h * a.vdim + c0 + tid]) : 0.f;
    if (a.taps) { cv.row = p % a.taps; cv.seen = min(p, a.taps - 1); }
    float qq = 0.f, kk = 0.f, kq = 0.f;
    if (tid < 128) {             // queries and keys; the other half brings the values
#pragma unroll 1
      for (int d = tid; d < a.dim; d += 128) {
        const int cq = hk * a.dim + d, ck = a.G * a.dim + cq;
        float q, k;
        if (a.taps) {
          ConvIn<T> vq, vk;
          conv_start(vq, cv, xr[cq], cq);
          conv_start(vk, cv, xr[ck], ck);
          q = conv_finish(vq, cv, cq);
          k = conv_finish(vk, cv, ck);
          if (keeper) { conv_keep(vq, cv, cq); conv_keep(vk, cv, ck); }
        } else {
          q = Elem<T>::to_f32(xr[cq]);
          k = Elem<T>::to_f32(xr[ck]);
        }
        sq_[d] = q; sk[d] = k;
        qq = fmaf(q, q, qq); kk = fmaf(k, k, kk); kq = fmaf(k, q, kq);
      }
    } else if (tid - 128 < a.VT) {
      const int c = tid - 128, ch = 2 * a.G * a.dim + h * a.vdim + c0 + c;
      float v = 0.f;
      if (c0 + c < a.vdim) {
        if (a.taps) {
          ConvIn<T> vv;
          conv_start(vv, cv, xr[ch], ch);
          v = conv_finish(vv, cv, ch);
          conv_keep(vv, cv, ch);
        } else {
          v = Elem<T>::to_f32(xr[ch]);
        }
      }
      sv[c] = v;
    }
    const float g = expf(delta_log_decay(a, row, h)), beta = delta_beta(a, row, h);
    qq = warp_sum(qq); kk = warp_sum(kk); kq = warp_sum(kq);
    if (lane == 0) { red[0][warp] = qq; red[1][warp] = kk; red[2][warp] = kq; }
    __syncthreads();
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * nrg;
      if (r < a.dim) {
        const float kr = sk[r], qr = sq_[r];
        ak.x = fmaf(s[i].x, kr, ak.x); ak.y = fmaf(s[i].y, kr, ak.y); ak.z = fmaf(s[i].z, kr, ak.z); ak.w = fmaf(s[i].w, kr, ak.w);
        aq.x = fmaf(s[i].x, qr, aq.x); aq.y = fmaf(s[i].y, qr, aq.y); aq.z = fmaf(s[i].z, qr, aq.z); aq.w = fmaf(s[i].w, qr, aq.w);
      }
    }
    for (int o = 16; o >= ncg; o >>= 1) {     // the row groups of a warp
      ak.x += __shfl_xor_sync(0xffffffffu, ak.x, o); ak.y += __shfl_xor_sync(0xffffffffu, ak.y, o);
      ak.z += __shfl_xor_sync(0xffffffffu, ak.z, o); ak.w += __shfl_xor_sync(0xffffffffu, ak.w, o);
      aq.x += __shfl_xor_sync(0xffffffffu, aq.x, o); aq.y += __shfl_xor_sync(0xffffffffu, aq.y, o);
      aq.z += __shfl_xor_sync(0xffffffffu, aq.z, o); aq.w += __shfl_xor_sync(0xffffffffu, aq.w, o);
    }
    if (lane < ncg) {
      *reinterpret_cast<float4*>(part + warp * a.VT + 4 * cg) = ak;
      *reinterpret_cast<float4*>(part + (8 + warp) * a.VT + 4 * cg) = aq;
    }
    __syncthreads();
    float o = 0.f;               // column tid of the tile
    if (tid < a.VT) {
      qq = kk = kq = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) { qq += red[0][w]; kk += red[1][w]; kq += red[2][w]; }
      const float rq = qscale / sqrtf(qq + DELTA_UNIT_EPS), rk = 1.f / sqrtf(kk + DELTA_UNIT_EPS);
      float kS = 0.f, qS = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) { kS += part[w * a.VT + tid]; qS += part[(8 + w) * a.VT + tid]; }
      const float u = beta * (sv[tid] - g * rk * kS);
      o = fmaf(g * rq, qS, rk * rq * kq * u);
      su[tid] = rk * u;
    }
    float ss = warp_sum(o * o);
    if (lane == 0) red2[warp] = ss;
    __syncthreads();
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
      const int r = rg + i * nrg;
      if (r < a.dim) {
        const float kr = sk[r];
        const float4 u = *reinterpret_cast<const float4*>(su + 4 * cg);
        s[i].x = fmaf(kr, u.x, g * s[i].x); s[i].y = fmaf(kr, u.y, g * s[i].y);
        s[i].z = fmaf(kr, u.z, g * s[i].z); s[i].w = fmaf(kr, u.w, g * s[i].w);
        if (t + 1 == sq.count && mine) *reinterpret_cast<float4*>(S + (int64_t)r * a.VP) = s[i];
      }
    }
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) ss += red2[w];            // (columns: the first 128 threads)
    if (cluster_size() > 1) {
      if (tid == 0) xsum[t & 1] = ss;
      cluster_sync();
      ss = 0.f;
      for (uint32_t r = 0; r < cluster_size(); ++r) ss += ld_cluster(&xsum[t & 1], r);
    }
    if (out_col) {
      const float rr = a.out_scale / sqrtf(ss / (float)a.vdim + a.eps);
      reinterpret_cast<T*>(a.out)[row * a.out_stride + (int64_t)h * a.vdim + c0 + tid] = Elem<T>::from_f32(o * rr * nw * (z / (1.f + expf(-z))));
    }
    if (t + 1 < sq.count) __syncthreads();   // q, k and u are rewritten by the next token
  }
  if (cluster_size() > 1) cluster_sync();   // peers may still be reading xsum
}

template <typename T, int RPT>
static int launch_recurrent(const DeltaArgs& a, int tiles, cudaStream_t st) {
  const size_t smem = sizeof(float) * (((2 * a.dim + 3) & ~3) + 18 * (size_t)a.VT);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles, a.H, a.B);
  cfg.blockDim = dim3(DR_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = tiles; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  cudaError_t e = cudaLaunchKernelEx(&cfg, delta_recurrent_kernel<T, RPT>, a);
  if (e != cudaSuccess) { set_error("zp_gated_delta: %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  return check_launch("zp_gated_delta");
}

// value columns of a block: as many as keep the state in registers, fewer when the batch leaves SMs without a block
static int recurrent_tile(const DeltaArgs& a) {
  int VT = 128;
  while (VT > 4 && (VT / 2 >= a.VP || (a.dim + DR_THREADS / (VT / 4) - 1) / (DR_THREADS / (VT / 4)) > 16)) VT /= 2;
  auto tiles = [&](int w) { return (a.VP + w - 1) / w; };
  while (VT > 16 && tiles(VT / 2) <= 8 && (int64_t)a.B * a.H * tiles(VT) < 148 * 2) VT /= 2;
  return VT;
}

template <typename T>
static int delta_recurrent(DeltaArgs a, cudaStream_t st) {
  a.VT = recurrent_tile(a);
  const int tiles = (a.VP + a.VT - 1) / a.VT, nrg = DR_THREADS / (a.VT / 4), rpt = (a.dim + nrg - 1) / nrg;
  if (tiles > 8 || rpt > 16) {
    set_error("zp_gated_delta: a state of %d x %d does not fit the registers of eight blocks", a.dim, a.vdim);
    return ZP_ERR_UNSUPPORTED;
  }
  if (rpt <= 4) return launch_recurrent<T, 4>(a, tiles, st);
  if (rpt <= 8) return launch_recurrent<T, 8>(a, tiles, st);
  return launch_recurrent<T, 16>(a, tiles, st);
}

}  // namespace zp

extern "C" size_t zp_gated_delta_workspace_bytes(int total_rows, int B, int H) {
  return total_rows > 0 && B > 0 && H > 0 ? zp::delta_chunk_workspace(total_rows, B, H) : 0;
}

extern "C" int zp_gated_delta(const void* x, int64_t x_stride, const void* gate, int64_t gate_stride, const float* ab,
                              int64_t ab_stride, const float* A_log, const float* dt_bias, const float* norm_weight,
                              const float* conv_weight, void* ring, int taps, const int32_t* cu_seqlens_q,
                              const int32_t* context_lens, const int32_t* slots, float* state, void* out, int64_t out_stride,
                              int B, int H, int G, int dim, int vdim, int VP, int n_slots, float eps, float out_scale,
                              int total_rows, int impl, int dtype, void* workspace, size_t workspace_bytes, void* stream) {
  if (B == 0) return ZP_OK;
  ZP_REQUIRE(x && gate && ab && A_log && dt_bias && norm_weight && context_lens && slots && state && out, "zp_gated_delta: null pointer");
  ZP_REQUIRE(taps >= 0 && (taps == 0 || (conv_weight && ring && !cu_seqlens_q)),
             "zp_gated_delta: the convolution is part of the launch for single rows only");
  ZP_REQUIRE(G > 0 && H % G == 0 && H <= 65535 && B <= 65535 && dim > 0 && dim <= 2048 && vdim > 0 && VP >= vdim && VP % 4 == 0 && n_slots > 0,
             "zp_gated_delta: bad sizes");
  ZP_REQUIRE((uintptr_t)state % 16 == 0, "zp_gated_delta: the state must be 16-byte aligned");
  zp::DeltaArgs a;
  a.x = x; a.gate = gate; a.ab = ab; a.A_log = A_log; a.dt_bias = dt_bias; a.norm_weight = norm_weight; a.conv_w = conv_weight;
  a.ring = ring; a.cu_q = cu_seqlens_q; a.context_lens = context_lens; a.slots = slots; a.S = state; a.out = out; a.B = B; a.H = H;
  a.G = G; a.dim = dim; a.vdim = vdim; a.VP = VP; a.n_slots = n_slots; a.taps = taps; a.VT = 0; a.x_stride = x_stride;
  a.gate_stride = gate_stride; a.ab_stride = ab_stride; a.out_stride = out_stride; a.eps = eps; a.out_scale = out_scale;
  cudaStream_t st = (cudaStream_t)stream;
  const bool tc = cu_seqlens_q && total_rows > 0 && zp::delta_chunk_supports(a, dtype);
  if (impl == ZP_IMPL_TCGEN05 && !tc) {
    zp::set_error("zp_gated_delta: the tcgen05 kernels need bf16 portions, head sizes that are multiples of 8, keys up to 128, values up to 256, "
                  "and 16-byte aligned rows");
    return ZP_ERR_UNSUPPORTED;
  }
  if (tc && (impl == ZP_IMPL_TCGEN05 || (impl == ZP_IMPL_AUTO && total_rows >= 8 * B))) {
    const size_t need = zp::delta_chunk_workspace(total_rows, B, H);
    ZP_REQUIRE(workspace && workspace_bytes >= need && (uintptr_t)workspace % 16 == 0, "zp_gated_delta: workspace of %zu bytes, %zu needed",
               workspace_bytes, need);
    return zp::delta_chunk(a, total_rows, workspace, st);
  }
  ZP_DISPATCH_DTYPE(dtype, T, { return zp::delta_recurrent<T>(a, st); });
  return ZP_OK;
}
