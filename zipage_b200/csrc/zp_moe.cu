// Mixture of experts: routing (softmax scores over all experts or over the chosen ones, or sigmoid scores, the largest `top` of a token) with the
// bookkeeping that sorts (token, expert) pairs by expert, and matrix products of the sorted rows with their
// expert's weights.  This file has the routing kernels, the SIMT product for fp32 and odd sizes, and the entry
// points; zp_moe_tc.cu has the tensor-core product.
//
// Places: the pairs of expert e take places offsets[e] .. offsets[e + 1] in an order that may differ
// between runs; a pair's results do not depend on its place.
#include "zp_moe.cuh"

namespace zp {

constexpr int RT_MAXE = 1024;

// fp32 -> unsigned with the same order (NaNs of either sign sort above or below all numbers)
__device__ __forceinline__ unsigned order_key(float v) {
  const unsigned u = __float_as_uint(v);
  return (u & 0x80000000u) ? ~u : u | 0x80000000u;
}

// The `top` largest of one token's logits by one warp: lane holds experts lane, lane + 32, ...  Ties: the lower
// expert.  Choice k is returned by lane k % 32 of round k / 32 (emit(k, expert, score) is called by that lane,
// all lanes of a round at once).
// Returns the sum that ZP_SCORE_SOFTMAX_TOP divides by (its scores are emitted without).
template <int VPL, typename F>
__device__ __forceinline__ float top_experts(const float* __restrict__ z, const float* __restrict__ bias, int E, int top, int score_kind, F&& emit) {
  const int lane = threadIdx.x & 31;
  float v[VPL], mx = -INFINITY;
  unsigned key[VPL];                        // 0: taken, or no expert
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
    const bool in = lane + 32 * i < E;
    v[i] = in ? z[lane + 32 * i] + (bias ? bias[lane + 32 * i] : 0.f) : -INFINITY;
    key[i] = in ? max(order_key(v[i]), 1u) : 0u;
    mx = fmaxf(mx, v[i]);
  }
  mx = warp_max(mx);
  float sum = 0.f;
#pragma unroll
  for (int i = 0; i < VPL; ++i) sum += lane + 32 * i < E ? expf(v[i] - mx) : 0.f;
  sum = score_kind == ZP_SCORE_SOFTMAX ? warp_sum(sum) : 1.f;
  float chosen = 0.f;
  for (int k0 = 0; k0 < top; k0 += 32) {
    int mine = 0;
    float score = 0.f;
    for (int k = k0; k < min(top, k0 + 32); ++k) {
      unsigned bk = 0, bi = 0xffffffffu;
      float bv = 0.f;
#pragma unroll
      for (int i = 0; i < VPL; ++i)
        if (key[i] > bk) { bk = key[i]; bi = lane + 32 * i; bv = v[i]; }
      const unsigned best = __reduce_max_sync(0xffffffffu, bk);
      const unsigned at = __reduce_min_sync(0xffffffffu, bk == best ? bi : 0xffffffffu);
      bv = __shfl_sync(0xffffffffu, bv, at & 31);
      if (score_kind == ZP_SCORE_SOFTMAX_TOP) chosen += expf(bv - mx);
      if ((int)(at & 31) == lane) {
#pragma unroll
        for (int i = 0; i < VPL; ++i)
          if ((int)(at >> 5) == i) key[i] = 0u;
      }
      if (lane == k - k0) { mine = (int)at; score = bv; }
    }
    if (lane < top - k0) emit(k0 + lane, mine, score_kind == ZP_SCORE_SIGMOID ? 1.f / (1.f + expf(-score)) : expf(score - mx) / sum);
  }
  return chosen;
}

// exclusive scan of counts[0 .. E) into offs[0 .. E] by the first warp of the block
__device__ __forceinline__ void scan_counts(const int* counts, int* offs, int E) {
  if (threadIdx.x < 32) {
    int base = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x, c = e < E ? counts[e] : 0;
      int s = c;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int t = __shfl_up_sync(0xffffffffu, s, o);
        if ((int)threadIdx.x >= o) s += t;
      }
      if (e < E) offs[e] = base + s - c;
      base += __shfl_sync(0xffffffffu, s, 31);
    }
    if (threadIdx.x == 0) offs[E] = base;
  }
}

struct RouteArgs {
  const float* logits;
  int64_t ld;
  int N, E, top;
  float* wts;          // [N, top]
  int32_t *idx, *pos;  // [N, top]; between the two kernels pos holds ranks within the expert
  int32_t *rows, *offsets, *counts;
  float* place_wts;    // [N * top] or NULL: the weights in the order of the places
  int score;
  const float* bias;   // [E] or NULL
};

// One block does everything (ONE; at most RT_ONE pairs), or several blocks choose and count and route_place_kernel places.
constexpr int RT_ONE = 4096;
template <int VPL, bool ONE>
__global__ void __launch_bounds__(ONE ? 1024 : 256) route_kernel(const RouteArgs a) {
  __shared__ int hist[RT_MAXE], offs[RT_MAXE + 1];
  __shared__ int2 picks[ONE ? RT_ONE : 1];                     // expert and rank within it
  for (int e = threadIdx.x; e < a.E; e += blockDim.x) hist[e] = 0;
  __syncthreads();
  const int nw = blockDim.x >> 5, per = ONE ? a.N : 32;        // tokens of a block
  const int t0 = blockIdx.x * per, t1 = min(a.N, t0 + per);
  for (int t = t0 + (threadIdx.x >> 5); t < t1; t += nw) {
    const float chosen = top_experts<VPL>(a.logits + (int64_t)t * a.ld, a.bias, a.E, a.top, a.score, [&](int k, int e, float s) {
      const int64_t at = (int64_t)t * a.top + k;
      a.wts[at] = s;
      a.idx[at] = e;
      const int rank = atomicAdd(&hist[e], 1);
      if constexpr (ONE) picks[at] = make_int2(e, rank);
      else a.pos[at] = rank;
    });
    if (a.score == ZP_SCORE_SOFTMAX_TOP)       // (a lane divides what it has written)
      for (int k = threadIdx.x & 31; k < a.top; k += 32) a.wts[(int64_t)t * a.top + k] /= chosen;
  }
  __syncthreads();
  if constexpr (ONE) {
    scan_counts(hist, offs, a.E);
    __syncthreads();
    for (int e = threadIdx.x; e <= a.E; e += blockDim.x) a.offsets[e] = offs[e];
    for (int i = threadIdx.x; i < a.N * a.top; i += blockDim.x) {
      const int p = offs[picks[i].x] + picks[i].y;
      a.pos[i] = p;
      a.rows[p] = i / a.top;
      if (a.place_wts) a.place_wts[p] = a.wts[i];
    }
  } else {
    for (int e = threadIdx.x; e < a.E; e += blockDim.x) offs[e] = hist[e] ? atomicAdd(&a.counts[e], hist[e]) : 0;
    __syncthreads();
    for (int i = t0 * a.top + threadIdx.x; i < t1 * a.top; i += blockDim.x) a.pos[i] += offs[a.idx[i]];
  }
}

__global__ void __launch_bounds__(256) route_place_kernel(const RouteArgs a) {
  __shared__ int offs[RT_MAXE + 1];
  scan_counts(a.counts, offs, a.E);
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = threadIdx.x; e <= a.E; e += blockDim.x) a.offsets[e] = offs[e];
  const int64_t n = (int64_t)a.N * a.top;
  for (int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x; i < n; i += (int64_t)gridDim.x * blockDim.x) {
    const int p = offs[a.idx[i]] + a.pos[i];
    a.pos[i] = p;
    a.rows[p] = (int32_t)(i / a.top);
    if (a.place_wts) a.place_wts[p] = a.wts[i];
  }
}

template <int VPL> static int launch_route(const RouteArgs& a, cudaStream_t st) {
  if (a.N <= 512 && a.N * a.top <= RT_ONE) {
    route_kernel<VPL, true><<<1, 1024, 0, st>>>(a);
  } else {
    cudaError_t e = cudaMemsetAsync(a.counts, 0, (size_t)a.E * sizeof(int), st);
    if (e != cudaSuccess) { set_error("zp_moe_route: %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
    route_kernel<VPL, false><<<(a.N + 31) / 32, 256, 0, st>>>(a);
    const int64_t want = ((int64_t)a.N * a.top + 255) / 256;
    route_place_kernel<<<(int)(want < 592 ? want : 592), 256, 0, st>>>(a);
  }
  return check_launch("zp_moe_route");
}

// ---------------------------------------------------------------------------------------------
// SIMT product: 64 x 64 tiles of out[place, n] = act(sum_k x[row(place), k] w[e, n, k]), fp32 accumulation.
// ---------------------------------------------------------------------------------------------
constexpr int GS_T = 64, GS_K = 16;

template <typename T> __global__ void __launch_bounds__(256) grouped_gemm_simt_kernel(const GroupedArgs a) {
  __shared__ float sx[GS_K][GS_T + 4], sw[GS_K][GS_T + 4];
  __shared__ int src[GS_T], s_e, s_first, s_count;
  if (threadIdx.x == 0) {
    int tile = blockIdx.x, e = 0;
    for (; e < a.E; ++e) {
      const int n = a.offsets[e + 1] - a.offsets[e], t = (n + GS_T - 1) / GS_T;
      if (tile < t) break;
      tile -= t;
    }
    s_e = e;
    if (e < a.E) { s_first = a.offsets[e] + tile * GS_T; s_count = min(GS_T, a.offsets[e + 1] - s_first); }
  }
  __syncthreads();
  if (s_e >= a.E) return;
  const int first = s_first, count = s_count, n0 = blockIdx.y * GS_T;
  if (threadIdx.x < GS_T) {
    const int p = first + min((int)threadIdx.x, count - 1);
    src[threadIdx.x] = a.rows ? min(max(a.rows[p], 0), a.src_rows - 1) : p;
  }
  __syncthreads();
  const T* x = reinterpret_cast<const T*>(a.x);
  const T* w = reinterpret_cast<const T*>(a.w) + (int64_t)s_e * a.Nout * a.K;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += GS_K) {
    for (int i = threadIdx.x; i < GS_T * GS_K; i += 256) {
      const int r = i / GS_K, k = i % GS_K;
      const bool in = k0 + k < a.K;
      sx[k][r] = in ? Elem<T>::to_f32(x[(int64_t)src[r] * a.x_stride + k0 + k]) : 0.f;
      sw[k][r] = in && n0 + r < a.Nout ? Elem<T>::to_f32(w[(int64_t)(n0 + r) * a.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GS_K; ++k) {
      const float4 p = *reinterpret_cast<const float4*>(&sx[k][4 * ty]), q = *reinterpret_cast<const float4*>(&sw[k][4 * tx]);
      const float pr[4] = {p.x, p.y, p.z, p.w}, qr[4] = {q.x, q.y, q.z, q.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(pr[i], qr[j], acc[i][j]);
    }
    __syncthreads();
  }
  if (a.act == ZP_ACT_SILU_MUL) {      // threads 0-3 of eight hold gates, the other four the matching entries of `up`
    const int col = (n0 >> 1) + (tx >> 3) * 16 + (tx & 3) * 4;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float f = 4 * ty + i < count && a.row_scale ? a.row_scale[first + 4 * ty + i] : 1.f;
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float up = __shfl_down_sync(0xffffffffu, acc[i][j], 4) * f, g = acc[i][j] * f;
        if ((tx & 4) == 0 && 4 * ty + i < count && col + j < a.Nout / 2)
          reinterpret_cast<T*>(a.out)[(int64_t)(first + 4 * ty + i) * (a.Nout / 2) + col + j] = Elem<T>::from_f32(g / (1.f + expf(-g)) * up);
      }
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < 4; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (4 * ty + i < count && n0 + 4 * tx + j < a.Nout) {
        float v = acc[i][j];
        if (a.act == ZP_ACT_RELU_SQUARED) { v = fmaxf(v, 0.f); v *= v; }
        reinterpret_cast<T*>(a.out)[(int64_t)(first + 4 * ty + i) * a.Nout + n0 + 4 * tx + j] = Elem<T>::from_f32(v);
      }
}

}  // namespace zp

extern "C" int zp_moe_route(const float* logits, int64_t row_stride, const float* bias, int n_tokens, int n_experts, int top, float* weights,
                            int32_t* experts, int32_t* places, int32_t* rows, int32_t* offsets, int32_t* counts, float* place_weights,
                            int score, void* stream) {
  if (n_tokens == 0) return ZP_OK;
  ZP_REQUIRE(logits && weights && experts && places && rows && offsets && counts, "zp_moe_route: null pointer");
  ZP_REQUIRE(n_experts > 0 && n_experts <= zp::RT_MAXE && top > 0 && top <= n_experts && row_stride >= n_experts,
             "zp_moe_route: %d of %d experts (at most %d)", top, n_experts, zp::RT_MAXE);
  ZP_REQUIRE(score == ZP_SCORE_SOFTMAX || score == ZP_SCORE_SIGMOID || score == ZP_SCORE_SOFTMAX_TOP, "zp_moe_route: unknown score %d", score);
  zp::RouteArgs a{logits, row_stride, n_tokens, n_experts, top, weights, experts, places, rows, offsets, counts, place_weights,
                  score, bias};
  cudaStream_t st = (cudaStream_t)stream;
  if (n_experts <= 32) return zp::launch_route<1>(a, st);
  if (n_experts <= 64) return zp::launch_route<2>(a, st);
  if (n_experts <= 128) return zp::launch_route<4>(a, st);
  if (n_experts <= 256) return zp::launch_route<8>(a, st);
  return zp::launch_route<32>(a, st);
}

extern "C" int zp_grouped_gemm(const void* x, int64_t x_stride, const int32_t* rows, int src_rows, const void* weight,
                               const int32_t* offsets, const float* row_scale, void* out, int n_places, int n_experts, int n_out, int k,
                               int act, int impl, int dtype, void* stream) {
  if (n_places == 0) return ZP_OK;
  ZP_REQUIRE(x && weight && offsets && out, "zp_grouped_gemm: null pointer");
  ZP_REQUIRE(n_experts > 0 && n_out > 0 && k > 0 && src_rows > 0 && x_stride >= k, "zp_grouped_gemm: bad sizes");
  ZP_REQUIRE(act == ZP_ACT_NONE || act == ZP_ACT_RELU_SQUARED || act == ZP_ACT_SILU_MUL, "zp_grouped_gemm: unknown activation %d", act);
  ZP_REQUIRE(act == ZP_ACT_SILU_MUL ? n_out % 32 == 0 : !row_scale,
             "zp_grouped_gemm: gated products take blocks of 16 + 16 rows, and only they take row factors");
  ZP_REQUIRE((n_out + zp::GS_T - 1) / zp::GS_T <= 65535, "zp_grouped_gemm: %d outputs", n_out);
  zp::GroupedArgs a{x, rows, weight, offsets, row_scale, out, x_stride, src_rows, n_places, n_experts, n_out, k, act};
  cudaStream_t st = (cudaStream_t)stream;
  const bool tc = zp::grouped_tc_supports(a, dtype);
  if (impl == ZP_IMPL_TCGEN05 && !tc) {
    zp::set_error("zp_grouped_gemm: the tcgen05 kernel needs bf16, rows of whole 16-byte pieces and 16-byte aligned tensors");
    return ZP_ERR_UNSUPPORTED;
  }
  if (tc && impl != ZP_IMPL_SIMT) return zp::grouped_gemm_tc(a, st);
  const dim3 grid((n_places + zp::GS_T - 1) / zp::GS_T + n_experts, (n_out + zp::GS_T - 1) / zp::GS_T);
  ZP_DISPATCH_DTYPE(dtype, T, { zp::grouped_gemm_simt_kernel<T><<<grid, 256, 0, st>>>(a); });
  return zp::check_launch("zp_grouped_gemm");
}
