// Sliding-window attention with soft-capped scores over paged K/V whose key and value sizes differ:
// the cache write, the fp32 / any-size SIMT kernel, and the entry points (zp_window_attn_mma.cu holds
// the tensor-core kernels for 16-bit caches).
//
// Cache rows are padded to KP / VP elements (multiples of 16; the padding stays zero), so that every
// row starts on a 16-byte boundary whatever the head sizes.
#include "zp_window_attn.cuh"

namespace zp {

// One block per token: k [Hkv, D] -> slot of [P*BS, Hkv, KP], v [Hkv, DV] -> slot of [P*BS, Hkv, VP].
template <typename T>
__global__ void __launch_bounds__(128)
store_kv_padded_kernel(const T* __restrict__ k, const T* __restrict__ v, T* __restrict__ k_cache,
                       T* __restrict__ v_cache, const int32_t* __restrict__ slot_mapping, int64_t stride,
                       int Hkv, int D, int DV, int KP, int VP, int64_t n_slots, int vec_ok) {
  const int64_t i = blockIdx.x;
  const int64_t slot = slot_mapping[i];
  if (slot < 0 || slot >= n_slots) return;
  constexpr int EPV = 16 / sizeof(T);
  const T* src[2] = {k + i * stride, v + i * stride};
  T* dst[2] = {k_cache + slot * Hkv * KP, v_cache + slot * Hkv * VP};
  const int dim[2] = {D, DV}, pad[2] = {KP, VP};
#pragma unroll
  for (int t = 0; t < 2; ++t) {
    if (vec_ok) {
      const int per = dim[t] / EPV, n = Hkv * per;
      for (int c = threadIdx.x; c < n; c += blockDim.x) {
        const int h = c / per, o = (c - h * per) * EPV;
        st16(dst[t] + h * pad[t] + o, ld16(src[t] + h * dim[t] + o));
      }
    } else {
      const int n = Hkv * dim[t];
      for (int c = threadIdx.x; c < n; c += blockDim.x) {
        const int h = c / dim[t];
        dst[t][h * pad[t] + c - h * dim[t]] = src[t][c];
      }
    }
  }
}

// ---------------------------------------------------------------------------------------------
// SIMT kernel: one warp per (query row, query head).  32 keys at a time: lane = key for the scores
// (fp32 dot products over the padded row), lane = value dim for the weighted sum.
// ---------------------------------------------------------------------------------------------
constexpr int WS_WARPS = 4;

template <typename T, int VPL>   // VPL: value dims per lane
__global__ void __launch_bounds__(WS_WARPS * 32) window_attn_simt_kernel(const WinArgs a) {
  extern __shared__ float sq[];   // [WS_WARPS][KP]
  const int b = blockIdx.z, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const WinSeq sq_ = win_seq(a, b);
  const int r = blockIdx.x * WS_WARPS + warp;
  if (r >= sq_.count) return;
  const int hk = h / (a.Hq / a.Hkv), pos = sq_.pos0 + r;
  float* q = sq + warp * a.KP;
  const T* qp = reinterpret_cast<const T*>(a.q) + (int64_t)(sq_.row0 + r) * a.q_stride + (int64_t)h * a.D;
  for (int d = lane; d < a.KP; d += 32) q[d] = d < a.D ? Elem<T>::to_f32(qp[d]) : 0.f;
  __syncwarp();
  const T* kc = reinterpret_cast<const T*>(a.k);
  const T* vc = reinterpret_cast<const T*>(a.v);
  float o[VPL], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int j = 0; j < VPL; ++j) o[j] = 0.f;
  constexpr int EPV = 16 / sizeof(T);
  const int lo = win_first(a, pos), near = lo & ~31;
  const float slope = a.slopes ? a.slopes[h] : 0.f;
  for (int k0 = min(near, a.keep > 0 ? 0 : near); k0 <= pos; k0 += 32) {
    if (k0 >= a.keep && k0 < near) k0 = near;      // between the kept keys and the window
    const int key = k0 + lane;
    const bool seen = (key >= lo || key < a.keep) && key <= pos;
    // the page size is a multiple of 32: the 32 keys share a page
    const int64_t slot0 = (int64_t)win_page(a, b, k0) * a.BS + k0 % a.BS;
    float s = -INFINITY;
    if (seen) {
      const T* kr = kc + ((slot0 + lane) * a.Hkv + hk) * a.KP;
      float acc = 0.f;
      for (int d = 0; d < a.KP; d += EPV) {
        const int4 raw = ld16(kr + d);
        const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
        for (int j = 0; j < EPV; ++j) acc = fmaf(q[d + j], Elem<T>::to_f32(e[j]), acc);
      }
      s = acc * a.scale;
      if (a.softcap > 0.f) s = a.softcap * tanhf(s / a.softcap);
      s = fmaf(-slope, (float)(pos - key), s);
    }
    const float mx = fmaxf(m, warp_max(s));
    const float corr = m == -INFINITY ? 0.f : expf(m - mx);
    const float p = (seen && mx != -INFINITY) ? expf(s - mx) : 0.f;
    l = l * corr + warp_sum(p);
    m = mx;
#pragma unroll
    for (int j = 0; j < VPL; ++j) o[j] *= corr;
    const int first = k0 < a.keep ? 0 : max(lo - k0, 0), last = min(pos - k0, 31);
    for (int t = first; t <= last; ++t) {
      const float pt = __shfl_sync(0xffffffffu, p, t);
      if (pt == 0.f) continue;
      const T* vr = vc + ((slot0 + t) * a.Hkv + hk) * a.VP;
#pragma unroll
      for (int j = 0; j < VPL; ++j) {
        const int d = lane + 32 * j;
        if (d < a.DV) o[j] = fmaf(pt, Elem<T>::to_f32(vr[d]), o[j]);
      }
    }
  }
  if (a.sink) l += expf(a.sink[h] - m);
  const float f = l > 0.f ? win_head_factor<T>(a, sq_.row0 + r, h) / l : 0.f;
  T* op = reinterpret_cast<T*>(a.out) + (int64_t)(sq_.row0 + r) * a.out_stride + (int64_t)h * a.DV;
#pragma unroll
  for (int j = 0; j < VPL; ++j) {
    const int d = lane + 32 * j;
    if (d < a.DV) op[d] = Elem<T>::from_f32(o[j] * f * win_entry_factor<T>(a, sq_.row0 + r, h, d));
  }
}

template <typename T>
static int launch_simt(const WinArgs& a, int max_q, cudaStream_t st) {
  const dim3 grid((max_q + WS_WARPS - 1) / WS_WARPS, a.Hq, a.B);
  const size_t smem = sizeof(float) * WS_WARPS * a.KP;
  if (a.DV <= 64) window_attn_simt_kernel<T, 2><<<grid, WS_WARPS * 32, smem, st>>>(a);
  else if (a.DV <= 128) window_attn_simt_kernel<T, 4><<<grid, WS_WARPS * 32, smem, st>>>(a);
  else if (a.DV <= 256) window_attn_simt_kernel<T, 8><<<grid, WS_WARPS * 32, smem, st>>>(a);
  else if (a.DV <= 512) window_attn_simt_kernel<T, 16><<<grid, WS_WARPS * 32, smem, st>>>(a);
  else window_attn_simt_kernel<T, 32><<<grid, WS_WARPS * 32, smem, st>>>(a);
  return check_launch("zp_window_attention");
}

// tensor-core kernels for 16-bit caches (zp_window_attn_mma.cu)
bool window_mma_supports(const WinArgs& a);
int window_prefill_mma(const WinArgs& a, int max_q, int dtype, cudaStream_t st);
int window_decode_mma(const WinArgs& a, int dtype, cudaStream_t st);
int window_decode_splits(int B, int Hkv, int span);
// tcgen05 prefill kernel (zp_window_attn_tc.cu)
bool window_tc_supports(const WinArgs& a, int total_q, int dtype);
int window_prefill_tc(const WinArgs& a, int max_q, int total_q, cudaStream_t st);

}  // namespace zp

extern "C" int zp_store_kv_padded(const void* k, const void* v, void* k_cache, void* v_cache,
                                  const int32_t* slot_mapping, int n_tokens, int Hkv, int D, int DV,
                                  int KP, int VP, int64_t row_stride, int64_t n_slots, int dtype, void* stream) {
  if (n_tokens == 0) return ZP_OK;
  ZP_REQUIRE(k && v && k_cache && v_cache && slot_mapping, "zp_store_kv_padded: null pointer");
  ZP_REQUIRE(Hkv > 0 && D > 0 && DV > 0 && KP >= D && VP >= DV, "zp_store_kv_padded: bad sizes");
  const int es = (int)zp::dtype_size(dtype), epv = 16 / es;
  const int vec = D % epv == 0 && DV % epv == 0 && KP % epv == 0 && VP % epv == 0 && row_stride % epv == 0 &&
                  ((uintptr_t)k | (uintptr_t)v | (uintptr_t)k_cache | (uintptr_t)v_cache) % 16 == 0;
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::store_kv_padded_kernel<T><<<n_tokens, 128, 0, (cudaStream_t)stream>>>(
        (const T*)k, (const T*)v, (T*)k_cache, (T*)v_cache, slot_mapping, row_stride, Hkv, D, DV, KP, VP, n_slots, vec);
  });
  return zp::check_launch("zp_store_kv_padded");
}

extern "C" size_t zp_window_attention_workspace_bytes(int B, int Hq, int Hkv, int VP, int span) {
  if (B < 1 || Hkv < 1 || Hq < Hkv) return 0;
  const int ns = zp::window_decode_splits(B, Hkv, span);
  return ns > 1 ? (size_t)B * Hq * ns * (VP + 2) * sizeof(float) : 0;
}

extern "C" int zp_window_attention(const void* q, const void* k_cache, const void* v_cache,
                                   const int32_t* cu_seqlens_q, const int32_t* context_lens,
                                   const int32_t* block_table, void* out, int B, int max_seqlen_q, int NBmax,
                                   int Hq, int Hkv, int D, int DV, int KP, int VP, int BS, int n_pages,
                                   int64_t q_stride, int64_t out_stride, float scale, float softcap, int window, int chunk, int keep,
                                   const float* slopes, const float* sink, const void* gate, int64_t gate_stride, int gate_mode, float out_scale,
                                   int total_q, int impl, int dtype, void* workspace, size_t workspace_bytes, void* stream) {
  if (B == 0 || (cu_seqlens_q && max_seqlen_q == 0)) return ZP_OK;
  ZP_REQUIRE(q && k_cache && v_cache && context_lens && block_table && out, "zp_window_attention: null pointer");
  ZP_REQUIRE(Hkv > 0 && Hq % Hkv == 0, "zp_window_attention: Hq must be a multiple of Hkv");
  ZP_REQUIRE(BS > 0 && BS % 64 == 0, "zp_window_attention: page size must be a multiple of 64");
  ZP_REQUIRE(D > 0 && D <= KP && DV > 0 && DV <= VP && KP % 16 == 0 && VP % 16 == 0 && DV <= 1024 && VP <= 2048 && KP <= 2048,
             "zp_window_attention: head sizes %d / %d (padded %d / %d) not supported", D, DV, KP, VP);
  ZP_REQUIRE(NBmax > 0 && n_pages > 0 && B <= 65535, "zp_window_attention: bad sizes");
  ZP_REQUIRE(((uintptr_t)k_cache | (uintptr_t)v_cache) % 16 == 0, "zp_window_attention: caches must be 16-byte aligned");
  ZP_REQUIRE(chunk >= 0 && window >= 0 && keep >= 0 && gate_mode >= 0 && gate_mode <= 2 && (gate_mode == 0 || gate),
             "zp_window_attention: bad mask or gate");
  zp::WinArgs a;
  a.q = q; a.k = k_cache; a.v = v_cache; a.cu_q = cu_seqlens_q; a.context_lens = context_lens; a.table = block_table;
  a.out = out; a.part = nullptr; a.B = B; a.NBmax = NBmax; a.Hq = Hq; a.Hkv = Hkv; a.D = D; a.DV = DV; a.KP = KP;
  a.VP = VP; a.BS = BS; a.window = window; a.n_pages = n_pages; a.nsplit = 1; a.q_stride = q_stride;
  a.out_stride = out_stride; a.scale = scale; a.softcap = softcap; a.chunk = chunk; a.keep = keep; a.slopes = slopes; a.sink = sink; a.gate = gate;
  a.gate_stride = gate_stride; a.gate_mode = gate_mode; a.out_scale = out_scale;
  cudaStream_t st = (cudaStream_t)stream;
  const bool half = dtype == ZP_DTYPE_BF16 || dtype == ZP_DTYPE_F16;
  // portions long enough to fill 128-row query tiles
  const bool tc = cu_seqlens_q && zp::window_tc_supports(a, total_q, dtype);
  if (impl == ZP_IMPL_TCGEN05 && !tc) {
    zp::set_error("zp_window_attention: the tcgen05 kernel needs bf16 portions, head sizes that are multiples of 8 up to 128, 16-byte "
                  "aligned rows and no soft cap or one of at most 69 without slopes");
    return ZP_ERR_UNSUPPORTED;
  }
  if (tc && (impl == ZP_IMPL_TCGEN05 || (impl == ZP_IMPL_AUTO && max_seqlen_q >= 96 && KP + VP > 128)))
    return zp::window_prefill_tc(a, max_seqlen_q, total_q, st);
  if (half && impl != ZP_IMPL_SIMT && zp::window_mma_supports(a)) {
    if (cu_seqlens_q) return zp::window_prefill_mma(a, max_seqlen_q, dtype, st);
    int span = NBmax * BS;
    if (window > 0 && window + keep < span) span = window + keep;
    if (chunk > 0 && chunk + keep < span) span = chunk + keep;
    a.nsplit = zp::window_decode_splits(B, Hkv, span);
    if (a.nsplit > 1) {
      const size_t need = (size_t)B * Hq * a.nsplit * (VP + 2) * sizeof(float);
      ZP_REQUIRE(workspace && workspace_bytes >= need, "zp_window_attention: workspace of %zu bytes, %zu needed",
                 workspace_bytes, need);
      a.part = reinterpret_cast<float*>(workspace);
    }
    return zp::window_decode_mma(a, dtype, st);
  }
  const int max_q = cu_seqlens_q ? max_seqlen_q : 1;
  ZP_DISPATCH_DTYPE(dtype, T, { return zp::launch_simt<T>(a, max_q, st); });
  return ZP_OK;
}
