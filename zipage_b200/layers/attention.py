"""Attention over the paged (compressed) KV cache.

`Attention` keeps the reference layer's contract (zipage/layers/attention.py:53-104): store this
step's K/V, store the window queries, then varlen causal attention (prefill; paged when a prefix
was cached) or paged decode attention — with the two flash-attn calls and both Triton store
kernels replaced by libzipage_b200 kernels.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _lib as L
from ..kernel import _count, store_kvcache, store_query_cache
from ..utils.context import get_context
from .rotary import rotate_store

_ws_cache: dict = {}
_ws_kept: list = []   # outgrown buffers stay: a captured graph may still name them


def _workspace(device, nbytes):
    key = (device.index, torch.cuda.current_stream().cuda_stream)
    buf = _ws_cache.get(key)
    if buf is None or buf.numel() < nbytes:
        if buf is not None:
            _ws_kept.append(buf)
        buf = torch.empty(max(nbytes, 1 << 20), dtype=torch.uint8, device=device)
        _ws_cache[key] = buf
    return buf


def paged_decode_attention(q, k_cache, v_cache, cache_seqlens, block_table, softmax_scale=None):
    """Replaces flash_attn_with_kvcache(q[B,1,Hq,D], k_cache, v_cache, cache_seqlens=...,
    block_table=..., causal=True) as called at zipage/layers/attention.py:95-103."""
    L.require_cuda(q, k_cache, v_cache, cache_seqlens, block_table)
    B, one, Hq, D = q.shape
    assert one == 1 and q.is_contiguous()
    _, BS, Hkv, _ = k_cache.shape
    assert k_cache.stride(2) == D and k_cache.stride(1) == Hkv * D and v_cache.stride() == k_cache.stride()
    if softmax_scale is None:
        softmax_scale = D ** (-0.5)
    out = torch.empty_like(q)
    lib = L.load()
    ws = _workspace(q.device, lib.zp_paged_decode_workspace_bytes(B, Hq, D, 32))
    L.check(lib.zp_paged_decode(L.ptr(q), L.ptr(k_cache), L.ptr(v_cache), L.ptr(cache_seqlens),
                                L.ptr(block_table), L.ptr(out), B, block_table.shape[1], Hq, Hkv, D,
                                BS, k_cache.stride(0), float(softmax_scale), L.dtype_code(q),
                                L.ptr(ws), ws.numel(), L.stream_ptr()), "paged_decode_attention")
    _count(1)
    return out


def varlen_prefill_attention(q, k, v, max_seqlen_q, cu_seqlens_q, max_seqlen_k, cu_seqlens_k,
                             softmax_scale=None, block_table=None, impl="auto"):
    """Replaces flash_attn_varlen_func(..., causal=True, block_table=...) as called at
    zipage/layers/attention.py:82-93.  q [sum_q,Hq,D]; k,v dense [sum_k,Hkv,D] or, with
    block_table, the paged caches [P,BS,Hkv,D]."""
    L.require_cuda(q, k, v, cu_seqlens_q, cu_seqlens_k, block_table)
    _, Hq, D = q.shape
    Hkv = k.shape[-2]
    assert q.is_contiguous()
    if softmax_scale is None:
        softmax_scale = D ** (-0.5)
    if block_table is None:
        assert k.is_contiguous() and v.is_contiguous()
        BS, stride_page, nbmax = 0, 0, 0
    else:
        BS = k.shape[1]
        assert k.stride(2) == D and k.stride(1) == Hkv * D and v.stride() == k.stride()
        stride_page, nbmax = k.stride(0), block_table.shape[1]
    out = torch.empty_like(q)
    B = cu_seqlens_q.numel() - 1
    total_k = 0 if block_table is not None else k.shape[0]
    L.check(L.load().zp_varlen_prefill_ex(L.ptr(q), L.ptr(k), L.ptr(v), L.ptr(cu_seqlens_q),
                                          L.ptr(cu_seqlens_k), L.ptr(block_table), L.ptr(out), B,
                                          int(max_seqlen_q), nbmax, Hq, Hkv, D, BS, stride_page,
                                          float(softmax_scale), q.shape[0], total_k, L.IMPL[impl],
                                          L.dtype_code(q), L.stream_ptr()),
            "varlen_prefill_attention")
    _count(1)
    return out


class Attention(nn.Module):
    """Drop-in for zipage.layers.attention.Attention (same constructor, same cache attributes)."""

    def __init__(self, num_heads, head_dim, scale, num_kv_heads):
        super().__init__()
        self.num_heads = num_heads
        self.head_dim = head_dim
        self.scale = scale
        self.num_kv_heads = num_kv_heads
        self.k_cache = self.v_cache = torch.tensor([])
        self.q_cache = torch.tensor([])

    def forward(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor):
        context = get_context()
        k_cache, v_cache = self.k_cache, self.v_cache
        if k_cache.numel() and v_cache.numel():
            store_kvcache(k, v, k_cache, v_cache, context.slot_mapping)
        if context.query_slot_mapping is not None:
            # a device-built triple list has fixed capacity; only its first query_slot_count rows count
            store_query_cache(q, self.q_cache, context.query_slot_mapping,
                              getattr(context, "query_slot_count", None))
        return self.attend(q, k, v)

    def attend(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor):
        """The attention call alone, for callers that wrote the caches already (the fused
        q/k normalisation + rotation + store launch)."""
        context = get_context()
        k_cache, v_cache = self.k_cache, self.v_cache
        if context.is_prefill:
            if context.block_tables is not None:  # prefix cache: keys come from the pages
                k, v = k_cache, v_cache
            return varlen_prefill_attention(
                q.contiguous(), k if context.block_tables is not None else k.contiguous(),
                v if context.block_tables is not None else v.contiguous(),
                context.max_seqlen_q, context.cu_seqlens_q, context.max_seqlen_k,
                context.cu_seqlens_k, self.scale, context.block_tables)
        return paged_decode_attention(q.contiguous().unsqueeze(1), k_cache, v_cache,
                                      context.context_lens, context.block_tables, self.scale)


def window_attention(q, k_cache, v_cache, context_lens, block_table, num_heads, head_dim, v_dim, scale,
                     window=0, softcap=0.0, cu_seqlens_q=None, max_seqlen_q=0, out=None, impl="auto", chunk=0, sink=None,
                     gate=None, gate_mode=None, out_scale=1.0, keep=0, slopes=None):
    """Attention with a sliding window or chunks, `keep` first tokens that are always seen, soft cap, distance biases
    (`slopes` [Hq] fp32 times the distance, off the scores), sink [Hq] (fp32) and output gate (`gate_mode` "head": one
    logit per head, "entry": one per entry of the result) over paged caches whose rows are padded to multiples of 16
    (k_cache [P, BS, Hkv, KP], v_cache [P, BS, Hkv, VP]).  q [rows, Hq * D] may be a column view of a
    projection.  One row per sequence without `cu_seqlens_q`."""
    L.require_cuda(q, k_cache, v_cache, context_lens, block_table, cu_seqlens_q, sink, gate, slopes)
    P, BS, Hkv, KP = k_cache.shape
    VP = v_cache.shape[3]
    assert all(t is None or t.dtype == torch.float32 and t.is_contiguous() and t.numel() == num_heads for t in (sink, slopes))
    assert gate is None or gate.dtype == q.dtype and gate.stride(1) == 1
    assert k_cache.is_contiguous() and v_cache.is_contiguous() and q.stride(1) == 1 and block_table.stride(1) == 1
    if out is None:
        out = torch.empty((q.shape[0], num_heads * v_dim), dtype=q.dtype, device=q.device)
    B, NB = block_table.shape
    assert block_table.stride(0) == NB or B == 1
    lib = L.load()
    ws = None
    if cu_seqlens_q is None:
        span = min([NB * BS] + [n + int(keep) for n in (window, chunk) if n])
        need = lib.zp_window_attention_workspace_bytes(B, num_heads, Hkv, VP, span)
        ws = _workspace(q.device, need) if need else None
    L.check(lib.zp_window_attention(
        L.ptr(q), L.ptr(k_cache), L.ptr(v_cache), L.ptr(cu_seqlens_q), L.ptr(context_lens), L.ptr(block_table),
        L.ptr(out), B, int(max_seqlen_q), NB, num_heads, Hkv, head_dim, v_dim, KP, VP, BS, P, q.stride(0),
        out.stride(0), float(scale), float(softcap or 0.0), int(window or 0), int(chunk or 0),
        int(keep), L.ptr(slopes), L.ptr(sink), L.ptr(gate), 0 if gate is None else gate.stride(0), L.GATE[gate_mode], float(out_scale), q.shape[0],
        L.IMPL[impl], L.dtype_code(q),
        L.ptr(ws), 0 if ws is None else ws.numel(), L.stream_ptr()), "window_attention")
    _count(1)
    return out


def store_kv_padded(k, v, k_cache, v_cache, slot_mapping, head_dim, v_dim):
    """k [N, Hkv * D], v [N, Hkv * DV] (column views of one projection) into padded paged caches."""
    L.require_cuda(k, v, k_cache, v_cache, slot_mapping)
    assert k.stride(0) == v.stride(0) and k.stride(1) == v.stride(1) == 1
    P, BS, Hkv, KP = k_cache.shape
    L.check(L.load().zp_store_kv_padded(
        L.ptr(k), L.ptr(v), L.ptr(k_cache), L.ptr(v_cache), L.ptr(slot_mapping), k.shape[0], Hkv, head_dim, v_dim,
        KP, v_cache.shape[3], k.stride(0), P * BS, L.dtype_code(k), L.stream_ptr()), "store_kv_padded")
    _count(1)


def distance_slopes(heads):
    """Slopes of linear distance biases, a geometric sequence that ends at 2^-8."""
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


class WindowAttentionMixer(nn.Module):
    """Grouped-query attention without rotation, with a sliding window and a soft cap on the scores;
    h -> head outputs [rows, heads * vdim] before the output projection.  `run` selects the cache of
    this pass when the layer runs several times.  Optional: `keep` first tokens that stay visible behind the window, distance
    biases (`slopes`, one per head), biases of the projections (named as their weights with '.b' added)."""

    def __init__(self, width, heads, kv_heads, dim, vdim, scale, softcap, window, dtype, device, keep=0, slopes=None, bias=False):
        super().__init__()
        self.keep = keep
        self.slopes = None if slopes is None else nn.Parameter(torch.tensor(slopes, dtype=torch.float32, device=device), requires_grad=False)
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.softcap, self.window = scale, softcap, window
        e = lambda *s: nn.Parameter(torch.empty(*s, dtype=dtype, device=device), requires_grad=False)
        self.qkv = e(heads * dim + kv_heads * (dim + vdim), width)
        self.qkv_bias = e(heads * dim + kv_heads * (dim + vdim)) if bias else None
        self.out_proj = e(width, heads * vdim)
        self.caches = []                                       # one (k_cache, v_cache) per pass

    def load(self, get):
        self.qkv.copy_(torch.cat([get(n) for n in "qkv"], 0))
        if self.qkv_bias is not None:
            self.qkv_bias.copy_(torch.cat([get(n + ".b") for n in "qkv"], 0))
        self.out_proj.copy_(get("o"))

    def forward(self, h, run):
        ctx = get_context()
        x = torch.mm(h, self.qkv.t()) if self.qkv_bias is None else torch.addmm(self.qkv_bias, h, self.qkv.t())
        nq, nk = self.heads * self.dim, self.kv_heads * self.dim
        q, k, v = x[:, :nq], x[:, nq:nq + nk], x[:, nq + nk:]
        kc, vc = self.caches[run]
        store_kv_padded(k, v, kc, vc, ctx.slot_mapping, self.dim, self.vdim)
        out = torch.empty((h.shape[0], self.heads * self.vdim), dtype=h.dtype, device=h.device)
        nd = ctx.decode_rows()
        shape = (self.heads, self.dim, self.vdim, self.scale, self.window, self.softcap)
        kw = dict(out=out, keep=self.keep, slopes=self.slopes)
        if nd:
            window_attention(q, kc, vc, ctx.context_lens[:nd], ctx.block_tables[:nd], *shape, **kw)
        if ctx.is_prefill and nd < ctx.context_lens.shape[0]:
            window_attention(q, kc, vc, ctx.context_lens[nd:], ctx.block_tables[nd:], *shape,
                             cu_seqlens_q=ctx.cu_seqlens_q[nd:], max_seqlen_q=ctx.max_seqlen_q, **kw)
        return out


class RotaryHeads(nn.Module):
    """The heads of grouped-query attention with rotary positions, from a projection's columns [q | k | v | gate] to
    outputs; see `HeadsMixer`.  Optional: an RMS norm per head of queries and keys (`qk_norm`), values that are the keys as
    projected (`shared_kv`: no columns of their own), a soft cap, chunks, a sink per head, an output gate per head or entry."""

    def __init__(self, heads, kv_heads, dim, vdim, scale, rotary, eps, dtype, device, qk_norm=False, shared_kv=False, softcap=0.0,
                 chunk=0, sink=False, gate=None, out_scale=1.0):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.rotary, self.eps, self.shared_kv, self.softcap, self.chunk = scale, rotary, eps, shared_kv, softcap, chunk
        self.gate, self.out_scale = gate, out_scale
        if shared_kv and dim != vdim:
            raise ValueError(f"keys of {dim} entries as values of {vdim}")
        self.nk, self.nv = kv_heads * dim, 0 if shared_kv else kv_heads * vdim
        self.columns = heads * dim + self.nk + self.nv + {None: 0, "head": heads, "entry": heads * vdim}[gate]
        self.out_columns = heads * vdim
        e = lambda n: nn.Parameter(torch.empty(n, dtype=torch.float32, device=device), requires_grad=False)
        self.q_norm, self.k_norm = (e(dim), e(dim)) if qk_norm else (None, None)
        self.sink = e(heads) if sink else None
        self.k_cache = self.v_cache = None                # bound by the cache

    def load(self, get):
        """-> rows of the projection."""
        if self.q_norm is not None:
            self.q_norm.copy_(get("q.norm"))
            self.k_norm.copy_(get("k.norm"))
        if self.sink is not None:
            self.sink.copy_(get("sink"))
        return torch.cat([get(n) for n in ("q", "k") + (() if self.shared_kv else ("v",)) + (("g",) if self.gate else ())], 0)

    def forward(self, y, positions, out):
        ctx = get_context()
        nq = self.heads * self.dim
        q, k = y[:, :nq], y[:, nq:nq + self.nk]
        v = k if self.shared_kv else y[:, nq + self.nk:nq + self.nk + self.nv]
        gate = y[:, nq + self.nk + self.nv:self.columns] if self.gate else None
        rotate_store(q, k, v, positions, self.rotary, self.k_cache, self.v_cache, ctx.slot_mapping, self.dim, self.vdim,
                     self.q_norm, self.k_norm, self.eps)
        nd = ctx.decode_rows()
        shape = (self.heads, self.dim, self.vdim, self.scale, 0, self.softcap)
        kw = dict(out=out, chunk=self.chunk, sink=self.sink, gate=gate, gate_mode=self.gate, out_scale=self.out_scale)
        if nd:
            window_attention(q, self.k_cache, self.v_cache, ctx.context_lens[:nd], ctx.block_tables[:nd], *shape, **kw)
        if ctx.is_prefill and nd < ctx.context_lens.shape[0]:
            window_attention(q, self.k_cache, self.v_cache, ctx.context_lens[nd:], ctx.block_tables[nd:], *shape,
                             cu_seqlens_q=ctx.cu_seqlens_q[nd:], max_seqlen_q=ctx.max_seqlen_q, **kw)
