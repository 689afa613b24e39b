"""Latent attention on libzipage_b200: keys and values of all heads are products of one latent per token,
and the cache holds only the latent and one rotated key part.

Two forms of the same attention:
  * direct: the per-head key product moves to the query side (q_lat = W_uk^T q), so every head meets the cached
    rows themselves: multi-query attention with keys [latent | rotated part] and the latent as value, then
    W_uv on the result.  Decoded tokens and short portions take it: it reads a cached row once for all heads.
  * expanded: keys and values of the step's sequences are computed from their latents by one product.  Longer
    portions take it: fewer operations per score.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _lib as L
from ..kernel import _count
from ..utils.context import get_context
from .attention import _workspace
from .rotary import rotary_turns
from .row_ops import project


def latent_prepare(y, positions, turns, q_weight, kv_weight, cache, slot_mapping, q_rank, kv_rank, rot, eps, dense=None):
    """y [N, q_rank (+ kv_rank + rot)] -> normed query latent [N, q_rank]; with kv_rank > 0 the token's cache row
    (cache [P, BS, 1, KP]) and its row of `dense` [N, KP]."""
    L.require_cuda(y, positions, turns, q_weight, kv_weight, cache, slot_mapping, dense)
    N = y.shape[0]
    cq = torch.empty((N, q_rank), dtype=y.dtype, device=y.device)
    KP, slots = (cache.shape[3], cache.shape[0] * cache.shape[1]) if kv_rank else (0, 0)
    L.check(L.load().zp_latent_prepare(
        L.ptr(y), y.stride(0), L.ptr(positions), L.ptr(turns), L.ptr(q_weight), L.ptr(kv_weight), L.ptr(cq), L.ptr(cache),
        L.ptr(dense), L.ptr(slot_mapping), N, q_rank, kv_rank, rot, KP, slots, float(eps), L.dtype_code(y), L.stream_ptr()),
        "latent_prepare")
    _count(1)
    return cq


def latent_rotate_q(q, positions, turns, heads, dim, rot, q_lat=None, kv_rank=0):
    """Rotates the last `rot` entries of every head of q [N, heads * (dim + rot)] in place, or into q_lat [N, heads, KP]."""
    L.require_cuda(q, positions, turns, q_lat)
    assert q.stride(1) == 1 and (q_lat is None or q_lat.is_contiguous())
    L.check(L.load().zp_latent_rotate_q(
        L.ptr(q), q.stride(0), L.ptr(positions), L.ptr(turns), L.ptr(q_lat), q.shape[0], heads, dim, rot, kv_rank,
        0 if q_lat is None else q_lat.shape[2], L.dtype_code(q), L.stream_ptr()), "latent_rotate_q")
    _count(1)


def gather_rows(cache, block_table, cu_seqlens_k, total):
    """The cached rows of every sequence one after the other, [total, KP]."""
    L.require_cuda(cache, block_table, cu_seqlens_k)
    P, BS, _, KP = cache.shape
    assert block_table.is_contiguous()
    out = torch.empty((total, KP), dtype=cache.dtype, device=cache.device)
    B, NB = block_table.shape
    L.check(L.load().zp_gather_rows(L.ptr(cache), L.ptr(block_table), L.ptr(cu_seqlens_k), L.ptr(out), B, NB, BS, P,
                                    KP * cache.element_size(), total, L.stream_ptr()), "gather_rows")
    _count(1)
    return out


def latent_attention(q_lat, cache, context_lens, block_table, rank, scale, cu_seqlens_q=None, max_seqlen_q=1, out=None, impl="auto"):
    """q_lat [rows, H, KP] over cached rows [P, BS, 1, KP] whose first `rank` entries are the values -> [rows, H, rank].
    One row per sequence without `cu_seqlens_q`."""
    L.require_cuda(q_lat, cache, context_lens, block_table, cu_seqlens_q)
    N, H, KP = q_lat.shape
    P, BS, _, row = cache.shape
    B, NB = block_table.shape
    assert q_lat.is_contiguous() and cache.is_contiguous() and row == KP and block_table.is_contiguous()
    if out is None:
        out = torch.empty((N, H, rank), dtype=q_lat.dtype, device=q_lat.device)
    assert out.is_contiguous()
    lib = L.load()
    need = lib.zp_latent_attention_workspace_bytes(N, B, max_seqlen_q, H, rank, NB * BS)
    ws = _workspace(q_lat.device, need) if need else None
    L.check(lib.zp_latent_attention(
        L.ptr(q_lat), L.ptr(cache), L.ptr(cu_seqlens_q), L.ptr(context_lens), L.ptr(block_table), L.ptr(out), B,
        int(max_seqlen_q), N, NB, H, rank, KP, BS, P, float(scale), L.IMPL[impl], L.dtype_code(q_lat), L.ptr(ws),
        0 if ws is None else ws.numel(), L.stream_ptr()), "latent_attention")
    _count(1)
    return out


def latent_prefill(q, kv, latent, cu_seqlens_q, cu_seqlens_k, max_seqlen_q, out, heads, dim, rot, vdim, rank, scale):
    """Causal attention of q [rows, heads * (dim + rot)] over kv [keys, heads * (dim + vdim)] (keys of all heads, then
    values) and the rotated parts in latent [keys, KP] at `rank`; writes out [rows, heads * vdim]."""
    L.require_cuda(q, kv, latent, cu_seqlens_q, cu_seqlens_k, out)
    assert q.stride(1) == out.stride(1) == 1 and kv.is_contiguous() and latent.is_contiguous()
    L.check(L.load().zp_latent_prefill(
        L.ptr(q), q.stride(0), L.ptr(kv), L.ptr(latent), L.ptr(cu_seqlens_q), L.ptr(cu_seqlens_k), L.ptr(out), out.stride(0),
        cu_seqlens_q.numel() - 1, int(max_seqlen_q), q.shape[0], kv.shape[0], heads, dim, rot, vdim, rank, latent.shape[1],
        float(scale), L.dtype_code(q), L.stream_ptr()), "latent_prefill")
    _count(1)
    return out


# portions whose longest has at least this many tokens take the expanded form
EXPAND_FROM = 64


class LatentAttentionMixer(nn.Module):
    """h -> W_o of the head outputs [rows, width].  `shares`: the layer keeps nothing of its own and reads another
    layer's cache (`cache` is bound to that one's)."""

    def __init__(self, width, heads, dim, rot, vdim, q_rank, kv_rank, base, scale, eps, shares, dtype, device):
        super().__init__()
        self.heads, self.dim, self.rot, self.vdim = heads, dim, rot, vdim
        self.q_rank, self.kv_rank, self.scale, self.eps, self.shares = q_rank, kv_rank, scale, eps, shares
        e = lambda *s, dt=dtype: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.down = e(q_rank + (0 if shares else kv_rank + rot), width)      # queries' rows, then keys' and values'
        self.q_norm = e(q_rank, dt=torch.float32)
        self.kv_norm = None if shares else e(kv_rank, dt=torch.float32)
        self.q_up = e(heads * (dim + rot), q_rank)
        self.kv_up = e(heads * (dim + vdim), kv_rank)                        # all keys' rows, then all values'
        self.out_proj = e(width, heads * vdim)
        self.turns = rotary_turns(rot, base, device)
        self.cache = None                                                    # [pages, page size, 1, KP]

    def load(self, get):
        self.down.copy_(get("dq") if self.shares else torch.cat([get("dq"), get("dkv")], 0))
        self.q_norm.copy_(get("dq.norm"))
        if not self.shares:
            self.kv_norm.copy_(get("dkv.norm"))
        self.q_up.copy_(get("uq"))
        self.kv_up.copy_(torch.cat([get("uk"), get("uv")], 0))
        self.out_proj.copy_(get("o"))

    def forward(self, h, positions):
        ctx = get_context()
        N, nd = h.shape[0], ctx.decode_rows()
        expand = ctx.is_prefill and nd < ctx.context_lens.shape[0] and self._expands(h, ctx)
        dense = None
        if expand and not self.shares and ctx.total_k == N - nd:      # no earlier context: the step's own rows are the keys
            dense = torch.empty((N, self.cache.shape[3]), dtype=h.dtype, device=h.device)
            ctx.scratch[id(self.cache)] = dense[nd:]
        cq = latent_prepare(project(h, self.down), positions, self.turns, self.q_norm, self.kv_norm, self.cache,
                            ctx.slot_mapping, self.q_rank, 0 if self.shares else self.kv_rank, self.rot, self.eps, dense)
        q = project(cq, self.q_up)
        out = torch.empty((N, self.heads * self.vdim), dtype=h.dtype, device=h.device)
        if expand:
            if nd:
                self._direct(q[:nd], positions[:nd], out[:nd], ctx, nd, False)
            self._expanded(q[nd:], positions[nd:], out[nd:], ctx, nd)
        else:
            self._direct(q, positions, out, ctx, nd, ctx.is_prefill and nd < ctx.context_lens.shape[0])
        return project(out, self.out_proj)

    def _expands(self, h, ctx):
        return ctx.max_seqlen_q >= EXPAND_FROM and ctx.cu_seqlens_k is not None and L.load().zp_latent_prefill_supported(
            self.dim, self.rot, self.vdim, self.kv_rank, self.cache.shape[3], L.dtype_code(h)) == 1

    def _expanded(self, q, positions, out, ctx, nd):
        latent = ctx.scratch.get(id(self.cache))        # (layers that share latents share their dense copy)
        if latent is None:
            latent = ctx.scratch[id(self.cache)] = gather_rows(self.cache, ctx.block_tables[nd:], ctx.cu_seqlens_k, ctx.total_k)
        kv = project(latent[:, :self.kv_rank], self.kv_up)
        latent_rotate_q(q, positions, self.turns, self.heads, self.dim, self.rot)
        if "cu_q" not in ctx.scratch:                   # rows counted from the first portion's
            ctx.scratch["cu_q"] = ctx.cu_seqlens_q[nd:] - nd if nd else ctx.cu_seqlens_q
        latent_prefill(q, kv, latent, ctx.scratch["cu_q"], ctx.cu_seqlens_k, ctx.max_seqlen_q, out,
                       self.heads, self.dim, self.rot, self.vdim, self.kv_rank, self.scale)

    def _direct(self, q, positions, out, ctx, nd, portions):
        """`nd` leading rows are sequences of one row each; with `portions`, the rest are portions."""
        H, R, N = self.heads, self.kv_rank, q.shape[0]
        q_lat = torch.empty((N, H, self.cache.shape[3]), dtype=q.dtype, device=q.device)
        latent_rotate_q(q, positions, self.turns, H, self.dim, self.rot, q_lat, R)
        nk = H * self.dim
        torch.bmm(q.view(N, H, -1)[:, :, :self.dim].transpose(0, 1), self.kv_up[:nk].view(H, self.dim, R),
                  out=q_lat.transpose(0, 1)[:, :, :R])
        o_lat = torch.empty((N, H, R), dtype=q.dtype, device=q.device)
        if nd:
            latent_attention(q_lat, self.cache, ctx.context_lens[:nd], ctx.block_tables[:nd], R, self.scale, out=o_lat)
        if portions:
            latent_attention(q_lat, self.cache, ctx.context_lens[nd:], ctx.block_tables[nd:], R, self.scale,
                             cu_seqlens_q=ctx.cu_seqlens_q[nd:], max_seqlen_q=ctx.max_seqlen_q, out=o_lat)
        torch.bmm(o_lat.transpose(0, 1), self.kv_up[nk:].view(H, self.vdim, R).transpose(1, 2),
                  out=out.view(N, H, self.vdim).transpose(0, 1))
