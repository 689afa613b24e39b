"""The gated delta rule on libzipage_b200: decoded tokens take one launch from projections and state to gated outputs, prompt
portions a short convolution and the chunked tensor-core kernels (fp32 and other sizes: the recurrent one).

State per sequence, in the slot that the context's `state_slots` names: the fp32 matrix S of every head and a
ring of the convolution's last inputs.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _lib as L
from ..kernel import _count
from ..utils.context import get_context
from .short_conv import short_conv


def gated_delta(x, gate, ab, A_log, dt_bias, norm_weight, state, out, context_lens, slots, heads, kv_heads, dim, vdim, eps,
                out_scale=1.0, conv_weight=None, ring=None, cu_seqlens_q=None, impl="auto"):
    """x [rows, q | k | v]: the projection itself with `conv_weight` and `ring` (single rows), or its convolution; gate [rows,
    H * vdim]; ab [rows, 2 H] fp32; state [slots, H, dim, VP] fp32, in place; out [rows, H * vdim] (column view)."""
    L.require_cuda(x, gate, ab, A_log, dt_bias, norm_weight, state, out, context_lens, slots, conv_weight, ring, cu_seqlens_q)
    assert x.stride(1) == gate.stride(1) == ab.stride(1) == out.stride(1) == 1 and ab.dtype == state.dtype == torch.float32
    assert state.is_contiguous() and state.shape[1:3] == (heads, dim) and x.dtype == gate.dtype == out.dtype
    lib, B = L.load(), context_lens.shape[0]
    ws = None                # (portions never run inside a graph: an allocation of this call's size)
    if cu_seqlens_q is not None and x.dtype == torch.bfloat16 and impl != "simt":
        ws = torch.empty(lib.zp_gated_delta_workspace_bytes(x.shape[0], B, heads), dtype=torch.uint8, device=x.device)
    L.check(lib.zp_gated_delta(
        L.ptr(x), x.stride(0), L.ptr(gate), gate.stride(0), L.ptr(ab), ab.stride(0), L.ptr(A_log), L.ptr(dt_bias), L.ptr(norm_weight),
        L.ptr(conv_weight), L.ptr(ring), 0 if conv_weight is None else conv_weight.shape[0], L.ptr(cu_seqlens_q), L.ptr(context_lens),
        L.ptr(slots), L.ptr(state), L.ptr(out), out.stride(0), B, heads, kv_heads, dim, vdim, state.shape[3], state.shape[0],
        float(eps), float(out_scale), x.shape[0], L.IMPL[impl], L.dtype_code(x), L.ptr(ws), 0 if ws is None else ws.numel(),
        L.stream_ptr()), "gated_delta")
    _count(1)
    return out


class DeltaHeads(nn.Module):
    """The heads of a gated delta rule, from a projection's columns [q | k | v | gate] to outputs; see `HeadsMixer`."""

    def __init__(self, width, heads, kv_heads, dim, vdim, taps, eps, dtype, device, out_scale=1.0):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps, self.out_scale = heads, kv_heads, dim, vdim, eps, out_scale
        self.channels = 2 * kv_heads * dim + heads * vdim
        self.columns, self.out_columns = self.channels + heads * vdim, heads * vdim
        e = lambda *s, dt=torch.float32: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.ab = e(2 * heads, width, dt=dtype)           # decays' rows, then steps': the product's results stay fp32
        self.A_log, self.dt_bias, self.norm = e(heads), e(heads), e(vdim)
        self.conv = e(taps, self.channels)
        self.state = self.ring = None                     # bound by the cache

    def load(self, get):
        """-> rows of the projection."""
        self.ab.copy_(torch.cat([get("a"), get("b")], 0))
        self.A_log.copy_(get("A_log"))
        self.dt_bias.copy_(get("dt_bias"))
        self.norm.copy_(get("norm"))
        self.conv.copy_(torch.cat([get(n + ".conv") for n in "qkv"], 0).t())
        return torch.cat([get(n) for n in "qkvg"], 0)

    def forward(self, y, ab, positions, out):
        ctx = get_context()
        x, gate = y[:, :self.channels], y[:, self.channels:self.columns]
        nd = ctx.decode_rows()
        common = (ab, self.A_log, self.dt_bias, self.norm, self.state, out)
        sizes = (self.heads, self.kv_heads, self.dim, self.vdim, self.eps, self.out_scale)
        if nd:
            gated_delta(x, gate, *common, ctx.context_lens[:nd], ctx.state_slots[:nd], *sizes, conv_weight=self.conv, ring=self.ring)
        if ctx.is_prefill and nd < ctx.context_lens.shape[0]:
            seqs = (ctx.context_lens[nd:], ctx.state_slots[nd:])
            z = torch.empty((x.shape[0], self.channels), dtype=x.dtype, device=x.device)
            short_conv(x, self.conv, self.ring, *seqs, ctx.cu_seqlens_q[nd:], ctx.max_seqlen_q, z)
            gated_delta(z, gate, *common, *seqs, *sizes, cu_seqlens_q=ctx.cu_seqlens_q[nd:])
