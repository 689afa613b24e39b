"""The matrix-memory (mLSTM) mixer on libzipage_b200: one launch from projections and state to the
normalised, gated head outputs.

Decoded tokens take the recurrent kernel, prompt portions the chunked tensor-core kernel (fp32: the
recurrent one).  Recurrent state is fp32, one slot per running sequence, named by the context's
`state_slots`.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _lib as L
from ..kernel import _count
from ..utils.context import get_context
from .row_ops import project


def mlstm_step(q, k, v, g, gates, gate_bias, norm_weight, state, out, context_lens, slots, heads, dim, vdim,
               gate_cap, eps, cu_seqlens_q=None, qscale=None, impl="auto"):
    """q, k, v, g: column views of one [rows, ...] projection; state = (S [slots, H, dim, VP], n [slots, H,
    dim], m [slots, H]) fp32, updated in place; out [rows, H * vdim]."""
    S, n, m = state
    L.require_cuda(q, k, v, g, gates, S, n, m, out, context_lens, slots, cu_seqlens_q)
    assert q.stride(0) == k.stride(0) == v.stride(0) == g.stride(0) and gates.dtype == torch.float32
    assert S.is_contiguous() and n.is_contiguous() and m.is_contiguous() and S.shape[1:3] == (heads, dim)
    B = context_lens.shape[0]
    L.check(L.load().zp_mlstm(
        L.ptr(q), L.ptr(k), L.ptr(v), L.ptr(g), L.ptr(gates), L.ptr(gate_bias), L.ptr(norm_weight),
        L.ptr(cu_seqlens_q), L.ptr(context_lens), L.ptr(slots), L.ptr(S), L.ptr(n), L.ptr(m), L.ptr(out),
        B, heads, dim, vdim, S.shape[3], S.shape[0], q.stride(0), gates.stride(0), out.stride(0),
        float(dim ** -0.5 if qscale is None else qscale), float(gate_cap), float(eps), q.shape[0], L.IMPL[impl],
        L.dtype_code(out), L.stream_ptr()), "mlstm")
    _count(1)
    return out


class MLSTMMixer(nn.Module):
    """h -> head outputs [rows, heads * vdim] before the output projection (whose product adds to the
    residual stream).  `run` selects the state of this pass when the layer runs several times."""

    def __init__(self, width, heads, dim, vdim, gate_cap, eps, dtype, device):
        super().__init__()
        self.heads, self.dim, self.vdim, self.gate_cap, self.eps = heads, dim, vdim, gate_cap, eps
        e = lambda *s, dt=dtype: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.qkvg = e(2 * heads * (dim + vdim), width)
        self.gates = e(2 * heads, width)                       # input gates, then forget gates
        self.gate_bias = e(2 * heads, dt=torch.float32)
        self.norm = e(heads * vdim, dt=torch.float32)
        self.out_proj = e(width, heads * vdim)
        self.states = []                                       # one (S, n, m) per pass, bound by the cache

    def load(self, get):
        """`get(name)` -> tensor of this mixer."""
        self.qkvg.copy_(torch.cat([get(n) for n in "qkvg"], 0))
        self.gates.copy_(torch.cat([get("i"), get("f")], 0))
        self.gate_bias.copy_(torch.cat([get("i.b"), get("f.b")], 0))
        self.norm.copy_(get("norm"))
        self.out_proj.copy_(get("o"))

    def forward(self, h, run):
        ctx = get_context()
        H, dk, dv = self.heads, self.dim, self.vdim
        x = project(h, self.qkvg)
        gates = project(h, self.gates, fp32=True)
        q, k, v, g = x[:, :H * dk], x[:, H * dk:2 * H * dk], x[:, 2 * H * dk:2 * H * dk + H * dv], x[:, 2 * H * dk + H * dv:]
        out = torch.empty((h.shape[0], H * dv), dtype=h.dtype, device=h.device)
        args = (q, k, v, g, gates, self.gate_bias, self.norm, self.states[run], out)
        nd = ctx.decode_rows()
        if nd:
            mlstm_step(*args, ctx.context_lens[:nd], ctx.state_slots[:nd], H, dk, dv, self.gate_cap, self.eps)
        if ctx.is_prefill and nd < ctx.context_lens.shape[0]:
            mlstm_step(*args, ctx.context_lens[nd:], ctx.state_slots[nd:], H, dk, dv, self.gate_cap, self.eps,
                       cu_seqlens_q=ctx.cu_seqlens_q[nd:])
        return out
