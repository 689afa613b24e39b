"""Linear attention with decaying matrix states on libzipage_b200: decoded tokens take one launch from projections and state to
outputs, prompt portions the chunked tensor-core kernels (fp32 and other sizes: the recurrent one); the norm with its gates
is the launch after it.

State per sequence, in the slot that the context's `state_slots` names: the fp32 matrix S of every head and, for mixers with a
convolution, a ring of its last inputs.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _lib as L
from ..kernel import _count
from ..utils.context import get_context
from .row_ops import project
from .short_conv import short_conv

KIND = {"forget": 0, "power": 1, "scalar": 2}


def linear_state(kind, q, k, v, gate, gate_bias, state, out, context_lens, slots, heads, kv_heads, dim, vdim, lower=None, rtau=1.0,
                 qscale=1.0, A_log=None, D=None, conv_weight=None, conv_bias=None, ring=None, cu_seqlens_q=None, impl="auto"):
    """S <- diag(a) S + key v^T, o = S^T query token after token; `kind`: "forget", "power" or "scalar" (where decays, keys and
    queries come from).  q, k, v: column views of one [rows, ...] projection (k None: "forget"); gate fp32 [rows, heads * dim]
    or [rows, heads]; state [slots, H, dim, VP] fp32, in place; out [rows, H * vdim] (column view).  With `conv_weight` and `ring`
    (single rows) the convolution is part of the launch."""
    params = (gate_bias, lower, A_log, D, conv_weight, conv_bias)
    L.require_cuda(q, k, v, gate, state, out, context_lens, slots, ring, cu_seqlens_q, *params)
    assert all(t is None or t.stride(1) == 1 and t.stride(0) == q.stride(0) and t.dtype == out.dtype for t in (q, k, v))
    assert gate.dtype == state.dtype == torch.float32 and gate.stride(1) == out.stride(1) == 1
    assert all(t is None or t.dtype == torch.float32 and t.is_contiguous() for t in params)
    assert state.is_contiguous() and state.shape[1:3] == (heads, dim)
    assert all(t is None or t.dtype == torch.int32 for t in (context_lens, slots, cu_seqlens_q))
    lib, B, rows = L.load(), context_lens.shape[0], q.shape[0]
    ws = None                # (portions never run inside a graph: an allocation of this call's size)
    if cu_seqlens_q is not None and q.dtype == torch.bfloat16 and impl != "simt":
        ws = torch.empty(lib.zp_linear_state_workspace_bytes(rows, B, heads, dim), dtype=torch.uint8, device=q.device)
    p = L.LinearStateParams(
        kind=KIND[kind], B=B, H=heads, G=kv_heads, dim=dim, vdim=vdim, VP=state.shape[3], n_slots=state.shape[0],
        taps=0 if conv_weight is None else conv_weight.shape[0], total_rows=rows, q=L.ptr(q), k=L.ptr(k), v=L.ptr(v), x_stride=q.stride(0),
        gate=L.ptr(gate), gate_stride=gate.stride(0), gate_bias=L.ptr(gate_bias), lower=L.ptr(lower), A_log=L.ptr(A_log), D=L.ptr(D),
        conv_weight=L.ptr(conv_weight), conv_bias=L.ptr(conv_bias), ring=L.ptr(ring), cu_seqlens_q=L.ptr(cu_seqlens_q),
        context_lens=L.ptr(context_lens), slots=L.ptr(slots), state=L.ptr(state), out=L.ptr(out), out_stride=out.stride(0),
        rtau=float(rtau), qscale=float(qscale), workspace=L.ptr(ws), workspace_bytes=0 if ws is None else ws.numel())
    L.check(lib.zp_linear_state(L.C.byref(p), L.IMPL[impl], L.dtype_code(q), L.stream_ptr()), "linear_state")
    _count(1)
    return out


def group_norm_gate(x, weight, parts, eps, pre_gate=None, post_gate=None, out=None):
    """RMS norm of `parts` equal parts of every row of silu(pre_gate) * x, times weight ([part width] or a whole row's), times
    silu(post_gate)."""
    L.require_cuda(x, weight, pre_gate, post_gate, out)
    N, W = x.shape
    assert W % parts == 0 and weight.dtype == torch.float32 and weight.is_contiguous() and weight.numel() in (W, W // parts)
    assert all(t is None or t.stride(1) == 1 and t.dtype == x.dtype for t in (x, pre_gate, post_gate, out))
    if out is None:
        out = torch.empty((N, W), dtype=x.dtype, device=x.device)
    st = lambda t: 0 if t is None else t.stride(0)
    L.check(L.load().zp_group_norm_gate(
        L.ptr(x), x.stride(0), L.ptr(pre_gate), st(pre_gate), L.ptr(post_gate), st(post_gate), L.ptr(weight), int(weight.numel() == W),
        L.ptr(out), out.stride(0), N, parts, W // parts, float(eps), L.dtype_code(x), L.stream_ptr()), "group_norm_gate")
    _count(1)
    return out


class LinearMixer(nn.Module):
    """h -> head outputs [rows, heads * vdim] before the output projection.  `run` selects the state of this pass when the
    layer runs several times.  Subclasses name their columns of one projection (`columns`: name -> size, in order; each starts at
    a multiple of 8, so that rows and groups are aligned) and make the fp32 gates."""

    def __init__(self, width, columns, heads, dim, vdim, eps, dtype, device):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.at, n = {}, 0
        for name, size in columns.items():
            self.at[name] = (n, n + size)
            n += (size + 7) // 8 * 8
        self._e = lambda *s, dt=torch.float32: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.proj = self._e(n, width, dt=dtype)
        self.out_proj = self._e(width, heads * vdim, dt=dtype)
        self.states = []                                       # one entry per pass, bound by the cache

    def _load(self, weights):
        """weights: name of the columns -> rows of the projection."""
        self.proj.zero_()
        for name, (a, b) in self.at.items():
            self.proj[a:b].copy_(weights[name])

    def _columns(self, y):
        return {name: y[:, a:b] for name, (a, b) in self.at.items()}

    def _recur(self, kind, q, k, v, gate, run, kv_heads, conv=None, **kw):
        """Decoded rows, then portions.  conv: (weight, bias, x) of the convolution that comes first, x its input columns
        (v | k | q)."""
        ctx = get_context()
        out = torch.empty((v.shape[0], self.heads * self.vdim), dtype=v.dtype, device=v.device)
        sizes = (self.heads, kv_heads, self.dim, self.vdim)
        state, nd = self.states[run][0], ctx.decode_rows()
        if nd:
            more = {} if conv is None else dict(conv_weight=conv[0], conv_bias=conv[1], ring=self.states[run][1])
            linear_state(kind, q, k, v, gate, self.gate_bias, state, out, ctx.context_lens[:nd], ctx.state_slots[:nd], *sizes, **kw, **more)
        if ctx.is_prefill and nd < ctx.context_lens.shape[0]:
            seqs, cu = (ctx.context_lens[nd:], ctx.state_slots[nd:]), ctx.cu_seqlens_q[nd:]
            if conv is not None:
                w, b, x = conv
                z = torch.empty((x.shape[0], (x.shape[1] + 7) // 8 * 8), dtype=x.dtype, device=x.device)
                short_conv(x, w, self.states[run][1], *seqs, cu, ctx.max_seqlen_q, z, bias=b)
                nv, nk = self.heads * self.vdim, kv_heads * self.dim
                v, k, q = z[:, :nv], z[:, nv:nv + nk], z[:, nv + nk:nv + 2 * nk]
            linear_state(kind, q, k, v, gate, self.gate_bias, state, out, *seqs, *sizes, cu_seqlens_q=cu, **kw)
        return out


class HGRN2Mixer(LinearMixer):
    """HGRN2: forget gates, bounded below, whose complement is the key."""

    def __init__(self, width, heads, dim, vdim, eps, dtype, device):
        super().__init__(width, {"q": heads * dim, "v": heads * vdim}, heads, dim, vdim, eps, dtype, device)
        self.forget = self._e(heads * dim, width, dt=dtype)    # (the product's results stay fp32)
        self.gate_bias, self.lower, self.norm = self._e(heads * dim), self._e(heads * dim), self._e(vdim)

    def load(self, get):
        self._load({n: get(n) for n in "qv"})
        self.forget.copy_(get("f"))
        self.gate_bias.copy_(get("f.b"))
        self.lower.copy_(get("lower"))
        self.norm.copy_(get("norm"))
        self.out_proj.copy_(get("o"))

    def forward(self, h, run):
        y = self._columns(project(h, self.proj))
        o = self._recur("forget", y["q"], None, y["v"], project(h, self.forget, fp32=True), run, self.heads, lower=self.lower)
        return group_norm_gate(o, self.norm, self.heads, self.eps, out=o)


class GLAMixer(LinearMixer):
    """Decays per key channel from a low-rank projection, sigmoid(z)^(1/tau), and an output gate (gated linear attention)."""

    def __init__(self, width, heads, dim, vdim, rank, tau, eps, dtype, device):
        super().__init__(width, {"q": heads * dim, "k": heads * dim, "v": heads * vdim, "g": heads * vdim, "a1": rank}, heads, dim, vdim, eps,
                         dtype, device)
        self.tau = tau
        self.a2 = self._e(heads * dim, rank, dt=dtype)
        self.gate_bias, self.norm = self._e(heads * dim), self._e(vdim)

    def load(self, get):
        self._load({n: get(n) for n in self.at})
        self.a2.copy_(get("a2"))
        self.gate_bias.copy_(get("a2.b"))
        self.norm.copy_(get("norm"))
        self.out_proj.copy_(get("o"))

    def forward(self, h, run):
        y = self._columns(project(h, self.proj))
        o = self._recur("power", y["q"], y["k"], y["v"], project(y["a1"], self.a2, fp32=True), run, self.heads, rtau=1.0 / self.tau,
                        qscale=self.dim ** -0.5)
        return group_norm_gate(o, self.norm, self.heads, self.eps, post_gate=y["g"], out=o)


class SSDMixer(LinearMixer):
    """Mamba-2: one decay per head and token, keys and queries shared by `groups` of heads, a short convolution ahead of
    them and of the values, the gate before a norm of `norm_groups` parts.  `dim` is the state's size."""

    def __init__(self, width, heads, groups, dim, vdim, taps, norm_groups, eps, dtype, device):
        self.channels = heads * vdim + 2 * groups * dim
        super().__init__(width, {"z": heads * vdim, "x": self.channels}, heads, dim, vdim, eps, dtype, device)
        self.groups, self.norm_groups = groups, norm_groups
        self.step = self._e(heads, width, dt=dtype)            # step sizes' rows: the product's results stay fp32
        self.gate_bias, self.A_log, self.D, self.norm = self._e(heads), self._e(heads), self._e(heads), self._e(heads * vdim)
        self.conv, self.conv_bias = self._e(taps, self.channels), self._e(self.channels)

    def load(self, get):
        w, n = get("in"), self.heads * self.vdim
        self._load({"z": w[:n], "x": w[n:n + self.channels]})
        self.step.copy_(w[n + self.channels:])
        self.conv.copy_(get("conv").t())
        self.conv_bias.copy_(get("conv.b"))
        self.gate_bias.copy_(get("dt_bias"))
        for p, name in ((self.A_log, "A_log"), (self.D, "D"), (self.norm, "norm"), (self.out_proj, "o")):
            p.copy_(get(name))

    def forward(self, h, run):
        y = self._columns(project(h, self.proj))
        x, nv, nk = y["x"], self.heads * self.vdim, self.groups * self.dim
        o = self._recur("scalar", x[:, nv + nk:], x[:, nv:nv + nk], x[:, :nv], project(h, self.step, fp32=True), run, self.groups,
                        conv=(self.conv, self.conv_bias, x), A_log=self.A_log, D=self.D)
        return group_norm_gate(o, self.norm, self.norm_groups, self.eps, pre_gate=y["z"], out=o)
