"""Feed-forward blocks whose result joins the residual stream at the layer boundary (`row_ops.join_norms`):
a gated dense block and a mixture of experts, on libzipage_b200 kernels and the library's matrix product.

Each block returns the keyword arguments that `join_norms` takes for its result, so that the experts'
weighting, the shared expert's gate and the sum are part of that launch.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import _lib as L
from ..kernel import _count
from .row_ops import project
from .step_ops import silu_and_mul


def gelu_tanh_and_mul(x):
    """gate | up [N, 2 F] -> gelu_tanh(gate) * up [N, F]."""
    L.require_cuda(x)
    assert x.is_contiguous()
    N, F = x.shape[0], x.shape[1] // 2
    out = torch.empty((N, F), dtype=x.dtype, device=x.device)
    L.check(L.load().zp_gelu_tanh_and_mul(L.ptr(x), L.ptr(out), N, F, L.dtype_code(x), L.stream_ptr()), "gelu_tanh_and_mul")
    _count(1)
    return out


def relu_squared_(x):
    L.require_cuda(x)
    assert x.is_contiguous()
    L.check(L.load().zp_relu_squared(L.ptr(x), L.ptr(x), x.numel(), L.dtype_code(x), L.stream_ptr()), "relu_squared")
    _count(1)
    return x


def moe_route(logits, n_experts, top, score="softmax", by_place=False, bias=None):
    """logits [N, >= n_experts] fp32 -> (weights [N, top] fp32, experts [N, top], places [N, top],
    rows [N * top], offsets [n_experts + 1]): scores of logits + bias (softmax over all experts or, "softmax_top", over the
    chosen ones; or sigmoid), the `top` largest of a
    token, and the (token, expert) pairs sorted by expert.  `by_place`: the weights in that order instead, [N * top]."""
    L.require_cuda(logits, bias)
    assert bias is None or bias.dtype == torch.float32 and bias.is_contiguous()
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    N, dev = logits.shape[0], logits.device
    w = torch.empty((N, top), dtype=torch.float32, device=dev)
    ints = torch.empty(3 * N * top + 2 * n_experts + 1, dtype=torch.int32, device=dev)
    experts, places, rows, offsets, counts = ints.split([N * top] * 3 + [n_experts + 1, n_experts])
    pw = torch.empty(N * top, dtype=torch.float32, device=dev) if by_place else None
    L.check(L.load().zp_moe_route(L.ptr(logits), logits.stride(0), L.ptr(bias), N, n_experts, top, L.ptr(w), L.ptr(experts), L.ptr(places),
                                  L.ptr(rows), L.ptr(offsets), L.ptr(counts), L.ptr(pw), L.SCORE[score], L.stream_ptr()), "moe_route")
    _count(1 if N <= 512 and N * top <= 4096 else 2)
    return w if pw is None else pw, experts.view(N, top), places.view(N, top), rows, offsets


def grouped_gemm(x, weight, offsets, n_places, rows=None, act=None, impl="auto", row_scale=None):
    """out[p] = act(x[rows[p]] @ weight[e].T) for the places p of every expert e; x [src, K] (rows None:
    place p is row p), weight [E, n_out, K].  act "silu_mul": weight as `interleave_gate_up` makes it, out [places, n_out / 2] =
    silu(s gate) * (s up) with s = row_scale[p]."""
    L.require_cuda(x, weight, offsets, rows, row_scale)
    assert row_scale is None or row_scale.dtype == torch.float32 and row_scale.is_contiguous()
    E, n_out, K = weight.shape
    assert x.stride(1) == 1 and weight.is_contiguous() and x.dtype == weight.dtype and x.shape[1] == K
    out = torch.empty((n_places, n_out // 2 if act == "silu_mul" else n_out), dtype=x.dtype, device=x.device)
    L.check(L.load().zp_grouped_gemm(L.ptr(x), x.stride(0), L.ptr(rows), x.shape[0], L.ptr(weight), L.ptr(offsets), L.ptr(row_scale), L.ptr(out),
                                     n_places, E, n_out, K, L.ACT[act], L.IMPL[impl], L.dtype_code(x), L.stream_ptr()),
            "grouped_gemm")
    _count(1)
    return out


class GatedFF(nn.Module):
    """W_down (gelu_tanh(W_gate h) * (W_up h))."""

    def __init__(self, width, ff, dtype, device):
        super().__init__()
        e = lambda *s: nn.Parameter(torch.empty(*s, dtype=dtype, device=device), requires_grad=False)
        self.gate_up, self.down = e(2 * ff, width), e(width, ff)

    def load(self, get):
        self.gate_up.copy_(torch.cat([get("gate"), get("up")], 0))
        self.down.copy_(get("down"))

    def forward(self, h):
        return {"b": project(gelu_tanh_and_mul(project(h, self.gate_up)), self.down)}


class SquaredReluFF(nn.Module):
    """W_down max(W_up h, 0)^2."""

    def __init__(self, width, ff, dtype, device):
        super().__init__()
        e = lambda *s: nn.Parameter(torch.empty(*s, dtype=dtype, device=device), requires_grad=False)
        self.up, self.down = e(ff, width), e(width, ff)

    def load(self, get):
        self.up.copy_(get("up"))
        self.down.copy_(get("down"))

    def forward(self, h):
        return {"b": project(relu_squared_(project(h, self.up)), self.down)}


class MixtureFF(nn.Module):
    """`top` of `experts` squared-ReLU blocks per token, weighted by their softmax scores, and (shared_ff > 0)
    a shared block scaled by a sigmoid gate.  The gate's row follows the experts' in the router product."""

    def __init__(self, width, experts, top, ff, shared_ff, dtype, device):
        super().__init__()
        self.experts, self.top, self.shared = experts, top, shared_ff > 0
        e = lambda *s: nn.Parameter(torch.empty(*s, dtype=dtype, device=device), requires_grad=False)
        # rows: experts, the gate, zeros up to a multiple of 8 (aligned rows of logits)
        self.router = e((experts + int(self.shared) + 7) // 8 * 8, width)
        self.up, self.down = e(experts, ff, width), e(experts, width, ff)
        if self.shared:
            self.shared_up, self.shared_down = e(shared_ff, width), e(width, shared_ff)

    def load(self, get):
        for i in range(self.experts):
            self.up[i].copy_(get(f"e{i}.up"))
            self.down[i].copy_(get(f"e{i}.down"))
        self.router.zero_()
        self.router[:self.experts].copy_(get("router"))
        if self.shared:
            self.router[self.experts:self.experts + 1].copy_(get("shared.sg"))
            self.shared_up.copy_(get("shared.up"))
            self.shared_down.copy_(get("shared.down"))

    def forward(self, h):
        N = h.shape[0]
        z = project(h, self.router, fp32=True)
        w, _, places, rows, offsets = moe_route(z, self.experts, self.top)
        mid = grouped_gemm(h, self.up, offsets, N * self.top, rows=rows, act="relu_squared")
        out = {"y": grouped_gemm(mid, self.down, offsets, N * self.top), "pos": places, "weights": w}
        if self.shared:
            out["b"] = project(relu_squared_(project(h, self.shared_up)), self.shared_down)
            out["gate"] = z[:, self.experts]
        return out


def padded_ff(ff):
    """Width that gated experts of width `ff` are stored with (whole blocks of 16)."""
    return (ff + 15) // 16 * 16


def interleave_gate_up(out, gate, up):
    """out [2 * padded_ff, width]: blocks of 16 rows of gate and of up in turn, zeros past the last."""
    ff, blocks = gate.shape[0], out.view(-1, 2, 16, out.shape[1])
    out.zero_()
    for i, w in enumerate((gate, up)):
        whole = ff // 16
        blocks[:whole, i].copy_(w[:whole * 16].view(whole, 16, w.shape[1]))
        if ff % 16:
            blocks[whole, i, :ff % 16].copy_(w[whole * 16:])


class GatedMixtureFF(nn.Module):
    """`top` of `experts` SiLU-gated blocks per token, W_down (silu(W_gate z) * (W_up z)).  weigh "input": each on z = s h with
    its own score s (the score joins the gate and up products' epilogue); "output": on z = h, and the scores weight the sum.
    `score` as in `moe_route`.  Optional: a bias of the router's logits, a shared block of the same form that every token takes."""

    def __init__(self, width, experts, top, ff, dtype, device, score="sigmoid", weigh="input", bias=False, shared_ff=0):
        super().__init__()
        self.experts, self.top, self.ff, self.score, self.weigh, self.shared_ff = experts, top, ff, score, weigh, shared_ff
        self.bias = nn.Parameter(torch.empty(experts, dtype=torch.float32, device=device), requires_grad=False) if bias else None
        e = lambda *s: nn.Parameter(torch.empty(*s, dtype=dtype, device=device), requires_grad=False)
        self.router = e((experts + 7) // 8 * 8, width)      # (zero rows up to a multiple of 8: aligned rows of logits)
        self.gate_up, self.down = e(experts, 2 * padded_ff(ff), width), e(experts, width, padded_ff(ff))
        if shared_ff:                                       # (gate rows, then up rows, each with zeros past the last)
            self.shared_gate_up, self.shared_down = e(2, padded_ff(shared_ff), width), e(width, padded_ff(shared_ff))

    def load(self, get):
        self.down.zero_()
        for i in range(self.experts):
            interleave_gate_up(self.gate_up[i], get(f"e{i}.gate"), get(f"e{i}.up"))
            self.down[i, :, :self.ff].copy_(get(f"e{i}.down"))
        self.router.zero_()
        self.router[:self.experts].copy_(get("router"))
        if self.bias is not None:
            self.bias.copy_(get("router.b"))
        if self.shared_ff:
            self.shared_gate_up.zero_()
            self.shared_down.zero_()
            for i, n in enumerate(("gate", "up")):
                self.shared_gate_up[i, :self.shared_ff].copy_(get("shared." + n))
            self.shared_down[:, :self.shared_ff].copy_(get("shared.down"))

    def forward(self, h):
        places, early = h.shape[0] * self.top, self.weigh == "input"
        w, _, pos, rows, offsets = moe_route(project(h, self.router, fp32=True), self.experts, self.top, self.score, by_place=early,
                                             bias=self.bias)
        mid = grouped_gemm(h, self.gate_up, offsets, places, rows=rows, act="silu_mul", row_scale=w if early else None)
        out = {"y": grouped_gemm(mid, self.down, offsets, places), "pos": pos}
        if not early:
            out["weights"] = w
        if self.shared_ff:
            out["b"] = project(silu_and_mul(project(h, self.shared_gate_up.view(-1, h.shape[1]))), self.shared_down)
        return out
