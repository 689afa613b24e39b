"""Row ops of decoders whose residual stream stays in fp32 between 16-bit matrix products.

`embed_position`, `rms_norm_f32`, `join_norms`, `soft_cap_` and `gelu_tanh` are single launches of libzipage_b200 kernels;
`project` and `project_add` are the library's matrix product with fp32 accumulation and, where the
result joins the fp32 stream, an fp32 result (the residual add is the product's epilogue).
"""
from __future__ import annotations

import math

import torch

from .. import _lib as L
from ..kernel import _count


def sinusoid_turns(width, device, base=10000.0):
    """Frequencies of a sinusoidal position vector in turns per position, fp64 [(width + 1) // 2]."""
    i = torch.arange((width + 1) // 2, dtype=torch.float64)
    return (base ** (-2.0 * i / width) / (2.0 * math.pi)).to(device)


def embed_position(tokens, positions, table, scale, turns=None, want_t=False, learned=None):
    """-> x fp32 [N, width] (and its copy in the table's dtype when `want_t`).  Positions: sinusoids (`turns`) or rows of the
    table `learned`."""
    L.require_cuda(tokens, positions, table, turns, learned)
    assert learned is None or learned.is_contiguous() and learned.dtype == table.dtype and learned.shape[1] == table.shape[1]
    assert tokens.dtype == positions.dtype == torch.int64 and table.is_contiguous()
    N, H = tokens.shape[0], table.shape[1]
    x = torch.empty((N, H), dtype=torch.float32, device=table.device)
    x_t = torch.empty((N, H), dtype=table.dtype, device=table.device) if want_t else None
    L.check(L.load().zp_embed_position(L.ptr(tokens), L.ptr(positions), L.ptr(table), L.ptr(turns), float(scale),
                                       L.ptr(learned), 0 if learned is None else learned.shape[0], L.ptr(x), L.ptr(x_t), N, H, table.shape[0], L.dtype_code(table),
                                       L.stream_ptr()), "embed_position")
    _count(1)
    return (x, x_t) if want_t else x


def rms_norm_f32(x, weight, eps, dtype, offset=0.0):
    """fp32 rows x -> dtype(x * rsqrt(mean(x^2) + eps) * (weight + offset)); weight None: the conversion alone."""
    L.require_cuda(x, weight)
    assert x.dtype == torch.float32 and x.is_contiguous() and (weight is None or weight.dtype == torch.float32)
    out = torch.empty(x.shape, dtype=dtype, device=x.device)
    L.check(L.load().zp_rms_norm_f32(L.ptr(x), L.ptr(weight), float(offset), L.ptr(out), x.shape[0], x.shape[1],
                                     float(eps), L.dtype_code(out), L.stream_ptr()), "rms_norm_f32")
    _count(1)
    return out


def join_norms(x, norms, eps, dtype, a=None, ls_a=None, b=None, ls_b=None, gate=None, y=None, pos=None, weights=None, rms=False, pair=None,
               pair_scale=0.5):
    """The boundary between sublayers.  x fp32 [N, width], in place:
    x += ls_a * a + ls_b * (sigmoid(gate) * b + sum_k weights[:, k] * y[pos[:, k]]) (weights None: ones) and, with `pair` = ((m1, w1),
    (m2, w2)), pair_scale * (RMS norm of m1 * w1 + RMS norm of m2 * w2); then one layer
    norm (`rms`: RMS norm) of x per (weight, bias) of `norms` (at most two), each as `dtype`."""
    (m1, mw1), (m2, mw2) = pair or ((None, None), (None, None))
    L.require_cuda(x, a, ls_a, b, ls_b, gate, y, pos, weights, m1, mw1, m2, mw2, *(t for n in norms for t in n))
    assert x.dtype == torch.float32 and x.is_contiguous() and len(norms) <= 2
    assert all(t is None or t.dtype == dtype and t.is_contiguous() for t in (a, b, y, m1, m2))
    outs = [torch.empty(x.shape, dtype=dtype, device=x.device) for _ in norms]
    flat = [p for n, o in zip(norms, outs) for p in (L.ptr(n[0]), L.ptr(n[1]), L.ptr(o))]
    flat += [None] * (6 - len(flat))
    L.check(L.load().zp_join_norms(
        L.ptr(x), L.ptr(a), L.ptr(ls_a), L.ptr(b), L.ptr(ls_b), L.ptr(gate), 0 if gate is None else gate.stride(0), L.ptr(y),
        0 if y is None else y.shape[0], L.ptr(pos), L.ptr(weights), 0 if y is None else pos.shape[1], L.ptr(m1), L.ptr(mw1), L.ptr(m2),
        L.ptr(mw2), float(pair_scale), *flat, x.shape[0],
        x.shape[1], float(eps), int(rms), L.ZP_DTYPE[dtype], L.stream_ptr()), "join_norms")
    _count(1)
    return outs


def soft_cap_(z, cap):
    """z = cap tanh(z / cap), fp32, in place."""
    L.require_cuda(z)
    assert z.dtype == torch.float32 and z.is_contiguous()
    L.check(L.load().zp_soft_cap(L.ptr(z), z.numel(), float(cap), L.stream_ptr()), "soft_cap")
    _count(1)
    return z


def gelu_tanh(x):
    L.require_cuda(x)
    assert x.is_contiguous()
    out = torch.empty_like(x)
    L.check(L.load().zp_gelu_tanh(L.ptr(x), L.ptr(out), x.numel(), L.dtype_code(x), L.stream_ptr()), "gelu_tanh")
    _count(1)
    return out


def project(h, weight, fp32=False):
    """h [N, in] @ weight [out, in]^T in h's dtype, or with an fp32 result."""
    if not fp32 or h.dtype == torch.float32:
        return torch.mm(h, weight.t())
    return torch.mm(h, weight.t(), out_dtype=torch.float32)


def project_add(x, h, weight):
    """fp32 x + h @ weight^T, accumulated and kept in fp32."""
    if h.dtype == torch.float32:
        return torch.addmm(x, h, weight.t())
    return torch.addmm(x, h, weight.t(), out_dtype=torch.float32)
