"""The short causal convolution of recurrent mixers over prompt portions, with a ring of its last inputs per state slot."""
from __future__ import annotations

from .. import _lib as L
from ..kernel import _count


def short_conv(x, weight, ring, context_lens, slots, cu_seqlens_q, max_seqlen_q, out, bias=None):
    """Causal convolution with silu over portions; x [rows, >= channels] (column view), weight [taps, channels] and bias [channels] fp32,
    ring [slots, taps, channels], out [rows, channels]."""
    L.require_cuda(x, weight, ring, context_lens, slots, cu_seqlens_q, out, bias)
    taps, C = weight.shape
    assert x.stride(1) == out.stride(1) == 1 and ring.is_contiguous() and ring.shape[1:] == (taps, C) and x.dtype == ring.dtype == out.dtype
    L.check(L.load().zp_short_conv(
        L.ptr(x), x.stride(0), L.ptr(weight), L.ptr(bias), L.ptr(ring), L.ptr(cu_seqlens_q), L.ptr(context_lens), L.ptr(slots), L.ptr(out),
        out.stride(0), context_lens.shape[0], int(max_seqlen_q), C, taps, ring.shape[0], L.dtype_code(x), L.stream_ptr()), "short_conv")
    _count(2)
    return out
