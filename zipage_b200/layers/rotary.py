"""Rotary positions: frequencies of the pairs, plain or stretched for long contexts, and the launch that norms and
rotates queries and keys and stores keys and values."""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .. import _lib as L
from ..kernel import _count


def rotary_turns(dims, base, device):
    """Frequencies of the pairs of a rotated vector in turns per position, fp64 [dims / 2]."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    return (float(base) ** (-2.0 * i / dims) / (2.0 * math.pi)).to(device)


def yarn_turns(dims, base, factor, original, fast, slow, device):
    """YaRN: pairs that turn more than `fast` times within `original` positions keep their frequency, those that turn less
    than `slow` times have it divided by `factor`, with a linear ramp over the pairs between.  -> (turns, the
    factor of cosine and sine)."""
    pair_of = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
    ramp = ((torch.arange(dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    t = rotary_turns(dims, base, "cpu")
    return (t / factor * ramp + t * (1.0 - ramp)).to(device), 0.1 * math.log(factor) + 1.0


@dataclass
class Rotary:
    """Rotation of the first `dims` entries of every head; interleaved: pairs (2t, 2t + 1), else (t, t + dims / 2)."""
    dims: int
    turns: torch.Tensor
    interleaved: bool
    mul: float = 1.0

    @classmethod
    def from_config(cls, rot, interleaved, device):
        """rot: dims, base and (or None) scaling with factor, original, fast and slow."""
        s, dims, base = rot.get("scaling"), int(rot["dims"]), float(rot["base"])
        if not s:
            return cls(dims, rotary_turns(dims, base, device), interleaved)
        turns, mul = yarn_turns(dims, base, float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"]), device)
        return cls(dims, turns, interleaved, mul)


def rotate_store(q, k, v, positions, rotary, k_cache, v_cache, slot_mapping, head_dim, v_dim, q_weight=None, k_weight=None, eps=0.0):
    """q [N, Hq * D] in place, k [N, Hkv * D] into k_cache [P, BS, Hkv, KP], both normed per head (weights given) and
    rotated; v [N, Hkv * DV] (possibly k itself) into v_cache as it is.  q, k, v: column views of one projection."""
    L.require_cuda(q, k, v, positions, rotary.turns, k_cache, v_cache, slot_mapping, q_weight, k_weight)
    assert q.stride(0) == k.stride(0) == v.stride(0) and q.stride(1) == k.stride(1) == v.stride(1) == 1
    P, BS, Hkv, KP = k_cache.shape
    L.check(L.load().zp_rotate_store(
        L.ptr(q), L.ptr(k), L.ptr(v), q.stride(0), L.ptr(positions), L.ptr(rotary.turns), rotary.dims, int(rotary.interleaved),
        float(rotary.mul), L.ptr(q_weight), L.ptr(k_weight), float(eps), L.ptr(k_cache), L.ptr(v_cache), L.ptr(slot_mapping),
        q.shape[0], q.shape[1] // head_dim, Hkv, head_dim, v_dim, KP, v_cache.shape[3], P * BS, L.dtype_code(q), L.stream_ptr()),
        "rotate_store")
    _count(1)
