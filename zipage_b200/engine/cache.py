"""Device memory of models that describe what each layer keeps: paged keys and values or latents, and
recurrent state in slots.  Pages and slots are handed out by the native scheduler (block tables, query_id);
this only owns the storage.

A page id or slot means the same row range in every entry, so one block table and one slot number per
sequence serve all layers, whatever their head sizes.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class KVSpec:
    """Keys and values of one attention layer (run): rows padded to multiples of 16 elements."""
    kv_heads: int
    dim: int
    vdim: int

    def allocate(self, pages, block_size, slots, dtype, device):
        pad = lambda n: (n + 15) // 16 * 16
        z = lambda d: torch.zeros((pages, block_size, self.kv_heads, pad(d)), dtype=dtype, device=device)
        return z(self.dim), z(self.vdim)

    def bytes(self, pages, block_size, slots, itemsize):
        return pages * block_size * self.kv_heads * ((self.dim + 15) // 16 + (self.vdim + 15) // 16) * 16 * itemsize


@dataclass(frozen=True)
class LatentSpec:
    """One row per token for all heads of a latent-attention layer: the latent and the rotated key part, padded
    to a multiple of 16 elements (the padding stays zero)."""
    rank: int
    rot: int

    @property
    def row(self):
        return (self.rank + self.rot + 15) // 16 * 16

    def allocate(self, pages, block_size, slots, dtype, device):
        return (torch.zeros((pages, block_size, 1, self.row), dtype=dtype, device=device),)

    def bytes(self, pages, block_size, slots, itemsize):
        return pages * block_size * self.row * itemsize


@dataclass(frozen=True)
class StateSpec:
    """fp32 matrix memory of one mLSTM layer (run): S [slots, heads, dim, vdim padded to 4], n, m.
    A sequence that starts in a slot reads none of what the slot held before."""
    heads: int
    dim: int
    vdim: int

    def allocate(self, pages, block_size, slots, dtype, device):
        z = lambda *s: torch.zeros(s, dtype=torch.float32, device=device)
        return (z(slots, self.heads, self.dim, (self.vdim + 3) // 4 * 4), z(slots, self.heads, self.dim),
                z(slots, self.heads))

    def bytes(self, pages, block_size, slots, itemsize):
        return slots * self.heads * (self.dim * ((self.vdim + 3) // 4 * 4) + self.dim + 1) * 4


@dataclass(frozen=True)
class DeltaSpec:
    """What a gated delta rule keeps per slot: the fp32 matrix S [heads, dim, vdim padded to 4] and a ring of the last `taps`
    inputs of its convolution, [taps, channels] in the model's dtype."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self):
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    def allocate(self, pages, block_size, slots, dtype, device):
        return (torch.zeros((slots, self.heads, self.dim, (self.vdim + 3) // 4 * 4), dtype=torch.float32, device=device),
                torch.zeros((slots, self.taps, self.channels), dtype=dtype, device=device))

    def bytes(self, pages, block_size, slots, itemsize):
        return slots * (self.heads * self.dim * ((self.vdim + 3) // 4 * 4) * 4 + self.taps * self.channels * itemsize)


@dataclass(frozen=True)
class LinearStateSpec:
    """What a linear-attention mixer keeps per slot: the fp32 matrix S [heads, dim, vdim padded to 4] and, with a convolution
    (taps > 0), a ring of its last `taps` inputs, [taps, channels] in the model's dtype."""
    heads: int
    dim: int
    vdim: int
    channels: int = 0
    taps: int = 0

    def allocate(self, pages, block_size, slots, dtype, device):
        out = (torch.zeros((slots, self.heads, self.dim, (self.vdim + 3) // 4 * 4), dtype=torch.float32, device=device),)
        return out + ((torch.zeros((slots, self.taps, self.channels), dtype=dtype, device=device),) if self.taps else ())

    def bytes(self, pages, block_size, slots, itemsize):
        return slots * (self.heads * self.dim * ((self.vdim + 3) // 4 * 4) * 4 + self.taps * self.channels * itemsize)


class PagedStateCache:
    def __init__(self, specs, pages, block_size, slots, dtype, device):
        if block_size % 64:
            raise ValueError("the page size must be a multiple of 64 tokens")
        self.pages, self.block_size, self.slots = pages, block_size, slots
        self.dtype, self.device = dtype, torch.device(device)
        self.entries = [s.allocate(pages, block_size, slots, dtype, device) for s in specs]
        self.nbytes = sum(t.numel() * t.element_size() for e in self.entries for t in e)
