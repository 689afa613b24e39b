"""A mixer made of one or several groups of heads side by side that read the same input: one product makes the columns of
all of them, each writes its outputs (already gated and scaled) into its columns, one product joins them."""
from __future__ import annotations

import torch
from torch import nn

from ..utils.context import get_context
from .gated_delta import DeltaHeads
from .row_ops import project


class HeadsMixer(nn.Module):
    """`parts`: (name prefix of the weights, heads) pairs, heads a `RotaryHeads` or a `DeltaHeads`.  `side`: a stream for the
    second part of a decode step, whose launches are short."""

    def __init__(self, width, parts, dtype, device, side=None):
        super().__init__()
        self.prefixes, self.parts, self.side = [p for p, _ in parts], nn.ModuleList([h for _, h in parts]), side
        self.first, at = [], 0
        for h in self.parts:                              # (each part's columns start at a multiple of 8: aligned rows)
            self.first.append(at)
            at += (h.columns + 7) // 8 * 8
        e = lambda *s: nn.Parameter(torch.empty(*s, dtype=dtype, device=device), requires_grad=False)
        self.proj, self.out_proj = e(at, width), e(width, sum(h.out_columns for h in self.parts))

    def load(self, get):
        self.proj.zero_()
        outs = []
        for prefix, h, at in zip(self.prefixes, self.parts, self.first):
            self.proj[at:at + h.columns].copy_(h.load(lambda n: get(prefix + n)))
            outs.append(get(prefix + "o"))
        self.out_proj.copy_(torch.cat(outs, 1))

    def forward(self, h, positions):
        y = project(h, self.proj)
        out = torch.empty((h.shape[0], self.out_proj.shape[1]), dtype=h.dtype, device=h.device)
        main, fork = None, self.side is not None and len(self.parts) > 1 and not get_context().is_prefill
        if fork:
            main = torch.cuda.current_stream()
            self.side.wait_stream(main)
        at = 0
        for i, (part, first) in enumerate(zip(self.parts, self.first)):
            with torch.cuda.stream(self.side if fork and i else None):
                args = (y[:, first:first + part.columns],)
                if isinstance(part, DeltaHeads):
                    args += (project(h, part.ab, fp32=True),)
                part(*args, positions, out[:, at:at + part.out_columns])
            at += part.out_columns
        if fork:
            main.wait_stream(self.side)
        return project(out, self.out_proj)
