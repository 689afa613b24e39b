"""Tukarax: a decoder of chunked attention and of layers that run softmax attention and a gated delta rule side by side,
with a mixture of experts after each and an fp32 residual stream.

Every sublayer reads an RMS norm of the stream; the launch that adds a sublayer's result also takes the norm that the
next one reads (`join_norms`).  The configuration names every layer on its own.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..engine.cache import DeltaSpec, KVSpec
from ..layers.attention import RotaryHeads
from ..layers.feed_forward import GatedMixtureFF
from ..layers.gated_delta import DeltaHeads
from ..layers.heads_mixer import HeadsMixer
from ..layers.rotary import Rotary
from ..layers.row_ops import embed_position, join_norms


@dataclass(frozen=True)
class LayerConfig:
    type: str            # "attention" or "parallel"
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class TukaraxConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple

    @classmethod
    def from_dict(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            mix, mlp = dict(e["mixer"]), e.get("mlp")
            if e["type"] not in ("attention", "parallel"):
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            if mlp is not None and mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            for m in [mix] if e["type"] == "attention" else [mix["left"], mix["right"]]:
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"layer {i}: {m['heads']} heads over {m['kv_heads']} key/value heads")
                if "rot" in m and (m["rot"]["dims"] % 2 or m["rot"]["dims"] > m["dim"]):
                    raise ValueError(f"layer {i}: {m['rot']['dims']} rotated entries of {m['dim']}")
            if e["type"] == "parallel" and mix["left"]["dim"] != mix["left"]["vdim"]:
                raise ValueError(f"layer {i}: keys of {mix['left']['dim']} entries as values of {mix['left']['vdim']}")
            if mlp is not None and not 0 < mlp["router"]["top"] <= mlp["router"]["experts"]:
                raise ValueError(f"layer {i}: {mlp['router']['top']} of {mlp['router']['experts']} experts")
            layers.append(LayerConfig(e["type"], mix, None if mlp is None else dict(mlp)))
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), tuple(layers))


class TukaraxLayer(nn.Module):
    def __init__(self, c: TukaraxConfig, lc: LayerConfig, dtype, device, side=None):
        super().__init__()
        m, f = lc.mixer, lc.mlp
        if lc.type == "attention":
            parts = [("", RotaryHeads(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"],
                                      Rotary.from_config(m["rot"], False, device), c.eps, dtype, device,
                                      softcap=m.get("softcap") or 0.0, chunk=int((m.get("mask") or {}).get("size") or 0),
                                      sink=True, gate="head"))]
        else:
            l, r = m["left"], m["right"]
            parts = [("left.", RotaryHeads(l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["scale"],
                                           Rotary.from_config(l["rot"], True, device), c.eps, dtype, device, qk_norm=True,
                                           shared_kv=True, gate="entry", out_scale=m["left_scale"])),
                     ("right.", DeltaHeads(c.width, r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"], c.eps, dtype, device,
                                           out_scale=m["right_scale"]))]
        self.mixer = HeadsMixer(c.width, parts, dtype, device, side)
        self.ff = None if f is None else GatedMixtureFF(c.width, f["router"]["experts"], f["router"]["top"], f["expert"]["ff"],
                                                        dtype, device)
        v = lambda: nn.Parameter(torch.empty(c.width, dtype=torch.float32, device=device), requires_grad=False)
        self.norm1, self.norm2 = v(), v() if self.ff is not None else None

    def load(self, get):
        self.norm1.copy_(get("norm1"))
        self.mixer.load(lambda n: get("mix." + n))
        if self.ff is not None:
            self.norm2.copy_(get("norm2"))
            self.ff.load(lambda n: get("mlp." + n))


class TukaraxModel(nn.Module):
    fp32_logits = True   # the engine keeps this model's logits in fp32

    def __init__(self, c: TukaraxConfig, dtype, device):
        super().__init__()
        self.config, self.dtype = c, dtype
        e = lambda *s, dt=dtype: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.embed = e(c.vocab, c.width)
        side = torch.cuda.Stream(device) if device.type == "cuda" else None
        self.layers = nn.ModuleList([TukaraxLayer(c, lc, dtype, device, side) for lc in c.layers])
        self.norm = e(c.width, dt=torch.float32)
        self.head = e(c.vocab, c.width)
        self.trail = None      # optional list: the residual stream after every layer

    @torch.no_grad()
    def load_weights(self, w):
        self.embed.copy_(w["embed"])
        self.head.copy_(w["head"])
        self.norm.copy_(w["final.norm"])
        for i, layer in enumerate(self.layers):
            layer.load(lambda n, p=f"l{i}.": w[p + n])

    def _heads(self):
        return [h for layer in self.layers for h in layer.mixer.parts]

    def cache_spec(self):
        """What each group of heads keeps, in order."""
        return [DeltaSpec(h.heads, h.kv_heads, h.dim, h.vdim, h.conv.shape[0]) if isinstance(h, DeltaHeads)
                else KVSpec(h.kv_heads, h.dim, h.vdim) for h in self._heads()]

    def bind_cache(self, cache):
        for h, entry in zip(self._heads(), cache.entries):
            if isinstance(h, DeltaHeads):
                h.state, h.ring = entry
            else:
                h.k_cache, h.v_cache = entry

    def forward(self, input_ids, positions):
        c = self.config
        join = lambda norm, **parts: join_norms(x, [(norm, None)], c.eps, self.dtype, rms=True, **parts)[0]
        after = [layer.norm1 for layer in self.layers] + [self.norm]
        x = embed_position(input_ids, positions, self.embed, 1.0)
        h = join(after[0])
        for layer, norm in zip(self.layers, after[1:]):
            a = layer.mixer(h, positions)
            h = join(norm, a=a) if layer.ff is None else join(norm, **layer.ff(join(layer.norm2, a=a)))
            if self.trail is not None:
                self.trail.append(x.clone())
        return h
