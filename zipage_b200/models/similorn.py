"""Similorn: a decoder of matrix-memory (mLSTM) and windowed-attention layers with an fp32 residual
stream, sinusoidal positions at the embedding, and a run of layers that is repeated with shared weights.

The configuration names every layer on its own, so sizes, window, cap and feed-forward may differ from
layer to layer.  A layer inside the repeated run keeps one cache or state per pass; `cache_spec()` lists
what each needs and the engine's cache manager provides it.

The residual stream x is fp32.  Each sublayer is norm -> projections -> mixer kernels -> a matrix
product that accumulates onto x.  Ahead of every pass of the repeated run x becomes
W_in [x; x0], x0 the embedding output; W_in's right half meets the same x0 in every pass, so that product
is taken once per step and each pass adds the left half's to it.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..engine.cache import KVSpec, StateSpec
from ..layers.attention import WindowAttentionMixer
from ..layers.mlstm import MLSTMMixer
from ..layers.row_ops import embed_position, gelu_tanh, project, project_add, rms_norm_f32, sinusoid_turns


@dataclass(frozen=True)
class LayerConfig:
    type: str            # "mlstm" or "attention"
    mixer: dict
    ff: int              # feed-forward width, 0 = the layer has none


@dataclass(frozen=True)
class SimilornConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    layers: tuple
    loop: tuple          # (start, stop, times); (0, 0, 0) = no layer is repeated

    @classmethod
    def from_dict(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            mix, mlp = dict(e["mixer"]), e.get("mlp")
            if e["type"] == "attention":
                mask = mix.pop("mask", None) or {}
                mix["window"] = int(mask.get("size") or 0)
                if mix["heads"] % mix["kv_heads"]:
                    raise ValueError(f"layer {i}: {mix['heads']} heads over {mix['kv_heads']} key/value heads")
            elif e["type"] != "mlstm":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(e["type"], mix, int(mlp["ff"]) if mlp is not None else 0))
        lp = c.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else (0, 0, 0)
        if not 0 <= loop[0] <= loop[1] <= len(layers):
            raise ValueError(f"loop {loop} over {len(layers)} layers")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c["embedding"]["scale"]),
                   tuple(layers), loop)

    def runs(self):
        """The forward's layer runs in order: (layer, pass, whether the run opens a pass)."""
        a, b, times = self.loop
        out = [(i, 0, False) for i in range(a)]
        for t in range(times):
            out += [(i, t, i == a) for i in range(a, b)]
        return out + [(i, 0, False) for i in range(b, len(self.layers))]


class DenseFF(nn.Module):
    def __init__(self, width, ff, dtype, device):
        super().__init__()
        self.up = nn.Parameter(torch.empty(ff, width, dtype=dtype, device=device), requires_grad=False)
        self.down = nn.Parameter(torch.empty(width, ff, dtype=dtype, device=device), requires_grad=False)

    def load(self, get):
        self.up.copy_(get("up"))
        self.down.copy_(get("down"))

    def forward(self, x, h):
        return project_add(x, gelu_tanh(project(h, self.up)), self.down)


class SimilornLayer(nn.Module):
    def __init__(self, c: SimilornConfig, lc: LayerConfig, dtype, device):
        super().__init__()
        self.eps, self.dtype = c.eps, dtype
        m = lc.mixer
        if lc.type == "mlstm":
            self.mixer = MLSTMMixer(c.width, m["heads"], m["dim"], m["vdim"], m["gate_cap"], c.eps, dtype, device)
        else:
            self.mixer = WindowAttentionMixer(c.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"],
                                              m.get("softcap") or 0.0, m["window"], dtype, device)
        w = lambda: nn.Parameter(torch.empty(c.width, dtype=torch.float32, device=device), requires_grad=False)
        self.norm1 = w()
        self.ff, self.norm2 = (DenseFF(c.width, lc.ff, dtype, device), w()) if lc.ff else (None, None)

    def load(self, get):
        self.norm1.copy_(get("norm1"))
        self.mixer.load(lambda n: get("mix." + n))
        if self.ff is not None:
            self.norm2.copy_(get("norm2"))
            self.ff.load(lambda n: get("mlp." + n))

    def forward(self, x, run):
        h = rms_norm_f32(x, self.norm1, self.eps, self.dtype, offset=1.0)
        x = project_add(x, self.mixer(h, run), self.mixer.out_proj)
        if self.ff is not None:
            x = self.ff(x, rms_norm_f32(x, self.norm2, self.eps, self.dtype, offset=1.0))
        return x


class SimilornModel(nn.Module):
    fp32_logits = True   # the engine keeps this model's logits in fp32

    def __init__(self, c: SimilornConfig, dtype, device):
        super().__init__()
        self.config, self.dtype = c, dtype
        e = lambda *s, dt=dtype: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.embed = e(c.vocab, c.width)
        self.turns = sinusoid_turns(c.width, device)
        self.looped = c.loop[1] > c.loop[0] and c.loop[2] > 0
        if self.looped:
            self.loop_x, self.loop_x0 = e(c.width, c.width), e(c.width, c.width)
        self.layers = nn.ModuleList([SimilornLayer(c, lc, dtype, device) for lc in c.layers])
        self.norm = e(c.width, dt=torch.float32)
        self.head = e(c.vocab, c.width)
        self.runs = c.runs()
        self.trail = None      # optional list: the residual stream after every layer run

    @torch.no_grad()
    def load_weights(self, w):
        self.embed.copy_(w["embed"])
        self.head.copy_(w["head"])
        self.norm.copy_(w["final.norm"])
        if self.looped:
            W = self.config.width
            self.loop_x.copy_(w["loop.in"][:, :W])
            self.loop_x0.copy_(w["loop.in"][:, W:])
        for i, layer in enumerate(self.layers):
            layer.load(lambda n, p=f"l{i}.": w[p + n])

    def cache_spec(self):
        """What each layer run keeps, in the order of `runs`."""
        out = []
        for i, _, _ in self.runs:
            m = self.layers[i].mixer
            if isinstance(m, MLSTMMixer):
                out.append(StateSpec(m.heads, m.dim, m.vdim))
            else:
                out.append(KVSpec(m.kv_heads, m.dim, m.vdim))
        return out

    def bind_cache(self, cache):
        for layer in self.layers:
            if isinstance(layer.mixer, MLSTMMixer):
                layer.mixer.states = []
            else:
                layer.mixer.caches = []
        for (i, _, _), entry in zip(self.runs, cache.entries):
            m = self.layers[i].mixer
            (m.states if isinstance(m, MLSTMMixer) else m.caches).append(entry)

    def forward(self, input_ids, positions):
        c = self.config
        if self.looped:
            x, x0 = embed_position(input_ids, positions, self.embed, c.embed_scale, self.turns, want_t=True)
            from_x0 = project(x0, self.loop_x0, fp32=True)
        else:
            x = embed_position(input_ids, positions, self.embed, c.embed_scale, self.turns)
        for i, run, opens in self.runs:
            if opens:
                x = project_add(from_x0, rms_norm_f32(x, None, 0.0, self.dtype), self.loop_x)
            x = self.layers[i](x, run)
            if self.trail is not None:
                self.trail.append(x.clone())
        return rms_norm_f32(x, self.norm, c.eps, self.dtype, offset=1.0)
