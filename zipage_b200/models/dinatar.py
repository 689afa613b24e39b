"""Dinatar: a decoder of linear-attention layers (HGRN2, gated linear attention) and of layers that run windowed attention with distance
biases beside a state-space mixer, with learned positions, tied embeddings and a run of layers that is repeated.

Mixer and feed-forward of a layer read the same layer norm of the fp32 residual stream; the launch that adds both results
(`join_norms`) also norms the two halves of a parallel mixer and takes the norm that the next layer reads.  The configuration
names every layer on its own; a layer inside the repeated run keeps one cache or state per pass.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..engine.cache import KVSpec, LinearStateSpec
from ..layers.attention import WindowAttentionMixer, distance_slopes
from ..layers.feed_forward import GatedMixtureFF, SquaredReluFF
from ..layers.linear_state import GLAMixer, HGRN2Mixer, SSDMixer
from ..layers.row_ops import embed_position, join_norms, project
from ..utils.context import get_context


@dataclass(frozen=True)
class LayerConfig:
    type: str            # "hgrn2", "gla" or "parallel"
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class DinatarConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    logit_scale: float
    max_positions: int
    layers: tuple
    loop: tuple          # (start, stop, times); (0, 0, 0) = no layer is repeated

    @classmethod
    def from_dict(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            mix, mlp = dict(e["mixer"]), e.get("mlp")
            if e["type"] not in ("hgrn2", "gla", "parallel"):
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            if mlp is not None and mlp["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            if e["type"] == "parallel":
                l, r = mix["left"], mix["right"]
                if l["heads"] % l["kv_heads"]:
                    raise ValueError(f"layer {i}: {l['heads']} heads over {l['kv_heads']} key/value heads")
                if r["heads"] % r["groups"]:
                    raise ValueError(f"layer {i}: {r['heads']} heads in {r['groups']} groups")
                if r["heads"] * r["vdim"] % r["norm_groups"]:
                    raise ValueError(f"layer {i}: {r['heads'] * r['vdim']} entries normed in {r['norm_groups']} parts")
            if mlp is not None and mlp["kind"] == "moe" and not 0 < mlp["router"]["top"] <= mlp["router"]["experts"]:
                raise ValueError(f"layer {i}: {mlp['router']['top']} of {mlp['router']['experts']} experts")
            layers.append(LayerConfig(e["type"], mix, None if mlp is None else dict(mlp)))
        lp = c.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else (0, 0, 0)
        if not 0 <= loop[0] <= loop[1] <= len(layers):
            raise ValueError(f"loop {loop} over {len(layers)} layers")
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c["embedding"]["scale"]), float(c["logit_scale"]),
                   int(c["max_positions"]), tuple(layers), loop)

    def runs(self):
        """The forward's layer runs in order: (layer, pass)."""
        a, b, times = self.loop
        if a == b:
            return [(i, 0) for i in range(len(self.layers))]
        return [(i, 0) for i in range(a)] + [(i, t) for t in range(times) for i in range(a, b)] + [(i, 0) for i in range(b, len(self.layers))]


class DinatarLayer(nn.Module):
    """`rank`: of a gla layer's decay projection."""

    def __init__(self, c: DinatarConfig, lc: LayerConfig, rank, dtype, device, sides=(None, None)):
        super().__init__()
        m, f, self.sides = lc.mixer, lc.mlp, sides
        v = lambda: nn.Parameter(torch.empty(c.width, dtype=torch.float32, device=device), requires_grad=False)
        if lc.type == "hgrn2":
            mixers = [("", HGRN2Mixer(c.width, m["heads"], m["dim"], m["vdim"], c.eps, dtype, device))]
        elif lc.type == "gla":
            mixers = [("", GLAMixer(c.width, m["heads"], m["dim"], m["vdim"], rank, m["tau"], c.eps, dtype, device))]
        else:
            l, r = m["left"], m["right"]
            mask = l.get("mask") or {}
            mixers = [("left.", WindowAttentionMixer(c.width, l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["scale"], 0.0,
                                                     int(mask.get("size") or 0), dtype, device, keep=int(mask.get("keep_first") or 0),
                                                     slopes=distance_slopes(l["heads"]), bias=True)),
                      ("right.", SSDMixer(c.width, r["heads"], r["groups"], r["state"], r["vdim"], r["conv"], r["norm_groups"], c.eps, dtype,
                                          device))]
        self.prefixes, self.mixers = [p for p, _ in mixers], nn.ModuleList([x for _, x in mixers])
        self.mix_norms = nn.ParameterList([v() for _ in mixers] if len(mixers) == 2 else [])
        if f is None:
            self.ff = None
        elif f["kind"] == "dense":
            self.ff = SquaredReluFF(c.width, f["ff"], dtype, device)
        else:
            self.ff = GatedMixtureFF(c.width, f["router"]["experts"], f["router"]["top"], f["expert"]["ff"], dtype, device, score="softmax_top",
                                     weigh="output", bias=True, shared_ff=(f.get("shared") or {}).get("ff", 0))
        self.norm, self.norm_bias = v(), v()

    def load(self, get):
        self.norm.copy_(get("norm1"))
        self.norm_bias.copy_(get("norm1.b"))
        for p, x in zip(self.prefixes, self.mixers):
            x.load(lambda n: get("mix." + p + n))
        for p, w in zip(self.prefixes, self.mix_norms):
            w.copy_(get("mix." + p + "out"))
        if self.ff is not None:
            self.ff.load(lambda n: get("mlp." + n))

    def forward(self, h, run):
        """h: the layer's norm of x.  -> this layer's summands, as `join_norms` takes them."""
        mix = lambda x: project(x(h, run), x.out_proj)
        jobs = [lambda x=x: mix(x) for x in self.mixers] + ([] if self.ff is None else [lambda: self.ff(h)])
        if len(jobs) > 1 and self.sides[0] is not None and not get_context().is_prefill:
            # a decode step's launches are short: mixers and feed-forward run side by side (the next layer's fork waits for
            # this layer's boundary, so memory that crosses the streams is not reused before its last reader)
            main, out = torch.cuda.current_stream(), [None] * len(jobs)
            for i, side in zip(range(1, len(jobs)), self.sides):
                side.wait_stream(main)
                with torch.cuda.stream(side):
                    out[i] = jobs[i]()
            out[0] = jobs[0]()
            for _, side in zip(jobs[1:], self.sides):
                main.wait_stream(side)
        else:
            out = [j() for j in jobs]
        parts = dict(out.pop()) if self.ff is not None else {}
        if len(out) == 2:
            parts["pair"] = tuple(zip(out, self.mix_norms))
        else:
            parts["a"] = out[0]
        return parts


class DinatarModel(nn.Module):
    fp32_logits = True   # the engine keeps this model's logits in fp32

    def __init__(self, c: DinatarConfig, dtype, device, ranks=None):
        """ranks: layer -> rank of its decays' projection (gla layers)."""
        super().__init__()
        self.config, self.dtype, self.max_positions = c, dtype, c.max_positions
        e = lambda *s, dt=dtype: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.embed, self.pos = e(c.vocab, c.width), e(c.max_positions, c.width)
        sides = tuple(torch.cuda.Stream(device) if device.type == "cuda" else None for _ in range(2))
        self.layers = nn.ModuleList([DinatarLayer(c, lc, (ranks or {}).get(i, 0), dtype, device, sides) for i, lc in enumerate(c.layers)])
        # the scale of the logits is part of the last norm's weights, in fp32
        self.norm, self.norm_bias = e(c.width, dt=torch.float32), e(c.width, dt=torch.float32)
        self.runs = c.runs()
        self.trail = None      # optional list: the residual stream after every layer run

    @property
    def head(self):
        return self.embed

    @staticmethod
    def ranks_of(weights):
        """What the configuration does not give: rank of the decays' projection, layer by layer."""
        return {int(n[1:].split(".")[0]): w.shape[0] for n, w in weights.items() if n.endswith(".mix.a1")}

    @torch.no_grad()
    def load_weights(self, w):
        self.embed.copy_(w["embed"])
        self.pos.copy_(w["pos"])
        for p, name in ((self.norm, "final.norm"), (self.norm_bias, "final.norm.b")):
            p.copy_(w[name].float() * self.config.logit_scale)
        for i, layer in enumerate(self.layers):
            layer.load(lambda n, p=f"l{i}.": w[p + n])

    def _mixers(self):
        """Mixers of every layer run in order."""
        return [x for i, _ in self.runs for x in self.layers[i].mixers]

    def cache_spec(self):
        """What each mixer keeps in each layer run, in order."""
        out = []
        for x in self._mixers():
            if isinstance(x, WindowAttentionMixer):
                out.append(KVSpec(x.kv_heads, x.dim, x.vdim))
            elif isinstance(x, SSDMixer):
                out.append(LinearStateSpec(x.heads, x.dim, x.vdim, x.channels, x.conv.shape[0]))
            else:
                out.append(LinearStateSpec(x.heads, x.dim, x.vdim))
        return out

    def bind_cache(self, cache):
        kept = lambda x: "caches" if isinstance(x, WindowAttentionMixer) else "states"
        for x in self._mixers():
            setattr(x, kept(x), [])
        for x, entry in zip(self._mixers(), cache.entries):
            getattr(x, kept(x)).append(entry)

    def forward(self, input_ids, positions):
        c = self.config
        norm_of = lambda m: [(m.norm, m.norm_bias)]
        x = embed_position(input_ids, positions, self.embed, c.embed_scale, learned=self.pos)
        order = [self.layers[i] for i, _ in self.runs]
        h = join_norms(x, norm_of(order[0] if order else self), c.eps, self.dtype)[0]
        for (_, run), layer, after in zip(self.runs, order, order[1:] + [self]):
            h = join_norms(x, norm_of(after), c.eps, self.dtype, **layer(h, run))[0]
            if self.trail is not None:
                self.trail.append(x.clone())
        return h
