"""Dobedra: a decoder of latent attention and mixtures of experts with an fp32 residual stream.

A layer's mixer and feed-forward read the same x through two layer norms, and both results, each with its
layer scale, are added to it; the launch that adds them also takes the norms of the next layer
(`join_norms`), so x crosses memory once per layer.  A layer may keep no latents of its own and attend to an
earlier layer's.  The configuration names every layer on its own.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
from torch import nn

from ..engine.cache import LatentSpec
from ..layers.feed_forward import GatedFF, MixtureFF
from ..layers.latent_attention import LatentAttentionMixer
from ..layers.row_ops import embed_position, join_norms
from ..utils.context import get_context


@dataclass(frozen=True)
class LayerConfig:
    mixer: dict
    mlp: dict | None


@dataclass(frozen=True)
class DobedraConfig:
    vocab: int
    width: int
    eps: float
    softcap: float       # of the logits, 0 = none
    layers: tuple

    @classmethod
    def from_dict(cls, c):
        layers = []
        for i, e in enumerate(c["layers"]):
            mix, mlp = dict(e["mixer"]), e.get("mlp")
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            if mix["rot"]["dims"] != mix["rot_dim"] or mix["rot_dim"] % 2:
                raise ValueError(f"layer {i}: {mix['rot']['dims']} rotated dimensions of {mix['rot_dim']}")
            j = mix.get("kv_from")
            if j is not None:
                if not 0 <= j < i or layers[j].mixer.get("kv_from") is not None:
                    raise ValueError(f"layer {i}: layer {j} keeps no latents before it")
                src = layers[j].mixer
                if any(src[k] != mix[k] for k in ("kv_rank", "rot_dim", "rot")):
                    raise ValueError(f"layer {i}: its latent sizes or rotation are not those of layer {j}")
            if mlp is not None and mlp["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerConfig(mix, None if mlp is None else dict(mlp)))
        return cls(int(c["vocab"]), int(c["width"]), float(c["norm"]["eps"]), float(c.get("logit_softcap") or 0.0),
                   tuple(layers))


class DobedraLayer(nn.Module):
    def __init__(self, c: DobedraConfig, lc: LayerConfig, dtype, device, side=None):
        super().__init__()
        m, f = lc.mixer, lc.mlp
        self.kv_from = m.get("kv_from")
        self.mixer = LatentAttentionMixer(c.width, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"],
                                          m["rot"]["base"], m["scale"], c.eps, self.kv_from is not None, dtype, device)
        if f is None:
            self.ff = None
        elif f["kind"] == "dense":
            self.ff = GatedFF(c.width, f["ff"], dtype, device)
        else:
            self.ff = MixtureFF(c.width, f["router"]["experts"], f["router"]["top"], f["expert"]["ff"],
                                (f.get("shared") or {}).get("ff", 0), dtype, device)
        v = lambda: nn.Parameter(torch.empty(c.width, dtype=torch.float32, device=device), requires_grad=False)
        self.side = side
        self.norm1, self.bias1, self.scale1 = v(), v(), v()
        self.norm2, self.bias2, self.scale2 = (v(), v(), v()) if self.ff is not None else (None, None, None)

    def load(self, get):
        self.norm1.copy_(get("norm1"))
        self.bias1.copy_(get("norm1.b"))
        self.scale1.copy_(get("ls1"))
        self.mixer.load(lambda n: get("mix." + n))
        if self.ff is not None:
            self.norm2.copy_(get("norm2"))
            self.bias2.copy_(get("norm2.b"))
            self.scale2.copy_(get("ls2"))
            self.ff.load(lambda n: get("mlp." + n))

    def norms(self):
        """What the launch ahead of this layer takes of x."""
        return [(self.norm1, self.bias1)] + ([(self.norm2, self.bias2)] if self.ff is not None else [])

    def forward(self, h, positions):
        """h: the outputs of `norms`.  -> this layer's summands, as `join_norms` takes them."""
        parts = {"ls_a": self.scale1, "ls_b": self.scale2}
        if self.ff is not None and self.side is not None and not get_context().is_prefill:
            # a decode step's launches are short: the two sublayers run side by side (the next layer's fork waits for
            # this layer's boundary, so memory that crosses the streams is not reused before its last reader)
            main = torch.cuda.current_stream()
            self.side.wait_stream(main)
            with torch.cuda.stream(self.side):
                parts.update(self.ff(h[1]))
            parts["a"] = self.mixer(h[0], positions)
            main.wait_stream(self.side)
            return parts
        if self.ff is not None:
            parts.update(self.ff(h[1]))
        parts["a"] = self.mixer(h[0], positions)
        return parts


class DobedraModel(nn.Module):
    fp32_logits = True   # the engine keeps this model's logits in fp32

    def __init__(self, c: DobedraConfig, dtype, device):
        super().__init__()
        self.config, self.dtype, self.logit_softcap = c, dtype, c.softcap
        e = lambda *s, dt=dtype: nn.Parameter(torch.empty(*s, dtype=dt, device=device), requires_grad=False)
        self.embed = e(c.vocab, c.width)
        side = torch.cuda.Stream(device) if device.type == "cuda" else None
        self.layers = nn.ModuleList([DobedraLayer(c, lc, dtype, device, side) for lc in c.layers])
        self.norm, self.norm_bias = e(c.width, dt=torch.float32), e(c.width, dt=torch.float32)
        self.head = e(c.vocab, c.width)
        self.trail = None      # optional list: the residual stream after every layer

    @torch.no_grad()
    def load_weights(self, w):
        self.embed.copy_(w["embed"])
        self.head.copy_(w["head"])
        self.norm.copy_(w["final.norm"])
        self.norm_bias.copy_(w["final.norm.b"])
        for i, layer in enumerate(self.layers):
            layer.load(lambda n, p=f"l{i}.": w[p + n])

    def cache_spec(self):
        """What each layer with latents of its own keeps, in order."""
        return [LatentSpec(l.mixer.kv_rank, l.mixer.rot) for l in self.layers if l.kv_from is None]

    def bind_cache(self, cache):
        entries = iter(cache.entries)
        for layer in self.layers:
            layer.mixer.cache = next(entries)[0] if layer.kv_from is None else self.layers[layer.kv_from].mixer.cache

    def forward(self, input_ids, positions):
        c = self.config
        final = [(self.norm, self.norm_bias)]
        after = [layer.norms() for layer in self.layers] + [final]
        x = embed_position(input_ids, positions, self.embed, 1.0)
        h = join_norms(x, after[0], c.eps, self.dtype)
        for layer, norms in zip(self.layers, after[1:]):
            h = join_norms(x, norms, c.eps, self.dtype, **layer(h, positions))
            if self.trail is not None:
                self.trail.append(x.clone())
        return h[0]
