"""Small Dinatar configurations with random weights for the tests."""
import torch

from dobedra_cases import all_chosen, for_dtype  # noqa: F401  (shared helpers)
from similorn_cases import tokens, write_model  # noqa: F401


def hgrn2(heads, dim, vdim, mlp=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": mlp}


def gla(heads, dim, vdim, tau, rank, mlp=None):
    """rank: of the decays' projection (a shape, not part of the configuration)."""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp, "rank": rank}


def parallel(left, right, mlp=None, scale=None):
    """left: heads, kv heads, dim, vdim, window, kept tokens; right: heads, groups, state, vdim, taps, norm groups."""
    l = dict(zip(("heads", "kv_heads", "dim", "vdim"), left))
    l.update(mask={"size": left[4], "keep_first": left[5]}, scale=scale or left[2] ** -0.5)
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": l, "right": dict(zip(("heads", "groups", "state", "vdim", "conv", "norm_groups"), right))}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return m | ({"shared": {"ff": shared}} if shared else {})


RANKS = {}


def config(name, layers, width, vocab, eps=1e-5, loop=None, embed=1.0, logits=1.0, positions=600):
    """The ranks of `gla` layers are kept beside the configuration, by name."""
    RANKS[name] = {i: e["rank"] for i, e in enumerate(layers) if "rank" in e}
    layers = [{k: v for k, v in e.items() if k != "rank"} for e in layers]
    return {"architecture": "Dinatar", "name": name, "embedding": {"scale": embed}, "layers": layers, "logit_scale": logits,
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None, "max_positions": positions, "norm": {"eps": eps},
            "vocab": vocab, "width": width}


_ALL = [
    config("mixed", [gla(3, 40, 24, 8.0, 12, moe(7, 3, 40, 56)), parallel((6, 2, 40, 24, 70, 5), (4, 2, 24, 56, 3, 1), moe(5, 2, 24)),
                     hgrn2(5, 24, 40, dense(72)), parallel((5, 1, 24, 48, 33, 65), (6, 1, 40, 16, 4, 3), None, scale=0.3),
                     hgrn2(2, 56, 32, None), gla(2, 16, 72, 1.0, 24, dense(40))],
           width=136, vocab=151, eps=1e-3, loop=(1, 3, 3), embed=3.0, logits=0.5),
    config("large_heads", [hgrn2(3, 128, 128, moe(9, 2, 72, 40)), parallel((4, 2, 128, 96, 100, 3), (4, 4, 128, 128, 2, 4), dense(96)),
                           gla(2, 96, 200, 16.0, 32, moe(6, 1, 48, 24)), parallel((8, 4, 112, 128, 128, 64), (2, 1, 96, 136, 4, 1), None)],
           width=208, vocab=90, loop=(0, 4, 2), logits=2.0),
    config("wide_state", [gla(1, 160, 40, 4.0, 8, dense(48)), parallel((3, 3, 176, 144, 64, 1), (3, 3, 136, 24, 4, 2), moe(4, 4, 32, 16)),
                          hgrn2(2, 200, 64, None)], width=120, vocab=77),
    # sizes that are not multiples of eight: kernels for any size
    config("odd_sizes", [hgrn2(3, 9, 7, moe(5, 2, 27, 11)), gla(2, 7, 13, 3.0, 5, dense(19)),
                         parallel((3, 1, 13, 11, 21, 2), (6, 3, 5, 7, 5, 3), moe(3, 1, 10)), parallel((2, 2, 15, 9, 40, 1), (1, 1, 11, 19, 1, 1), None)],
           width=58, vocab=101, eps=1e-2, loop=(1, 2, 2), embed=0.5),
    config("one_hgrn2", [hgrn2(1, 8, 8, None)], width=16, vocab=33),
    config("one_gla", [gla(1, 8, 8, 2.0, 1, moe(1, 1, 8, 8))], width=24, vocab=35),
    config("one_parallel", [parallel((1, 1, 8, 8, 5, 1), (1, 1, 8, 8, 2, 1), dense(8))], width=24, vocab=35, loop=(0, 1, 1)),
]
# name -> configuration: every branch of the design, sizes that are equal elsewhere kept apart here
CONFIGS = {c["name"]: c for c in _ALL}
CONFIGS.update({n + ", all chosen": all_chosen(c) for n, c in list(CONFIGS.items())})


def weights(c, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).to(dtype)
    u = lambda n, lo, hi: (torch.rand(n, generator=g) * (hi - lo) + lo).to(dtype)
    W = c["width"]
    lin = lambda o, i, k=1.0: r(o, i, k=k / i ** 0.5)
    near1 = lambda n: (1 + r(n, k=0.2).float()).to(dtype)
    w = {"embed": r(c["vocab"], W), "pos": r(c["max_positions"], W, k=0.5), "final.norm": near1(W), "final.norm.b": r(W, k=0.2)}
    for i, e in enumerate(c["layers"]):
        m, p = e["mixer"], f"l{i}."
        w.update({p + "norm1": near1(W), p + "norm1.b": r(W, k=0.2)})
        q = p + "mix."
        if e["type"] == "hgrn2":
            H, d, v = m["heads"], m["dim"], m["vdim"]
            w.update({q + "q": lin(H * d, W, 1.5), q + "f": lin(H * d, W, 2.0), q + "f.b": r(H * d) + 1, q + "lower": u(H * d, 0.0, 0.95),
                      q + "v": lin(H * v, W), q + "norm": near1(v), q + "o": lin(W, H * v, 1.5)})
        elif e["type"] == "gla":
            H, d, v, rank = m["heads"], m["dim"], m["vdim"], RANKS[c["name"]][i]
            w.update({q + "q": lin(H * d, W, 1.5), q + "k": lin(H * d, W, 1.5), q + "v": lin(H * v, W), q + "g": lin(H * v, W, 1.5),
                      q + "o": lin(W, H * v, 2.0), q + "norm": near1(v), q + "a1": lin(rank, W, 2.0), q + "a2": lin(H * d, rank, 2.0),
                      q + "a2.b": r(H * d)})
        else:
            l, t, s = m["left"], m["right"], q + "left."
            H, G, d, v = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            for n, rows, k in (("q", H * d, 2.0), ("k", G * d, 1.5), ("v", G * v, 1.0)):
                w.update({s + n: lin(rows, W, k), s + n + ".b": r(rows, k=0.5)})
            w.update({s + "o": lin(W, H * v, 2.0), s + "out": near1(W)})
            H, G, N, v, s = t["heads"], t["groups"], t["state"], t["vdim"], q + "right."
            ch = H * v + 2 * G * N
            # decays from nearly none to a few tokens
            w.update({s + "in": lin(2 * H * v + 2 * G * N + H, W, 1.5), s + "conv": r(ch, t["conv"], k=0.7), s + "conv.b": r(ch, k=0.3),
                      s + "dt_bias": u(H, -4.0, 0.5), s + "A_log": u(H, -3.0, 1.0), s + "D": r(H), s + "norm": near1(H * v),
                      s + "o": lin(W, H * v, 2.0), s + "out": near1(W)})
        f = e["mlp"]
        if f is None:
            continue
        if f["kind"] == "dense":
            w.update({p + "mlp.up": lin(f["ff"], W), p + "mlp.down": lin(W, f["ff"])})
            continue
        blocks = [(f"e{x}.", f["expert"]["ff"]) for x in range(f["router"]["experts"])] + ([("shared.", f["shared"]["ff"])] if "shared" in f else [])
        for n, ff in blocks:
            w.update({p + f"mlp.{n}gate": lin(ff, W, 1.5), p + f"mlp.{n}up": lin(ff, W, 1.5), p + f"mlp.{n}down": lin(W, ff, 1.5)})
        # logits far apart: 16-bit and 64-bit forwards choose the same experts except in close calls
        w.update({p + "mlp.router": lin(f["router"]["experts"], W, 2.0), p + "mlp.router.b": r(f["router"]["experts"])})
    return w
