"""Small Tukarax configurations with random weights for the tests."""
import torch

from dobedra_cases import all_chosen, for_dtype  # noqa: F401  (shared helpers)
from similorn_cases import tokens, write_model  # noqa: F401


def attention(heads, kv, dim, vdim, chunk, rot, mlp=None, base=10000.0, scaling=None, softcap=20.0, scale=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": {"size": chunk}, "rot": {"base": base, "dims": rot},
         "scale": scale or dim ** -0.5, "softcap": softcap}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": m, "mlp": mlp}


def parallel(left, right, scales, mlp=None, base=10000.0, scale=None):
    """left: heads, kv heads, dim, rotated entries; right: heads, kv heads, dim, vdim, taps."""
    h, g, d, rot = left
    r = dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": h, "kv_heads": g, "dim": d, "vdim": d, "rot": {"base": base, "dims": rot}, "scale": scale or d ** -0.5},
        "left_scale": scales[0], "right": r, "right_scale": scales[1]}}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(layers, width, vocab, eps=1e-5):
    return {"architecture": "Tukarax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# name -> configuration: every branch of the design, sizes that are equal elsewhere kept apart here
CONFIGS = {
    "mixed": config([attention(5, 1, 40, 24, 70, 16, moe(7, 3, 40), scaling=(8.0, 64, 4.0, 0.5)),
                     parallel((4, 2, 48, 20), (6, 2, 40, 56, 4), (0.7, 1.3), moe(5, 2, 24)),
                     attention(4, 2, 32, 48, 33, 32, None, base=500.0, softcap=5.0, scale=0.3),
                     parallel((6, 1, 24, 8), (4, 4, 24, 16, 2), (1.0, 0.4), None, base=1e6)], width=136, vocab=151, eps=1e-3),
    "large_heads": config([parallel((8, 2, 128, 128), (6, 3, 128, 128, 3), (0.8, 0.9), moe(9, 2, 72)),
                           attention(4, 2, 128, 96, 100, 64, moe(6, 1, 48), softcap=45.0, scaling=(2.0, 2048, 32.0, 1.0)),
                           parallel((10, 5, 96, 32), (4, 1, 112, 80, 4), (1.2, 1.0), moe(4, 3, 56))], width=208, vocab=90),
    "wide_state": config([parallel((3, 1, 160, 40), (3, 1, 160, 200, 4), (0.5, 1.0), moe(5, 2, 32)),
                          attention(3, 3, 176, 144, 64, 100, moe(4, 4, 32), softcap=30.0)], width=120, vocab=77),
    # sizes that are not multiples of eight: kernels for any size
    "odd_sizes": config([attention(3, 1, 13, 11, 21, 6, moe(5, 2, 27), softcap=8.0),
                         parallel((3, 3, 9, 4), (6, 3, 7, 5, 5), (0.6, 1.1), moe(3, 1, 10), base=100.0),
                         parallel((2, 1, 15, 14), (1, 1, 11, 19, 3), (1.0, 1.0), None)], width=58, vocab=101, eps=1e-2),
    "one_attention": config([attention(1, 1, 8, 8, 5, 2, moe(1, 1, 8), softcap=None)], width=16, vocab=33),
    "one_parallel": config([parallel((1, 1, 8, 8), (1, 1, 8, 8, 2), (0.5, 0.5), None)], width=24, vocab=35),
}
CONFIGS.update({n + ", all chosen": all_chosen(c) for n, c in list(CONFIGS.items())})


def weights(c, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).to(dtype)
    u = lambda n, lo, hi: (torch.rand(n, generator=g) * (hi - lo) + lo).to(dtype)
    W = c["width"]
    lin = lambda o, i, k=1.0: r(o, i, k=k / i ** 0.5)
    near1 = lambda n: (1 + r(n, k=0.2).float()).to(dtype)
    w = {"embed": r(c["vocab"], W), "head": lin(c["vocab"], W, 3.0), "final.norm": near1(W)}
    for i, e in enumerate(c["layers"]):
        m, p = e["mixer"], f"l{i}."
        w[p + "norm1"] = near1(W)
        if e["type"] == "attention":
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({p + "mix.q": lin(H * d, W, 2.0), p + "mix.k": lin(G * d, W, 1.5), p + "mix.v": lin(G * v, W),
                      p + "mix.sink": r(H), p + "mix.g": lin(H, W, 1.5), p + "mix.o": lin(W, H * v, 2.0)})
        else:
            l, t, q = m["left"], m["right"], p + "mix.left."
            H, G, d = l["heads"], l["kv_heads"], l["dim"]
            w.update({q + "q": lin(H * d, W), q + "k": lin(G * d, W), q + "q.norm": near1(d) * 1.5, q + "k.norm": near1(d),
                      q + "g": lin(H * d, W, 1.5), q + "o": lin(W, H * d, 2.0)})
            q, H, G, d, v = p + "mix.right.", t["heads"], t["kv_heads"], t["dim"], t["vdim"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * v)):
                w[q + n] = lin(rows, W, 1.5)
                w[q + n + ".conv"] = r(rows, t["conv"], k=0.7)
            # decays from nearly none to a few tokens
            w.update({q + "b": lin(H, W, 1.5), q + "a": lin(H, W), q + "A_log": u(H, -3.0, 1.0), q + "dt_bias": u(H, -4.0, 0.5),
                      q + "norm": near1(v), q + "g": lin(H * v, W, 1.5), q + "o": lin(W, H * v, 2.0)})
        f = e["mlp"]
        if f is None:
            continue
        w[p + "norm2"] = near1(W)
        for x in range(f["router"]["experts"]):
            w.update({p + f"mlp.e{x}.gate": lin(f["expert"]["ff"], W, 1.5), p + f"mlp.e{x}.up": lin(f["expert"]["ff"], W, 1.5),
                      p + f"mlp.e{x}.down": lin(W, f["expert"]["ff"], 1.5)})
        # logits far apart: 16-bit and 64-bit forwards choose the same experts except in close calls
        w[p + "mlp.router"] = lin(f["router"]["experts"], W, 2.0)
    return w
