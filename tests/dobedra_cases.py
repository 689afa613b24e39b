"""Small Dobedra configurations with random weights for the tests."""
import torch

from similorn_cases import tokens, write_model  # noqa: F401  (shared helpers)


def layer(heads, dim, rot, vdim, q_rank, kv_rank, mlp=None, kv_from=None, base=10000.0, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "rot": {"base": base, "dims": rot}, "scale": scale or (dim + rot) ** -0.5}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=0):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(layers, width, vocab, eps=1e-5, softcap=20.0):
    return {"architecture": "Dobedra", "layers": layers, "logit_softcap": softcap, "norm": {"eps": eps}, "vocab": vocab,
            "width": width}


# name -> configuration: every branch of the design, sizes that are equal elsewhere kept apart here
CONFIGS = {
    "mixed": config([layer(3, 40, 8, 24, 56, 48, dense(72)),
                     layer(5, 32, 8, 48, 40, 48, moe(7, 3, 40, 56), kv_from=0),
                     layer(2, 64, 24, 32, 64, 80, None, base=500.0),
                     layer(4, 24, 8, 72, 48, 48, moe(5, 1, 24, 40), kv_from=0, scale=0.3),
                     layer(6, 16, 24, 16, 32, 80, moe(9, 9, 16, 24), kv_from=2, base=500.0)], width=136, vocab=151),
    "sharing_far_back": config([layer(2, 72, 32, 40, 24, 120, moe(16, 4, 64, 32), base=1e6),
                                layer(2, 48, 16, 88, 72, 96, dense(56)),
                                layer(1, 80, 16, 120, 40, 96, dense(48), kv_from=1),
                                layer(3, 56, 32, 64, 32, 120, moe(6, 2, 48), kv_from=0, base=1e6),
                                layer(9, 32, 16, 24, 48, 96, None, kv_from=1)], width=104, vocab=97, eps=1e-2, softcap=5.0),
    "large_heads": config([layer(20, 128, 64, 128, 96, 256, moe(11, 2, 72, 128)),
                           layer(40, 64, 64, 96, 64, 256, dense(128), kv_from=0)], width=192, vocab=90, softcap=30.0),
    # sizes that are not multiples of eight: kernels for any size
    "odd_sizes": config([layer(3, 13, 6, 11, 21, 19, moe(5, 2, 27, 13)), layer(2, 9, 6, 15, 17, 19, dense(23), kv_from=0),
                         layer(1, 7, 10, 5, 9, 33, moe(3, 1, 10, 7), base=100.0)], width=58, vocab=101),
    "one_layer": config([layer(1, 8, 2, 8, 8, 8, moe(1, 1, 8, 8))], width=16, vocab=33, softcap=None),
}


def weights(c, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).to(dtype)
    W = c["width"]
    lin = lambda o, i, k=1.0: r(o, i, k=k / i ** 0.5)
    near1 = lambda n: (1 + r(n, k=0.2).float()).to(dtype)
    w = {"embed": r(c["vocab"], W), "head": lin(c["vocab"], W, 3.0), "final.norm": near1(W), "final.norm.b": r(W, k=0.2)}
    for i, e in enumerate(c["layers"]):
        m, p = e["mixer"], f"l{i}."
        H, R = m["heads"], m["kv_rank"]
        w.update({p + "norm1": near1(W), p + "norm1.b": r(W, k=0.2), p + "ls1": near1(W),
                  p + "mix.dq": lin(m["q_rank"], W), p + "mix.dq.norm": near1(m["q_rank"]),
                  p + "mix.uq": lin(H * (m["dim"] + m["rot_dim"]), m["q_rank"], 2.0),
                  p + "mix.uk": lin(H * m["dim"], R, 1.5), p + "mix.uv": lin(H * m["vdim"], R),
                  p + "mix.o": lin(W, H * m["vdim"], 1.5)})
        if "kv_from" not in m:
            w[p + "mix.dkv"] = lin(R + m["rot_dim"], W, 1.5)
            w[p + "mix.dkv.norm"] = near1(R)
        f = e["mlp"]
        if f is None:
            continue
        w.update({p + "norm2": near1(W), p + "norm2.b": r(W, k=0.2), p + "ls2": near1(W)})
        if f["kind"] == "dense":
            w.update({p + "mlp.gate": lin(f["ff"], W), p + "mlp.up": lin(f["ff"], W), p + "mlp.down": lin(W, f["ff"])})
        else:
            for x in range(f["router"]["experts"]):
                w[p + f"mlp.e{x}.up"] = lin(f["expert"]["ff"], W)
                w[p + f"mlp.e{x}.down"] = lin(W, f["expert"]["ff"])
            # logits far apart: 16-bit and 64-bit forwards choose the same experts except in close calls
            w[p + "mlp.router"] = lin(f["router"]["experts"], W, 3.0)
            if f.get("shared"):
                w.update({p + "mlp.shared.up": lin(f["shared"]["ff"], W), p + "mlp.shared.down": lin(W, f["shared"]["ff"]),
                          p + "mlp.shared.sg": lin(1, W, 2.0)})
    return w


def all_chosen(c):
    """The configuration with every expert chosen: its forward is continuous, so 16-bit rounding cannot turn a close
    call of the router into another expert's output."""
    def one(e):
        f = e["mlp"]
        return {**e, "mlp": {**f, "router": {**f["router"], "top": f["router"]["experts"]}}} if f and f["kind"] == "moe" else e
    return {**c, "layers": [one(e) for e in c["layers"]]}


CONFIGS.update({n + ", all chosen": all_chosen(c) for n, c in list(CONFIGS.items())})


def for_dtype(name, dtype):
    return name if dtype == torch.float32 else name + ", all chosen"
