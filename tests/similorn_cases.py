"""Small Similorn configurations with random weights for the tests."""
import json
import struct
from pathlib import Path

import torch


def mlstm(heads, dim, vdim, cap=10.0, ff=0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention(heads, kv_heads, dim, vdim, window, softcap=15.0, scale=None, ff=0):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                           "scale": scale or dim ** -0.5, "softcap": softcap, "mask": {"size": window}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width, vocab, loop=None, eps=1e-5, embed_scale=2.0):
    c = {"architecture": "Similorn", "embedding": {"scale": embed_scale}, "layers": layers,
         "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# name -> configuration: every branch of the design, sizes that are equal elsewhere kept apart here
CONFIGS = {
    "mixed": config([mlstm(3, 24, 40), attention(6, 2, 40, 56, 70, ff=200), mlstm(2, 48, 32, cap=4.0, ff=96)],
                    width=96, vocab=151, loop=(0, 2, 2)),
    "loop_in_the_middle": config([attention(4, 4, 16, 24, 33), mlstm(1, 64, 72, ff=80), attention(4, 1, 32, 16, 130, softcap=40.0, ff=64),
                                  mlstm(4, 16, 16)], width=132, vocab=97, loop=(1, 3, 3), eps=1e-3, embed_scale=1.0),
    "no_loop": config([mlstm(2, 32, 96), attention(8, 8, 20, 36, 1, ff=72), attention(2, 1, 64, 128, 64, softcap=5.0)],
                      width=80, vocab=64),
    "one_pass_over_all": config([attention(5, 5, 48, 16, 65, softcap=30.0, ff=40), mlstm(2, 20, 28, cap=30.0)], width=72,
                                vocab=203, loop=(0, 2, 1), embed_scale=9.5),
    # head sizes of the tcgen05 kernels
    "large_heads": config([mlstm(1, 128, 128), attention(2, 1, 128, 128, 100, softcap=30.0, ff=64), mlstm(2, 128, 256)], width=64,
                          vocab=90, loop=(1, 3, 2)),
    "odd_sizes": config([mlstm(3, 17, 23), attention(3, 1, 13, 19, 77, ff=61)], width=58, vocab=101, loop=(1, 2, 2)),
}


def weights(c, seed=0, dtype=torch.bfloat16):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s, k=1.0: (torch.randn(*s, generator=g) * k).to(dtype)
    W = c["width"]
    lin = lambda o, i, k=1.0: r(o, i, k=k / i ** 0.5)
    w = {"embed": r(c["vocab"], W), "head": lin(c["vocab"], W), "final.norm": r(W, k=0.2)}
    if "loop" in c:
        w["loop.in"] = lin(W, 2 * W, 1.2)
    for i, e in enumerate(c["layers"]):
        m, p = e["mixer"], f"l{i}."
        w[p + "norm1"] = r(W, k=0.2)
        if e["type"] == "mlstm":
            H, dk, dv = m["heads"], m["dim"], m["vdim"]
            w.update({p + "mix.q": lin(H * dk, W), p + "mix.k": lin(H * dk, W), p + "mix.v": lin(H * dv, W),
                      p + "mix.g": lin(H * dv, W), p + "mix.o": lin(W, H * dv, 1.5),
                      p + "mix.norm": (1 + r(H * dv, k=0.2).float()).to(dtype),
                      p + "mix.i": lin(H, W), p + "mix.i.b": r(H, k=0.5), p + "mix.f": lin(H, W, 2.0),
                      p + "mix.f.b": (r(H).float() + 3.0).to(dtype)})
        else:
            H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            w.update({p + "mix.q": lin(H * dk, W, 2.0), p + "mix.k": lin(G * dk, W, 1.5), p + "mix.v": lin(G * dv, W),
                      p + "mix.o": lin(W, H * dv, 2.0)})
        if e["mlp"]:
            w[p + "norm2"] = r(W, k=0.2)
            w[p + "mlp.up"] = lin(e["mlp"]["ff"], W)
            w[p + "mlp.down"] = lin(W, e["mlp"]["ff"])
    return w


def write_safetensors(path, tensors):
    header, blobs, at = {}, [], 0
    code = {torch.bfloat16: "BF16", torch.float32: "F32", torch.int32: "I32"}
    for n, t in tensors.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes() if t.numel() else b""
        header[n] = {"dtype": code[t.dtype], "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    h = json.dumps(header).encode()
    Path(path).write_bytes(struct.pack("<Q", len(h)) + h + b"".join(blobs))


def write_model(folder, c, w):
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(c))
    write_safetensors(folder / "model.safetensors", w)
    return folder


def tokens(c, n, seed=0):
    return torch.randint(0, c["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
