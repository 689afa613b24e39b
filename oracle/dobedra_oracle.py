"""CPU restatement of the Dobedra decoder, one function per mechanism (test infrastructure only).

Written for clarity, not speed: keys and values of every head spelled out, dense masks, one expert at a
time, no cache.  Everything is computed in the dtype of the inputs (float64 unless a caller asks
otherwise), so a comparison shows the error of the kernels and not of this file.  Shares no code with
the product path.
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, b, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def rotate_pairs(x, positions, base):
    """x [T, ..., n]: entries (2i, 2i + 1) of the last dimension turned by p * base^(-2i / n)."""
    n = x.shape[-1]
    out = torch.empty_like(x)
    for i in range(n // 2):
        angle = positions.to(x.dtype) * float(base) ** (-2.0 * i / n)
        c, s = torch.cos(angle), torch.sin(angle)
        for _ in range(x.dim() - 2):
            c, s = c.unsqueeze(-1), s.unsqueeze(-1)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def latent_of(h, w, cfg, positions, eps):
    """What a layer keeps per token: the normed latent [T, kv_rank] and the rotated shared key part [T, rot_dim]."""
    y = h @ w["dkv"].T
    c = rms_norm(y[:, :cfg["kv_rank"]], w["dkv.norm"], eps)
    return c, rotate_pairs(y[:, cfg["kv_rank"]:], positions, cfg["rot"]["base"])


def queries(h, w, cfg, positions, eps):
    """-> unrotated part [T, H, dim], rotated part [T, H, rot_dim]."""
    q = rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T
    q = q.view(len(h), cfg["heads"], cfg["dim"] + cfg["rot_dim"])
    return q[..., :cfg["dim"]], rotate_pairs(q[..., cfg["dim"]:], positions, cfg["rot"]["base"])


def softmax_attention(q, k, v, scale):
    """q [T, H, d], k [S, H, d], v [S, H, vd]; row r of q is the token at position S - T + r.  -> [T, H, vd]."""
    T, S = q.shape[0], k.shape[0]
    s = torch.einsum("thd,shd->hts", q, k) * scale
    ahead = torch.arange(S)[None, :] > torch.arange(S - T, S)[:, None]
    return torch.einsum("hts,shd->thd", torch.softmax(s.masked_fill(ahead[None], float("-inf")), dim=-1), v)


def latent_attention(h, w, cfg, positions, eps, kept=None):
    """`kept`: another layer's (latent, rotated key part), or None.  -> mixer output [T, width], what was kept."""
    H = cfg["heads"]
    c, kr = latent_of(h, w, cfg, positions, eps) if kept is None else kept
    qn, qr = queries(h, w, cfg, positions, eps)
    k = (c @ w["uk"].T).view(len(c), H, cfg["dim"])
    v = (c @ w["uv"].T).view(len(c), H, cfg["vdim"])
    q = torch.cat([qn, qr], dim=-1)
    k = torch.cat([k, kr[:, None, :].expand(-1, H, -1)], dim=-1)
    return softmax_attention(q, k, v, cfg["scale"]).flatten(1) @ w["o"].T, (c, kr)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_ff(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def squared_relu_ff(h, up, down):
    return torch.clamp(h @ up.T, min=0.0) ** 2 @ down.T


def route(logits, top):
    """-> chosen experts [T, top], their softmax scores (over all experts, not renormalised)."""
    s, i = torch.softmax(logits, dim=-1).topk(top, dim=-1)
    return i, s


def mixture_ff(h, w, cfg):
    idx, score = route(h @ w["router"].T, cfg["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(idx[t].tolist(), score[t]):
            out[t] += s * squared_relu_ff(h[t:t + 1], w[f"e{e}.up"], w[f"e{e}.down"])[0]
    if cfg.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * squared_relu_ff(h, w["shared.up"], w["shared.down"])
    return out


def feed_forward(h, w, cfg):
    return gated_ff(h, w) if cfg["kind"] == "dense" else mixture_ff(h, w, cfg)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(config, weights, tokens, dtype=torch.float64):
    """Whole-prompt forward of one sequence.  -> logits [T, vocab], the residual stream after every
    layer (list of [T, width])."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(tokens))
    eps = config["norm"]["eps"]
    x = W["embed"][tokens]
    trail, kept = [], {}
    for li, spec in enumerate(config["layers"]):
        p = f"l{li}."
        part = lambda s: {n[len(p + s):]: t for n, t in W.items() if n.startswith(p + s)}
        if spec["type"] != "latent_attention":
            raise ValueError(spec["type"])
        source = spec["mixer"].get("kv_from")
        a, k = latent_attention(layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps), part("mix."), spec["mixer"],
                                positions, eps, None if source is None else kept[source])
        if source is None:
            kept[li] = k
        new = x + W[p + "ls1"] * a
        if spec["mlp"] is not None:
            new = new + W[p + "ls2"] * feed_forward(layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps), part("mlp."),
                                                    spec["mlp"])
        x = new
        trail.append(x)
    return soft_cap(layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T, config["logit_softcap"]), trail
