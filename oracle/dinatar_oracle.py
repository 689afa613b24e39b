"""CPU restatement of the Dinatar decoder, one function per mechanism (test infrastructure only).

Written for clarity, not speed: dense masks, one recurrence step per token, one expert at a time, no cache.
Everything is computed in the dtype of the inputs (float64 unless a caller asks otherwise), so a comparison
shows the error of the kernels and not of this file.  Shares no code with the product path.
"""
from __future__ import annotations

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


# -- attention with distance biases ------------------------------------------------------------------
def visible(T, S, window=0, first=0):
    """[T, S]: whether row r, at position S - T + r, sees key j: the last `window` positions and the first `first`."""
    p, j = torch.arange(S - T, S)[:, None], torch.arange(S)[None, :]
    near = p - j < window if window else torch.ones(T, S, dtype=torch.bool)
    return (j <= p) & (near | (j < first))


def slopes(heads, dtype=torch.float64):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=dtype)


def biased_attention(q, k, v, scale, window=0, first=0, slope=None):
    """q [T, H, d], k [S, G, d], v [S, G, vd], slope [H] or None; the rows of q are the newest tokens.  -> [T, H, vd]."""
    T, H = q.shape[:2]
    S, G = k.shape[:2]
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("thd,shd->hts", q, k) * scale
    if slope is not None:
        distance = torch.arange(S - T, S)[:, None] - torch.arange(S)[None, :]
        s = s - slope[:, None, None] * distance[None].to(s.dtype)
    s = s.masked_fill(~visible(T, S, window, first)[None], float("-inf"))
    return torch.einsum("hts,shd->thd", torch.softmax(s, dim=-1), v)


def attention_mixer(h, w, m):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    lin = lambda n: h @ w[n].T + w[n + ".b"]
    q, k, v = lin("q").view(T, H, m["dim"]), lin("k").view(T, G, m["dim"]), lin("v").view(T, G, m["vdim"])
    o = biased_attention(q, k, v, m["scale"], m["mask"]["size"], m["mask"]["keep_first"], slopes(H, h.dtype))
    return o.flatten(1) @ w["o"].T


# -- recurrences whose state decays and takes an outer product per token ---------------------------------
def decayed_recurrence(q, k, v, a, S=None):
    """S <- diag(a) S + k v^T, o = S^T q.  q, k, a [T, H, dim], v [T, H, vdim], S [H, dim, vdim] or None.
    -> o [T, H, vdim], S after the last token."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        S = a[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def hgrn2_gates(z, bias, lower):
    """z [T, H * dim] -> forget gates."""
    return lower + (1 - lower) * torch.sigmoid(z + bias)


def hgrn2_mixer(h, w, m, eps):
    T, H, d = len(h), m["heads"], m["dim"]
    f = hgrn2_gates(h @ w["f"].T, w["f.b"], w["lower"]).view(T, H, d)
    q, v = silu(h @ w["q"].T).view(T, H, d), (h @ w["v"].T).view(T, H, m["vdim"])
    o, _ = decayed_recurrence(q, 1 - f, v, f)
    return (rms(o, eps) * w["norm"]).flatten(1) @ w["o"].T


def gla_decay(z, tau):
    return torch.sigmoid(z) ** (1.0 / tau)


def gla_mixer(h, w, m, eps):
    T, H, d = len(h), m["heads"], m["dim"]
    a = gla_decay((h @ w["a1"].T) @ w["a2"].T + w["a2.b"], m["tau"]).view(T, H, d)
    q, k = (h @ w["q"].T).view(T, H, d) * d ** -0.5, (h @ w["k"].T).view(T, H, d)
    o, _ = decayed_recurrence(q, k, (h @ w["v"].T).view(T, H, m["vdim"]), a)
    return ((rms(o, eps) * w["norm"]).flatten(1) * silu(h @ w["g"].T)) @ w["o"].T


def short_conv(x, w, bias, before=None):
    """x [T, channels], w [channels, taps] -> silu of the causal convolution; `before`: the taps - 1 inputs ahead of x."""
    taps = w.shape[1]
    if before is None:
        before = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    x = torch.cat([before, x])
    out = bias.expand(len(x) - taps + 1, -1).clone()
    for t in range(len(out)):
        for j in range(taps):
            out[t] += w[:, j] * x[t + j]
    return silu(out)


def ssd_mixer(h, w, m, eps):
    """State-space duality: one decay per head and token, keys and queries shared by groups of heads."""
    T, H, vd, N, G = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * vd
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=1)
    x, B, C = torch.split(short_conv(xbc, w["conv"], w["conv.b"]), [inner, G * N, G * N], dim=1)
    x = x.view(T, H, vd)
    B, C = (t.view(T, G, N).repeat_interleave(H // G, dim=1) for t in (B, C))
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    a = torch.exp(-torch.exp(w["A_log"]) * dt)
    y, _ = decayed_recurrence(C, B * dt[:, :, None], x, a[:, :, None].expand(T, H, N))
    y = (y + w["D"][:, None] * x).flatten(1) * silu(z)
    parts = m["norm_groups"]
    return (rms(y.view(T, parts, inner // parts), eps).flatten(1) * w["norm"]) @ w["o"].T


def parallel_mixer(h, w, m, eps):
    part = lambda s: {n[len(s):]: t for n, t in w.items() if n.startswith(s)}
    l, r = attention_mixer(h, part("left."), m["left"]), ssd_mixer(h, part("right."), m["right"], eps)
    return 0.5 * (rms(l, eps) * w["left.out"] + rms(r, eps) * w["right.out"])


# -- feed-forward ------------------------------------------------------------------------------------
def dense_ff(h, w):
    return torch.relu(h @ w["up"].T) ** 2 @ w["down"].T


def gated_ff(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def route(logits, top):
    """-> chosen experts [T, top], softmax over the chosen logits alone."""
    z, i = logits.topk(top, dim=-1)
    return i, torch.softmax(z, dim=-1)


def mixture_ff(h, w, cfg):
    idx, weight = route(h @ w["router"].T + w["router.b"], cfg["router"]["top"])
    out = gated_ff(h, w, "shared.") if cfg.get("shared") else torch.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(idx[t].tolist(), weight[t]):
            out[t] += s * gated_ff(h[t:t + 1], w, f"e{e}.")[0]
    return out


# -- the whole decoder ---------------------------------------------------------------------------------
def layer_runs(config):
    n, lp = len(config["layers"]), config.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def forward(config, weights, tokens, dtype=torch.float64):
    """Whole-prompt forward of one sequence.  -> logits [T, vocab], the residual stream after every
    layer run (list of [T, width])."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = W["embed"][tokens] * config["embedding"]["scale"] + W["pos"][:len(tokens)]
    trail = []
    for li in layer_runs(config):
        spec, p = config["layers"][li], f"l{li}."
        part = lambda s: {n[len(p + s):]: t for n, t in W.items() if n.startswith(p + s)}
        h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
        mix = {"hgrn2": hgrn2_mixer, "gla": gla_mixer, "parallel": parallel_mixer}[spec["type"]]
        y = mix(h, part("mix."), spec["mixer"], eps)
        if spec["mlp"] is not None:
            y = y + (dense_ff(h, part("mlp.")) if spec["mlp"]["kind"] == "dense" else mixture_ff(h, part("mlp."), spec["mlp"]))
        x = x + y
        trail.append(x)
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["embed"].T * config["logit_scale"], trail
