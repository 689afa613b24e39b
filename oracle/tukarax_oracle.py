"""CPU restatement of the Tukarax decoder, one function per mechanism (test infrastructure only).

Written for clarity, not speed: dense masks, one recurrence step per token, one expert at a time, no cache.
Everything is computed in the dtype of the inputs (float64 unless a caller asks otherwise), so a comparison
shows the error of the kernels and not of this file.  Shares no code with the product path.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def frequencies(rot):
    """-> angle per position of each pair [dims / 2], factor of cos and sin."""
    n, base, s = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not s:
        return f, 1.0
    turn_dim = lambda t: n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turn_dim(s["fast"])), 0), min(math.ceil(turn_dim(s["slow"])), n - 1)
    out = []
    for i, w in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(w / s["factor"] * ramp + w * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot, interleaved):
    """x [T, heads, dim]: the pairs of the first rot["dims"] entries of every head turned."""
    n = rot["dims"]
    f, mul = frequencies(rot)
    out = x.clone()
    for i in range(n // 2):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n // 2)
        angle = positions.to(x.dtype)[:, None] * f[i]
        c, s = torch.cos(angle) * mul, torch.sin(angle) * mul
        out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def visible(T, S, chunk=0):
    """[T, S]: whether row r, at position S - T + r, sees key j."""
    p, j = torch.arange(S - T, S)[:, None], torch.arange(S)[None, :]
    ok = j <= p
    return ok & (torch.div(p, chunk, rounding_mode="floor") == torch.div(j, chunk, rounding_mode="floor")) if chunk else ok


def softmax_attention(q, k, v, scale, softcap=0.0, chunk=0, sink=None):
    """q [T, H, d], k [S, G, d], v [S, G, vd], sink [H] or None; the rows of q are the newest tokens.  -> [T, H, vd]."""
    T, H = q.shape[:2]
    S, G = k.shape[:2]
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("thd,shd->hts", q, k) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    s = s.masked_fill(~visible(T, S, chunk)[None], float("-inf"))
    if sink is not None:
        s = torch.cat([s, sink[:, None, None].expand(H, T, 1)], dim=-1)
    w = torch.softmax(s, dim=-1)[..., :S]
    return torch.einsum("hts,shd->thd", w, v)


def chunked_attention(h, w, m, positions):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q = rotate((h @ w["q"].T).view(T, H, m["dim"]), positions, m["rot"], False)
    k = rotate((h @ w["k"].T).view(T, G, m["dim"]), positions, m["rot"], False)
    v = (h @ w["v"].T).view(T, G, m["vdim"])
    o = softmax_attention(q, k, v, m["scale"], m.get("softcap") or 0.0, m["mask"]["size"], w["sink"])
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.flatten(1) @ w["o"].T


def key_value_attention(h, w, m, positions, eps):
    """Normed and rotated queries and keys; the values are the raw keys."""
    T, H, G = len(h), m["heads"], m["kv_heads"]
    q, k = (h @ w["q"].T).view(T, H, m["dim"]), (h @ w["k"].T).view(T, G, m["dim"])
    v = k
    q = rotate(rms(q, eps) * w["q.norm"], positions, m["rot"], True)
    k = rotate(rms(k, eps) * w["k.norm"], positions, m["rot"], True)
    o = softmax_attention(q, k, v, m["scale"]).flatten(1)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def short_conv(x, w, before=None):
    """x [T, channels], w [channels, taps] -> silu of the causal convolution; `before`: the taps - 1 inputs ahead of x."""
    taps = w.shape[1]
    if before is None:
        before = torch.zeros(taps - 1, x.shape[1], dtype=x.dtype)
    x = torch.cat([before, x])
    out = torch.zeros(len(x) - taps + 1, x.shape[1], dtype=x.dtype)
    for t in range(len(out)):
        for j in range(taps):
            out[t] += w[:, j] * x[t + j]
    return silu(out)


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, g, beta, S=None):
    """q, k [T, H, dim], v [T, H, vdim], g, beta [T, H]; S [H, dim, vdim] or None.  -> o [T, H, vdim], S after the last."""
    T, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if S is None else S.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for t in range(T):
        for i in range(H):
            S[i] = g[t, i] * S[i]
            u = beta[t, i] * (v[t, i] - S[i].T @ k[t, i])
            S[i] = S[i] + torch.outer(k[t, i], u)
            out[t, i] = S[i].T @ q[t, i]
    return out, S


def gated_delta(h, w, m, eps):
    T, H, G = len(h), m["heads"], m["kv_heads"]
    conv = lambda n, heads, d: short_conv(h @ w[n].T, w[n + ".conv"]).view(T, heads, d)
    q, k, v = conv("q", G, m["dim"]), conv("k", G, m["dim"]), conv("v", H, m["vdim"])
    q, k = unit(q) * m["dim"] ** -0.5, unit(k)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * torch.nn.functional.softplus(h @ w["a"].T + w["dt_bias"], threshold=1e9))
    o, _ = delta_recurrence(q, k, v, g, beta)
    o = rms(o, eps) * w["norm"] * silu(h @ w["g"].T).view(T, H, m["vdim"])
    return o.flatten(1) @ w["o"].T


def parallel(h, w, m, positions, eps):
    part = lambda s: {n[len(s):]: t for n, t in w.items() if n.startswith(s)}
    return m["left_scale"] * key_value_attention(h, part("left."), m["left"], positions, eps) + \
        m["right_scale"] * gated_delta(h, part("right."), m["right"], eps)


def route(logits, top):
    """-> chosen experts [T, top], their sigmoid scores."""
    s, i = torch.sigmoid(logits).topk(top, dim=-1)
    return i, s


def expert(z, w, e):
    return (silu(z @ w[f"e{e}.gate"].T) * (z @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T


def mixture_ff(h, w, cfg):
    idx, score = route(h @ w["router"].T, cfg["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(len(h)):
        for e, s in zip(idx[t].tolist(), score[t]):
            out[t] += expert(s * h[t:t + 1], w, e)[0]
    return out


def forward(config, weights, tokens, dtype=torch.float64):
    """Whole-prompt forward of one sequence.  -> logits [T, vocab], the residual stream after every
    layer (list of [T, width])."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    positions = torch.arange(len(tokens))
    eps = config["norm"]["eps"]
    x = W["embed"][tokens]
    trail = []
    for li, spec in enumerate(config["layers"]):
        p = f"l{li}."
        part = lambda s: {n[len(p + s):]: t for n, t in W.items() if n.startswith(p + s)}
        h = rms(x, eps) * W[p + "norm1"]
        if spec["type"] == "attention":
            x = x + chunked_attention(h, part("mix."), spec["mixer"], positions)
        elif spec["type"] == "parallel":
            x = x + parallel(h, part("mix."), spec["mixer"], positions, eps)
        else:
            raise ValueError(spec["type"])
        if spec["mlp"] is not None:
            x = x + mixture_ff(rms(x, eps) * W[p + "norm2"], part("mlp."), spec["mlp"])
        trail.append(x)
    return (rms(x, eps) * W["final.norm"]) @ W["head"].T, trail
