"""CPU restatement of the Similorn decoder, one function per mechanism (test infrastructure only).

Written for clarity, not speed: dense masks, one recurrence step per token, no cache.  Everything
is computed in the dtype of `DT` (float64 unless a caller asks otherwise), so a comparison shows the
error of the kernels and not of the checker.  Shares no code with the product path.
"""
from __future__ import annotations

import math

import torch

DT = torch.float64


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm_about_one(x, w, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sinusoid(positions, width):
    """[T, width]: sin in the even entries, cos in the odd ones, wavelengths 2 pi 10000^(2i/width)."""
    out = torch.zeros(len(positions), width, dtype=DT)
    for col in range(width):
        freq = 10000.0 ** (-(2.0 * (col // 2)) / width)
        angle = positions.to(DT) * freq
        out[:, col] = torch.sin(angle) if col % 2 == 0 else torch.cos(angle)
    return out


def embedding(tokens, positions, table, scale):
    return table[tokens].to(DT) * scale + sinusoid(positions, table.shape[1])


def mlstm_gates(h, w_i, b_i, w_f, b_f, cap):
    """-> log input gate, log forget gate, both [T, heads]."""
    i = cap * torch.tanh((h @ w_i.T + b_i) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w_f.T + b_f) / cap))
    return i, f


def mlstm_recurrence(q, k, v, i, f, state=None):
    """q, k [T, H, dim] (q already scaled), v [T, H, vdim], i, f [T, H].  state = (S [H, dim, vdim],
    n [H, dim], m [H]) or None for a fresh sequence.  -> o [T, H, vdim], the state after the last token."""
    T, H, dk = q.shape
    dv = v.shape[2]
    if state is None:
        state = (torch.zeros(H, dk, dv, dtype=q.dtype), torch.zeros(H, dk, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    S, n, m = (t.clone() for t in state)
    out = torch.zeros(T, H, dv, dtype=q.dtype)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep = torch.exp(f[t] + m - m_new)
        add = torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        num = torch.einsum("hkv,hk->hv", S, q[t])
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = num / den[:, None]
    return out, (S, n, m)


def mlstm_output(o, gate, w_norm, eps):
    """o [T, H, vdim], gate = W_g h [T, H*vdim]: per-head unit RMS, the weight, the sigmoid gate."""
    return rms(o, eps).flatten(1) * w_norm * torch.sigmoid(gate)


def mlstm_mixer(h, w, cfg, eps):
    H, dk, dv = cfg["heads"], cfg["dim"], cfg["vdim"]
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, H, dk) * dk ** -0.5
    k = (h @ w["k"].T).view(T, H, dk)
    v = (h @ w["v"].T).view(T, H, dv)
    i, f = mlstm_gates(h, w["i"], w["i.b"], w["f"], w["f.b"], cfg["gate_cap"])
    o, _ = mlstm_recurrence(q, k, v, i, f)
    return mlstm_output(o, h @ w["g"].T, w["norm"], eps) @ w["o"].T


def window_attention(q, k, v, scale, softcap, window):
    """q [T, H, dim], k [S, G, dim], v [S, G, vdim]; query row r is the token at position S - T + r.
    -> [T, H, vdim]."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    kk = k.repeat_interleave(H // G, dim=1)
    vv = v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("thd,shd->hts", q, kk) * scale
    if softcap:
        s = softcap * torch.tanh(s / softcap)
    back = torch.arange(S - T, S)[:, None] - torch.arange(S)[None, :]
    seen = (back >= 0) & (back < window) if window else back >= 0
    s = s.masked_fill(~seen[None], float("-inf"))
    return torch.einsum("hts,shd->thd", torch.softmax(s, dim=-1), vv)


def attention_mixer(h, w, cfg):
    T = h.shape[0]
    q = (h @ w["q"].T).view(T, cfg["heads"], cfg["dim"])
    k = (h @ w["k"].T).view(T, cfg["kv_heads"], cfg["dim"])
    v = (h @ w["v"].T).view(T, cfg["kv_heads"], cfg["vdim"])
    return window_attention(q, k, v, cfg["scale"], cfg["softcap"], cfg["mask"]["size"]).flatten(1) @ w["o"].T


def dense_ff(h, up, down):
    return gelu_tanh(h @ up.T) @ down.T


def run_order(n_layers, loop):
    """The layers of one forward in order, as (layer, opens a pass of the loop)."""
    if not loop:
        return [(i, False) for i in range(n_layers)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    order = [(i, False) for i in range(a)]
    for _ in range(times):
        order += [(i, i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n_layers)]


def forward(config, weights, tokens, dtype=DT):
    """Whole-prompt forward of one sequence.  -> logits [T, vocab], the residual stream after every
    layer run (list of [T, width])."""
    global DT
    before, DT = DT, dtype
    try:
        W = {n: t.to(dtype) for n, t in weights.items()}
        tokens = torch.as_tensor(tokens, dtype=torch.long)
        x0 = x = embedding(tokens, torch.arange(len(tokens)), W["embed"], config["embedding"]["scale"])
        eps = config["norm"]["eps"]
        trail = []
        for li, opens in run_order(len(config["layers"]), config.get("loop")):
            if opens:
                x = torch.cat([x, x0], dim=-1) @ W["loop.in"].T
            spec, p = config["layers"][li], f"l{li}."
            mix = {n[len(p) + 4:]: t for n, t in W.items() if n.startswith(p + "mix.")}
            h = norm_about_one(x, W[p + "norm1"], eps)
            if spec["type"] == "mlstm":
                x = x + mlstm_mixer(h, mix, spec["mixer"], eps)
            elif spec["type"] == "attention":
                x = x + attention_mixer(h, mix, spec["mixer"])
            else:
                raise ValueError(spec["type"])
            if spec["mlp"] is not None:
                x = x + dense_ff(norm_about_one(x, W[p + "norm2"], eps), W[p + "mlp.up"], W[p + "mlp.down"])
            trail.append(x)
        return norm_about_one(x, W["final.norm"], eps) @ W["head"].T, trail
    finally:
        DT = before
