"""Kernels of the Dinatar decoder against the plain fp64 functions, one mechanism at a time."""
import pytest
import torch

from oracle import dinatar_oracle as O

pytestmark = pytest.mark.gpu
F64, BF = torch.float64, torch.bfloat16
DTYPES = [torch.float32, BF]


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _r(g, *s, k=1.0):
    return torch.randn(*s, generator=g) * k


def _u(g, n, lo, hi):
    return torch.rand(n, generator=g) * (hi - lo) + lo


def _dev(t, dtype=None):
    return None if t is None else (t if dtype is None else t.to(dtype)).cuda()


def _i32(v):
    return torch.tensor(v, dtype=torch.int32).cuda()


def _close(got, want, dtype, k=1.0):
    """Largest error over the size of the values: one rounding of the result (bf16) or fp32 sums."""
    err = (got.double().cpu() - want.double()).abs().max().item() / want.double().abs().max().item()
    assert err < k * (4e-3 if dtype == BF else 1e-5), err


def _check_device():
    from zipage_b200 import _lib as L
    torch.cuda.synchronize()
    assert L.device_error(reset=True) == 0


# -- embedding, boundary ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [40, 77, 2048])
def test_embedding_with_learned_positions(W, dtype):
    from zipage_b200.layers.row_ops import embed_position
    g = _gen(W)
    table, pos = _r(g, 50, W).to(dtype), _r(g, 300, W).to(dtype)
    tok, at = torch.randint(50, (23,), generator=g), torch.randint(300, (23,), generator=g)
    at[:3] = torch.tensor([0, 299, 1])
    x, x_t = embed_position(_dev(tok), _dev(at), _dev(table), 7.5, learned=_dev(pos), want_t=True)
    want = table.to(F64)[tok] * 7.5 + pos.to(F64)[at]
    _close(x, want, torch.float32)
    _close(x_t, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [136, 58, 2052, 8192])
def test_boundary_with_a_pair_of_normed_rows(W, dtype):
    from zipage_b200.layers.row_ops import join_norms
    g = _gen(W)
    N, top, eps = 7, 3, 1e-2
    x, b, y, m1, m2 = _r(g, N, W) + 3.0, *(_r(g, n, W).to(dtype) for n in (N, N * top, N, N))
    m2 = (m2 * 30).to(dtype)                                               # of very different sizes before their norms
    w1, w2, wn, bn, wt = _r(g, W), _r(g, W), _r(g, W), _r(g, W), torch.rand(N, top, generator=g)
    pos = torch.randperm(N * top, generator=g).view(N, top).to(torch.int32)
    D = lambda t: t.to(F64)
    pair = 0.5 * (O.rms(D(m1), eps) * D(w1) + O.rms(D(m2), eps) * D(w2))
    moe = (D(wt)[:, :, None] * D(y)[pos.long()]).sum(1)
    for kw, want in (({}, D(x) + pair), ({"b": b}, D(x) + pair + D(b)),
                     ({"b": b, "y": y, "pos": pos, "weights": wt}, D(x) + pair + D(b) + moe)):
        xd = _dev(x.clone())
        out, = join_norms(xd, [(_dev(wn), _dev(bn))], eps, dtype, pair=((_dev(m1), _dev(w1)), (_dev(m2), _dev(w2))),
                          **{k: _dev(t) for k, t in kw.items()})
        _close(xd, want, torch.float32)
        _close(out, O.layer_norm(want, D(wn), D(bn), eps), dtype)
    xd = _dev(x.clone())
    out, = join_norms(xd, [(_dev(wn), _dev(bn))], eps, dtype, a=_dev(b), y=_dev(y), pos=_dev(pos), weights=_dev(wt))
    _close(out, O.layer_norm(D(x) + D(b) + moe, D(wn), D(bn), eps), dtype)


# -- attention with kept tokens and distance biases --------------------------------------------------------
def _paged(rows, BS, g):
    """rows: list of [ctx, heads, width] -> (cache with pages in random order and others' rows around, table)."""
    need = [(len(r) + BS - 1) // BS for r in rows]
    P = sum(need) + 3
    _, H, d = rows[0].shape
    cache = torch.zeros(P, BS, H, (d + 15) // 16 * 16)
    cache[..., :d] = torch.randn(P, BS, H, d, generator=g) * 5
    order = torch.randperm(P, generator=_gen(5)).tolist()
    table = torch.full((len(rows), max(need) + 1), -1, dtype=torch.int32)
    for b, r in enumerate(rows):
        for i in range(need[b]):
            table[b, i] = order.pop()
            part = r[i * BS:(i + 1) * BS]
            cache[table[b, i], :len(part), :, :d] = part
    return cache.to(rows[0].dtype), table


def _attend(dtype, impl, H, G, d, dv, ctxs, counts, window, keep, sloped, decode=False, steep=0.0, BS=64, softcap=0.0):
    from zipage_b200.layers.attention import distance_slopes, window_attention
    g = _gen(H * 100 + d + window)
    ks, vs = [_r(g, c, G, d).to(dtype) for c in ctxs], [_r(g, c, G, dv).to(dtype) for c in ctxs]
    q = _r(g, sum(counts), H * d + 8, k=2.0).to(dtype)
    if steep:      # scores that climb along the sequence by far more than fp32 exponents absorb
        for k in ks:
            k[..., 0] = (torch.arange(len(k)) * steep)[:, None].to(dtype)
        q[:, 0:H * d:d] = 1.0
    kc, table = _paged(ks, BS, g)
    vc, _ = _paged(vs, BS, g)
    slope = torch.tensor(distance_slopes(H)) if sloped else None
    if sloped:
        assert torch.equal(slope.to(F64), O.slopes(H).to(torch.float32).to(F64))
    scale, at, want = d ** -0.5, 0, []
    for k, v, n in zip(ks, vs, counts):
        want.append(O.biased_attention(q[at:at + n, :H * d].to(F64).reshape(n, H, d), k.to(F64), v.to(F64), scale, window, keep,
                                       O.slopes(H) if sloped else None).flatten(1))
        at += n
    cu = None if decode else _i32([0] + torch.tensor(counts).cumsum(0).tolist())
    out = torch.full((sum(counts), H * dv + 8), 9.0, dtype=dtype, device="cuda")
    window_attention(_dev(q)[:, :H * d], _dev(kc), _dev(vc), _i32(ctxs), _dev(table), H, d, dv, scale, window, softcap, cu_seqlens_q=cu,
                     max_seqlen_q=max(counts), out=out[:, :H * dv], impl=impl, keep=keep, slopes=_dev(slope))
    _check_device()
    assert (out[:, H * dv:] == 9).all()
    _close(out[:, :H * dv], torch.cat(want), dtype)


MASKS = [(0, 0, True), (70, 5, True), (33, 65, True), (64, 64, False), (1, 1, True), (130, 3, True), (100, 200, True), (20, 129, False), (50, 0, True)]


@pytest.mark.parametrize("window,keep,sloped", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 48, 40), (8, 1, 128, 128), (3, 3, 13, 11), (2, 1, 176, 208)])
def test_attention_of_portions(H, G, d, dv, window, keep, sloped):
    ctxs, counts = [200, 71, 2, 130, 64, 1, 400], [200, 3, 2, 66, 2, 1, 131]
    for dtype, impl in ((torch.float32, "auto"), (BF, "auto"), (BF, "simt")):
        _attend(dtype, impl, H, G, d, dv, ctxs, counts, window, keep, sloped)


@pytest.mark.parametrize("window,keep,sloped", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 48, 40), (8, 1, 128, 128), (6, 3, 96, 128), (2, 2, 72, 16)])
def test_attention_of_portions_tcgen05(H, G, d, dv, window, keep, sloped):
    ctxs, counts = [200, 71, 2, 130, 64, 1, 700], [200, 3, 2, 66, 2, 1, 290]
    for steep in (0.0, 1.5, 40.0):                                         # (references that move)
        _attend(BF, "tcgen05", H, G, d, dv, ctxs, counts, window, keep, sloped, steep=steep)


@pytest.mark.parametrize("window,keep,sloped", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 48, 40), (8, 1, 128, 128), (3, 3, 13, 11), (2, 1, 176, 208), (20, 1, 32, 16), (15, 1, 24, 24)])
def test_attention_of_decoded_tokens(H, G, d, dv, window, keep, sloped):
    ctxs = [1, 2, 63, 64, 65, 70, 71, 140, 141, 128, 129, 1000]
    for dtype in DTYPES:
        _attend(dtype, "auto", H, G, d, dv, ctxs, [1] * len(ctxs), window, keep, sloped, decode=True)


def test_slopes_beside_a_cap_are_refused_by_the_tcgen05_kernel():
    from zipage_b200._lib import ZipageError
    with pytest.raises(ZipageError):
        _attend(BF, "tcgen05", 2, 1, 64, 64, [70], [70], 0, 0, True, softcap=20.0)


@pytest.mark.parametrize("window,keep", [(64, 5), (70, 64), (33, 130), (128, 1)])
def test_keys_at_the_edges_of_the_window_and_of_the_kept_tokens(window, keep):
    """A key whose score stands out is the output of the rows that see it, and of no other row."""
    from zipage_b200.layers.attention import window_attention
    d, T = 128, 330
    g = _gen(window)
    for place in (0, keep - 1, keep, 63, 64, 127, 128, 129, 200, 256):
        q = torch.zeros(T, d)
        q[:, 0] = 1.0
        k, v = torch.zeros(T, 1, d), _r(g, T, 1, d)
        k[place, 0, 0] = 300.0
        v[:, 0, 5] = 0.0
        v[place, 0, 5] = 1.0
        kc, table = _paged([k.to(BF)], 64, g)
        vc, _ = _paged([v.to(BF)], 64, g)
        p = torch.arange(T)
        sees = (p >= place) & ((p - place < window) | (place < keep))
        for dtype, impl in ((BF, "tcgen05"), (BF, "auto"), (torch.float32, "simt")):
            args = _dev(q, dtype), _dev(kc, dtype), _dev(vc, dtype)
            o = window_attention(*args, _i32([T]), _dev(table), 1, d, d, 0.1, window, cu_seqlens_q=_i32([0, T]), max_seqlen_q=T, keep=keep, impl=impl)
            assert torch.equal(o[:, 5].float().cpu() > 0.5, sees) and (o[~sees.cuda(), 5] == 0).all()
            last = [c for c in (place, place + 1, place + 2, place + window, place + window + 1, place + window + 2, T) if 0 < c <= T]
            o = window_attention(args[0][:len(last)], *args[1:], _i32(last), _dev(table).expand(len(last), -1).contiguous(), 1, d, d, 0.1, window,
                                 keep=keep)
            assert torch.equal(o[:, 5].float().cpu() > 0.5, sees[torch.tensor(last) - 1])
    _check_device()


# -- linear attention with decaying states -------------------------------------------------------------------
KINDS = ["forget", "power", "scalar"]


def _case(kind, H, G, dk, dv, T, seed, span, dtype):
    """Inputs of one sequence.  span: "mixed" decays; "slow": next to none; "fast": states forgotten within a token or two."""
    g = _gen(seed)
    c = {"q": _r(g, T, G * dk).to(dtype), "k": _r(g, T, G * dk).to(dtype), "v": _r(g, T, H * dv).to(dtype)}
    shift = {"mixed": 0.0, "slow": 7.0, "fast": -9.0}[span]
    if kind == "scalar":
        c.update(z=_r(g, T, H, k=2.0), bias=_u(g, H, -3.0, 0.5), A_log=_u(g, H, -3.0, 1.0) - shift / 3, D=_r(g, H))
    else:
        c.update(z=_r(g, T, H * dk, k=2.0), bias=_r(g, H * dk) + shift)
        if kind == "forget":
            c["lower"] = _u(g, H * dk, 0.0, 0.9) * (span != "fast")
    return c


def _want(kind, c, H, G, dk, dv, tau, S=None, v=None, k=None, q=None):
    """-> outputs [T, H * dv], state, of fp64 inputs (v, k, q: instead of the case's)."""
    D = lambda n, alt: (c[n] if alt is None else alt).to(F64)
    q, k, v, z, T = D("q", q), D("k", k), D("v", v), c["z"].to(F64), len(c["z"])
    if kind == "forget":
        a = O.hgrn2_gates(z, c["bias"].to(F64), c["lower"].to(F64)).view(T, H, dk)
        q, k = O.silu(q).view(T, H, dk), 1 - a
    elif kind == "power":
        a = O.gla_decay(z + c["bias"].to(F64), tau).view(T, H, dk)
        q, k = q.view(T, H, dk) * dk ** -0.5, k.view(T, H, dk)
    else:
        dt = torch.nn.functional.softplus(z + c["bias"].to(F64), threshold=1e9)
        a = torch.exp(-torch.exp(c["A_log"].to(F64)) * dt)[:, :, None].expand(T, H, dk)
        q, k = (t.reshape(T, G, dk).repeat_interleave(H // G, 1) for t in (q, k))
        k = k * dt[:, :, None]
    o, S = O.decayed_recurrence(q, k, v.reshape(T, H, dv), a, S)
    if kind == "scalar":
        o = o + c["D"].to(F64)[:, None] * v.reshape(T, H, dv)
    return o.flatten(1), S


def _shared(kind, c, tau, dk):
    kw = {"rtau": 1 / tau, "qscale": dk ** -0.5} if kind == "power" else {}
    return kw | {n: _dev(c[n]) for n in ("lower", "A_log", "D") if n in c}


SIZES = [(6, 2, 40, 56), (4, 4, 128, 128), (3, 3, 9, 7), (2, 1, 160, 200), (1, 1, 300, 33), (2, 2, 16, 304), (8, 1, 8, 8), (2, 1, 96, 256), (3, 1, 128, 72),
         (4, 2, 64, 64), (2, 2, 48, 136)]


@pytest.mark.parametrize("span", ["mixed", "slow", "fast"])
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,G,dk,dv", SIZES)
def test_linear_state_portions(H, G, dk, dv, kind, span):
    """Portions of unequal length, each on the state that the one before left, in slots that held others' numbers."""
    from zipage_b200.layers.linear_state import linear_state
    G, tau = G if kind == "scalar" else H, 5.0
    plans = [[130, 64, 2], [2, 63, 70], [65, 1, 200]]
    impls = [(torch.float32, "auto"), (BF, "simt")]
    if dk % 8 == dv % 8 == 0 and dk <= 128:
        impls.append((BF, "tcgen05"))
    wants = {}
    for dtype, impl in impls:
        cases = [_case(kind, H, G, dk, dv, sum(p), 10 + i, span, dtype) for i, p in enumerate(plans)]
        for c in cases[1:]:
            c.update({n: cases[0][n] for n in ("bias", "lower", "A_log", "D") if n in c})
        state = torch.full((5, H, dk, (dv + 3) // 4 * 4), 3.0, device="cuda")
        slots, done, outs = [3, 0, 4], [0, 0, 0], [[], [], []]
        shared, nq, nv = _shared(kind, cases[0], tau, dk), (G * dk + 7) // 8 * 8, (H * dv + 7) // 8 * 8
        for step in range(3):
            n, lead = [p[step] for p in plans], 4                  # rows of other sequences ahead of the portions'
            total = lead + sum(n)
            x = torch.zeros(total, 2 * nq + nv + 8, dtype=dtype)   # columns of one projection
            z = torch.zeros(total, cases[0]["z"].shape[1])
            at = lead
            for c, d, m in zip(cases, done, n):
                for key, lo in (("q", 0), ("k", nq), ("v", 2 * nq)):
                    x[at:at + m, lo:lo + c[key].shape[1]] = c[key][d:d + m]
                z[at:at + m] = c["z"][d:d + m]
                at += m
            x, done = _dev(x), [d + m for d, m in zip(done, n)]
            out = torch.full((total, (H * dv + 15) // 8 * 8), 9.0, dtype=dtype, device="cuda")
            cu = _i32([lead] + [lead + v for v in torch.tensor(n).cumsum(0).tolist()])
            linear_state(kind, x[:, :G * dk], None if kind == "forget" else x[:, nq:nq + G * dk], x[:, 2 * nq:2 * nq + H * dv], _dev(z),
                         _dev(cases[0]["bias"]), state, out[:, :H * dv], _i32(done), _i32(slots), H, G, dk, dv, cu_seqlens_q=cu, impl=impl, **shared)
            _check_device()
            assert (out[:lead] == 9).all() and (out[:, H * dv:] == 9).all()
            for i, part in enumerate(out[lead:, :H * dv].split(n)):
                outs[i].append(part.cpu())
        for i, c in enumerate(cases):
            if (dtype, i) not in wants:
                wants[dtype, i] = _want(kind, c, H, G, dk, dv, tau)
            want, S = wants[dtype, i]
            _close(torch.cat(outs[i]), want, dtype, 1 if dtype == BF else 5)
            _close(state[slots[i]][..., :dv], S, torch.float32, 5 if impl == "auto" else 10)
        assert (state[[1, 2]] == 3).all()


@pytest.mark.parametrize("kind", KINDS)
def test_linear_state_of_jumps(kind):
    """Decays that jump between none and all, channel by channel: exponents taken against any one token would leave fp32's range."""
    from zipage_b200.layers.linear_state import linear_state
    H, d, T, tau = 2, 128, 300, 1.0
    g = _gen(3)
    for dtype, impl in ((BF, "tcgen05"), (BF, "simt"), (torch.float32, "auto")):
        c = _case(kind, H, H, d, d, T, 7, "mixed", dtype)
        z = torch.where(torch.rand(c["z"].shape, generator=g) < 0.2, -60.0, 15.0)       # (forget, power: decays of e^-60 and of e^-3e-7)
        c["z"] = z if kind != "scalar" else -z * 0.5
        c["bias"], want_k = torch.zeros_like(c["bias"]), 1
        if kind == "forget":
            c["lower"] = torch.zeros_like(c["lower"])
        state, out = torch.zeros(1, H, d, d, device="cuda"), torch.empty(T, H * d, dtype=dtype, device="cuda")
        for a, b in ((0, 150), (150, 300)):
            xs = [_dev(torch.cat([c["q"], c["k"], c["v"]], 1)[a:b]).split(H * d, dim=1)][0]
            linear_state(kind, xs[0], None if kind == "forget" else xs[1], xs[2], _dev(c["z"][a:b]), _dev(c["bias"]), state, out[a:b], _i32([b]),
                         _i32([0]), H, H, d, d, cu_seqlens_q=_i32([0, b - a]), impl=impl, **_shared(kind, c, tau, d))
        _check_device()
        want, S = _want(kind, c, H, H, d, d, tau)
        _close(out, want, dtype, 5 if dtype != BF else 1)
        _close(state[0], S, torch.float32, 10)


@pytest.mark.parametrize("kind", KINDS)
def test_linear_state_keeps_a_far_write(kind):
    """With next to no decay a value written once comes back hundreds of tokens later, across chunks, portions and slots."""
    from zipage_b200.layers.linear_state import linear_state
    T, d = 400, 64
    g = _gen(4)
    for dtype, impl in ((BF, "tcgen05"), (BF, "simt"), (torch.float32, "auto")):
        for place in (0, 7, 8, 15, 31, 32, 63, 64, 100):
            q, k, v, z = torch.zeros(T, d), torch.zeros(T, d), _r(g, T, d), torch.full((T, d), 30.0)
            k[:, 1:], q[:, 1:] = _r(g, T, d - 1), _r(g, T, d - 1)
            k[place, 0] = 4.0
            q[T - 1] = 0.0
            q[T - 1, 0] = 3.0
            c = {"q": q.to(dtype), "k": k.to(dtype), "v": v.to(dtype), "z": z, "bias": torch.zeros(d)}
            if kind == "forget":
                z[place, 0] = -30.0                        # written where the channel forgets
                c["lower"] = torch.zeros(d)
            if kind == "scalar":
                c.update(z=torch.zeros(T, 1), bias=torch.zeros(1), A_log=torch.full((1,), -20.0), D=torch.zeros(1))
            state, out = torch.zeros(1, 1, d, d, device="cuda"), torch.empty(T, d, dtype=dtype, device="cuda")
            for a, b in ((0, 150), (150, 400)):
                part = lambda n: _dev(c[n][a:b])
                linear_state(kind, part("q"), None if kind == "forget" else part("k"), part("v"), part("z"), _dev(c["bias"]), state, out[a:b],
                             _i32([b]), _i32([0]), 1, 1, d, d, cu_seqlens_q=_i32([0, b - a]), impl=impl, **_shared(kind, c, 1.0, d))
            want, _ = _want(kind, c, 1, 1, d, d, 1.0)
            _close(out[-1], want[-1], dtype, 5 if dtype != BF else 1.5)
            assert torch.nn.functional.cosine_similarity(out[-1].double().cpu(), v[place].to(F64), dim=0) > 0.99
    _check_device()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["forget", "power"])
@pytest.mark.parametrize("H,dk,dv", [(6, 40, 56), (4, 128, 128), (3, 9, 7), (2, 160, 200), (1, 300, 33), (64, 16, 48), (40, 128, 64)])
def test_linear_state_decoding(H, dk, dv, kind, dtype):
    """Single rows of a batch whose sequences start at different steps, on what a prompt left; a padding row."""
    from zipage_b200.layers.linear_state import linear_state
    tau, T, first = 7.0, 14, [0, 5, 9]
    cases = [_case(kind, H, H, dk, dv, T, 50 + i, "mixed", dtype) for i in range(3)]
    for c in cases[1:]:
        c.update({n: cases[0][n] for n in ("bias", "lower") if n in c})
    state = torch.full((4, H, dk, (dv + 3) // 4 * 4), 3.0, device="cuda")
    slots, outs = [2, 0, 3], [[], [], []]
    sh = _shared(kind, cases[0], tau, dk)

    def run(rows, ctx, sl, cu=None):
        x = _dev(torch.cat([torch.cat([c["q"], c["k"], c["v"]], 1)[a:b] for c, a, b in rows]))
        q, k, v = x.split([H * dk, H * dk, H * dv], dim=1)
        out = torch.full((len(x), H * dv), 9.0, dtype=dtype, device="cuda")
        linear_state(kind, q, None if kind == "forget" else k, v, _dev(torch.cat([c["z"][a:b] for c, a, b in rows])), _dev(cases[0]["bias"]), state, out,
                     _i32(ctx), _i32(sl), H, H, dk, dv, cu_seqlens_q=cu, **sh)
        _check_device()
        return out
    outs[0].append(run([(cases[0], 0, 4)], [4], [2], _i32([0, 4])).cpu())
    for t in range(T):
        live = [i for i in range(3) if first[i] <= t and (i or t >= 4)]
        if not live:
            continue
        rows = [(cases[i], t - first[i], t - first[i] + 1) for i in live]
        out = run(rows + [(cases[0], 0, 1)], [t - first[i] + 1 for i in live] + [0], [slots[i] for i in live] + [-1])
        assert (out[-1] == 9).all()
        for i, o in zip(live, out):
            outs[i].append(o[None].cpu())
    for i, c in enumerate(cases):
        n = T - first[i]
        cut = {k: v[:n] if len(v) == T and k in "qkvz" else v for k, v in c.items()}
        want, S = _want(kind, cut, H, H, dk, dv, tau)
        _close(torch.cat(outs[i]), want, dtype, 1 if dtype == BF else 2)
        _close(state[slots[i]][..., :dv], S, torch.float32, 2)
    assert (state[1] == 3).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,taps", [(6, 2, 40, 56, 4), (4, 4, 128, 128, 3), (3, 3, 9, 7, 5), (2, 1, 160, 200, 2), (1, 1, 8, 12, 1), (32, 16, 64, 64, 4)])
def test_scalar_state_convolution_prompts_and_decoding(H, G, dk, dv, taps, dtype):
    """Prompts through the convolution, then single rows with the convolution in the launch, then portions again: outputs, state and
    the convolution's memory carry over; a batch of two sequences out of step, and a padding row."""
    from zipage_b200.layers.short_conv import short_conv
    from zipage_b200.layers.linear_state import linear_state
    g = _gen(taps)
    T, nv, nk = [41, 30], H * dv, G * dk
    C = nv + 2 * nk
    cases = [_case("scalar", H, G, dk, dv, t, 20 + i, "mixed", dtype) | {"x": _r(g, t, C).to(dtype)} for i, t in enumerate(T)]
    cases[1].update({n: cases[0][n] for n in ("bias", "A_log", "D")})
    w, b = _r(g, C, taps, k=0.7), _r(g, C, k=0.5)
    wd, bd = _dev(w.t().contiguous()), _dev(b)
    state, ring = torch.full((4, H, dk, (dv + 3) // 4 * 4), 3.0, device="cuda"), torch.full((4, taps, C), 5.0, dtype=dtype, device="cuda")
    sh = {n: _dev(cases[0][n]) for n in ("A_log", "D")}
    slots, at, outs = [2, 0], [0, 0], [[], []]

    def run(n, decode):
        x, z = (torch.cat([c[key][a:a + m] for c, a, m in zip(cases, at, n)]) for key in ("x", "z"))
        live = [i for i in range(2) if n[i]]
        for i in live:
            at[i] += n[i]
        ctx, sl = [at[i] for i in live], [slots[i] for i in live]
        wide = torch.zeros(len(x) + decode, (C + 15) // 8 * 8, dtype=dtype, device="cuda")       # rows of a wider projection
        wide[:len(x), :C] = _dev(x)
        out = torch.full((len(x) + decode, nv), 9.0, dtype=dtype, device="cuda")
        cols = lambda y: (y[:, nv + nk:C], y[:, nv:nv + nk], y[:, :nv])
        if decode:                                                                   # (the last row pads the batch)
            linear_state("scalar", *cols(wide), _dev(torch.cat([z, z[:1]])), _dev(cases[0]["bias"]), state, out, _i32(ctx + [0]), _i32(sl + [-1]),
                         H, G, dk, dv, conv_weight=wd, conv_bias=bd, ring=ring, **sh)
            assert (out[-1] == 9).all()
        else:
            m = [n[i] for i in live]
            cu = _i32([0] + torch.tensor(m).cumsum(0).tolist())
            y = torch.empty(len(x), wide.shape[1], dtype=dtype, device="cuda")
            short_conv(wide[:, :C], wd, ring, _i32(ctx), _i32(sl), cu, max(m), y, bias=bd)
            linear_state("scalar", *cols(y), _dev(z), _dev(cases[0]["bias"]), state, out, _i32(ctx), _i32(sl), H, G, dk, dv, cu_seqlens_q=cu, **sh)
        _check_device()
        o = 0
        for i in live:
            outs[i].append(out[o:o + n[i]].cpu())
            o += n[i]
    run([1, 0], True)
    run([19, 2], False)
    for _ in range(3):
        run([1, 1], True)
    run([2, 17], False)
    run([1, 0], True)
    run([0, 2], False)
    run([T[0] - at[0] - 1, T[1] - at[1] - 1], False)
    run([1, 1], True)
    for i, c in enumerate(cases):
        assert at[i] == T[i]
        conv = O.short_conv(c["x"].to(F64), w.to(F64), b.to(F64))
        want, S = _want("scalar", c, H, G, dk, dv, 1.0, v=conv[:, :nv], k=conv[:, nv:nv + nk], q=conv[:, nv + nk:])
        _close(torch.cat(outs[i]), want, dtype, 4 if dtype == BF else 5)
        _close(state[slots[i]][..., :dv], S, torch.float32, 30 if dtype == torch.float32 else 600)       # (bf16: rounded inputs of prompts)
        for p in range(max(0, T[i] - taps), T[i]):
            assert torch.equal(ring[slots[i], p % taps].cpu(), c["x"][p])
    assert (state[[1, 3]] == 3).all() and (ring[[1, 3]] == 5).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps", [(96, 2), (100, 3), (37, 4), (2056, 4), (40, 8), (16, 1)])
def test_short_convolution_with_a_bias(C, taps, dtype):
    from zipage_b200.layers.short_conv import short_conv
    g = _gen(C)
    plan = [2, 1, 16, 17, 3, 33, 5]
    x, w, b = _r(g, sum(plan), C).to(dtype), _r(g, C, taps), _r(g, C)
    ring, at, outs = torch.full((2, taps, C), 5.0, dtype=dtype, device="cuda"), 0, []
    for n in plan:
        y = torch.empty(n, C, dtype=dtype, device="cuda")
        short_conv(_dev(x[at:at + n]), _dev(w.t().contiguous()), ring, _i32([at + n]), _i32([1]), _i32([0, n]), n, y, bias=_dev(b))
        outs.append(y.cpu())
        at += n
    _close(torch.cat(outs), O.short_conv(x.to(F64), w.to(F64), b.to(F64)), dtype)
    assert (ring[0] == 5).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("parts,width", [(6, 56), (1, 4096), (2, 1048), (3, 7), (1, 1031), (8, 128), (4, 256), (2, 6144), (1, 9000), (16, 8)])
def test_group_norms_with_gates(parts, width, dtype):
    from zipage_b200.layers.linear_state import group_norm_gate
    g = _gen(width)
    N, W, eps = 9, parts * width, 1e-2
    x = (_r(g, N, W) * torch.repeat_interleave(_u(g, parts, 0.1, 5.0), width)).to(dtype)        # parts of different sizes
    gates = [_r(g, N, W + 8, k=2.0).to(dtype) for _ in range(2)]
    for weight in (1 + _r(g, width, k=0.3), 1 + _r(g, W, k=0.3)):
        for pre, post in ((False, False), (True, False), (False, True), (True, True)):
            xd = _dev(x)
            o = group_norm_gate(xd, _dev(weight), parts, eps, _dev(gates[0])[:, :W] if pre else None, _dev(gates[1])[:, :W] if post else None,
                                out=xd if pre else None)
            y = x.to(F64) * (O.silu(gates[0][:, :W].to(F64)) if pre else 1)
            y = O.rms(y.view(N, parts, width), eps).flatten(1) * (weight if len(weight) == W else weight.repeat(parts)).to(F64)
            _close(o, y * (O.silu(gates[1][:, :W].to(F64)) if post else 1), dtype)


# -- feed-forward --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,E,top", [(1, 11, 2), (7, 5, 5), (300, 64, 6), (513, 11, 2), (3000, 300, 8), (700, 1, 1), (20, 40, 40)])
def test_routing_by_softmax_over_the_chosen(N, E, top):
    from zipage_b200.layers.feed_forward import moe_route
    g = _gen(N)
    z, b = _r(g, N, E + 3, k=3.0), _r(g, E, k=3.0)
    i, s = O.route(z[:, :E].to(F64) + b.to(F64), top)
    w, experts, places, rows, offsets = moe_route(_dev(z), E, top, "softmax_top", bias=_dev(b))
    assert torch.equal(experts.cpu().long(), i)
    _close(w, s, torch.float32)
    p = places.cpu().long()
    assert torch.equal(rows.cpu().long()[p], torch.arange(N)[:, None].expand(N, top))
    assert torch.equal(torch.bincount(i.flatten(), minlength=E).cumsum(0), offsets[1:].cpu().long())
    pw, _, places, *_ = moe_route(_dev(z), E, top, "softmax_top", bias=_dev(b), by_place=True)
    assert torch.equal(pw.cpu()[places.cpu().long()], w.cpu())


@pytest.mark.parametrize("N,E,top,ff,shared,W", [(1, 5, 2, 40, 24, 136), (90, 7, 3, 24, 0, 64), (700, 3, 2, 136, 72, 128), (40, 6, 6, 11, 13, 58),
                                                 (300, 12, 1, 16, 200, 200)])
def test_experts_weighted_at_the_output_beside_a_shared_one(N, E, top, ff, shared, W):
    from zipage_b200.layers.feed_forward import GatedMixtureFF, moe_route
    from zipage_b200.layers.row_ops import join_norms
    g = _gen(N)
    for dtype in DTYPES:
        shapes = [("gate", lambda f: (f, W)), ("up", lambda f: (f, W)), ("down", lambda f: (W, f))]
        w = {f"e{e}.{n}": (_r(g, *s(ff)) / W ** 0.5 * 2).to(dtype) for e in range(E) for n, s in shapes}
        if shared:
            w.update({f"shared.{n}": (_r(g, *s(shared)) / W ** 0.5 * 2).to(dtype) for n, s in shapes})
        w["router"], w["router.b"] = (_r(g, E, W) / W ** 0.5 * 3).to(dtype), _r(g, E, k=2.0).to(dtype)
        m = GatedMixtureFF(W, E, top, ff, dtype, torch.device("cuda"), score="softmax_top", weigh="output", bias=True, shared_ff=shared)
        m.load(lambda n: w[n])
        h = _r(g, N, W).to(dtype)
        x = torch.zeros(N, W, device="cuda")
        join_norms(x, [], 1e-5, dtype, **m(_dev(h)))
        # the kernels' own choice: rounding may turn a close call
        z = _dev(h).float() @ _dev(w["router"]).float().t()
        _, experts, *_ = moe_route(z, E, top, "softmax_top", bias=_dev(w["router.b"].float()))
        H, W64 = h.to(F64), {k: v.to(F64) for k, v in w.items()}
        s = torch.softmax((H @ W64["router"].T + W64["router.b"]).gather(1, experts.cpu().long()), dim=-1)
        want = O.gated_ff(H, W64, "shared.") if shared else torch.zeros_like(H)
        for t in range(N):
            for e, v in zip(experts[t].tolist(), s[t]):
                want[t] += v * O.gated_ff(H[t:t + 1], W64, f"e{e}.")[0]
        _close(x, want, dtype, 3 if dtype == BF else 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("N,ff,W", [(5, 40, 136), (130, 11, 58)])
def test_squared_relu_block(N, ff, W, dtype):
    from zipage_b200.layers.feed_forward import SquaredReluFF
    g = _gen(N)
    w = {"up": (_r(g, ff, W) / W ** 0.5).to(dtype), "down": (_r(g, W, ff) / ff ** 0.5).to(dtype)}
    m = SquaredReluFF(W, ff, dtype, torch.device("cuda"))
    m.load(lambda n: w[n])
    h = _r(g, N, W).to(dtype)
    _close(m(_dev(h))["b"], O.dense_ff(h.to(F64), {k: v.to(F64) for k, v in w.items()}), dtype, 2)
