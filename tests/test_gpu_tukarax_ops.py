"""Kernels of the Tukarax decoder against the plain fp64 functions, one mechanism at a time."""
import pytest
import torch

from oracle import tukarax_oracle as O

pytestmark = pytest.mark.gpu
F64, BF = torch.float64, torch.bfloat16
DTYPES = [torch.float32, BF]


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _r(g, *s, k=1.0):
    return torch.randn(*s, generator=g) * k


def _dev(t, dtype=None):
    return (t if dtype is None else t.to(dtype)).cuda()


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


# -- queries and keys on their way to attention ----------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Hkv,D,DV,dims,inter,norm,scaled", [
    (4, 2, 40, 24, 16, False, False, True), (6, 1, 128, 128, 128, True, True, False), (3, 3, 13, 11, 6, False, True, True),
    (5, 1, 72, 72, 20, True, True, True), (2, 2, 176, 48, 176, False, True, False), (10, 5, 9, 9, 2, True, False, False)])
def test_norm_rotation_and_store(Hq, Hkv, D, DV, dims, inter, norm, scaled, dtype):
    from zipage_b200.layers.rotary import Rotary, rotate_store
    g = _gen(D)
    N, eps, shared = 23, 1e-2, DV == D and norm
    rot = {"dims": dims, "base": 3000.0}
    if scaled:
        rot["scaling"] = {"factor": 5.0, "original": 100, "fast": 6.0, "slow": 0.7}
    y = _r(g, N, 3 + Hq * D + Hkv * (D + DV), k=0.3).to(dtype)
    pos = torch.cat([torch.arange(12), torch.tensor([100003, 77, 5000, 64, 63, 1, 0, 2, 999, 31, 12345])])
    slots = torch.randperm(128, generator=g)[:N].to(torch.int32)
    slots[3], slots[7] = -1, 128
    wq, wk = (1 + _r(g, D, k=0.3), 1 + _r(g, D, k=0.3)) if norm else (None, None)
    KP, VP = (D + 15) // 16 * 16, (DV + 15) // 16 * 16
    kc, vc = (torch.full((2, 64, Hkv, p), 7.0, dtype=dtype, device="cuda") for p in (KP, VP))
    yd = _dev(y.clone())
    nq, nk = Hq * D, Hkv * D
    q, k, v = yd[:, :nq], yd[:, nq:nq + nk], yd[:, nq:nq + nk] if shared else yd[:, nq + nk:nq + nk + Hkv * DV]
    R = Rotary.from_config(rot, inter, "cuda")
    rotate_store(q, k, v, _dev(pos), R, kc, vc, _dev(slots), D, DV, *(None if w is None else _dev(w) for w in (wq, wk)), eps)
    Y = y.to(F64)

    def want(x, heads, w):
        x = x.reshape(N, heads, D)
        return O.rotate(x if w is None else O.rms(x, eps) * w.to(F64), pos, rot, inter)
    _close(yd[:, :nq].reshape(N, Hq, D), want(Y[:, :nq], Hq, wq), dtype)
    assert torch.equal(yd[:, nq:].cpu(), y[:, nq:])                        # keys and values as they were
    keep = (slots >= 0) & (slots < 128)
    at = slots[keep].long().cuda()
    _close(kc.view(128, Hkv, KP)[at][..., :D], want(Y[:, nq:nq + nk], Hkv, wk)[keep], dtype)
    values = y[:, nq:nq + nk] if shared else y[:, nq + nk:nq + nk + Hkv * DV]
    assert torch.equal(vc.view(128, Hkv, VP)[at][..., :DV].cpu(), values.reshape(N, Hkv, DV)[keep])
    rest = torch.ones(128, dtype=torch.bool, device="cuda")
    rest[at] = False
    for c, d in ((kc, D), (vc, DV)):
        flat = c.view(128, Hkv, -1)
        assert (flat[rest] == 7).all() and (flat[..., d:] == 7).all()


# -- attention with masks, soft cap, sink and gates --------------------------------------------------------
def _paged(rows, BS, g):
    """rows: list of [ctx, heads, width] -> (cache with pages in random order and others' rows around, table)."""
    need = [(len(r) + BS - 1) // BS for r in rows]
    P = sum(need) + 3
    _, H, d = rows[0].shape
    pad = (d + 15) // 16 * 16
    cache = torch.zeros(P, BS, H, pad)
    cache[..., :d] = torch.randn(P, BS, H, d, generator=g) * 5
    order = torch.randperm(P, generator=_gen(5)).tolist()
    table = torch.full((len(rows), max(need) + 1), -1, dtype=torch.int32)
    for b, r in enumerate(rows):
        for i in range(need[b]):
            page = order.pop()
            table[b, i] = page
            part = r[i * BS:(i + 1) * BS]
            cache[page, :len(part), :, :d] = part
    return cache.to(rows[0].dtype), table


def _attend(dtype, impl, H, G, d, dv, ctxs, counts, chunk, softcap, sink, mode, seed=0, decode=False, steep=0.0, BS=64, out_scale=0.7):
    from zipage_b200.layers.attention import window_attention
    g = _gen(seed)
    ks, vs = [_r(g, c, G, d).to(dtype) for c in ctxs], [_r(g, c, G, dv).to(dtype) for c in ctxs]
    q = _r(g, sum(counts), H * d + (8 if impl == "tcgen05" else 5), k=2.0).to(dtype)
    if steep:      # scores that climb along the sequence by far more than fp32 exponents absorb
        for k in ks:
            k[..., 0] = (torch.arange(len(k)) * steep)[:, None].to(dtype)
        q[:, 0:H * d:d] = 1.0
    kc, table = _paged(ks, BS, g)
    vc, _ = _paged(vs, BS, g)
    width = {None: 1, "head": H, "entry": H * dv}[mode]
    gate = _r(g, sum(counts), width + 8, k=2.0).to(dtype)
    s = _r(g, H, k=2.0) if sink else None
    scale, at, want = d ** -0.5, 0, []
    for k, v, n in zip(ks, vs, counts):
        o = O.softmax_attention(q[at:at + n, :H * d].to(F64).reshape(n, H, d), k.to(F64), v.to(F64), scale, softcap, chunk,
                                None if s is None else s.to(F64))
        z = torch.sigmoid(gate[at:at + n, :width].to(F64))
        if mode:
            o = o * (z[:, :, None] if mode == "head" else z.view(n, H, dv))
        want.append(o.flatten(1) * out_scale)
        at += n
    cu = None if decode else _i32([0] + torch.tensor(counts).cumsum(0).tolist())
    out = torch.full((sum(counts), H * dv + 8), 9.0, dtype=dtype, device="cuda")
    window_attention(_dev(q)[:, :H * d], _dev(kc), _dev(vc), _i32(ctxs), _dev(table), H, d, dv, scale, 0, softcap, cu_seqlens_q=cu,
                     max_seqlen_q=max(counts), out=out[:, :H * dv], impl=impl, chunk=chunk, sink=None if s is None else _dev(s),
                     gate=_dev(gate)[:, :width] if mode else None, gate_mode=mode, out_scale=out_scale)
    _check_device()
    assert (out[:, H * dv:] == 9).all()
    _close(out[:, :H * dv], torch.cat(want), dtype)


MASKS = [(0, 0.0, False, "entry"), (70, 20.0, True, "head"), (33, 50.0, True, None), (64, 0.0, True, "entry"), (0, 90.0, True, "head"),
         (1, 30.0, True, "head"), (128, 0.0, False, None)]


@pytest.mark.parametrize("chunk,softcap,sink,mode", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 48, 40), (8, 1, 128, 128), (3, 3, 13, 11), (2, 1, 176, 208)])
def test_attention_of_portions(H, G, d, dv, chunk, softcap, sink, mode):
    ctxs, counts = [200, 71, 2, 130, 64, 1, 300], [200, 3, 2, 66, 2, 1, 131]
    for dtype, impl in ((torch.float32, "auto"), (BF, "auto"), (BF, "simt")):
        _attend(dtype, impl, H, G, d, dv, ctxs, counts, chunk, softcap, sink, mode)


@pytest.mark.parametrize("chunk,softcap,sink,mode", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 48, 40), (8, 1, 128, 128), (6, 3, 96, 128), (2, 2, 72, 16)])
def test_attention_of_portions_tcgen05(H, G, d, dv, chunk, softcap, sink, mode):
    if softcap > 69:
        pytest.skip("the kernel takes caps up to 69")
    ctxs, counts = [200, 71, 2, 130, 64, 1, 400], [200, 3, 2, 66, 2, 1, 290]
    _attend(BF, "tcgen05", H, G, d, dv, ctxs, counts, chunk, softcap, sink, mode)
    for steep in (1.5, 40.0):                             # (without a cap, references that move)
        if not softcap:
            _attend(BF, "tcgen05", H, G, d, dv, ctxs, counts, chunk, softcap, sink, mode, steep=steep)


@pytest.mark.parametrize("chunk,softcap,sink,mode", MASKS)
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 48, 40), (8, 1, 128, 128), (3, 3, 13, 11), (2, 1, 176, 208), (20, 1, 32, 16)])
def test_attention_of_decoded_tokens(H, G, d, dv, chunk, softcap, sink, mode):
    ctxs = [1, 2, 63, 64, 65, 70, 71, 140, 141, 128, 129, 1000]
    for dtype in DTYPES:
        _attend(dtype, "auto", H, G, d, dv, ctxs, [1] * len(ctxs), chunk, softcap, sink, mode, decode=True)


def test_attention_limits_of_the_tcgen05_kernel():
    from zipage_b200._lib import ZipageError
    for kw in (dict(softcap=90.0), dict(d=13), dict(d=144)):
        with pytest.raises(ZipageError):
            _attend(BF, "tcgen05", 2, 1, kw.get("d", 64), 32, [70], [70], 0, kw.get("softcap", 0.0), True, None)


@pytest.mark.parametrize("chunk", [64, 70, 100])
def test_keys_at_the_edges_of_chunks(chunk):
    """A key whose score stands out is the output of the rows of its chunk that follow it, and of no other row."""
    from zipage_b200.layers.attention import window_attention
    d, T = 128, 250
    g = _gen(chunk)
    for place in (0, chunk - 1, chunk, 2 * chunk - 1, 2 * chunk, 63, 64, 127, 128):
        q = torch.zeros(T, d)
        q[:, 0] = 1.0
        k, v = torch.zeros(T, 1, d), _r(g, T, 1, d)
        k[place, 0, 0] = 300.0
        v[:, 0, 5] = 0.0
        v[place, 0, 5] = 1.0
        kc, table = _paged([k.to(BF)], 64, g)
        vc, _ = _paged([v.to(BF)], 64, g)
        p = torch.arange(T)
        sees = (p >= place) & (p // chunk == place // chunk)
        for dtype, impl in ((BF, "tcgen05"), (BF, "auto"), (torch.float32, "simt")):
            args = _dev(q, dtype), _dev(kc, dtype), _dev(vc, dtype)
            o = window_attention(*args, _i32([T]), _dev(table), 1, d, d, 0.1, cu_seqlens_q=_i32([0, T]), max_seqlen_q=T, chunk=chunk, impl=impl)
            assert torch.equal(o[:, 5].float().cpu() > 0.5, sees) and (o[~sees.cuda(), 5] == 0).all()
            last = [c for c in (place, place + 1, place + 2, chunk, chunk + 1, 2 * chunk, 2 * chunk + 1, T) if 0 < c <= T]
            o = window_attention(args[0][:len(last)], *args[1:], _i32(last), _dev(table).expand(len(last), -1).contiguous(), 1, d, d, 0.1, chunk=chunk)
            assert torch.equal(o[:, 5].float().cpu() > 0.5, sees[torch.tensor(last) - 1])
    _check_device()


# -- gated delta rule -----------------------------------------------------------------------------------------
def _delta_case(H, G, dk, dv, T, seed=0, fast=False):
    """Inputs of one sequence (fp64) and what they give: rows of q | k | v before the convolution, ..."""
    g = _gen(seed)
    C = 2 * G * dk + H * dv
    return {"x": _r(g, T, C), "gate": _r(g, T, H * dv, k=2.0), "ab": torch.cat([_r(g, T, H), _r(g, T, H, k=2.0)], 1),
            "A_log": torch.rand(H, generator=g) * (2 if fast else 4) - (0 if fast else 3), "dt": torch.rand(H, generator=g) * 4 - (0 if fast else 4),
            "norm": 1 + _r(g, dv, k=0.2)}


def _delta_want(cs, H, G, dk, dv, eps, x=None, S=None):
    """-> gated output [T, H * dv], state.  x: rows after the convolution."""
    x = cs["x"].to(F64) if x is None else x
    T = len(x)
    q, k = O.unit(x[:, :G * dk].reshape(T, G, dk)) * dk ** -0.5, O.unit(x[:, G * dk:2 * G * dk].reshape(T, G, dk))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    ab = cs["ab"].to(F64)
    dec = torch.exp(-torch.exp(cs["A_log"].to(F64)) * torch.nn.functional.softplus(ab[:, :H] + cs["dt"].to(F64)))
    o, S = O.delta_recurrence(q, k, x[:, 2 * G * dk:].reshape(T, H, dv), dec, torch.sigmoid(ab[:, H:]), S)
    o = O.rms(o, eps) * cs["norm"].to(F64) * O.silu(cs["gate"].to(F64)).view(T, H, dv)
    return o.flatten(1), S


SIZES = [(6, 2, 40, 56), (4, 4, 128, 128), (6, 3, 64, 120), (3, 3, 9, 7), (2, 1, 160, 200), (1, 1, 300, 33), (2, 2, 16, 304), (8, 1, 8, 8), (2, 1, 96, 256), (3, 1, 128, 72)]


@pytest.mark.parametrize("fast", [False, True])
@pytest.mark.parametrize("H,G,dk,dv", SIZES)
def test_delta_portions(H, G, dk, dv, fast):
    """Portions of unequal length, each on the state that the one before left, in slots that held others' numbers."""
    from zipage_b200.layers.gated_delta import gated_delta
    eps, sc = 1e-3, 0.8
    plans = [[130, 64, 2], [2, 63, 70], [65, 1, 200]]
    cases = [_delta_case(H, G, dk, dv, sum(p), 10 + i, fast) for i, p in enumerate(plans)]
    impls = [(torch.float32, "auto"), (BF, "simt")]
    if dk % 8 == dv % 8 == 0 and dk <= 128 and dv <= 256:
        impls.append((BF, "tcgen05"))
    for dtype, impl in impls:
        for c in cases:
            c["x"], c["gate"] = c["x"].to(dtype).float(), c["gate"].to(dtype).float()
        VP = (dv + 3) // 4 * 4
        state = torch.full((5, H, dk, VP), 3.0, device="cuda")
        slots, done, outs = [3, 0, 4], [0, 0, 0], [[], [], []]
        shared = {n: _dev(cases[0][n]) for n in ("A_log", "dt", "norm")}
        for step in range(3):
            n = [p[step] for p in plans]
            rows = lambda key: torch.cat([c[key][d:d + m] for c, d, m in zip(cases, done, n)])
            lead = 4                                               # rows of other sequences ahead of the portions'
            pad = lambda t: torch.cat([torch.zeros(lead, t.shape[1]), t])
            x, gate, ab = (_dev(pad(rows(k)), dt) for k, dt in (("x", dtype), ("gate", dtype), ("ab", torch.float32)))
            done = [d + m for d, m in zip(done, n)]
            out = torch.full((x.shape[0], H * dv), 9.0, dtype=dtype, device="cuda")
            cu = _i32([lead] + [lead + v for v in torch.tensor(n).cumsum(0).tolist()])
            gated_delta(x, gate, ab, shared["A_log"], shared["dt"], shared["norm"], state, out, _i32(done), _i32(slots), H, G, dk, dv, eps, sc,
                        cu_seqlens_q=cu, impl=impl)
            _check_device()
            assert (out[:lead] == 9).all()
            for i, part in enumerate(out[lead:].split(n)):
                outs[i].append(part.cpu())
        for i, c in enumerate(cases):
            c0 = {**c, **{k: cases[0][k] for k in ("A_log", "dt", "norm")}}
            want, S = _delta_want(c0, H, G, dk, dv, eps)
            _close(torch.cat(outs[i]), want * sc, dtype, 2 if dtype == BF else 5)
            _close(state[slots[i]][..., :dv], S, torch.float32, 20 if dtype == torch.float32 else 40)
        assert (state[[1, 2]] == 3).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,dk,dv,taps", [(6, 2, 40, 56, 4), (4, 4, 128, 128, 3), (3, 3, 9, 7, 5), (2, 1, 160, 200, 2), (1, 1, 8, 12, 1), (32, 16, 64, 64, 4)])
def test_delta_convolution_prompts_and_decoding(H, G, dk, dv, taps, dtype):
    """Prompts through the convolution, then single rows with the convolution in the launch, then portions again: outputs, state and
    the convolution's memory carry over; a batch of two sequences out of step, and a padding row."""
    from zipage_b200.layers.gated_delta import gated_delta, short_conv
    g = _gen(taps)
    eps, T = 1e-3, [41, 30]
    C = 2 * G * dk + H * dv
    cases = [_delta_case(H, G, dk, dv, t, 20 + i) for i, t in enumerate(T)]
    for c in cases:
        c["x"], c["gate"] = c["x"].to(dtype).float(), c["gate"].to(dtype).float()
    w = _r(g, C, taps, k=0.7)
    wd = _dev(w.t().contiguous())
    VP = (dv + 3) // 4 * 4
    state, ring = torch.full((4, H, dk, VP), 3.0, device="cuda"), torch.full((4, taps, C), 5.0, dtype=dtype, device="cuda")
    sh = [_dev(cases[0][n]) for n in ("A_log", "dt", "norm")]
    slots, at, outs = [2, 0], [0, 0], [[], []]

    def run(n, decode):
        x, gate, ab = (_dev(torch.cat([c[k][a:a + m] for c, a, m in zip(cases, at, n)]), dt) for k, dt in (("x", dtype), ("gate", dtype), ("ab", torch.float32)))
        live = [i for i in range(2) if n[i]]
        for i in live:
            at[i] += n[i]
        ctx, sl = [at[i] for i in live], [slots[i] for i in live]
        wide = torch.zeros(len(x) + decode, C + 8, dtype=dtype, device="cuda")       # rows of a wider projection
        wide[:len(x), :C] = x
        out = torch.full((len(x) + decode, H * dv), 9.0, dtype=dtype, device="cuda")
        if decode:                                                                   # (the last row pads the batch)
            z = lambda t: torch.cat([t, torch.zeros_like(t[:1])])
            gated_delta(wide[:, :C], z(gate), z(ab), *sh, state, out, _i32(ctx + [0]), _i32(sl + [-1]), H, G, dk, dv, eps, conv_weight=wd, ring=ring)
            assert (out[-1] == 9).all()
        else:
            m = [n[i] for i in live]
            cu = _i32([0] + torch.tensor(m).cumsum(0).tolist())
            y = torch.empty(len(x), C, dtype=dtype, device="cuda")
            short_conv(wide[:, :C], wd, ring, _i32(ctx), _i32(sl), cu, max(m), y)
            gated_delta(y, gate, ab, *sh, state, out, _i32(ctx), _i32(sl), H, G, dk, dv, eps, cu_seqlens_q=cu)
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
        conv = O.short_conv(c["x"].to(F64), w.to(F64))
        want, S = _delta_want({**c, **{k: cases[0][k] for k in ("A_log", "dt", "norm")}}, H, G, dk, dv, eps, conv)
        _close(torch.cat(outs[i]), want, dtype, 4 if dtype == BF else 5)
        _close(state[slots[i]][..., :dv], S, torch.float32, 30 if dtype == torch.float32 else 600)       # (bf16: rounded q, k, v of prompts)
        held = torch.stack([c["x"][p] for p in range(T[i] - min(taps, T[i]), T[i])])
        for p, row in zip(range(T[i] - taps, T[i]), held):
            assert torch.equal(ring[slots[i], p % taps].float().cpu(), row)
    assert (state[[1, 3]] == 3).all() and (ring[[1, 3]] == 5).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,taps", [(96, 2), (100, 3), (37, 4), (2056, 4), (40, 8), (16, 1)])
def test_short_convolution(C, taps, dtype):
    """Portions of every length around the number of taps and the run of a thread, with what earlier portions left."""
    from zipage_b200.layers.gated_delta import short_conv
    g = _gen(C)
    plan = [[2, 1, 16, 17, 3, 33, 5], [70, 2, 1, 1, 1, 1, 1]]
    xs = [_r(g, sum(p), C).to(dtype) for p in plan]
    w = _r(g, C, taps)
    ring = torch.full((3, taps, C), 5.0, dtype=dtype, device="cuda")
    at, outs = [0, 0], [[], []]
    for step in zip(*plan):
        x = torch.cat([s[a:a + n] for s, a, n in zip(xs, at, step)])
        at = [a + n for a, n in zip(at, step)]
        y = torch.empty(len(x), C, dtype=dtype, device="cuda")
        short_conv(_dev(x), _dev(w.t().contiguous()), ring, _i32(at), _i32([1, 2]), _i32([0, step[0], sum(step)]), max(step), y)
        for o, part in zip(outs, y.split(step)):
            o.append(part.cpu())
    for o, x in zip(outs, xs):
        _close(torch.cat(o), O.short_conv(x.to(F64), w.to(F64)), dtype)
    assert (ring[0] == 5).all()


def test_delta_keeps_a_far_write():
    """With next to no decay a value written once comes back hundreds of tokens later, across chunks, portions and slots."""
    from zipage_b200.layers.gated_delta import gated_delta
    T, d = 400, 128
    g = _gen(4)
    for dtype, impl in ((BF, "tcgen05"), (BF, "simt"), (torch.float32, "auto")):
        for place in (0, 63, 64, 100):
            x = torch.zeros(T, 3 * d)
            k = torch.nn.functional.normalize(_r(g, d), dim=0)
            other = _r(g, T, d)
            x[:, d:2 * d] = other - (other @ k)[:, None] * k           # other keys: orthogonal to the one that counts
            x[place, d:2 * d] = k * 4
            x[:, 2 * d:] = _r(g, T, d, k=0.2)
            x[:, :d] = x[:, d:2 * d]
            x[T - 1, :d] = k * 3
            ab = torch.cat([torch.full((T, 1), -25.0), torch.full((T, 1), 20.0)], 1)
            state, slots = torch.zeros(1, 1, d, d, device="cuda"), _i32([0])
            out, o = [], torch.empty(T, d, dtype=dtype, device="cuda")
            for a, b in ((0, 150), (150, 399), (399, 400)) if impl != "tcgen05" else ((0, 150), (150, 400)):
                gated_delta(_dev(x[a:b], dtype), torch.ones(b - a, d, dtype=dtype, device="cuda"), _dev(ab[a:b]), torch.zeros(1, device="cuda"),
                            torch.zeros(1, device="cuda"), torch.ones(d, device="cuda"), state, o[a:b], _i32([b]), slots, 1, 1, d, d, 1e-6,
                            cu_seqlens_q=_i32([0, b - a]), impl=impl)
            _check_device()
            v = x[place, 2 * d:]
            want = O.rms(v.to(F64) * d ** -0.5, 1e-6) * O.silu(torch.ones((), dtype=F64))
            _close(o[-1], want, dtype, 4 if dtype == BF else 20)


def test_delta_with_repeated_keys_and_full_steps():
    """Steps near one on keys that repeat and alternate in sign: the worst case for the inverse of a chunk's system."""
    from zipage_b200.layers.gated_delta import gated_delta
    T, d = 192, 64
    g = _gen(9)
    for sign in (False, True):
        cs = _delta_case(2, 1, d, d, T, 3)
        base = _r(g, 1, d)
        cs["x"][:, d:2 * d] = base * (torch.where(torch.arange(T) % 2 == 0, 1.0, -1.0)[:, None] if sign else 1.0) + _r(g, T, d, k=0.02)
        cs["ab"][:, :2], cs["ab"][:, 2:] = -12.0, 9.0
        cs["x"], cs["gate"] = cs["x"].to(BF).float(), cs["gate"].to(BF).float()
        want, _ = _delta_want(cs, 2, 1, d, d, 1e-5)
        for impl in ("tcgen05", "simt"):
            state, out = torch.zeros(1, 2, d, d, device="cuda"), torch.empty(T, 2 * d, dtype=BF, device="cuda")
            gated_delta(_dev(cs["x"], BF), _dev(cs["gate"], BF), _dev(cs["ab"]), _dev(cs["A_log"]), _dev(cs["dt"]), _dev(cs["norm"]), state, out,
                        _i32([T]), _i32([0]), 2, 1, d, d, 1e-5, cu_seqlens_q=_i32([0, T]), impl=impl)
            _check_device()
            _close(out, want, BF, 3)


# -- boundary, experts -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [136, 58, 2052, 8192])
def test_boundary_with_rms_norms(W, dtype):
    from zipage_b200.layers.row_ops import join_norms
    g = _gen(W)
    N, top, eps = 7, 3, 1e-2
    x, a, y, w = _r(g, N, W) + 3.0, _r(g, N, W).to(dtype), _r(g, N * top, W).to(dtype), _r(g, W)
    pos = torch.randperm(N * top, generator=g).view(N, top).to(torch.int32)
    D = lambda t: t.to(F64)
    for kw, want in (({}, D(x)), ({"a": a}, D(x) + D(a)), ({"y": y, "pos": pos}, D(x) + D(y)[pos.long()].sum(1))):
        xd = _dev(x.clone())
        out, = join_norms(xd, [(_dev(w), None)], eps, dtype, rms=True, **{k: _dev(t) for k, t in kw.items()})
        _close(xd, want, torch.float32)
        _close(out, O.rms(want, eps) * D(w), dtype)


@pytest.mark.parametrize("N,E,top", [(1, 11, 2), (7, 5, 5), (300, 64, 6), (513, 11, 2), (3000, 300, 8), (700, 1, 1)])
def test_sigmoid_routing(N, E, top):
    from zipage_b200.layers.feed_forward import moe_route
    z = _r(_gen(N), N, E + 3, k=3.0)
    i, s = O.route(z[:, :E].to(F64), top)
    w, experts, places, rows, offsets = moe_route(_dev(z), E, top, "sigmoid")
    assert torch.equal(experts.cpu().long(), i)
    _close(w, s, torch.float32)
    pw, experts, places, rows, offsets = moe_route(_dev(z), E, top, "sigmoid", by_place=True)
    p = places.cpu().long()
    assert torch.equal(experts.cpu().long(), i) and torch.equal(rows.cpu().long()[p], torch.arange(N)[:, None].expand(N, top))
    assert torch.equal(pw.cpu()[p], w.cpu())


@pytest.mark.parametrize("N,E,top,ff,W", [(1, 5, 2, 40, 136), (90, 7, 3, 24, 64), (700, 3, 2, 136, 128), (40, 6, 6, 11, 58), (300, 12, 1, 16, 200)])
def test_gated_experts_on_scaled_inputs(N, E, top, ff, W):
    from zipage_b200.layers.feed_forward import GatedMixtureFF, grouped_gemm, moe_route, padded_ff
    g = _gen(N)
    for dtype in DTYPES:
        w = {f"e{e}.{n}": (_r(g, *s) / W ** 0.5 * 2).to(dtype) for e in range(E) for n, s in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff)))}
        w["router"] = (_r(g, E, W) / W ** 0.5 * 3).to(dtype)
        m = GatedMixtureFF(W, E, top, ff, dtype, torch.device("cuda"))
        m.load(lambda n: w[n])
        h = _r(g, N, W).to(dtype)
        out = m(_dev(h))
        pos = out["pos"].cpu().long()
        # the kernels' own choice: rounding may turn a close call
        got = out["y"].double().cpu()[pos].sum(1)
        z = _dev(h).float() @ _dev(w["router"]).float().t()
        _, experts, *_ = moe_route(z, E, top, "sigmoid")
        W64 = {k: v.to(F64) for k, v in w.items()}
        sc = torch.sigmoid(h.to(F64) @ W64["router"].T)
        want = torch.stack([sum(O.expert(sc[t, e] * h[t:t + 1].to(F64), W64, e)[0] for e in experts[t].tolist()) for t in range(N)])
        _close(got, want, dtype, 3 if dtype == BF else 1)
        if dtype == BF and W % 8 == 0:
            _, _, _, rows, off = moe_route(z, E, top, "sigmoid")
            s = torch.rand(N * top, generator=g)
            x, mid = _dev(h), []
            for impl in ("tcgen05", "simt"):
                mid.append(grouped_gemm(x, m.gate_up, off, N * top, rows=rows, act="silu_mul", row_scale=_dev(s), impl=impl))
            _check_device()
            assert mid[0].shape[1] == padded_ff(ff) and (mid[0][:, ff:] == 0).all()
            _close(mid[0], mid[1].double().cpu(), BF, 2)
