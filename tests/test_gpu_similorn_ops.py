"""Each mechanism of the Similorn decoder alone: the kernels against the plain fp64 equations.

Inputs are rounded to the tested dtype first, so what is measured is the kernels' arithmetic.
"""
import pytest
import torch

from oracle import similorn_oracle as O

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32
F64 = torch.float64


def _rand(*shape, seed=0, scale=1.0, dtype=F32):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype)


def _close(got, want, rel, what=""):
    err = (got.double().cpu() - want.double()).abs().max().item()
    size = want.double().abs().max().item()
    assert err <= rel * size, f"{what}: {err:.3e} of {size:.3e}"


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [58, 96, 131])
def test_embedding(dtype, width):
    from zipage_b200.layers.row_ops import embed_position, sinusoid_turns
    table = _rand(40, width, dtype=dtype)
    tok = torch.randint(0, 40, (9,), generator=torch.Generator().manual_seed(2))
    pos = torch.tensor([0, 1, 2, 63, 64, 100, 2047, 5000, 65535])
    x, xt = embed_position(tok.cuda(), pos.cuda(), table.cuda(), 7.5, sinusoid_turns(width, "cuda"), want_t=True)
    want = O.embedding(tok, pos, table.double(), 7.5)
    _close(x, want, 1e-6, "fp32")
    assert torch.equal(xt.cpu(), x.cpu().to(dtype))
    plain = embed_position(tok.cuda(), pos.cuda(), table.cuda(), 7.5)
    _close(plain, table[tok].double() * 7.5, 1e-6, "without positions")


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("width", [50, 128, 1028, 2048, 4100, 8192, 9001])
def test_norm_with_offset_weight(dtype, width):
    from zipage_b200.layers.row_ops import rms_norm_f32
    x, w = _rand(5, width, scale=3.0), _rand(width, seed=1, scale=0.3)
    x[3] *= 1e-3                                                    # eps matters here
    got = rms_norm_f32(x.cuda(), w.cuda(), 1e-3, dtype, offset=1.0)
    want = O.norm_about_one(x.double(), w.double(), 1e-3)
    _close(got[3], want[3], 5e-3 if dtype == BF else 1e-5)
    _close(got, want, 5e-3 if dtype == BF else 1e-5)
    assert torch.equal(rms_norm_f32(x.cuda(), None, 0.0, dtype).cpu(), x.to(dtype))


@pytest.mark.parametrize("dtype", [BF, F32])
def test_gelu(dtype):
    from zipage_b200.layers.row_ops import gelu_tanh
    x = torch.cat([torch.linspace(-30, 30, 4001), torch.tensor([0.0, 1e4, -1e4, 1e-6])]).to(dtype)
    got, want = gelu_tanh(x.cuda()).cpu().double(), O.gelu_tanh(x.double())
    assert ((got - want).abs() <= (4e-3 if dtype == BF else 1e-5) * want.abs() + 1e-6).all()


# (heads, kv heads, dim, vdim)
SHAPES = [(4, 2, 40, 56), (3, 1, 13, 19), (8, 8, 64, 32), (16, 1, 128, 128), (5, 5, 96, 256), (2, 1, 256, 72)]


def _paged(k, v, block, seed):
    """Scatter keys and values into padded caches at random pages, other rows filled with large values
    (a key that is read although nobody may see it changes the result)."""
    from zipage_b200.layers.attention import store_kv_padded
    S, G, dk = k.shape
    dv = v.shape[2]
    nb = (S + block - 1) // block
    pages = nb + 3
    g = torch.Generator().manual_seed(seed)
    table = torch.randperm(pages, generator=g)[:nb].to(torch.int32)
    pad = lambda n: (n + 15) // 16 * 16
    kc = torch.zeros(pages, block, G, pad(dk), dtype=k.dtype, device="cuda")
    vc = torch.zeros(pages, block, G, pad(dv), dtype=k.dtype, device="cuda")
    kc[..., :dk], vc[..., :dv] = 3.0, 50.0
    slots = (table.long().repeat_interleave(block)[:S] * block + torch.arange(S) % block).to(torch.int32)
    kv = torch.cat([k.reshape(S, -1), v.reshape(S, -1)], 1).cuda()
    store_kv_padded(kv[:, :G * dk], kv[:, G * dk:], kc, vc, slots.cuda(), dk, dv)
    return kc, vc, table


@pytest.mark.parametrize("dtype,impl", [(BF, "auto"), (BF, "simt"), (torch.float16, "auto"), (F32, "auto")])
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,softcap", [(70, 15.0), (64, 50.0), (1, 0.0), (0, 30.0), (129, 300.0)])
def test_window_attention(dtype, impl, shape, window, softcap):
    """Portions at several places of several sequences in one launch, then single rows; a key that
    dominates sits at the last visible and at the first hidden distance of some rows."""
    from zipage_b200.layers.attention import window_attention
    H, G, dk, dv = shape
    block, S = 64, 260
    # (context, rows): whole prompt, a portion over a page edge, two tokens, one token
    parts = [(200, 200), (S, 70), (131, 2), (65, 1), (64, 33)]
    caches, tables, qs, wants = None, [], [], []
    P = 0
    kcs, vcs = [], []
    for n, (ctx, rows) in enumerate(parts):
        q, k, v = (_rand(ctx, h, d, seed=10 * n + i) for i, (h, d) in enumerate([(H, dk), (G, dk), (G, dv)]))
        if window > 1:
            for edge, back in ((ctx - 1, window - 1), (ctx - 2, window)):   # just inside, just outside
                if 0 <= edge - back:
                    k[edge - back] = q[edge].view(G, H // G, dk)[:, 0] * 6.0 / q[edge].view(G, H // G, dk)[:, 0].norm(dim=-1, keepdim=True) * 4
                    v[edge - back] *= 4
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        kc, vc, t = _paged(k, v, block, n)
        tables.append(t + P)
        P += kc.shape[0]
        kcs.append(kc)
        vcs.append(vc)
        qs.append(q[ctx - rows:].reshape(rows, -1))
        wants.append(O.window_attention(q[ctx - rows:].double(), k.double(), v.double(), dk ** -0.5, softcap, window).flatten(1))
    kc, vc = torch.cat(kcs), torch.cat(vcs)
    nb = max(len(t) for t in tables)
    bt = torch.full((len(parts), nb), -1, dtype=torch.int32)
    for i, t in enumerate(tables):
        bt[i, :len(t)] = t
    rows = [r for _, r in parts]
    cu = torch.tensor([0] + torch.tensor(rows).cumsum(0).tolist(), dtype=torch.int32).cuda()
    ctx = torch.tensor([c for c, _ in parts], dtype=torch.int32).cuda()
    # q as a column view of a wider projection
    wide = torch.cat([torch.cat(qs), torch.zeros(sum(rows), 8, dtype=dtype)], 1).cuda()
    q = wide[:, :H * dk]
    got = window_attention(q, kc, vc, ctx, bt.cuda(), H, dk, dv, dk ** -0.5, window, softcap, cu_seqlens_q=cu,
                           max_seqlen_q=max(rows), impl=impl)
    tol = {BF: 6e-3, torch.float16: 1.5e-3, F32: 2e-6}[dtype]
    for i in range(len(parts)):
        _close(got[cu[i]:cu[i + 1]], wants[i], tol, f"portion {i}")
    last = cu[1:].long() - 1
    one = window_attention(q[last].contiguous(), kc, vc, ctx, bt.cuda(), H, dk, dv, dk ** -0.5, window, softcap, impl=impl)
    for i in range(len(parts)):
        _close(one[i], wants[i][-1], tol, f"single row {i}")


def test_window_attention_weights_are_not_rounded():
    """bf16 operands, fp32 softmax: with values that cancel, weights rounded to 8 bits would miss by far."""
    from zipage_b200.layers.attention import window_attention
    dk = dv = 32
    S = 192
    q, k = _rand(S, 1, dk, seed=1, dtype=BF), _rand(S, 1, dk, seed=2, scale=0.1, dtype=BF)
    v = torch.ones(S, 1, dv) * 64
    v[1::2] = -64
    v += _rand(S, 1, dv, seed=3) * 0.01
    v = v.to(BF)
    kc, vc, t = _paged(k, v, 64, 0)
    want = O.window_attention(q.double(), k.double(), v.double(), dk ** -0.5, 20.0, 128).flatten(1)
    ctx, cu = torch.tensor([S], dtype=torch.int32).cuda(), torch.tensor([0, S], dtype=torch.int32).cuda()
    got = window_attention(q.reshape(S, -1).cuda(), kc, vc, ctx, t[None].cuda(), 1, dk, dv, dk ** -0.5, 128, 20.0,
                           cu_seqlens_q=cu, max_seqlen_q=S).double().cpu()
    err = (got - want).abs()
    assert (err <= 2 ** -8 * want.abs() + 3e-3).all(), err.max()


# (heads, dim, vdim)
MEMORIES = [(3, 24, 40), (2, 64, 64), (1, 128, 256), (2, 17, 23), (1, 200, 72), (1, 256, 512), (4, 32, 130), (2, 80, 600)]


def _mlstm_inputs(H, dk, dv, n, seed, dtype, gate_scale=2.0):
    x = _rand(n, 2 * H * (dk + dv), seed=seed, dtype=dtype)
    gates = _rand(n, 2 * H, seed=seed + 1, scale=gate_scale)
    bias = torch.cat([_rand(H, seed=3), _rand(H, seed=4) + 2.0])
    norm = _rand(H * dv, seed=5, scale=0.3) + 1.0
    return x, gates, bias, norm


def _mlstm_want(x, gates, bias, norm, H, dk, dv, cap, eps, state=None):
    n = x.shape[0]
    x, g = x.double(), gates.double() + bias.double()
    q, k, v, og = x.split([H * dk, H * dk, H * dv, H * dv], 1)
    i = cap * torch.tanh(g[:, :H] / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(g[:, H:] / cap))
    o, state = O.mlstm_recurrence(q.view(n, H, dk) * dk ** -0.5, k.view(n, H, dk), v.view(n, H, dv), i, f, state)
    return O.mlstm_output(o, og, norm.double(), eps), state


def _mlstm_state(slots, H, dk, dv):
    junk = lambda *s: torch.full(s, 7.0, device="cuda")            # what an earlier owner left
    return junk(slots, H, dk, (dv + 3) // 4 * 4), junk(slots, H, dk), junk(slots, H)


def _mlstm_run(x, gates, bias, norm, state, ctx, slots, H, dk, dv, cap, eps, cu=None, impl="auto"):
    from zipage_b200.layers.mlstm import mlstm_step
    x = x.cuda()
    q, k, v, g = x[:, :H * dk], x[:, H * dk:2 * H * dk], x[:, 2 * H * dk:2 * H * dk + H * dv], x[:, 2 * H * dk + H * dv:]
    out = torch.empty(x.shape[0], H * dv, dtype=x.dtype, device="cuda")
    i32 = lambda a: torch.tensor(a, dtype=torch.int32).cuda()
    return mlstm_step(q, k, v, g, gates.cuda(), bias.cuda(), norm.cuda(), state, out, i32(ctx), i32(slots), H, dk, dv, cap,
                      eps, cu_seqlens_q=None if cu is None else i32(cu), impl=impl)


@pytest.mark.parametrize("dtype,impl", [(BF, "auto"), (BF, "simt"), (F32, "auto"), (torch.float16, "auto")])
@pytest.mark.parametrize("shape", MEMORIES)
def test_mlstm_portions_and_single_tokens(dtype, impl, shape):
    """Two sequences in one launch, cut into portions (one of two tokens, one over several chunks), then single
    tokens; outputs and the state itself against the recurrence, in slots that held something else."""
    H, dk, dv = shape
    cap, eps, lengths = 6.0, 1e-4, (150, 91)
    cuts = [(0, 0), (65, 2), (67, 90), (146, 91)]
    data = [_mlstm_inputs(H, dk, dv, n, 20 + n, dtype) for n in lengths]
    for d in data:
        d[2].copy_(data[0][2]), d[3].copy_(data[0][3])
    want = [_mlstm_want(*d, H, dk, dv, cap, eps) for d in data]
    state, slots = _mlstm_state(4, H, dk, dv), (2, 0)
    got = [[], []]
    for a, b in zip(cuts, cuts[1:]):
        rows = [b[i] - a[i] for i in range(2)]
        x, g = (torch.cat([data[i][j][a[i]:b[i]] for i in range(2)]) for j in (0, 1))
        o = _mlstm_run(x, g, *data[0][2:], state, list(b), slots, H, dk, dv, cap, eps, cu=[0, rows[0], sum(rows)], impl=impl)
        for i in range(2):
            got[i].append(o[sum(rows[:i]):sum(rows[:i + 1])].cpu())
    for t in range(146, 150):                                       # the second row pads the batch: context 0
        x, g = torch.cat([data[0][0][t:t + 1]] * 2), torch.cat([data[0][1][t:t + 1]] * 2)
        got[0].append(_mlstm_run(x, g, *data[0][2:], state, [t + 1, 0], (2, 1), H, dk, dv, cap, eps)[:1].cpu())
    tol = {BF: 6e-3, torch.float16: 1e-3, F32: 2e-5}[dtype]
    for i in range(2):
        _close(torch.cat(got[i]), want[i][0], tol, f"outputs {i}")
        S, n, m = want[i][1]
        _close(state[0][slots[i]][..., :dv], S, 1e-4, f"S {i}")
        _close(state[1][slots[i]], n, 1e-4, f"n {i}")
        assert (state[2][slots[i]].cpu().double() - m).abs().max() < 1e-3
    assert all(bool((s[3] == 7.0).all()) and bool((s[1] == 7.0).all()) for s in state)   # other slots untouched


@pytest.mark.parametrize("impl", ["auto", "simt"])
@pytest.mark.parametrize("fill", ["forget nothing", "forget all", "input shut", "input wide open"])
def test_mlstm_gate_extremes(impl, fill):
    H, dk, dv, n = 2, 32, 48, 200
    x, gates, bias, norm = _mlstm_inputs(H, dk, dv, n, 1, BF, gate_scale=0.5)
    col, value = {"forget nothing": (slice(H, None), 60.0), "forget all": (slice(H, None), -60.0),
                  "input shut": (slice(0, H), -60.0), "input wide open": (slice(0, H), 60.0)}[fill]
    gates[:, col] += value
    want, (S, nn, m) = _mlstm_want(x, gates, bias, norm, H, dk, dv, 15.0, 1e-5)
    state = _mlstm_state(1, H, dk, dv)
    got = _mlstm_run(x, gates, bias, norm, state, [n], [0], H, dk, dv, 15.0, 1e-5, cu=[0, n], impl=impl)
    assert torch.isfinite(got).all()
    _close(got, want, 8e-3, fill)
    _close(state[0][0][..., :dv], S, 3e-4, fill)


@pytest.mark.parametrize("impl", ["auto", "simt"])
def test_mlstm_recalls_a_far_token(impl):
    """A value written once behind an open input gate and kept for 900 tokens of shut ones: what is read
    there comes from the far token alone."""
    H, dk, dv, n = 1, 32, 24, 901
    x, gates, bias, norm = _mlstm_inputs(H, dk, dv, n, 7, BF)
    bias.zero_()
    gates[:, 0], gates[:, 1] = -8.0, 12.0
    gates[3, 0] = 8.0
    x[900, :dk] = x[3, dk:2 * dk] * 2                              # the last query asks for the key of token 3
    want, _ = _mlstm_want(x, gates, bias, norm, H, dk, dv, 12.0, 1e-5)
    state = _mlstm_state(1, H, dk, dv)
    got = _mlstm_run(x, gates, bias, norm, state, [n], [0], H, dk, dv, 12.0, 1e-5, cu=[0, n], impl=impl)
    _close(got[900], want[900], 6e-3)
    x[3, 2 * dk:2 * dk + dv] *= -1                                 # the checker would notice a lost token
    other, _ = _mlstm_want(x, gates, bias, norm, H, dk, dv, 12.0, 1e-5)
    assert (other[900] - want[900]).abs().max() > 0.5 * want[900].abs().max()


@pytest.mark.parametrize("window,softcap", [(1000, 30.0), (0, 20.0), (128, 30.0), (129, 5.0), (65, 34.0)])
@pytest.mark.parametrize("block", [64, 256])
def test_window_attention_on_long_portions(window, softcap, block):
    """Head sizes of 128 (the tcgen05 kernel): many key tiles, a portion after a long prefix, ragged ends; and
    the mma.sync kernel's numbers stand in for a second opinion through single rows."""
    from zipage_b200.layers.attention import window_attention
    H, G, d, S, rows = 4, 2, 128, 1111, 700
    q, k, v = (_rand(S, h, d, seed=i, dtype=BF) for i, h in enumerate((H, G, G)))
    k[S - 1 - 64] = q[S - 1].view(G, H // G, d)[:, 0]              # 64 back from the last row
    kc, vc, t = _paged(k, v, block, 3)
    want = O.window_attention(q[S - rows:].double(), k.double(), v.double(), d ** -0.5, softcap, window).flatten(1)
    i32 = lambda a: torch.tensor(a, dtype=torch.int32).cuda()
    qg = q[S - rows:].reshape(rows, -1).cuda()
    got = window_attention(qg, kc, vc, i32([S]), t[None].cuda(), H, d, d, d ** -0.5, window, softcap,
                           cu_seqlens_q=i32([0, rows]), max_seqlen_q=rows, impl="tcgen05")
    _close(got, want, 6e-3, "tcgen05")
    one = window_attention(qg[-1:], kc, vc, i32([S]), t[None].cuda(), H, d, d, d ** -0.5, window, softcap)
    _close(one[0], want[-1], 6e-3, "single row")


def test_mlstm_decode_of_a_large_batch():
    """Enough sequences for one block per head; two tokens each, odd slots."""
    H, dk, dv, B = 3, 40, 168, 110
    x, gates, bias, norm = _mlstm_inputs(H, dk, dv, 2 * B, 2, F32)
    state, slots = _mlstm_state(B + 1, H, dk, dv), [(7 * b + 3) % B for b in range(B)]
    got = [_mlstm_run(x[t * B:(t + 1) * B], gates[t * B:(t + 1) * B], bias, norm, state, [t + 1] * B, slots, H, dk, dv, 9.0, 1e-5).cpu()
           for t in range(2)]
    for b in (0, 1, 57, 109):
        want, (S, n, m) = _mlstm_want(x[b::B], gates[b::B], bias, norm, H, dk, dv, 9.0, 1e-5)
        _close(torch.stack([got[0][b], got[1][b]]), want, 2e-5)
        _close(state[0][slots[b]], S, 1e-5)
        _close(state[1][slots[b]], n, 1e-5)


@pytest.mark.parametrize("dv", [128, 256, 512])
@pytest.mark.parametrize("lengths", [(128,), (1, 300), (257, 128, 40)])
def test_mlstm_tcgen05_portions(dv, lengths):
    """Key size 128: 128-token chunks on tcgen05, one portion after another (whole chunks, ragged ends, two
    tokens), against the recurrence; what the other rows of the batch hold must not matter."""
    H, dk, cap, eps = 2, 128, 8.0, 1e-4
    data = [_mlstm_inputs(H, dk, dv, n, 40 + n, BF) for n in lengths]
    for d in data:
        d[2].copy_(data[0][2]), d[3].copy_(data[0][3])
    want = [_mlstm_want(*d, H, dk, dv, cap, eps) for d in data]
    B = len(lengths)
    state, slots = _mlstm_state(B + 1, H, dk, dv), [(i + 1) % (B + 1) for i in range(B)]
    got = [[] for _ in lengths]
    cuts = [[0] * B, [min(n, 130) for n in lengths], [min(n, 132) for n in lengths], list(lengths)]
    for a, b in zip(cuts, cuts[1:]):
        live = [i for i in range(B) if b[i] > a[i]]
        if not live:
            continue
        rows = [b[i] - a[i] for i in live]
        x, g = (torch.cat([data[i][j][a[i]:b[i]] for i in live] + [torch.full_like(data[0][j][:1], float("nan"))]) for j in (0, 1))
        cu = [0] + torch.tensor(rows).cumsum(0).tolist()
        o = _mlstm_run(x, g, *data[0][2:], state, [b[i] for i in live], [slots[i] for i in live], H, dk, dv, cap, eps, cu=cu,
                       impl="tcgen05")
        for k, i in enumerate(live):
            got[i].append(o[cu[k]:cu[k + 1]].cpu())
    for i in range(B):
        _close(torch.cat(got[i]), want[i][0], 6e-3, f"outputs {i}")
        S, n, m = want[i][1]
        _close(state[0][slots[i]], S, 1e-4, f"S {i}")
        _close(state[1][slots[i]], n, 1e-4, f"n {i}")
        assert (state[2][slots[i]].cpu().double() - m).abs().max() < 1e-3
