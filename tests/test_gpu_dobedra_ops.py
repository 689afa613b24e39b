"""Kernels of the Dobedra decoder against the plain fp64 functions, one mechanism at a time."""
import pytest
import torch

from oracle import dobedra_oracle as O

pytestmark = pytest.mark.gpu
F64 = torch.float64


def _gen(seed=0):
    return torch.Generator().manual_seed(seed)


def _r(g, *s, k=1.0):
    return torch.randn(*s, generator=g) * k


def _dev(t, dtype=None):
    return (t if dtype is None else t.to(dtype)).cuda()


def _close(got, want, dtype, k=1.0):
    """Largest error over the size of the values: one rounding of the result (bf16) or fp32 sums."""
    err = (got.double().cpu() - want.double()).abs().max().item() / want.double().abs().max().item()
    assert err < k * (4e-3 if dtype == torch.bfloat16 else 1e-5), err


def _check_device():
    from zipage_b200 import _lib as L
    torch.cuda.synchronize()
    assert L.device_error(reset=True) == 0


# -- attention over cached latents ---------------------------------------------------------------------
def _paged(rows, BS, g, extra=3):
    """rows: list of [ctx, KP] -> (cache [P, BS, 1, KP] with pages in random order, table)."""
    need = [(len(r) + BS - 1) // BS for r in rows]
    P = sum(need) + extra
    KP = rows[0].shape[1]
    cache = torch.randn(P, BS, 1, KP, generator=g).to(rows[0].dtype)      # what other sequences left
    order = torch.randperm(P, generator=g).tolist()
    table = torch.full((len(rows), max(need) + 2), -1, dtype=torch.int32)
    for b, r in enumerate(rows):
        for i in range(need[b]):
            page = order.pop()
            table[b, i] = page
            part = r[i * BS:(i + 1) * BS]
            cache[page, :len(part), 0] = part
    return cache, table


def _latent_case(H, R, rot, ctxs, counts, dtype, seed=0, qk=1.0, steep=0.0, BS=64):
    g = _gen(seed)
    KP = (R + rot + 15) // 16 * 16
    rows, qs = [], []
    for c, n in zip(ctxs, counts):
        kr = _r(g, c, KP)
        if steep:      # scores that climb along the sequence by far more than fp32 exponents absorb
            kr[:, 0] = torch.arange(c) * steep
        kr[:, R + rot:] = 0
        q = _r(g, n, H, KP, k=qk)
        if steep:
            q[..., 0] = 1.0 + 0.1 * torch.rand(n, H, generator=g)
        q[..., R + rot:] = 0
        rows.append(kr.to(dtype))
        qs.append(q.to(dtype))
    cache, table = _paged(rows, BS, g)
    scale = (R + rot) ** -0.5
    want = [O.softmax_attention(q.to(F64), r.to(F64)[:, None].expand(-1, H, -1), r.to(F64)[:, None, :R].expand(-1, H, -1), scale)
            for q, r in zip(qs, rows)]
    return cache, table, torch.cat(qs), torch.cat(want), scale


SIZES = [(7, 64, 16), (1, 48, 16), (16, 128, 8), (20, 160, 24), (40, 512, 64), (3, 96, 30), (5, 512, 0), (130, 64, 4)]


@pytest.mark.parametrize("impl", ["simt", "tcgen05"])
@pytest.mark.parametrize("H,R,rot", SIZES)
def test_decode_over_latents(H, R, rot, impl):
    from zipage_b200.layers.latent_attention import latent_attention
    for dtype in ((torch.bfloat16,) if impl == "tcgen05" else (torch.float32, torch.bfloat16)):
        ctxs = [1, 2, 63, 64, 65, 127, 128, 300, 129]
        cache, table, q, want, scale = _latent_case(H, R, rot, ctxs, [1] * len(ctxs), dtype, qk=3.0)
        got = latent_attention(_dev(q), _dev(cache), _dev(torch.tensor(ctxs, dtype=torch.int32)), _dev(table), R, scale, impl=impl)
        _check_device()
        _close(got, want, dtype)


@pytest.mark.parametrize("impl", ["simt", "tcgen05"])
@pytest.mark.parametrize("H,R,rot", SIZES)
def test_portions_over_latents(H, R, rot, impl):
    from zipage_b200.layers.latent_attention import latent_attention
    for dtype in ((torch.bfloat16,) if impl == "tcgen05" else (torch.float32, torch.bfloat16)):
        ctxs, counts = [2, 70, 64, 130, 200, 66], [2, 3, 64, 2, 17, 66]
        cache, table, q, want, scale = _latent_case(H, R, rot, ctxs, counts, dtype, seed=1, qk=3.0, BS=128)
        cu = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
        got = latent_attention(_dev(q), _dev(cache), _dev(torch.tensor(ctxs, dtype=torch.int32)), _dev(table), R, scale,
                               cu_seqlens_q=_dev(cu), max_seqlen_q=max(counts), impl=impl)
        _check_device()
        _close(got, want, dtype)


def test_decode_over_latents_long_spans_and_moving_references():
    """A span per block, spans without a key, and scores that climb by hundreds along the sequence."""
    from zipage_b200.layers.latent_attention import latent_attention
    for steep in (0.0, 1.5, 40.0):
        ctxs = [3000, 5, 700, 64]
        cache, table, q, want, scale = _latent_case(12, 128, 16, ctxs, [1] * 4, torch.bfloat16, seed=2, qk=2.0, steep=steep)
        got = latent_attention(_dev(q), _dev(cache), _dev(torch.tensor(ctxs, dtype=torch.int32)), _dev(table), 128, scale, impl="tcgen05")
        _check_device()
        _close(got, want, torch.bfloat16)
        counts = [40, 5, 7, 2]
        cache, table, q, want, scale = _latent_case(12, 128, 16, ctxs, counts, torch.bfloat16, seed=3, qk=2.0, steep=steep)
        cu = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
        got = latent_attention(_dev(q), _dev(cache), _dev(torch.tensor(ctxs, dtype=torch.int32)), _dev(table), 128, scale,
                               cu_seqlens_q=_dev(cu), max_seqlen_q=40, impl="tcgen05")
        _check_device()
        _close(got, want, torch.bfloat16)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_rows_too_long_for_the_tensor_core_kernel(dtype):
    from zipage_b200._lib import ZipageError
    from zipage_b200.layers.latent_attention import latent_attention
    cache, table, q, want, scale = _latent_case(3, 900, 40, [130, 7], [1, 1], dtype, seed=4)
    args = _dev(q), _dev(cache), _dev(torch.tensor([130, 7], dtype=torch.int32)), _dev(table), 900, scale
    _close(latent_attention(*args), want, dtype)
    with pytest.raises(ZipageError):
        latent_attention(*args, impl="tcgen05")


@pytest.mark.parametrize("place", [0, 63, 64, 447, 448, 500])
def test_one_far_key_decides(place):
    """A key whose score stands out by 30: the output is its value, wherever it lies and however the span is cut."""
    from zipage_b200.layers.latent_attention import latent_attention
    H, R, rot, ctx = 4, 64, 16, 501
    g = _gen(place)
    rows = _r(g, ctx, 80, k=0.1)
    q = _r(g, 1, H, 80)
    rows[place] = q[0].mean(0) * 30 / q[0].mean(0).pow(2).sum()
    q[:] = q.mean(1, keepdim=True)
    rows, q = rows.to(torch.bfloat16), q.to(torch.bfloat16)
    cache, table = _paged([rows], 64, g)
    for impl in ("tcgen05", "simt"):
        got = latent_attention(_dev(q), _dev(cache), _dev(torch.tensor([ctx], dtype=torch.int32)), _dev(table), R, 1.0, impl=impl)
        _check_device()
        _close(got, rows[place, :R].double().expand(1, H, R), torch.bfloat16, 2)


def test_rows_past_the_context_do_not_count():
    """What a page holds after the sequence's last key is another request's, here NaN."""
    from zipage_b200.layers.latent_attention import latent_attention
    cache, table, q, want, scale = _latent_case(7, 64, 24, [70], [1], torch.bfloat16, seed=5)
    cache[table[0, 1].item(), 6:] = float("nan")
    got = latent_attention(_dev(q), _dev(cache), _dev(torch.tensor([70], dtype=torch.int32)), _dev(table), 64, scale, impl="tcgen05")
    _check_device()
    _close(got, want, torch.bfloat16)


# -- expanded keys and values ----------------------------------------------------------------------------
@pytest.mark.parametrize("H,dim,rot,vdim,R", [(7, 64, 16, 56, 72), (2, 128, 64, 128, 512), (3, 48, 8, 32, 96), (4, 96, 32, 120, 128),
                                              (1, 192, 64, 72, 40), (2, 8, 0, 8, 64)])
def test_prompts_over_expanded_keys(H, dim, rot, vdim, R):
    from zipage_b200.layers.latent_attention import latent_prefill
    bf = torch.bfloat16
    KP = (R + rot + 15) // 16 * 16
    for steep in (0.0, 2.0):
        g = _gen(7)
        counts, ctxs = [128, 1, 70, 300, 129], [128, 1, 190, 300, 400]
        T, S = sum(counts), sum(ctxs)
        q = _r(g, T, H, dim + rot, k=2.0)
        kv = _r(g, S, H * (dim + vdim))
        lat = _r(g, S, KP)
        if steep:
            q[..., 0] = 1.0
            kv[:, 0:H * dim:dim] = torch.cat([torch.arange(c) for c in ctxs])[:, None] * steep
        q, kv, lat = q.to(bf), kv.to(bf), lat.to(bf)
        scale, want, a, b = (dim + rot) ** -0.5, [], 0, 0
        for n, c in zip(counts, ctxs):
            k = torch.cat([kv[b:b + c, :H * dim].view(c, H, dim), lat[b:b + c, None, R:R + rot].expand(-1, H, -1)], -1)
            want.append(O.softmax_attention(q[a:a + n].to(F64), k.to(F64), kv[b:b + c, H * dim:].view(c, H, vdim).to(F64), scale))
            a, b = a + n, b + c
        i32 = lambda v: torch.tensor([0] + v).cumsum(0).to(torch.int32).cuda()
        out = torch.full((T, H * vdim), float("nan"), dtype=bf, device="cuda")
        latent_prefill(_dev(q).view(T, -1), _dev(kv), _dev(lat), i32(counts), i32(ctxs), max(counts), out, H, dim, rot, vdim, R, scale)
        _check_device()
        _close(out.view(T, H, vdim), torch.cat(want), bf)


# -- row ops ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("q_rank,R,rot", [(40, 72, 16), (33, 21, 6), (256, 512, 64)])
def test_latent_rows(q_rank, R, rot, dtype):
    from zipage_b200.layers.latent_attention import gather_rows, latent_prepare, latent_rotate_q, rotary_turns
    g = _gen(1)
    N, base, eps, H, dim = 37, 12345.0, 1e-3, 3, 10
    KP = (R + rot + 15) // 16 * 16
    y = _r(g, N, q_rank + R + rot, k=0.1).to(dtype)
    pos = torch.randint(0, 5000, (N,), generator=g)
    wq, wk = 1 + _r(g, q_rank, k=0.2), 1 + _r(g, R, k=0.2)
    slots = torch.randperm(128, generator=g)[:N].to(torch.int32)
    slots[3] = -1
    cache = torch.zeros(2, 64, 1, KP, dtype=dtype, device="cuda")
    dense = torch.full((N, KP), 7.0, dtype=dtype, device="cuda")
    turns = rotary_turns(rot, base, "cuda")
    cq = latent_prepare(_dev(y), _dev(pos), turns, _dev(wq), _dev(wk), cache, _dev(slots), q_rank, R, rot, eps, dense)
    Y = y.to(F64)
    _close(cq, O.rms_norm(Y[:, :q_rank], wq.to(F64), eps), dtype)
    want = torch.cat([O.rms_norm(Y[:, q_rank:q_rank + R], wk.to(F64), eps), O.rotate_pairs(Y[:, q_rank + R:], pos, base)], -1)
    _close(dense[:, :R + rot], want, dtype)
    assert (dense[:, R + rot:] == 0).all()
    flat, keep = cache.view(128, KP), slots >= 0
    assert torch.equal(flat[slots[keep].long().cuda()], dense[keep.cuda()])
    assert flat.abs().sum(-1).count_nonzero() == keep.sum()
    only = latent_prepare(_dev(y[:, :q_rank].contiguous()), _dev(pos), turns, _dev(wq), None, cache, _dev(slots), q_rank, 0, rot, eps)
    assert torch.equal(only, cq)
    # queries
    q = _r(g, N, H * (dim + rot)).to(dtype)
    Q = q.to(F64).view(N, H, -1)
    turned = O.rotate_pairs(Q[..., dim:], pos, base)
    ql = torch.full((N, H, KP), 7.0, dtype=dtype, device="cuda")
    qd = _dev(q)
    latent_rotate_q(qd, _dev(pos), turns, H, dim, rot, ql, R)
    assert torch.equal(qd.cpu(), q) and (ql[..., R + rot:] == 0).all() and (ql[..., :R] == 7).all()
    _close(ql[..., R:R + rot], turned, dtype)
    latent_rotate_q(qd, _dev(pos), turns, H, dim, rot)
    _close(qd.view(N, H, -1)[..., dim:], turned, dtype)
    assert torch.equal(qd.view(N, H, -1)[..., :dim].cpu(), q.view(N, H, -1)[..., :dim])
    # cached rows of sequences, in order
    rows = [_r(g, c, KP).to(dtype) for c in (130, 1, 64)]
    pages, table = _paged(rows, 64, g)
    cu = torch.tensor([0, 130, 131, 195], dtype=torch.int32)
    assert torch.equal(gather_rows(_dev(pages), _dev(table), _dev(cu), 195).cpu(), torch.cat(rows))


def test_angles_stay_exact_far_from_the_start():
    from zipage_b200.layers.latent_attention import latent_rotate_q, rotary_turns
    q = torch.zeros(3, 8)
    q[:, ::2] = 1.0
    pos = torch.tensor([1, 100003, 1000003])
    d = _dev(q.clone())
    latent_rotate_q(d, _dev(pos), rotary_turns(8, 10000.0, "cuda"), 1, 0, 8)
    want = O.rotate_pairs(q.to(F64)[:, None], pos, 10000.0)[:, 0]
    assert (d.cpu().double() - want).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [260, 58, 2052, 8192, 9000])
def test_join_norms(W, dtype):
    from zipage_b200.layers.row_ops import join_norms
    g = _gen(W)
    N, top, eps = 9, 3, 1e-2
    x = _r(g, N, W) + 5.0
    a, b, y = (_r(g, n, W).to(dtype) for n in (N, N, N * top))
    v = [_r(g, W) for _ in range(6)]
    gate = _r(g, N, 5)
    pos = torch.randperm(N * top, generator=g).view(N, top).to(torch.int32)
    wts = torch.rand(N, top, generator=g)
    D = lambda t: t.to(F64)
    ff = torch.sigmoid(D(gate[:, 2:3])) * D(b) + torch.einsum("nk,nkw->nw", D(wts), D(y)[pos.long()])
    cases = [({}, D(x)),
             ({"a": a, "ls_a": v[0]}, D(x) + D(v[0]) * D(a)),
             ({"a": a, "ls_a": v[0], "b": b, "ls_b": v[1]}, D(x) + D(v[0]) * D(a) + D(v[1]) * D(b)),
             ({"b": b}, D(x) + D(b)),
             ({"a": a, "ls_a": v[0], "b": b, "ls_b": v[1], "gate": "gate", "y": y, "pos": pos, "weights": wts},
              D(x) + D(v[0]) * D(a) + D(v[1]) * ff)]
    for kw, want in cases:
        xd = _dev(x.clone())
        gd = _dev(gate)
        kw = {k: gd[:, 2] if k == "gate" else _dev(t) for k, t in kw.items()}
        for norms in ([], [(_dev(v[2]), _dev(v[3]))], [(_dev(v[2]), _dev(v[3])), (_dev(v[4]), _dev(v[5]))]):
            xd.copy_(x)
            outs = join_norms(xd, norms, eps, dtype, **kw)
            _close(xd, want, torch.float32)
            for o, (w, bias) in zip(outs, [(v[2], v[3]), (v[4], v[5])]):
                _close(o, O.layer_norm(want, D(w), D(bias), eps), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("F", [96, 37])
def test_activations_and_soft_cap(F, dtype):
    from zipage_b200.layers.feed_forward import gelu_tanh_and_mul, relu_squared_
    from zipage_b200.layers.row_ops import soft_cap_
    x = _r(_gen(F), 11, 2 * F, k=2.0).to(dtype)
    X = x.to(F64)
    _close(gelu_tanh_and_mul(_dev(x)), O.gelu_tanh(X[:, :F]) * X[:, F:], dtype)
    _close(relu_squared_(_dev(x)), torch.clamp(X, min=0) ** 2, dtype)
    z = _r(_gen(1), 7, 33, k=40.0)
    _close(soft_cap_(_dev(z.clone()), 11.0), O.soft_cap(z.to(F64), 11.0), torch.float32)


# -- experts -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("N,E,top", [(1, 11, 2), (7, 5, 5), (300, 64, 6), (513, 11, 2), (3000, 300, 8), (700, 1, 1), (600, 33, 1)])
def test_routing(N, E, top):
    from zipage_b200.layers.feed_forward import moe_route
    z = _r(_gen(N), N, E + 3, k=3.0)
    w, experts, places, rows, offsets = moe_route(_dev(z), E, top)
    i, s = O.route(z[:, :E].to(F64), top)
    assert torch.equal(experts.cpu().long(), i)
    _close(w, s, torch.float32)
    counts = torch.bincount(i.flatten(), minlength=E)
    assert torch.equal(offsets.cpu().long(), torch.cat([torch.zeros(1, dtype=torch.long), counts.cumsum(0)]))
    p = places.cpu().long()
    assert torch.equal(p.flatten().sort().values, torch.arange(N * top))
    assert torch.equal(rows.cpu().long()[p], torch.arange(N)[:, None].expand(N, top))
    lo, hi = offsets.cpu().long()[i], offsets.cpu().long()[i + 1]
    assert ((p >= lo) & (p < hi)).all()


def test_routing_ties_take_the_lower_expert():
    from zipage_b200.layers.feed_forward import moe_route
    z = torch.zeros(3, 40)
    z[1, 35] = z[1, 7] = 1.0
    _, experts, *_ = moe_route(_dev(z), 40, 3)
    assert experts.cpu().tolist() == [[0, 1, 2], [7, 35, 0], [0, 1, 2]]


@pytest.mark.parametrize("impl,dtype", [("simt", torch.float32), ("simt", torch.bfloat16), ("tcgen05", torch.bfloat16)])
@pytest.mark.parametrize("K,n_out,counts", [(112, 264, [3, 0, 130, 1, 0, 64]), (264, 112, [1] * 40 + [0]), (64, 40, [0, 0, 5]),
                                            (200, 520, [300, 128, 256, 0, 1]), (2048, 128, [2, 129]), (72, 77, [9, 4])])
def test_grouped_products(K, n_out, counts, impl, dtype):
    from zipage_b200.layers.feed_forward import grouped_gemm
    g = _gen(K)
    E, M, S = len(counts), sum(counts), 50
    w = (_r(g, E, n_out, K) / K ** 0.5).to(dtype)
    x, direct = _r(g, S, K).to(dtype), _r(g, M, K).to(dtype)
    rows = torch.randint(0, S, (M,), generator=g).to(torch.int32)
    off = torch.tensor([0] + counts).cumsum(0).to(torch.int32)
    owner = torch.repeat_interleave(torch.arange(E), torch.tensor(counts))
    for src, r in ((x, rows), (direct, None)):
        X = src[rows.long()] if r is not None else src
        want = torch.einsum("mk,mnk->mn", X.to(F64), w.to(F64)[owner])
        for act in (None, "relu_squared"):
            got = grouped_gemm(_dev(src), _dev(w), _dev(off), M, rows=None if r is None else _dev(r), act=act, impl=impl)
            _check_device()
            _close(got, torch.clamp(want, min=0) ** 2 if act else want, dtype)


def test_grouped_products_with_a_strided_source_and_spare_places():
    """Rows that are columns of a wider tensor, and a place count above what the offsets use."""
    from zipage_b200.layers.feed_forward import grouped_gemm
    g = _gen(3)
    wide, w = _r(g, 20, 160).to(torch.bfloat16), _r(g, 2, 64, 64).to(torch.bfloat16)
    off = torch.tensor([0, 3, 9], dtype=torch.int32)
    x = _dev(wide)[:, 32:96]
    got = grouped_gemm(x, _dev(w), _dev(off), 20, impl="tcgen05")
    want = torch.cat([wide[:3, 32:96].double() @ w[0].double().T, wide[3:9, 32:96].double() @ w[1].double().T])
    _check_device()
    _close(got[:9], want, torch.bfloat16)
