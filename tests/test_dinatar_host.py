"""Dinatar without a GPU: configuration, registry, what the layers keep, limits, and the oracle's own consistency."""
import json
import math

import pytest
import torch

import dinatar_cases as C
from oracle import dinatar_oracle as O

F64 = torch.float64


def _copy(name):
    return json.loads(json.dumps(C.CONFIGS[name]))


def _model(name):
    from zipage_b200.models.dinatar import DinatarConfig, DinatarModel
    return DinatarModel(DinatarConfig.from_dict(_copy(name)), torch.bfloat16, torch.device("cpu"), C.RANKS[name])


@pytest.mark.parametrize("name", [n for n in sorted(C.CONFIGS) if "," not in n])
def test_configurations_and_weights_load(name, tmp_path):
    from zipage_b200.models import registry
    from zipage_b200.models.dinatar import DinatarConfig, DinatarModel
    from zipage_b200.models.weights import read_model_weights
    c, w = C.CONFIGS[name], C.weights(C.CONFIGS[name])
    C.write_model(tmp_path, c, w)
    assert registry.read_config(tmp_path)[0] == "Dinatar" and registry.kernel_part(tmp_path) == "dinatar"
    assert "Dinatar" in registry.architectures()
    w = read_model_weights(tmp_path)
    assert DinatarModel.ranks_of(w) == C.RANKS[name]
    m = DinatarModel(DinatarConfig.from_dict(_copy(name)), torch.bfloat16, torch.device("cpu"), DinatarModel.ranks_of(w))
    seen = set()

    class Read(dict):
        def __getitem__(self, k):
            seen.add(k)
            return dict.__getitem__(self, k)
    m.load_weights(Read(w))
    assert seen == set(w)                     # every tensor is used, none is asked for that is not there
    assert m.head is m.embed and torch.allclose(m.norm, w["final.norm"].float() * c["logit_scale"])


def test_every_pass_of_every_mixer_keeps_what_it_needs():
    from zipage_b200.engine.cache import KVSpec, LinearStateSpec, PagedStateCache
    m = _model("mixed")
    assert m.runs == [(0, 0)] + [(1, 0), (2, 0), (1, 1), (2, 1), (1, 2), (2, 2)] + [(3, 0), (4, 0), (5, 0)]
    one = [KVSpec(2, 40, 24), LinearStateSpec(4, 24, 56, 4 * 56 + 2 * 2 * 24, 3), LinearStateSpec(5, 24, 40)]
    assert m.cache_spec() == [LinearStateSpec(3, 40, 24)] + 3 * one + [KVSpec(1, 24, 48), LinearStateSpec(6, 40, 16, 6 * 16 + 2 * 40, 4),
                                                                       LinearStateSpec(2, 56, 32), LinearStateSpec(2, 16, 72)]
    cache = PagedStateCache(m.cache_spec(), 5, 64, 3, torch.bfloat16, "cpu")
    m.bind_cache(cache)
    left, right = m.layers[1].mixers
    assert len(left.caches) == len(right.states) == 3 and len(m.layers[5].mixers[0].states) == 1
    state, ring = right.states[1]
    assert state.shape == (3, 4, 24, 56) and state.dtype == torch.float32 and ring.shape == (3, 3, 320) and ring.dtype == torch.bfloat16
    assert left.caches[2][0].shape == (5, 64, 2, 48) and left.caches[2][0].data_ptr() != left.caches[1][0].data_ptr()
    assert cache.nbytes == sum(s.bytes(5, 64, 3, 2) for s in m.cache_spec())
    m.bind_cache(cache)                       # binding again replaces
    assert len(left.caches) == 3


def test_runs_of_loops():
    from zipage_b200.models.dinatar import DinatarConfig
    for loop, want in ((None, [0, 1, 2, 3, 4, 5]), ((0, 6, 2), [0, 1, 2, 3, 4, 5] * 2), ((2, 3, 4), [0, 1, 2, 2, 2, 2, 3, 4, 5]), ((5, 6, 1), [0, 1, 2, 3, 4, 5]),
                       ((3, 3, 9), [0, 1, 2, 3, 4, 5])):
        c = _copy("mixed")
        c["loop"] = dict(zip(("start", "stop", "times"), loop)) if loop else None
        assert [i for i, _ in DinatarConfig.from_dict(c).runs()] == want == O.layer_runs(c)


def test_unknown_or_inconsistent_parts_are_refused():
    from zipage_b200.models.dinatar import DinatarConfig
    at = lambda c, i: c["layers"][i]
    changes = [lambda c: at(c, 0).update(type="other"), lambda c: at(c, 0)["mlp"].update(kind="other"),
               lambda c: at(c, 1)["mixer"]["left"].update(kv_heads=4), lambda c: at(c, 1)["mixer"]["right"].update(groups=3),
               lambda c: at(c, 1)["mixer"]["right"].update(norm_groups=9), lambda c: at(c, 0)["mlp"]["router"].update(top=8),
               lambda c: c["loop"].update(stop=7), lambda c: c["loop"].update(start=4)]
    DinatarConfig.from_dict(_copy("mixed"))
    for change in changes:
        c = _copy("mixed")
        change(c)
        with pytest.raises(ValueError):
            DinatarConfig.from_dict(c)


def test_positions_past_the_table_are_refused():
    from types import SimpleNamespace
    from zipage_b200.engine.native_engine import NativeEngine
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    eng = object.__new__(NativeEngine)
    eng.model, eng._fed = SimpleNamespace(max_positions=10), {}
    held = {}

    def feed(tokens, handle):
        handle = len(held) if handle < 0 else handle
        held[handle] = held.get(handle, 0) + len(tokens)
        return handle
    eng.scheduler = SimpleNamespace(add=lambda seq: setattr(seq, "_h", 0), feed=feed, close=held.pop)
    eng.add_request(Sequence([1] * 4, SamplingParams(1.0, 6)))
    with pytest.raises(ValueError):
        eng.add_request(Sequence([1] * 4, SamplingParams(1.0, 7)))
    h = eng.feed([1] * 9)
    other = eng.feed([1] * 10)
    assert eng.feed([1], h) == h and held == {h: 10, other: 10}
    for tokens, handle in (([1], h), ([1] * 11, -1)):
        with pytest.raises(ValueError):
            eng.feed(tokens, handle)
    assert held == {h: 10, other: 10}
    eng.close(h)
    assert eng._fed == {other: 10}


def test_the_family_library_has_what_it_needs():
    """Every kernel entry point the family's Python layers call is in the sources of its part."""
    import re
    from zipage_b200 import build as B
    text = "".join((B.CSRC / f"{n}.cu").read_text() for n in B.PARTS["dinatar"])
    used = {"zp_embed_position", "zp_join_norms", "zp_window_attention", "zp_store_kv_padded", "zp_prepare_decode", "zp_sample", "zp_last_error",
            "zp_device_error_async", "zp_moe_route", "zp_grouped_gemm", "zp_short_conv", "zp_silu_and_mul", "zp_relu_squared"}
    used |= set(re.findall(r"\.(zp_[a-z0-9_]+)\(", (B.PKG / "layers/linear_state.py").read_text()))
    used |= set(re.findall(r"\.(zp_[a-z0-9_]+)\(", (B.PKG / "layers/short_conv.py").read_text()))
    assert "zp_linear_state" in used and "zp_group_norm_gate" in used
    missing = [n for n in used if not re.search(r"extern \"C\"[^\n]*\b" + n + r"\(", text)]
    assert not missing, missing


def test_argument_errors_come_back_as_errors():
    from zipage_b200 import _lib as L
    from zipage_b200.build import build
    build()
    lib, one = L.load(), 16

    def state(impl=0, dtype=0, **kw):
        p = dict(kind=1, B=1, H=2, G=2, dim=8, vdim=8, VP=8, n_slots=1, taps=0, total_rows=64, q=one, k=one, v=one, x_stride=64, gate=one, gate_stride=16,
                 gate_bias=one, lower=one, A_log=one, D=one, conv_weight=one, conv_bias=one, ring=one, cu_seqlens_q=one, context_lens=one, slots=one,
                 state=one, out=one, out_stride=16, rtau=1.0, qscale=1.0, workspace=None, workspace_bytes=0)
        p.update(kw)
        return lib.zp_linear_state(L.C.byref(L.LinearStateParams(**p)), impl, dtype, None)
    assert state(kind=3) == -1 and state(k=None) == -1 and state(kind=0, lower=None) == -1 and state(kind=2, D=None) == -1
    assert state(G=1) == -1 and state(kind=2, G=1, H=0) == -1 and state(VP=10) == -1 and state(VP=4) == -1
    assert state(taps=3) == -1 and state(kind=2, taps=3) == -1                  # the fused convolution is for single rows of scalar decays
    assert state(impl=2, dim=136) == -3 and state(impl=2, cu_seqlens_q=None) == -3 and state(impl=2, dtype=1) == -3 and state(impl=2, v=8) == -3
    assert state(impl=2) == -1                                                  # no workspace
    assert state(B=0) == 0
    assert lib.zp_linear_state_workspace_bytes(0, 1, 1, 8) == 0
    small, large = (lib.zp_linear_state_workspace_bytes(200, 2, 3, d) for d in (64, 72))
    assert 0 < small < large
    norm = lambda parts, width, stride: lib.zp_group_norm_gate(16, stride, None, 0, None, 0, 16, 0, 16, stride, 4, parts, width, 1e-5, 0, None)
    assert norm(0, 8, 64) == -1 and norm(4, 32, 64) == -1
    assert lib.zp_join_norms(*[16] + [None] * 5, 0, None, 0, None, None, 0, 16, 16, None, None, 0.5, *[None] * 6, 1, 8, 1e-5, 0, 0, None) == -1
    assert lib.zp_embed_position(16, 16, 16, 16, 1.0, 16, 8, 16, None, 1, 8, 8, 0, None) == -1       # two kinds of positions


def test_oracle_chunked_form_of_the_decayed_recurrence():
    """The unrolled chunk equals the recurrence (two readings of the same mechanism)."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    T, dk, dv = 13, 5, 4
    q, k, v, S0 = r(T, 1, dk), r(T, 1, dk), r(T, 1, dv), r(1, dk, dv)
    a = torch.rand(T, 1, dk, generator=g, dtype=F64)
    o, S = O.decayed_recurrence(q, k, v, a, S0)
    L = a[:, 0].log().cumsum(0)
    E = (L[:, None] - L[None]).exp()                                # [t, s, d]
    P = torch.tril((q[:, 0][:, None] * k[:, 0][None] * E).sum(-1))
    assert torch.allclose((q[:, 0] * L.exp()) @ S0[0] + P @ v[:, 0], o[:, 0], rtol=1e-9)
    assert torch.allclose(L[-1].exp()[:, None] * S0[0] + (k[:, 0] * (L[-1] - L).exp()).T @ v[:, 0], S[0], rtol=1e-9)


def test_oracle_masks_slopes_and_gates():
    assert O.visible(3, 7, 2, 1).int().tolist() == [[1, 0, 0, 1, 1, 0, 0], [1, 0, 0, 0, 1, 1, 0], [1, 0, 0, 0, 0, 1, 1]]
    assert O.visible(2, 3).int().tolist() == [[1, 1, 0], [1, 1, 1]] and O.visible(1, 3, 1, 2).int().tolist() == [[1, 1, 1]]
    from zipage_b200.layers.attention import distance_slopes
    assert distance_slopes(8) == [2.0 ** -(i + 1) for i in range(8)] and O.slopes(2).tolist() == [2 ** -4, 2 ** -8]
    # equal scores: weights fall with the distance by the slope
    z, v = torch.zeros(1, 1, 2, dtype=F64), torch.eye(3, dtype=F64)[:, None]
    w = O.biased_attention(z, torch.zeros(3, 1, 2, dtype=F64), v, 1.0, slope=torch.tensor([math.log(2.0)], dtype=F64))
    assert torch.allclose(w[0, 0], torch.tensor([1.0, 2.0, 4.0], dtype=F64) / 7)
    f = O.hgrn2_gates(torch.tensor([-50.0, 0.0, 50.0], dtype=F64), torch.zeros(3, dtype=F64), torch.full((3,), 0.4, dtype=F64))
    assert torch.allclose(f, torch.tensor([0.4, 0.7, 1.0], dtype=F64))
    assert torch.allclose(O.gla_decay(torch.zeros(1, dtype=F64), 4.0), torch.tensor([0.5 ** 0.25], dtype=F64))
    i, s = O.route(torch.tensor([[1.0, 3.0, 2.0]], dtype=F64), 2)
    assert i.tolist() == [[1, 2]] and torch.allclose(s[0, 0] / s[0, 1], torch.tensor(math.e, dtype=F64)) and abs(s.sum() - 1) < 1e-12


def test_oracle_states_and_convolutions_carry_over():
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    x, w, b = r(11, 3), r(3, 4), r(3)
    whole = O.short_conv(x, w, b)
    assert torch.allclose(torch.cat([O.short_conv(x[:5], w, b), O.short_conv(x[5:], w, b, x[2:5])]), whole)
    assert torch.allclose(whole[0], O.silu(b + w[:, -1] * x[0]))          # nothing before the start
    q, k, v, a = r(9, 2, 3), r(9, 2, 3), r(9, 2, 4), torch.rand(9, 2, 3, generator=g, dtype=F64)
    o, S = O.decayed_recurrence(q, k, v, a)
    o1, S1 = O.decayed_recurrence(q[:4], k[:4], v[:4], a[:4])
    o2, S2 = O.decayed_recurrence(q[4:], k[4:], v[4:], a[4:], S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)
