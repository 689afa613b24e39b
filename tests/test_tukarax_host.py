"""Tukarax without a GPU: configuration, registry, what the layers keep, and the oracle's own consistency."""
import json
import math

import pytest
import torch

import tukarax_cases as C
from oracle import tukarax_oracle as O

F64 = torch.float64


def _copy(name):
    return json.loads(json.dumps(C.CONFIGS[name]))


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_configurations_and_weights_load(name, tmp_path):
    from zipage_b200.models import registry
    from zipage_b200.models.tukarax import TukaraxConfig, TukaraxModel
    from zipage_b200.models.weights import read_model_weights
    c, w = C.CONFIGS[name], C.weights(C.CONFIGS[name])
    C.write_model(tmp_path, c, w)
    assert registry.read_config(tmp_path)[0] == "Tukarax" and registry.kernel_part(tmp_path) == "tukarax"
    assert "Tukarax" in registry.architectures()
    m = TukaraxModel(TukaraxConfig.from_dict(_copy(name)), torch.bfloat16, torch.device("cpu"))
    seen = set()

    class Read(dict):
        def __getitem__(self, k):
            seen.add(k)
            return dict.__getitem__(self, k)
    m.load_weights(Read(read_model_weights(tmp_path)))
    assert seen == set(w)                     # every tensor is used, none is asked for that is not there


def test_every_group_of_heads_keeps_what_it_needs():
    from zipage_b200.engine.cache import DeltaSpec, KVSpec, PagedStateCache
    from zipage_b200.models.tukarax import TukaraxConfig, TukaraxModel
    m = TukaraxModel(TukaraxConfig.from_dict(_copy("mixed")), torch.bfloat16, torch.device("cpu"))
    assert m.cache_spec() == [KVSpec(1, 40, 24), KVSpec(2, 48, 48), DeltaSpec(6, 2, 40, 56, 4), KVSpec(2, 32, 48), KVSpec(1, 24, 24),
                              DeltaSpec(4, 4, 24, 16, 2)]
    cache = PagedStateCache(m.cache_spec(), 5, 64, 3, torch.bfloat16, "cpu")
    m.bind_cache(cache)
    d = m.layers[1].mixer.parts[1]
    assert d.state.shape == (3, 6, 40, 56) and d.state.dtype == torch.float32 and d.ring.shape == (3, 4, 2 * 2 * 40 + 6 * 56)
    assert m.layers[1].mixer.parts[0].k_cache.shape == (5, 64, 2, 48)
    assert cache.nbytes == sum(s.bytes(5, 64, 3, 2) for s in m.cache_spec())
    assert DeltaSpec(1, 1, 4, 5, 2).allocate(1, 64, 2, torch.float32, "cpu")[0].shape == (2, 1, 4, 8)


def test_unknown_or_inconsistent_parts_are_refused():
    from zipage_b200.models.tukarax import TukaraxConfig
    at = lambda c, i: c["layers"][i]
    changes = [lambda c: at(c, 0).update(type="other"), lambda c: at(c, 0)["mlp"].update(kind="dense"),
               lambda c: at(c, 2)["mixer"].update(kv_heads=3), lambda c: at(c, 1)["mixer"]["right"].update(kv_heads=4),
               lambda c: at(c, 0)["mixer"]["rot"].update(dims=15), lambda c: at(c, 1)["mixer"]["left"]["rot"].update(dims=50),
               lambda c: at(c, 1)["mixer"]["left"].update(vdim=32), lambda c: at(c, 1)["mlp"]["router"].update(top=6)]
    TukaraxConfig.from_dict(_copy("mixed"))
    for change in changes:
        c = _copy("mixed")
        change(c)
        with pytest.raises(ValueError):
            TukaraxConfig.from_dict(c)


def test_the_family_library_has_what_it_needs():
    """Every kernel entry point the family's Python layers call is in the sources of its part."""
    import re
    from zipage_b200 import build as B
    text = "".join((B.CSRC / f"{n}.cu").read_text() for n in B.PARTS["tukarax"])
    used = {"zp_embed_position", "zp_join_norms", "zp_window_attention", "zp_prepare_decode", "zp_sample", "zp_last_error",
            "zp_device_error_async"}
    for f in ("layers/gated_delta.py", "layers/short_conv.py", "layers/rotary.py"):
        used |= set(re.findall(r"\.(zp_[a-z0-9_]+)\(", (B.PKG / f).read_text()))
    used |= {"zp_moe_route", "zp_grouped_gemm"}
    assert "zp_gated_delta" in used and "zp_rotate_store" in used
    missing = [n for n in used if not re.search(r"extern \"C\"[^\n]*\b" + n + r"\(", text)]
    assert not missing, missing


def test_argument_errors_come_back_as_errors():
    from zipage_b200 import _lib as L
    from zipage_b200.build import build
    build()
    lib = L.load()
    one = L.C.c_void_p(16)
    conv = lambda taps: lib.zp_short_conv(one, 8, one, None, one, one, one, one, one, 8, 1, 1, 8, taps, 1, 0, None)
    assert conv(9) == -1 and conv(0) == -1
    delta = lambda taps, cu, H, G, impl, dim: lib.zp_gated_delta(one, 64, one, 64, one, 8, one, one, one, one, one, taps, cu, one, one, one,
                                                                 one, 64, 1, H, G, dim, 8, 8, 1, 1e-5, 1.0, 4, impl, 0, None, 0, None)
    assert delta(3, one, 2, 1, 0, 8) == -1            # the fused convolution is for single rows
    assert delta(0, one, 3, 2, 0, 8) == -1            # heads over key heads
    assert delta(0, one, 2, 1, 2, 136) == -3 and delta(0, None, 2, 1, 2, 8) == -3      # what the chunked kernels do not take
    assert delta(0, one, 2, 1, 2, 8) == -1            # no workspace
    rot = lambda dims, D: lib.zp_rotate_store(one, one, one, 64, one, one, dims, 0, 1.0, None, None, 0.0, one, one, one, 1, 1, 1, D, 8, 16, 16,
                                              64, 0, None)
    assert rot(10, 8) == -1 and rot(3, 8) == -1 and rot(8, 24) == -1
    grouped = lambda n_out, act, scale: lib.zp_grouped_gemm(one, 8, None, 4, one, one, scale, one, 4, 2, n_out, 8, act, 0, 1, None)
    assert grouped(48, 2, None) == -1 and grouped(64, 1, one) == -1
    assert lib.zp_moe_route(one, 8, None, 4, 8, 2, one, one, one, one, one, one, None, 7, None) == -1
    assert lib.zp_gated_delta_workspace_bytes(0, 1, 1) == 0 and lib.zp_gated_delta_workspace_bytes(200, 2, 3) > 0


@pytest.mark.parametrize("rot", [{"dims": 48, "base": 250.0}, {"dims": 16, "base": 1e4, "scaling": {"factor": 8.0, "original": 64, "fast": 4.0, "slow": 0.5}},
                                 {"dims": 64, "base": 5e5, "scaling": {"factor": 2.5, "original": 4096, "fast": 32.0, "slow": 1.0}},
                                 {"dims": 6, "base": 30.0, "scaling": {"factor": 4.0, "original": 7, "fast": 9.0, "slow": 5.0}}])
def test_frequencies(rot):
    from zipage_b200.layers.rotary import Rotary
    r = Rotary.from_config(rot, True, "cpu")
    f, mul = O.frequencies(rot)
    assert r.mul == pytest.approx(mul, abs=1e-12) and r.dims == rot["dims"] and r.interleaved
    assert torch.allclose(r.turns * 2 * math.pi, torch.tensor(f, dtype=F64), rtol=1e-12)
    if "scaling" in rot and rot["dims"] == 64:       # a ramp: some pairs keep their frequency, some are stretched, some lie between
        plain = torch.tensor(O.frequencies({"dims": 64, "base": 5e5})[0])
        q = (torch.tensor(f) / plain)
        assert (q > 0.999).any() and (q < 0.401).any() and ((q > 0.41) & (q < 0.99)).any()


def test_gate_and_up_rows_alternate_in_blocks():
    from zipage_b200.layers.feed_forward import interleave_gate_up, padded_ff
    for ff in (16, 5, 40):
        out = torch.full((2 * padded_ff(ff), 3), 7.0)
        gate, up = torch.randn(ff, 3), torch.randn(ff, 3)
        interleave_gate_up(out, gate, up)
        b = out.view(-1, 2, 16, 3)
        for i, w in enumerate((gate, up)):
            rows = b[:, i].reshape(-1, 3)
            assert torch.equal(rows[:ff], w) and (rows[ff:] == 0).all()


def test_oracle_chunked_form_of_the_delta_rule():
    """The unrolled chunk equals the recurrence (two readings of the same mechanism)."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    T, dk, dv = 13, 5, 4
    q, k, v = O.unit(r(T, 1, dk)), O.unit(r(T, 1, dk)), r(T, 1, dv)
    dec, beta, S0 = torch.rand(T, 1, generator=g, dtype=F64), torch.rand(T, 1, generator=g, dtype=F64), r(1, dk, dv)
    o, S = O.delta_recurrence(q, k, v, dec, beta, S0)
    L = dec[:, 0].log().cumsum(0)
    K, Q, V, b, G = k[:, 0], q[:, 0], v[:, 0], beta[:, 0], L.exp()
    E = (L[:, None] - L[None, :]).exp()
    A = torch.tril(b[:, None] * E * (K @ K.T), -1)
    W = torch.linalg.inv(torch.eye(T, dtype=F64) + A) * b[None, :]
    U = W @ (V - G[:, None] * (K @ S0[0]))
    assert torch.allclose(G[:, None] * (Q @ S0[0]) + torch.tril(E * (Q @ K.T)) @ U, o[:, 0], rtol=1e-9)
    assert torch.allclose(G[-1] * S0[0] + K.T @ ((G[-1] / G)[:, None] * U), S[0], rtol=1e-9)


def test_oracle_convolution_state_and_rotation():
    g = torch.Generator().manual_seed(1)
    x, w = torch.randn(11, 3, generator=g, dtype=F64), torch.randn(3, 4, generator=g, dtype=F64)
    whole = O.short_conv(x, w)
    assert torch.allclose(torch.cat([O.short_conv(x[:5], w), O.short_conv(x[5:], w, x[2:5])]), whole)
    assert torch.allclose(whole[0], O.silu(w[:, -1] * x[0]))          # nothing before the start
    rot = {"dims": 6, "base": 50.0}
    a, b = torch.randn(1, 1, 10, generator=g, dtype=F64), torch.randn(1, 1, 10, generator=g, dtype=F64)
    for inter in (True, False):
        at = lambda t, p: O.rotate(t, torch.tensor([p]), rot, inter)
        assert torch.allclose((at(a, 9) * at(b, 4)).sum(), (at(a, 105) * at(b, 100)).sum())
        assert torch.equal(at(a, 9)[..., 6:], a[..., 6:])
    assert not torch.allclose(O.rotate(a, torch.tensor([3]), rot, True), O.rotate(a, torch.tensor([3]), rot, False))


def test_oracle_masks_and_sinks():
    v = O.visible(4, 7, 3)      # positions 3 .. 6, chunks 0-2, 3-5, 6
    assert v.int().tolist() == [[0, 0, 0, 1, 0, 0, 0], [0, 0, 0, 1, 1, 0, 0], [0, 0, 0, 1, 1, 1, 0], [0, 0, 0, 0, 0, 0, 1]]
    q, k, val = torch.zeros(1, 1, 2, dtype=F64), torch.zeros(1, 1, 2, dtype=F64), torch.ones(1, 1, 2, dtype=F64)
    o = O.softmax_attention(q, k, val, 1.0, sink=torch.tensor([math.log(3.0)], dtype=F64))
    assert torch.allclose(o, torch.full_like(o, 0.25))                # one key of weight 1 beside a sink of weight 3
