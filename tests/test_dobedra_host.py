"""Dobedra without a GPU: configuration, registry, what the layers keep, and the oracle's own consistency."""
import json

import pytest
import torch

import dobedra_cases as C
from oracle import dobedra_oracle as O


def _copy(name):
    return json.loads(json.dumps(C.CONFIGS[name]))


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_configurations_and_weights_load(name, tmp_path):
    from zipage_b200.models import registry
    from zipage_b200.models.dobedra import DobedraConfig, DobedraModel
    from zipage_b200.models.weights import read_model_weights
    c, w = C.CONFIGS[name], C.weights(C.CONFIGS[name])
    C.write_model(tmp_path, c, w)
    assert registry.read_config(tmp_path)[0] == "Dobedra" and registry.kernel_part(tmp_path) == "dobedra"
    assert "Dobedra" in registry.architectures()
    m = DobedraModel(DobedraConfig.from_dict(_copy(name)), torch.bfloat16, torch.device("cpu"))
    seen = set()

    class Read(dict):
        def __getitem__(self, k):
            seen.add(k)
            return dict.__getitem__(self, k)
    m.load_weights(Read(read_model_weights(tmp_path)))
    assert seen == set(w)                     # every tensor is used, none is asked for that is not there
    assert m.logit_softcap == (c["logit_softcap"] or 0.0)


def test_layers_that_share_latents_are_bound_to_their_source():
    from zipage_b200.engine.cache import LatentSpec, PagedStateCache
    from zipage_b200.models.dobedra import DobedraConfig, DobedraModel
    m = DobedraModel(DobedraConfig.from_dict(_copy("sharing_far_back")), torch.bfloat16, torch.device("cpu"))
    assert m.cache_spec() == [LatentSpec(120, 32), LatentSpec(96, 16)]
    cache = PagedStateCache(m.cache_spec(), 5, 64, 2, torch.bfloat16, "cpu")
    m.bind_cache(cache)
    own = [l.mixer.cache for l in m.layers]
    assert own[3] is own[0] and own[2] is own[1] and own[4] is own[1] and own[0] is not own[1]
    assert own[0].shape == (5, 64, 1, 160) and own[1].shape == (5, 64, 1, 112)
    assert cache.nbytes == sum(s.bytes(5, 64, 2, 2) for s in m.cache_spec())


def test_unknown_or_inconsistent_parts_are_refused():
    from zipage_b200.models.dobedra import DobedraConfig
    changes = [lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
               lambda c: c["layers"][1]["mixer"].update(kv_from=1), lambda c: c["layers"][1]["mixer"].update(kv_from=4),
               lambda c: c["layers"][4]["mixer"].update(kv_from=3), lambda c: c["layers"][1]["mixer"].update(kv_rank=56),
               lambda c: c["layers"][4]["mixer"]["rot"].update(base=7.0), lambda c: c["layers"][0]["mixer"].update(rot_dim=10)]
    DobedraConfig.from_dict(_copy("mixed"))
    for change in changes:
        c = _copy("mixed")
        change(c)
        with pytest.raises(ValueError):
            DobedraConfig.from_dict(c)


def test_the_family_library_has_what_it_needs():
    """Every kernel entry point the family's Python layers call is in the sources of its part."""
    import re
    from zipage_b200 import build as B
    text = "".join((B.CSRC / f"{n}.cu").read_text() for n in B.PARTS["dobedra"])
    used = set()
    for f in ("layers/row_ops.py", "layers/feed_forward.py", "layers/latent_attention.py", "layers/step_ops.py"):
        used |= set(re.findall(r"\.(zp_[a-z0-9_]+)\(", (B.PKG / f).read_text()))
    assert "zp_latent_prefill" in used and "zp_grouped_gemm" in used
    missing = [n for n in used | {"zp_last_error", "zp_window_attention"} if not re.search(r"extern \"C\"[^\n]*\b" + n + r"\(", text)]
    assert not missing, missing


def test_argument_errors_come_back_as_errors():
    from zipage_b200 import _lib as L
    from zipage_b200.build import build
    build()
    lib = L.load()
    one = L.C.c_void_p(16)
    assert lib.zp_moe_route(one, 8, None, 4, 8, 9, one, one, one, one, one, one, None, 0, None) == -1      # more chosen than there are
    assert lib.zp_grouped_gemm(one, 8, None, 4, one, one, None, one, 4, 2, 8, 9, 0, 0, 1, None) == -1   # rows shorter than k
    assert lib.zp_latent_attention(one, one, None, one, one, one, 1, 1, 1, 1, 2, 1100, 1104, 64, 1, 1.0, 0, 0, None, 0, None) == -1
    assert lib.zp_latent_prefill_supported(128, 64, 128, 512, 576, 0) == 1
    assert lib.zp_latent_prefill_supported(128, 64, 128, 512, 576, 1) == 0
    assert lib.zp_latent_prefill_supported(13, 64, 128, 512, 576, 0) == 0
    assert lib.zp_latent_prefill_supported(128, 64, 136, 512, 576, 0) == 0


def test_oracle_moving_the_key_product_to_the_queries_changes_nothing():
    """The attention over expanded keys equals the one over latents (two readings of the same mechanism)."""
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    T, H, R, dim, rot, vd = 9, 3, 8, 5, 4, 6
    c, kr, uk, uv, qn, qr = r(T, R), r(T, rot), r(H * dim, R), r(H * vd, R), r(T, H, dim), r(T, H, rot)
    k = torch.cat([(c @ uk.T).view(T, H, dim), kr[:, None].expand(-1, H, -1)], -1)
    a = O.softmax_attention(torch.cat([qn, qr], -1), k, (c @ uv.T).view(T, H, vd), 0.3)
    q2 = torch.cat([torch.einsum("thd,hdr->thr", qn, uk.view(H, dim, R)), qr], -1)
    lat = torch.cat([c, kr], -1)[:, None].expand(-1, H, -1)
    b = torch.einsum("thr,hvr->thv", O.softmax_attention(q2, lat, c[:, None].expand(-1, H, -1), 0.3), uv.view(H, vd, R))
    assert torch.allclose(a, b, rtol=1e-10)


def test_oracle_rotation_depends_on_the_distance_only():
    g = torch.Generator().manual_seed(1)
    q, k = (torch.randn(1, 10, generator=g, dtype=torch.float64) for _ in range(2))
    at = lambda x, p: O.rotate_pairs(x, torch.tensor([p]), 50.0)
    assert torch.allclose((at(q, 9) * at(k, 4)).sum(), (at(q, 105) * at(k, 100)).sum())
    assert not torch.allclose((at(q, 9) * at(k, 4)).sum(), (at(q, 9) * at(k, 5)).sum())
