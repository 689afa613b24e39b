"""Similorn without a GPU: configuration, weight files, registry, and the native scheduler's portion steps."""
import json
import random
import types

import numpy as np
import pytest
import torch

import similorn_cases as C
from oracle import similorn_oracle as O


def _scheduler(pages=12, slots=3, block=64, budget=100, max_seqs=3):
    from zipage_b200.build import build
    from zipage_b200.engine.scheduler import Scheduler
    build()
    return Scheduler(types.SimpleNamespace(
        max_num_seqs=max_seqs, max_num_batched_tokens=budget, eos=None, num_kvcache_blocks=pages, kvcache_block_size=block,
        max_cache_blocks_per_seq=pages + 1, enable_prefix_cache=False, max_concurrency=slots, enable_hybrid_engine=False,
        query_cache_len=0))


def _sequence(n, new):
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    return Sequence(list(range(1, n + 1)), SamplingParams(1.0, new, True))


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_run_order_matches_the_oracle(name):
    from zipage_b200.models.similorn import SimilornConfig
    c = C.CONFIGS[name]
    cfg = SimilornConfig.from_dict(json.loads(json.dumps(c)))
    assert [(i, opens) for i, _, opens in cfg.runs()] == O.run_order(len(c["layers"]), c.get("loop"))
    passes = {}
    for i, t, _ in cfg.runs():           # a layer's passes are numbered from 0 in order
        assert t == passes.get(i, 0)
        passes[i] = t + 1


def test_unknown_parts_are_refused():
    from zipage_b200.models.similorn import SimilornConfig
    c = json.loads(json.dumps(C.CONFIGS["no_loop"]))
    c["layers"][0]["type"] = "something_else"
    with pytest.raises(ValueError):
        SimilornConfig.from_dict(c)
    c = json.loads(json.dumps(C.CONFIGS["mixed"]))
    c["layers"][1]["mlp"]["kind"] = "gated"
    with pytest.raises(ValueError):
        SimilornConfig.from_dict(c)


def test_registry_and_weight_files(tmp_path):
    from zipage_b200.models import registry
    from zipage_b200.models.weights import read_model_weights
    c = C.CONFIGS["odd_sizes"]
    w = C.weights(c)
    w["a.table"] = torch.arange(7, dtype=torch.int32)
    C.write_model(tmp_path, c, w)
    back = read_model_weights(tmp_path)
    assert set(back) == set(w) and all(torch.equal(back[n], w[n]) and back[n].dtype == w[n].dtype for n in w)
    assert registry.read_config(tmp_path)[0] == "Similorn" and registry.kernel_part(tmp_path) == "similorn"
    assert {"Similorn", "Qwen3ForCausalLM"} <= set(registry.architectures())
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError):
        registry.read_config(tmp_path)


def test_the_family_library_has_what_it_needs():
    """Every kernel entry point the family's Python layers call is in the sources of its part."""
    import re
    from zipage_b200 import build as B
    text = "".join((B.CSRC / f"{n}.cu").read_text() for n in B.PARTS["similorn"])
    used = set()
    for f in ("layers/row_ops.py", "layers/mlstm.py", "layers/step_ops.py"):
        used |= set(re.findall(r"\.(zp_[a-z0-9_]+)\(", (B.PKG / f).read_text()))
    used |= {"zp_window_attention", "zp_window_attention_workspace_bytes", "zp_store_kv_padded", "zp_last_error"}
    missing = [n for n in used if not re.search(r"extern \"C\"[^\n]*\b" + n + r"\(", text)]
    assert not missing, missing


def test_portions_respect_budget_order_and_pages():
    s = _scheduler(pages=12, slots=3, budget=100)
    seqs = [_sequence(n, 5) for n in (150, 30, 90, 40)]
    for q in seqs:
        s.add(q)
    seen, steps = {q._h: [] for q in seqs}, 0
    while not s.is_finished():
        handles, counts = s.schedule_portions()
        assert len(handles) and counts.min() >= 1 and len(set(handles.tolist())) == len(handles)
        assert counts.sum() <= 100
        p = s.portion_inputs(handles, counts, 12)
        assert p["cu_seqlens_q"].tolist() == [0] + np.cumsum(counts).tolist()
        used = []
        for i, (h, n) in enumerate(zip(handles.tolist(), counts.tolist())):
            a, b = p["cu_seqlens_q"][i:i + 2]
            pos = p["positions"][a:b].tolist()
            assert pos == list(range(len(seen[h]), len(seen[h]) + n)) and p["context_lens"][i] == pos[-1] + 1
            toks = seqs[h].token_ids
            assert p["input_ids"][a:b].tolist() == toks[pos[0]:pos[-1] + 1]
            table = [t for t in p["block_tables"][i].tolist() if t >= 0]
            used += table
            assert p["slot_mapping"][a:b].tolist() == [table[x // 64] * 64 + x % 64 for x in pos]
            seen[h] += pos
        assert len(used) == len(set(used)) and len(set(p["slots"].tolist())) == len(handles)
        s.commit_portions(handles, counts, np.full(len(handles), 7))
        steps += 1
        c = s.counts()
        assert c[2] + c[3] == 12
    assert all(q.completion_token_ids == [7] * 5 for q in seqs)
    assert s.counts()[3] == 0 and s.counts()[4] == 3
    assert steps >= 4


def test_running_out_of_pages_preempts_the_newest_and_recomputes_it():
    s = _scheduler(pages=4, slots=3, budget=1000)
    seqs = [_sequence(60, 80), _sequence(60, 80)]
    for q in seqs:
        s.add(q)
    starts = {q._h: 0 for q in seqs}
    while not s.is_finished():
        handles, counts = s.schedule_portions()
        p = s.portion_inputs(handles, counts, 8)
        for i, h in enumerate(handles.tolist()):
            starts[h] += int(p["positions"][p["cu_seqlens_q"][i]] == 0)
        s.commit_portions(handles, counts, np.full(len(handles), 3))
    assert starts[seqs[0]._h] == 1 and starts[seqs[1]._h] >= 2        # the second was computed again
    assert all(q.completion_token_ids == [3] * 80 for q in seqs)


def test_a_sequence_larger_than_the_pool_is_an_error():
    s = _scheduler(pages=2, slots=1, budget=1000)
    s.add(_sequence(200, 4))
    with pytest.raises(AssertionError, match="pool"):
        s.schedule_portions()


def test_fed_sequences_take_and_return_pages_and_slots():
    s = _scheduler(pages=6, slots=2)
    rng = random.Random(3)
    a, b = s.feed([1] * 65), s.feed([2])
    assert s.counts()[3] == 3 and s.counts()[4] == 0
    with pytest.raises(AssertionError, match="slots"):
        s.feed([3])
    assert s.pending([a, b]).tolist() == [65, 1]
    s.commit_portions(np.array([a, b], np.int32), np.array([65, 1], np.int32))
    s.feed([4] * 63, a)
    assert s.counts()[3] == 3
    s.feed([4], a)
    assert s.counts()[3] == 4
    with pytest.raises(AssertionError, match="pages"):
        s.feed([5] * 200, b)
    p = s.portion_inputs(np.array([a], np.int32), np.array([64], np.int32), 6)
    assert p["positions"].tolist() == list(range(65, 129)) and p["context_lens"].tolist() == [129]
    s.commit_portions(np.array([a], np.int32), np.array([64], np.int32))
    s.close(a)
    assert s.counts()[3] == 1 and s.counts()[4] == 1
    live, total = {b: 1}, 1
    for _ in range(300):                                          # random feeding and closing
        h = rng.choice(list(live) + [-1])
        n = rng.randint(1, 90)
        need = lambda t: (t + 63) // 64
        room = 6 - sum(need(t) for t in live.values())
        grow = need(live.get(h, 0) + n) - need(live.get(h, 0))
        if h == -1 and len(live) == 2 or grow > room:
            victim = rng.choice(list(live))
            s.close(victim)
            live.pop(victim)
        else:
            k = s.feed([9] * n, h)
            live[k] = live.get(k, 0) + n
            s.commit_portions(np.array([k], np.int32), np.array([n], np.int32))
        assert s.counts()[3] == sum(need(t) for t in live.values()) and s.counts()[5] == len(live)


def test_oracle_state_hand_over():
    """The recurrence carried over a cut gives the uncut result (the checker's own consistency)."""
    g = torch.Generator().manual_seed(1)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v, i, f = r(9, 2, 4), r(9, 2, 4), r(9, 2, 3), r(9, 2), -r(9, 2).abs()
    whole, end = O.mlstm_recurrence(q, k, v, i, f)
    a, mid = O.mlstm_recurrence(q[:4], k[:4], v[:4], i[:4], f[:4])
    b, end2 = O.mlstm_recurrence(q[4:], k[4:], v[4:], i[4:], f[4:], mid)
    assert torch.allclose(torch.cat([a, b]), whole, rtol=1e-12, atol=0) and all(torch.allclose(x, y) for x, y in zip(end, end2))
