"""Dinatar through the serving engine: pages, state slots, portion steps, graphs, scheduler, command line.

fp32 engines are compared with the plain fp64 forward at 1e-4 of the logits' size at the worst position, bf16 engines
at the error of 16-bit products.  The bf16 models choose all experts: where two scores all but tie, rounding may
choose the other expert, and the logits of that position and of those after it are then those of another function.
"""
import json
import random
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import dinatar_cases as C
from oracle import dinatar_oracle as O

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DTYPES = [torch.float32, torch.bfloat16]
NAMES = [n for n in sorted(C.CONFIGS) if "," not in n]
TOL = {torch.float32: 1e-4, torch.bfloat16: 6e-2}
_oracle_cache = {}


def _engine(name, dtype, max_tokens=1024, max_seqs=4, weights=None, **kw):
    from zipage_b200.models.registry import LoadedModel, engine_for
    from zipage_b200.models.dinatar import DinatarConfig, DinatarModel
    cfg = DinatarConfig.from_dict(C.CONFIGS[name])
    m = DinatarModel(cfg, dtype, torch.device("cuda"), C.RANKS[C.CONFIGS[name]["name"]])
    m.load_weights(weights or C.weights(C.CONFIGS[name]))
    return engine_for(LoadedModel("Dinatar", m, m.head, cfg.width, cfg.vocab, dtype, True), max_tokens=max_tokens, max_seqs=max_seqs, **kw)


def _oracle(name, tokens, weights=None):
    """-> logits, residual streams."""
    key = (name, tuple(tokens), id(weights))
    if key not in _oracle_cache:
        _oracle_cache[key] = O.forward(C.CONFIGS[name], weights or C.weights(C.CONFIGS[name]), tokens)
    return _oracle_cache[key]


def _errors(got, want):
    d = got.double().cpu() - want.double().cpu()
    return d.pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt().item()


def _ok(got, want, dtype, k=1.0):
    e = _errors(got, want).flatten()
    if dtype == torch.float32:
        assert e.max() < k * TOL[dtype], (e.max(), e.argmax())
    else:
        # norms of heads of a few entries: where one is short, the rounding of the projections alone shows several times larger
        assert e.max() < 4 * k * TOL[dtype] and (e > k * TOL[dtype]).sum() <= max(1, 0.05 * len(e)), (e.max(), e.argmax())


def _replay(eng, requests, steps):
    """steps: lists of (request, count); a request is closed when its tokens are used up.  -> logits of
    every position, per request."""
    at, handle, out = {i: 0 for i in requests}, {}, {i: [] for i in requests}
    for step in steps:
        hs, ns = [], []
        for i, n in step:
            handle[i] = eng.feed(requests[i][at[i]:at[i] + n], handle.get(i, -1))
            hs.append(handle[i])
            ns.append(n)
        lg = eng.run_fed(hs, ns, [list(range(n)) for n in ns])
        for (i, n), rows in zip(step, lg.split(ns)):
            out[i].append(rows.cpu())
            at[i] += n
            if at[i] == len(requests[i]):
                eng.close(handle.pop(i))
    assert eng.scheduler.counts()[3] == 0                          # every page came back
    return {i: torch.cat(o) for i, o in out.items()}


def _portions(n, sizes):
    out, left, k = [], n, 0
    while left:
        out.append(min(sizes[k % len(sizes)], left))
        left -= out[-1]
        k += 1
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_layers_and_every_cut(name, dtype):
    """One prompt whole, in portions of several sizes (down to two tokens, around the edges of pages, windows and the
    recurrences' chunks), and token by token through the decode graphs; the whole prompt also layer by layer."""
    name = C.for_dtype(name, dtype)
    eng = _engine(name, dtype)
    toks = C.tokens(C.CONFIGS[name], 200, 1)
    want, trail = _oracle(name, toks)
    eng.model.trail = []
    for sizes in ([200], [64], [63, 66], [2], [65, 1, 63, 2], [7, 3, 100], [99, 1, 1, 1], [1]):
        got = _replay(eng, {"a": toks}, [[("a", n)] for n in _portions(200, sizes)])["a"]
        if eng.model.trail is not None:
            assert len(trail) == len(eng.model.trail)
            for a, b in zip(eng.model.trail, trail):
                _ok(a, b, dtype)
            eng.model.trail = None
        _ok(got, want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "large_heads", "odd_sizes"])
def test_mixed_batches_with_reused_pages_and_slots(name, dtype):
    """Random batches of portions beside single tokens; requests pause, end and make room for others in
    a pool just large enough, so that pages and slots change hands."""
    name = C.for_dtype(name, dtype)
    c = C.CONFIGS[name]
    rng = random.Random(5)
    lengths = [130, 3, 200, 65, 1, 90, 64, 150, 40]
    requests = {k: C.tokens(c, n, 10 + k) for k, n in enumerate(lengths)}
    left, live, todo, steps = dict(enumerate(lengths)), [], list(requests), []
    pages = lambda: sum((lengths[k] + 63) // 64 for k in live)
    while todo or live:
        while todo and len(live) < 4 and pages() + (lengths[todo[0]] + 63) // 64 <= 8:
            live.append(todo.pop(0))
        step = []
        for k in live:
            if rng.random() < 0.8 or not step and k == live[-1]:
                step.append((k, min(left[k], rng.choice([1, 1, 1, 2, 3, 17, 64, 70]))))
        rng.shuffle(step)
        for k, n in step:
            left[k] -= n
        live = [k for k in live if left[k]]
        steps.append(step)
    got = _replay(_engine(name, dtype, max_tokens=8 * 64), requests, steps)
    alone = _engine(name, dtype)
    for k, toks in requests.items():
        _ok(got[k], _oracle(name, toks)[0], dtype)
        _ok(got[k], _replay(alone, {k: toks}, [[(k, len(toks))]])[k], dtype, 2)     # both sides carry the error


def test_far_and_edge_tokens_change_the_logits_as_they_should():
    """Changing one token moves the oracle's logits at the end; the engine follows the change exactly, in a prompt
    and decoded, wherever the token lies (page edges, a window's edges, the kept tokens and those after them, a portion's edges)."""
    name = "mixed"
    c = C.CONFIGS[name]
    toks = C.tokens(c, 150, 2)
    eng = _engine(name, torch.float32)
    moved, places = 0, (0, 1, 4, 5, 6, 63, 64, 65, 79, 80, 81, 116, 117, 119, 120, 127, 128, 148, 149)
    for place in places:
        other = list(toks)
        other[place] = (other[place] + 31) % c["vocab"]
        want = _oracle(name, other)[0]
        moved += _errors(want[-1:], _oracle(name, toks)[0][-1:]).max() > 3 * TOL[torch.float32]
        for steps in ([150], [120] + [1] * 30):
            _ok(_replay(eng, {"a": other}, [[("a", n)] for n in steps])["a"], want, torch.float32)
    assert moved == len(places)


def test_scores_that_stand_out_in_every_schedule():
    """Queries scaled so that the softmaxes lean on few keys and states that hardly decay: an error in a key's page, window or
    distance, or in what a state keeps, would replace the result."""
    name = "mixed, all chosen"
    c = C.CONFIGS[name]
    w = C.weights(c)
    for n in w:
        if n.endswith("left.q"):
            w[n] = w[n] * 2.5
        if n.endswith("f.b") or n.endswith("a2.b"):
            w[n] = w[n] + 4
        if n.endswith("dt_bias"):
            w[n] = w[n] - 2
    toks = C.tokens(c, 260, 3)
    want = _oracle(name, toks, w)[0]
    for dtype in DTYPES:
        eng = _engine(name, dtype, weights=w)
        for sizes in ([260], [100, 2], [230] + [1] * 30, [65]):
            _ok(_replay(eng, {"a": toks}, [[("a", n)] for n in _portions(260, sizes)])["a"], want, dtype, 3)


def test_sequences_longer_than_the_table_of_positions_are_refused():
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    name = "one_gla"
    limit = C.CONFIGS[name]["max_positions"]
    eng = _engine(name, torch.float32, max_tokens=2048)
    toks = C.tokens(C.CONFIGS[name], limit + 1)
    h = eng.feed(toks[:limit - 1])
    eng.run_fed([h], [limit - 1], [[]])
    eng.feed(toks[limit - 1:limit], h)
    last = eng.run_fed([h], [1], [[0]])
    _ok(last.cpu(), _oracle(name, toks[:limit])[0][-1:], torch.float32)
    with pytest.raises(ValueError):
        eng.feed(toks[limit:], h)
    eng.close(h)
    with pytest.raises(ValueError):
        eng.add_request(Sequence(toks[:limit], SamplingParams(1.0, 1)))


def _greedy_oracle(name, prompt, new):
    c, w = C.CONFIGS[name], C.weights(C.CONFIGS[name])
    toks = list(prompt)
    for _ in range(new):
        toks.append(int(O.forward(c, w, toks)[0][-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation_through_the_scheduler(graph):
    """More requests than slots, prompts longer than a step's budget: the engine's tokens are the oracle's."""
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    name = "odd_sizes"
    c = C.CONFIGS[name]
    eng = _engine(name, torch.float32, max_tokens=64 * 6, max_seqs=3, token_budget=40, greedy=True, graph=graph)
    prompts = [C.tokens(c, n, 30 + n) for n in (70, 1, 45, 5, 62)]
    seqs = [Sequence(p, SamplingParams(1.0, 8, True)) for p in prompts]
    out = eng.generate(seqs)
    for s, p in zip(seqs, prompts):
        assert out[s._h] == _greedy_oracle(name, p, 8)
    assert eng.scheduler.counts()[3] == 0


def test_generation_recomputes_what_it_had_to_give_back():
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    name = "mixed"
    c = C.CONFIGS[name]
    prompts = [C.tokens(c, n, 50 + n) for n in (60, 50)]
    runs = []
    for pool in (16, 3):
        eng = _engine(name, torch.float32, max_tokens=64 * pool, max_seqs=2, greedy=True)
        seqs = [Sequence(p, SamplingParams(1.0, 90, True)) for p in prompts]
        out = eng.generate(seqs)
        runs.append([out[s._h] for s in seqs])
    assert runs[0] == runs[1] and all(len(o) == 90 for o in runs[0])


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """500 decoded tokens (graphs), against the same tokens in one portion."""
    name = C.for_dtype("mixed", dtype)
    toks = C.tokens(C.CONFIGS[name], 540, 9)
    eng = _engine(name, dtype)
    whole = _replay(eng, {"a": toks}, [[("a", 540)]])["a"]
    steps = _replay(eng, {"a": toks}, [[("a", 40)]] + [[("a", 1)]] * 500)["a"]
    want = _oracle(name, toks)[0]
    _ok(steps, whole, dtype, 2)
    _ok(steps, want, dtype)


def test_sampled_tokens_follow_temperature_and_seed():
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    name = "large_heads"
    runs = []
    for seed, temp in ((1, 1.0), (1, 1.0), (2, 1.0), (3, 1e-4)):
        eng = _engine(name, torch.bfloat16, seed=seed)
        s = Sequence(C.tokens(C.CONFIGS[name], 9), SamplingParams(temp, 24, True))
        runs.append(eng.generate([s])[s._h])
    greedy = _engine(name, torch.bfloat16, greedy=True)
    s = Sequence(C.tokens(C.CONFIGS[name], 9), SamplingParams(1.0, 24, True))
    assert runs[0] == runs[1] != runs[2] and runs[3] == greedy.generate([s])[s._h]


def test_command_line_and_trace_replay(tmp_path):
    name = "mixed"
    c = C.CONFIGS[name]
    folder = C.write_model(tmp_path / "m", c, C.weights(c))
    r = subprocess.run([sys.executable, "-m", "zipage_b200", "generate", "--model", str(folder), "--dtype", "float32", "--greedy",
                        "--new-tokens", "6", "--max-tokens", "512", "--prompt", ",".join(map(str, C.tokens(c, 30, 4))), "--prompt", "5"],
                       capture_output=True, text=True, cwd=ROOT, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(x) for x in r.stdout.splitlines() if x.startswith("[")]
    assert lines == [_greedy_oracle(name, C.tokens(c, 30, 4), 6), _greedy_oracle(name, [5], 6)]

    a, b = C.tokens(c, 100, 5), C.tokens(c, 70, 6)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:80], "want": [0, 79]}, {"id": "b", "tokens": b[:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:3], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[80:81], "want": [0]}, {"id": "b", "tokens": b[3:], "want": [66, 1]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[81:], "want": [18]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": b, "want": [69]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                       text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    wa, wb = _oracle(name, a)[0], _oracle(name, b)[0]
    want = {0: wa[[0, 79]], 2: torch.stack([wa[80], wb[69], wb[4]]), 3: wa[[99]], 4: wb[[69]]}
    assert sorted(p.name for p in out.iterdir()) == sorted(f"{i}.f32" for i in want)
    for i, w in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{i}.f32", dtype="<f4")).view(len(w), -1)
        _ok(got, w, torch.float32)
