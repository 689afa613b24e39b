"""Model registry: config.json names the architecture, the architecture names a builder.

A builder takes (config dict, weights, dtype, device) and returns a `LoadedModel`: the module whose
forward(input_ids, positions) gives the final hidden states, the LM head, and which serving mode the
engine runs it in.  `build_engine` sizes caches and scheduler for it and returns the engine.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from types import SimpleNamespace

import torch

from .weights import read_model_weights


@dataclass
class LoadedModel:
    name: str
    model: torch.nn.Module
    lm_head: torch.Tensor
    hidden_size: int
    vocab_size: int
    dtype: torch.dtype
    portions: bool        # served in portion steps from `model.cache_spec()`; else prefill / decode with compression


_BUILDERS = {}
# kernel sources a family needs when the whole library is not built (zipage_b200.build.PARTS)
_PARTS = {}


def register(name, part=None):
    def add(fn):
        _BUILDERS[name] = fn
        _PARTS[name] = part
        return fn
    return add


def architectures():
    return sorted(_BUILDERS)


def read_config(model_dir):
    """-> (registered architecture name, config dict)."""
    config = json.loads((Path(model_dir) / "config.json").read_text())
    names = [config["architecture"]] if "architecture" in config else list(config.get("architectures") or [])
    for n in names:
        if n in _BUILDERS:
            return n, config
    raise ValueError(f"{model_dir}: architecture {names or '(none named)'} is not one of {architectures()}")


def kernel_part(model_dir):
    return _PARTS[read_config(model_dir)[0]]


def load_model(model_dir, dtype=torch.bfloat16, device="cuda") -> LoadedModel:
    name, config = read_config(model_dir)
    if dtype == torch.float32:     # true fp32 products
        torch.backends.cuda.matmul.allow_tf32 = False
    return _BUILDERS[name](config, read_model_weights(model_dir), dtype, torch.device(device))


@register("Similorn", part="similorn")
def _similorn(config, weights, dtype, device):
    from .similorn import SimilornConfig, SimilornModel
    cfg = SimilornConfig.from_dict(config)
    model = SimilornModel(cfg, dtype, device)
    model.load_weights(weights)
    return LoadedModel("Similorn", model, model.head, cfg.width, cfg.vocab, dtype, portions=True)


@register("Dobedra", part="dobedra")
def _dobedra(config, weights, dtype, device):
    from .dobedra import DobedraConfig, DobedraModel
    cfg = DobedraConfig.from_dict(config)
    model = DobedraModel(cfg, dtype, device)
    model.load_weights(weights)
    return LoadedModel("Dobedra", model, model.head, cfg.width, cfg.vocab, dtype, portions=True)


@register("Tukarax", part="tukarax")
def _tukarax(config, weights, dtype, device):
    from .tukarax import TukaraxConfig, TukaraxModel
    cfg = TukaraxConfig.from_dict(config)
    model = TukaraxModel(cfg, dtype, device)
    model.load_weights(weights)
    return LoadedModel("Tukarax", model, model.head, cfg.width, cfg.vocab, dtype, portions=True)


@register("Dinatar", part="dinatar")
def _dinatar(config, weights, dtype, device):
    from .dinatar import DinatarConfig, DinatarModel
    cfg = DinatarConfig.from_dict(config)
    model = DinatarModel(cfg, dtype, device, DinatarModel.ranks_of(weights))
    model.load_weights(weights)
    return LoadedModel("Dinatar", model, model.head, cfg.width, cfg.vocab, dtype, portions=True)


@register("Qwen3ForCausalLM")
def _qwen3(config, weights, dtype, device):
    from ..engine.native_engine import full_state_from_hf
    from ..layers.qwen3_block import Qwen3Model
    c = SimpleNamespace(**config)
    full, lm_head = full_state_from_hf(weights)
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        with device:
            model = Qwen3Model(c).eval()
    finally:
        torch.set_default_dtype(prev)
    model.load_full_state({k: v.to(device=device, dtype=dtype) for k, v in full.items()})
    return LoadedModel("Qwen3ForCausalLM", model, lm_head.to(device=device, dtype=dtype), c.hidden_size, c.vocab_size,
                       dtype, portions=False)


def build_engine(model_dir, dtype=torch.bfloat16, device="cuda", max_tokens=65536, max_seqs=8, block_size=None,
                 token_budget=8192, max_model_len=None, eos=None, greedy=False, graph=True, seed=0,
                 budget_blocks=8, query_cache_len=32):
    """An engine for the model in `model_dir` with pages for `max_tokens` tokens and slots for
    `max_seqs` running sequences.  The last two arguments are the page budget and window of the KV
    compression, for the architectures that are served with it."""
    return engine_for(load_model(model_dir, dtype, device), max_tokens, max_seqs, block_size, token_budget,
                      max_model_len, eos, greedy, graph, seed, budget_blocks, query_cache_len)


def engine_for(loaded, max_tokens=65536, max_seqs=8, block_size=None, token_budget=8192, max_model_len=None, eos=None,
               greedy=False, graph=True, seed=0, budget_blocks=8, query_cache_len=32):
    from ..engine.native_engine import NativeEngine
    m = loaded.model
    bs = block_size or (64 if loaded.portions else 256)
    pages = (max_tokens + bs - 1) // bs
    sched = SimpleNamespace(max_num_seqs=max_seqs, max_num_batched_tokens=token_budget, eos=eos, num_kvcache_blocks=pages,
                            kvcache_block_size=bs, enable_prefix_cache=False, max_concurrency=max_seqs,
                            enable_hybrid_engine=False)
    kw = dict(max_bs=max_seqs, max_model_len=max_model_len or max_tokens, greedy=greedy, graph=graph, seed=seed)
    if loaded.portions:
        from ..engine.cache import PagedStateCache
        sched.max_cache_blocks_per_seq, sched.query_cache_len = pages + 1, 0
        cache = PagedStateCache(m.cache_spec(), pages, bs, max_seqs, loaded.dtype, loaded.lm_head.device)
        m.bind_cache(cache)
        return NativeEngine(m, loaded.lm_head, None, None, sched, None, loaded.hidden_size, cache=cache, **kw)
    from ..compress import CompressConfig
    a = m.layers[0].self_attn
    L, dev, D = len(m.layers), loaded.lm_head.device, a.head_dim
    kv = torch.zeros((2, L, pages, bs, a.num_kv_heads, D), dtype=loaded.dtype, device=dev)
    qc = torch.zeros((L, max_seqs, query_cache_len, a.num_heads, D), dtype=loaded.dtype, device=dev)
    m.bind_caches(kv, qc)
    sched.max_cache_blocks_per_seq, sched.query_cache_len = budget_blocks, query_cache_len
    ccfg = CompressConfig(budget_blocks=budget_blocks, query_cache_len=query_cache_len, use_redudancy=True,
                          lightning_redudancy=True, redudancy_lambda=0.5, enable_pooling=True)
    return NativeEngine(m, loaded.lm_head, kv, qc, sched, ccfg, loaded.hidden_size, **kw)
