"""The registry's other architecture: a small Qwen3 folder in the Hugging Face layout through
`build_engine`, against the engine put together by hand from the same weights."""
import json
import types

import pytest
import torch

import similorn_cases as C

pytestmark = pytest.mark.gpu
HID, INTER, HQ, HKV, LAYERS, VOCAB = 256, 384, 4, 2, 2, 500
CONFIG = {"architectures": ["Qwen3ForCausalLM"], "hidden_size": HID, "intermediate_size": INTER, "num_attention_heads": HQ,
          "num_key_value_heads": HKV, "head_dim": 128, "num_hidden_layers": LAYERS, "vocab_size": VOCAB, "hidden_act": "silu",
          "rms_norm_eps": 1e-6, "max_position_embeddings": 4096, "rope_theta": 1e6}


def _weights():
    g = torch.Generator().manual_seed(0)
    r = lambda o, i: (torch.randn(o, i, generator=g) / i ** 0.5).to(torch.bfloat16)
    one = lambda n: torch.ones(n, dtype=torch.bfloat16)
    w = {"model.embed_tokens.weight": r(VOCAB, HID) * 10, "model.norm.weight": one(HID), "lm_head.weight": r(VOCAB, HID)}
    for i in range(LAYERS):
        p = f"model.layers.{i}."
        for n, o in (("q", HQ), ("k", HKV), ("v", HKV)):
            w[p + f"self_attn.{n}_proj.weight"] = r(o * 128, HID)
        w.update({p + "self_attn.o_proj.weight": r(HID, HQ * 128), p + "self_attn.q_norm.weight": one(128),
                  p + "self_attn.k_norm.weight": one(128), p + "mlp.gate_proj.weight": r(INTER, HID),
                  p + "mlp.up_proj.weight": r(INTER, HID), p + "mlp.down_proj.weight": r(HID, INTER),
                  p + "input_layernorm.weight": one(HID), p + "post_attention_layernorm.weight": one(HID)})
    return w


def test_qwen3_folder_through_the_registry(tmp_path):
    from zipage_b200.compress import CompressConfig
    from zipage_b200.engine.native_engine import NativeEngine, full_state_from_hf
    from zipage_b200.engine.scheduler import SamplingParams, Sequence
    from zipage_b200.layers.qwen3_block import Qwen3Model
    from zipage_b200.models.registry import build_engine
    w = _weights()
    (tmp_path / "config.json").write_text(json.dumps(CONFIG))
    C.write_safetensors(tmp_path / "model.safetensors", w)
    prompts = [torch.randint(0, VOCAB, (n,), generator=torch.Generator().manual_seed(n)).tolist() for n in (300, 17)]
    requests = lambda: [Sequence(p, SamplingParams(1.0, 20, True)) for p in prompts]

    eng = build_engine(tmp_path, max_tokens=4096, max_seqs=2, budget_blocks=3, query_cache_len=16, greedy=True)
    assert not eng.portions
    seqs = requests()
    got = eng.generate(seqs)
    got = [got[s._h] for s in seqs]

    full, head = full_state_from_hf(w)
    prev = torch.get_default_dtype()
    torch.set_default_dtype(torch.bfloat16)
    try:
        with torch.device("cuda"):
            m = Qwen3Model(types.SimpleNamespace(**CONFIG)).eval()
    finally:
        torch.set_default_dtype(prev)
    m.load_full_state({k: v.cuda() for k, v in full.items()})
    kv = torch.zeros((2, LAYERS, 16, 256, HKV, 128), dtype=torch.bfloat16, device="cuda")
    qc = torch.zeros((LAYERS, 2, 16, HQ, 128), dtype=torch.bfloat16, device="cuda")
    m.bind_caches(kv, qc)
    cfg = types.SimpleNamespace(max_num_seqs=2, max_num_batched_tokens=8192, eos=None, num_kvcache_blocks=16, kvcache_block_size=256,
                                max_cache_blocks_per_seq=3, enable_prefix_cache=False, max_concurrency=2,
                                enable_hybrid_engine=False, query_cache_len=16)
    ccfg = CompressConfig(budget_blocks=3, query_cache_len=16, use_redudancy=True, lightning_redudancy=True, redudancy_lambda=0.5,
                          enable_pooling=True)
    by_hand = NativeEngine(m, head.cuda(), kv, qc, cfg, ccfg, HID, max_bs=2, max_model_len=4096, greedy=True)
    seqs = requests()
    want = by_hand.generate(seqs)
    assert got == [want[s._h] for s in seqs] and all(len(t) == 20 for t in got)
