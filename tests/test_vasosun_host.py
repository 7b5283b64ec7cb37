"""Vasosun without a GPU: configuration reader, registry, weight table, cache shapes, oracle."""
import json
import math

import pytest
import torch

import _vasosun_oracle as oracle
from rhinoforge_b200.api.errors import UnsupportedModelError
from rhinoforge_b200.models.mixed import (DeltaRule, GatedMLP, GroupedAttention, LatentAttention, MixedConfig, MixedLayer, MoE, Rotary, TokenPairs,
                                          YarnScaling, random_weights, weight_shapes)
from rhinoforge_b200.runtime.mixed_cache import MixedCache

ROT = Rotary(6, 100.0, YarnScaling(2.0, 50.0, 8.0, 1.0))


def small_config(**kw) -> MixedConfig:
    window = GroupedAttention(4, 2, 8, 12, 0.4, qk_norm=False, sink=False, gate=False, log_bias=True, window=4, growth=0.3, growth_every=5)
    own = LatentAttention(3, 10, 7, 18, 0.5, q_rank=9, rot=ROT)
    other = LatentAttention(2, 4, 5, 18, 0.6, q_rank=11, rot=ROT, kv_from=1)
    experts = MoE(6, 2, 10, gated=False, identity=3, renormalise=False)
    return MixedConfig.vasosun("vasosun", 50, 24, 1e-5, (MixedLayer(DeltaRule(4, 2, 10, 6, 3), GatedMLP(30)), MixedLayer(own, experts),
                                                         MixedLayer(window), MixedLayer(other, experts)),
                               input_taps=3, pairs=TokenPairs(11, 3, 7), logit_softcap=4.0, **kw)


def all_weights(cfg, dtype=torch.float32):
    get = random_weights(cfg, dtype=dtype)
    return {n: get(n) for n, _, _ in weight_shapes(cfg)}


def test_config_round_trip_and_refusals():
    cfg = small_config()
    raw = json.loads(json.dumps(cfg.to_vasosun()))
    assert MixedConfig.from_vasosun(raw) == cfg
    bad = [(("layers", 0, "type"), "mamba1"), (("layers", 0, "mlp", "kind"), "relu"), (("layers", 0, "mlp", "ff"), 0), (("layers", 0, "mixer", "conv"), 0),
           (("layers", 0, "mixer", "scale"), 1.0), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "dim"), 257), (("layers", 0, "mixer", "vdim"), 513),
           (("layers", 1, "mixer", "rot", "dims"), 4), (("layers", 1, "mixer", "rot_dim"), 7), (("layers", 1, "mixer", "rot"), None),
           (("layers", 1, "mixer", "rot", "scaling"), {"factor": 2.0}), (("layers", 1, "mixer", "mask"), {"size": 4}), (("layers", 1, "mixer", "kv_from"), 0),
           (("layers", 1, "mixer", "q_rank"), 0), (("layers", 2, "mixer", "kv_heads"), 3), (("layers", 2, "mixer", "mask", "size"), 0),
           (("layers", 2, "mixer", "mask", "keep_first"), 1), (("layers", 2, "mixer", "q_temp", "every"), 0), (("layers", 2, "mixer", "rot"), {"dims": 2}),
           (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "kv_from"), 2), (("layers", 3, "mixer", "kv_rank"), 20),
           (("layers", 3, "mixer", "rot", "base"), 50.0), (("layers", 1, "mlp", "router", "top"), 10), (("layers", 1, "mlp", "router", "identity"), 251),
           (("layers", 1, "mlp", "router", "identity"), -1), (("layers", 1, "mlp", "shared"), {"ff": 4}), (("vocab",), "x"), (("layers",), []),
           (("norm", "eps"), None), (("embedding", "scale"), 1.0), (("embedding", "bigram", "buckets"), 0), (("canon", "taps"), 0), (("logit_softcap",), 0),
           (("tied",), True)]
    for path, value in bad:
        broken = json.loads(json.dumps(raw))
        d = broken
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            MixedConfig.from_vasosun(broken)
    # what may be left out: convolution, token pairs, soft cap, window, growth, stretch, identity experts
    lean = json.loads(json.dumps(raw))
    del lean["canon"], lean["embedding"], lean["logit_softcap"], lean["layers"][2]["mixer"]["mask"], lean["layers"][2]["mixer"]["q_temp"]
    del lean["layers"][1]["mlp"]["router"]["identity"], lean["layers"][1]["mixer"]["rot"]["scaling"], lean["layers"][3]
    got = MixedConfig.from_vasosun(lean)
    assert (got.input_taps, got.pairs, got.logit_softcap) == (0, None, None) and got.layers[1].mixer.rot == Rotary(6, 100.0)
    assert got.layers[2].mixer.window is None and got.layers[2].mixer.growth_every == 0 and got.layers[1].mlp.identity == 0
    assert not any("canon" in n or n == "bigram" for n, _, _ in weight_shapes(got))


def test_architecture_resolves_through_the_registry(tmp_path):
    from rhinoforge_b200.api._loading import local_native_config
    from rhinoforge_b200.api.causal_lm import RPUModelForCausalLM
    from rhinoforge_b200.runtime.registry import get_adapter
    (tmp_path / "config.json").write_text(json.dumps(small_config().to_vasosun()))
    got = local_native_config(str(tmp_path))
    adapter = get_adapter(got["architecture"])
    cfg = adapter.config_from_dict(got)
    assert adapter.ARCH == "Vasosun" and cfg.vocab_size == 50 and cfg.num_hidden_layers == 4 and cfg._mixed == small_config()
    assert cfg.model_type == "vasosun" and not cfg.tie_word_embeddings
    with pytest.raises(UnsupportedModelError, match="device='rpu'"):
        RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=torch.bfloat16)


def test_checkpoint_with_a_wrong_shape_is_refused(tmp_path):
    from safetensors.torch import save_file

    from rhinoforge_b200.adapters.vasosun import VasosunAdapter
    from rhinoforge_b200.api._loading import checkpoint_tensor_getter
    from rhinoforge_b200.api.errors import WeightShapeMismatchError
    cfg = small_config()
    w = all_weights(cfg)
    adapter = VasosunAdapter(None, config=VasosunAdapter.config_from_dict(cfg.to_vasosun()), get_weight=w.__getitem__)
    save_file(w, str(tmp_path / "model.safetensors"))
    adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))
    for name, broken in (("bigram", lambda t: t[:-1]), ("l0.norm1b", lambda t: t.reshape(1)), ("l3.mix.uq", None), ("l1.mlp.correction", lambda t: t[:6])):
        bad = dict(w)
        if broken is None:
            bad.pop(name)
        else:
            bad[name] = broken(w[name]).contiguous()
        save_file(bad, str(tmp_path / "model.safetensors"))
        with pytest.raises(WeightShapeMismatchError, match=name):
            adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))


def test_weight_table_names_every_tensor_once():
    shapes = {n: s for n, s, _ in weight_shapes(small_config())}
    assert len(shapes) == len(list(weight_shapes(small_config())))
    assert shapes["l0.norm1"] == shapes["l0.norm2b"] == shapes["final.norm"] == () and shapes["l0.canon1"] == shapes["l3.canon2"] == (24, 3)
    assert shapes["l0.mix.q"] == (20, 24) and shapes["l0.mix.v.conv"] == (24, 3) and shapes["l0.mix.norm"] == (6,) and shapes["l0.mix.o"] == (24, 24)
    assert shapes["l1.mix.dkv"] == (24, 24) and shapes["l1.mix.dkv.norm"] == (18,) and shapes["l1.mix.uq"] == (48, 9) and shapes["l1.mix.uv"] == (21, 18)
    assert shapes["l1.mlp.router"] == (9, 24) and shapes["l1.mlp.correction"] == (9,) and shapes["l2.mix.r1"] == (4,) and shapes["l3.mix.uk"] == (8, 18)
    absent = ("l2.norm2", "l2.norm2b", "l2.canon2", "l3.mix.dkv", "l3.mix.dkv.norm", "l1.mlp.e0.gate", "l1.mlp.e6.up", "l1.mix.q", "l2.mix.q.norm", "side.embed")
    assert not any(n in shapes for n in absent)


def test_cache_shapes_follow_the_layers():
    cfg = small_config()
    cache = MixedCache(cfg, 3, 64, device="cpu", dtype=torch.float32)
    assert tuple(cache.latent[1].shape) == (cache.num_pages, 16, 32 + 16) and cache.latent[3] is None
    assert cache.layer_state(3).latent_pool == cache.layer_state(1).latent_pool == cache.latent[1].data_ptr()
    assert tuple(cache.recurrent[0].shape) == (3, 4, 16, 8) and tuple(cache.conv[0].shape) == (3, 3, 2 * 2 * 16 + 4 * 8)
    assert tuple(cache.inputs.shape) == (4, 2, 3, 2, 24) and cache.layer_state(2).input_state[1] == cache.inputs[2, 1].data_ptr()
    assert tuple(cache.kv[2].shape) == (2, cache.num_pages, 2, 16, 16) and len(cache.state_tensors()) == 4
    half = MixedCache(cfg, 3, 64, device="cpu", dtype=torch.bfloat16)
    assert tuple(half.recurrent[0].shape) == (3, 4, 64, 32) and half.recurrent[0].dtype == torch.float32 and half.inputs.dtype == torch.bfloat16


def test_stretched_rotation_matches_the_definition():
    for rot in (ROT, Rotary(64, 1e6, YarnScaling(8.0, 128, 32.0, 1.0)), Rotary(2, 10.0), Rotary(20, 1e4, YarnScaling(1.0, 300, 16.0, 2.0))):
        y = rot.scaling
        f, amp = oracle.frequencies({"dims": rot.dims, "base": rot.base, "scaling": y and {"factor": y.factor, "original": y.original, "fast": y.fast, "slow": y.slow}})
        assert rot.frequencies().tolist() == pytest.approx(f, rel=1e-12)
        cos, sin = rot.tables(40, "cpu")
        assert cos[33].tolist() == pytest.approx([amp * math.cos(33 * x) for x in f], abs=1e-6) and sin[0].abs().max() == 0


def test_oracle_mechanisms_on_small_cases():
    assert [oracle.query_factor(p, {"coef": 0.5, "every": 4}) for p in (0, 2, 3, 11)] == pytest.approx([1, 1, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(4)])
    assert float(oracle.log_bias(torch.tensor(2.0), torch.tensor(3.0), torch.tensor(1.0))) == pytest.approx(2 * math.log(4))
    b = {"buckets": 11, "mul_prev": 3, "mul_cur": 7}
    assert [oracle.pair_row(p, 5, b) for p in (None, 0, 4)] == [11, 35 % 11, 47 % 11]
    x = torch.tensor([[1.0], [10.0], [100.0], [1000.0]])
    assert oracle.causal_convolution(x, torch.tensor([[1.0, 2.0, 3.0]])).flatten().tolist() == [3, 32, 321, 3210]
    y = oracle.rotate(torch.tensor([[[0.0, 0.0]], [[1.0, 0.0]]], dtype=torch.float64), {"dims": 2, "base": 5.0})
    assert y[1, 0].tolist() == pytest.approx([math.cos(1), math.sin(1)])
    picks, a = oracle.choose(torch.log(torch.tensor([0.1, 0.5, 0.4])), torch.tensor([0.6, 0.0, 0.0]), 2)
    assert picks == [0, 1] and a.tolist() == pytest.approx([0.1, 0.5])
    # one head, unit keys: the state forgets, then what the key already holds is taken off before the write
    q = k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]]], dtype=torch.float64)
    v = torch.tensor([[[4.0]], [[1.0]]], dtype=torch.float64)
    o, s = oracle.delta_rule(q, k, v, torch.tensor([[0.5], [0.25]], dtype=torch.float64), torch.tensor([[1.0], [0.5]], dtype=torch.float64))
    assert o.flatten().tolist() == pytest.approx([2.0, 1.0 + 0.25 * (1.0 - 1.0)]) and s[0, 1].abs().sum() == 0


def test_oracle_is_causal_and_shares_the_cache():
    cfg = small_config()
    w = all_weights(cfg)
    ids = torch.randint(0, 50, (13,), generator=torch.Generator().manual_seed(0))
    full = oracle.forward(cfg.to_vasosun(), w, ids)
    assert full.shape == (13, 50) and float(full.abs().max()) < 4.0
    for n in (1, 2, 7):
        torch.testing.assert_close(oracle.forward(cfg.to_vasosun(), w, ids[:n]), full[:n], rtol=1e-9, atol=1e-9)
    taps, other = [], []
    oracle.forward(cfg.to_vasosun(), w, ids, taps)
    w["l1.mix.dkv"] = w["l1.mix.dkv"] * 1.5
    oracle.forward(cfg.to_vasosun(), w, ids, other)
    assert torch.equal(taps[0], other[0]) and not torch.equal(taps[3], other[3])


def test_example_configuration_is_checked():
    import importlib.util
    from pathlib import Path
    root = Path(__file__).resolve().parents[1]
    spec = importlib.util.spec_from_file_location("vasosun_example", root / "examples" / "vasosun.py")
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    cfg = mod.load_config(root / "examples" / "configs" / "vasosun.toml")
    assert cfg["model"]["checkpoint"] == "models/vasosun" and cfg["generation"]["slots"] == 2
