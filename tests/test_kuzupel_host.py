"""Kuzupel without a GPU: configuration reader, registry, weight table, cache shapes, oracle."""
import json
import math

import pytest
import torch

import _kuzupel_oracle as oracle
from rhinoforge_b200.api.errors import UnsupportedModelError
from rhinoforge_b200.models.mixed import (ClippedGLU, GroupedAttention, MixedConfig, MixedLayer, MoE, Rotary, TokenPairs, random_weights,
                                          weight_shapes)
from rhinoforge_b200.runtime.mixed_cache import MixedCache


def small_config(**kw) -> MixedConfig:
    biased = GroupedAttention(4, 2, 8, 12, 0.4, sink=False, gate=False, window=4, distance_bias=True, norm_all=True)
    rotary = GroupedAttention(6, 3, 10, 7, 0.5, rot=Rotary(6, 100.0), sink=False, unit_sink=True, window=5, keep_first=2, conv=3, gate_by_head=True)
    experts = MoE(6, 2, 10, router="chosen", limit=1.5, shared_ff=7, shared_limit=0.5, shared_gate=True)
    return MixedConfig.kuzupel("kuzupel", 50, 24, 1e-5, (MixedLayer(biased, ClippedGLU(30, 2.0)), MixedLayer(rotary, experts), MixedLayer(rotary)),
                               pairs=TokenPairs(11, 3, 7), embed_scale=2.0, residual_mult=0.25, logit_softcap=4.0, **kw)


def all_weights(cfg, dtype=torch.float32):
    get = random_weights(cfg, dtype=dtype)
    return {n: get(n) for n, _, _ in weight_shapes(cfg)}


def test_config_round_trip_and_refusals():
    cfg = small_config()
    raw = json.loads(json.dumps(cfg.to_kuzupel()))
    assert MixedConfig.from_kuzupel(raw) == cfg
    bad = [(("layers", 0, "type"), "mamba1"), (("layers", 0, "mlp", "kind"), "relu"), (("layers", 0, "mlp", "limit"), 0), (("layers", 0, "mixer", "conv"), 4),
           (("layers", 0, "mixer", "mask", "keep_first"), 1), (("layers", 0, "mixer", "rot"), {"dims": 2, "base": 10.0}), (("layers", 1, "mixer", "conv"), 0),
           (("layers", 1, "mixer", "kv_heads"), 4), (("layers", 1, "mixer", "rot", "dims"), 7), (("layers", 1, "mixer", "rot", "dims"), 12),
           (("layers", 1, "mixer", "rot", "scaling"), {}), (("layers", 1, "mixer", "mask", "size"), 0), (("layers", 1, "mixer", "mask", "keep_first"), -1),
           (("layers", 1, "mlp", "router", "top"), 7), (("layers", 1, "mlp", "router", "groups"), {"count": 2}), (("layers", 1, "mlp", "shared", "act"), "x"),
           (("layers", 1, "mlp", "expert", "limit"), None), (("vocab",), "x"), (("layers",), []), (("norm", "eps"), None), (("embedding", "scale"), "1"),
           (("embedding", "bigram", "buckets"), 0), (("embedding", "bigram", "mul_cur"), -1), (("residual_mult",), 0), (("logit_softcap",), 0), (("tied",), True)]
    for path, value in bad:
        broken = json.loads(json.dumps(raw))
        d = broken
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            MixedConfig.from_kuzupel(broken)
    # what may be left out: mask, kept tokens, rotation, shared expert, token pairs, embedding scale, factor, soft cap
    lean = json.loads(json.dumps(raw))
    del lean["embedding"], lean["residual_mult"], lean["logit_softcap"], lean["layers"][1]["mlp"]["shared"], lean["layers"][1]["mixer"]["rot"]
    lean["layers"][0]["mixer"].update(mask=None)
    del lean["layers"][1]["mixer"]["mask"]["keep_first"]
    got = MixedConfig.from_kuzupel(lean)
    assert (got.embed_scale, got.residual_mult, got.logit_softcap, got.pairs) == (1.0, 1.0, None, None)
    assert got.layers[0].mixer.window is None and got.layers[1].mixer.keep_first == 0 and got.layers[1].mixer.rot is None
    assert got.layers[1].mlp == MoE(6, 2, 10, router="chosen", limit=1.5)


def test_architecture_resolves_through_the_registry(tmp_path):
    from rhinoforge_b200.api._loading import local_native_config
    from rhinoforge_b200.api.causal_lm import RPUModelForCausalLM
    from rhinoforge_b200.runtime.registry import get_adapter
    (tmp_path / "config.json").write_text(json.dumps(small_config().to_kuzupel()))
    got = local_native_config(str(tmp_path))
    adapter = get_adapter(got["architecture"])
    cfg = adapter.config_from_dict(got)
    assert adapter.ARCH == "Kuzupel" and cfg.vocab_size == 50 and cfg.num_hidden_layers == 3 and cfg._mixed == small_config()
    assert cfg.model_type == "kuzupel" and not cfg.tie_word_embeddings
    with pytest.raises(UnsupportedModelError, match="device='rpu'"):
        RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=torch.bfloat16)


def test_checkpoint_with_a_wrong_shape_is_refused(tmp_path):
    from safetensors.torch import save_file

    from rhinoforge_b200.adapters.kuzupel import KuzupelAdapter
    from rhinoforge_b200.api._loading import checkpoint_tensor_getter
    from rhinoforge_b200.api.errors import WeightShapeMismatchError
    cfg = small_config()
    w = all_weights(cfg)
    adapter = KuzupelAdapter(None, config=KuzupelAdapter.config_from_dict(cfg.to_kuzupel()), get_weight=w.__getitem__)
    save_file(w, str(tmp_path / "model.safetensors"))
    adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))
    for name, broken in (("bigram", lambda t: t[:-1]), ("l0.mix.q.norm", lambda t: t[:8]), ("l1.mlp.shared.sg", None)):
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
    assert shapes["bigram"] == (12, 24) and shapes["l0.mix.q.norm"] == (32,) and shapes["l0.mix.k.norm"] == (16,) and shapes["l1.mix.q.norm"] == (10,)
    assert shapes["l1.mix.q.conv"] == (60, 3) and shapes["l1.mix.v.conv"] == (21, 3) and shapes["l1.mix.g"] == (6, 24) and shapes["l0.mlp.gate"] == (30, 24)
    assert shapes["l1.mlp.router.b"] == (6,) and shapes["l1.mlp.shared.sg"] == (1, 24) and shapes["head"] == (50, 24) and shapes["l1.mix.o"] == (24, 42)
    assert not any(n.startswith(("l2.mlp", "l2.norm2", "side")) or n.endswith(("shift", "sink", "ls1", "correction", "l0.mix.g")) for n in shapes)


def test_cache_shapes_follow_the_layers():
    cfg = small_config()
    cache = MixedCache(cfg, 3, 64, device="cpu", dtype=torch.float32)
    assert tuple(cache.kv[0].shape) == (2, cache.num_pages, 2, 16, 16) and cache.conv[0] is None
    assert tuple(cache.conv[1].shape) == (3, 2, 12 * 16) and cache.recurrent == [None] * 3 and cache.shift is None
    assert cache.last_token.dtype == torch.int32 and len(cache.state_tensors()) == 3
    assert cache.layer_state(0).last_token == cache.layer_state(2).last_token == cache.last_token.data_ptr()
    plain = MixedCache(MixedConfig.kuzupel("x", 50, 24, 1e-5, (cfg.layers[0],)), 3, 64, device="cpu")
    assert plain.last_token is None and not plain.layer_state(0).last_token and plain.state_tensors() == []


def test_slopes_and_rotation_match_the_definition():
    for heads in (1, 3, 8, 20):
        got = GroupedAttention(heads, 1, 8, 8, 1.0, distance_bias=True).slopes()
        assert got.tolist() == pytest.approx([oracle.slope(h, heads) for h in range(heads)], rel=1e-12)
    x = torch.randn(5, 2, 9, dtype=torch.float64, generator=torch.Generator().manual_seed(0))
    y = oracle.rotate(x, 3, {"dims": 6, "base": 50.0})
    for t in range(5):
        for i in range(3):
            a = (3 + t) * 50.0 ** (-2 * i / 6)
            z = torch.complex(x[t, 0, i], x[t, 0, i + 3]) * complex(math.cos(a), math.sin(a))
            assert float(abs(torch.complex(y[t, 0, i], y[t, 0, i + 3]) - z)) < 1e-12
    assert torch.equal(y[..., 6:], x[..., 6:])


def test_oracle_mechanisms_on_small_cases():
    assert oracle.visible(6, {"size": 3, "keep_first": 2}) == [0, 1, 4, 5, 6] and oracle.visible(2, {"size": 2}) == [1, 2]
    assert oracle.visible(3, {"size": 9, "keep_first": 1}) == [0, 1, 2, 3] and oracle.visible(2, None) == [0, 1, 2]
    b = {"buckets": 11, "mul_prev": 3, "mul_cur": 7}
    assert [oracle.bigram_row(p, 5, b) for p in (None, 0, 4)] == [11, 35 % 11, 47 % 11]
    p = oracle.softmax(torch.zeros(3, dtype=torch.float64), True)
    assert p.tolist() == pytest.approx([0.25] * 3) and float(oracle.softmax(torch.tensor([900.0, 900.0]), True).sum()) == pytest.approx(1.0)
    picks, a = oracle.choose(torch.tensor([0.0, 2.0, -1.0, 2.0], dtype=torch.float64), 3)
    assert picks == [1, 3, 0] and a.tolist() == pytest.approx([1 / (2 + math.exp(-2))] * 2 + [math.exp(-2) / (2 + math.exp(-2))])
    one = {k: torch.ones(1, 1, dtype=torch.float64) for k in ("gate", "up", "down")}
    h = torch.tensor([[3.0], [-3.0]], dtype=torch.float64)
    got = oracle.clipped_glu(h, one, "", 2.0)
    assert got[0].item() == pytest.approx(2 / (1 + math.exp(-3.404)) * 3) and got[1].item() == pytest.approx(-3 / (1 + math.exp(5.106)) * -1)


def test_oracle_is_causal():
    cfg = small_config()
    w = all_weights(cfg)
    ids = torch.randint(0, 50, (13,), generator=torch.Generator().manual_seed(0))
    full = oracle.forward(cfg.to_kuzupel(), w, ids)
    assert full.shape == (13, 50) and float(full.abs().max()) < 4.0
    for n in (1, 2, 7):
        torch.testing.assert_close(oracle.forward(cfg.to_kuzupel(), w, ids[:n]), full[:n], rtol=1e-9, atol=1e-9)


def test_example_configuration_is_checked():
    import importlib.util
    from pathlib import Path
    root = Path(__file__).resolve().parents[1]
    spec = importlib.util.spec_from_file_location("kuzupel_example", root / "examples" / "kuzupel.py")
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    cfg = mod.load_config(root / "examples" / "configs" / "kuzupel.toml")
    assert cfg["model"]["checkpoint"] == "models/kuzupel" and cfg["generation"]["slots"] == 2
