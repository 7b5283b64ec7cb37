"""Zulopel without a GPU: configuration reader, registry, weight table, cache shapes, oracle."""
import json

import pytest
import torch

import _zulopel_oracle as oracle
from rhinoforge_b200.api.errors import UnsupportedModelError
from rhinoforge_b200.models.mixed import (GroupedAttention, Mamba1, MixedConfig, MixedLayer, MoE, Rotary, YarnScaling, random_weights,
                                          weight_shapes)
from rhinoforge_b200.runtime.mixed_cache import MixedCache, head_layout

YARN = Rotary(6, 100.0, YarnScaling(4.0, 32, 4.0, 0.5))


def small_config() -> MixedConfig:
    return MixedConfig.zulopel("zulopel", 50, 24, 1e-5, (
        MixedLayer(Mamba1(20, 5, 3, 3), MoE(6, 2, 10, 3, 2, 7)),
        MixedLayer(GroupedAttention(4, 2, 8, 12, 0.4, 4, YARN, True), MoE(4, 1, 9)),
        MixedLayer(GroupedAttention(2, 2, 10, 12, 0.5, None, None, True))), 3.0)


def all_weights(cfg, dtype=torch.float32):
    get = random_weights(cfg, dtype=dtype)
    return {n: get(n) for n, _, _ in weight_shapes(cfg)}


def test_config_round_trip_and_refusals():
    cfg = small_config()
    raw = json.loads(json.dumps(cfg.to_zulopel()))
    assert MixedConfig.from_zulopel(raw) == cfg
    bad = [(("layers", 0, "type"), "hgrn2"), (("layers", 0, "mlp", "kind"), "dense"), (("layers", 0, "mixer", "conv"), 0),
           (("layers", 1, "mixer", "window"), 4), (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "rot", "dims"), 7),
           (("layers", 1, "mixer", "rot", "dims"), 10), (("layers", 1, "mixer", "rot", "scaling", "factor"), 0),
           (("layers", 0, "mlp", "router", "groups", "count"), 4), (("layers", 0, "mlp", "router", "groups", "keep"), 4),
           (("layers", 0, "mlp", "router", "top"), 5), (("layers", 0, "mlp", "shared", "act"), "gelu"), (("vocab",), "x"), (("layers",), []),
           (("layers", 2, "mixer", "vdim"), 13), (("norm", "eps"), None), (("embedding", "scale"), "1"), (("tied",), True)]
    for path, value in bad:
        broken = json.loads(json.dumps(raw))
        d = broken
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            MixedConfig.from_zulopel(broken)
    # what may be left out: rotation, its scaling, mask, groups, shared expert, embedding scale
    lean = json.loads(json.dumps(raw))
    del lean["embedding"], lean["layers"][0]["mlp"]["router"]["groups"], lean["layers"][0]["mlp"]["shared"]
    lean["layers"][1]["mixer"].update(mask=None)
    lean["layers"][1]["mixer"]["rot"]["scaling"] = None
    got = MixedConfig.from_zulopel(lean)
    assert got.embed_scale == 1.0 and got.layers[0].mlp == MoE(6, 2, 10) and got.layers[1].mixer.chunk is None and got.layers[1].mixer.rot == Rotary(6, 100.0)


def test_architecture_resolves_through_the_registry(tmp_path):
    from rhinoforge_b200.api._loading import local_native_config
    from rhinoforge_b200.api.causal_lm import RPUModelForCausalLM
    from rhinoforge_b200.runtime.registry import get_adapter
    raw = small_config().to_zulopel()
    (tmp_path / "config.json").write_text(json.dumps(raw))
    got = local_native_config(str(tmp_path))
    adapter = get_adapter(got["architecture"])
    cfg = adapter.config_from_dict(got)
    assert adapter.ARCH == "Zulopel" and cfg.vocab_size == 50 and cfg.num_hidden_layers == 3 and cfg._mixed == small_config()
    assert cfg.model_type == "zulopel" and not cfg.tie_word_embeddings
    with pytest.raises(UnsupportedModelError, match="device='rpu'"):
        RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=torch.bfloat16)


def test_checkpoint_with_a_wrong_shape_is_refused(tmp_path):
    from safetensors.torch import save_file

    from rhinoforge_b200.adapters.zulopel import ZulopelAdapter
    from rhinoforge_b200.api._loading import checkpoint_tensor_getter
    from rhinoforge_b200.api.errors import WeightShapeMismatchError
    cfg = small_config()
    w = all_weights(cfg)
    adapter = ZulopelAdapter(None, config=ZulopelAdapter.config_from_dict(cfg.to_zulopel()), get_weight=w.__getitem__)
    save_file(w, str(tmp_path / "model.safetensors"))
    adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))
    w["l0.mlp.e5.down"] = w["l0.mlp.e5.down"][:, :-1].contiguous()
    save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(WeightShapeMismatchError, match="l0.mlp.e5.down"):
        adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))
    w.pop("l1.mix.sink")
    save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(WeightShapeMismatchError, match="l1.mix.sink"):
        adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))


def test_weight_table_names_every_tensor_once():
    shapes = {n: s for n, s, _ in weight_shapes(small_config())}
    assert len(shapes) == len(list(weight_shapes(small_config())))
    assert shapes["l0.mix.conv"] == (20, 3) and shapes["l0.mix.x"] == (13, 20) and shapes["l1.mix.vmix"] == () and shapes["l1.mix.g"] == (48, 24)
    assert shapes["head"] == (50, 24) and shapes["l0.mlp.shared.down"] == (24, 7) and shapes["l2.ls1"] == (24,)
    assert not any(n.startswith(("l1.mlp.shared", "l2.mlp", "l2.norm2", "l2.ls2", "side")) or n.endswith("shift") for n in shapes)


def test_cache_shapes_follow_the_layers():
    cfg = small_config()
    cache = MixedCache(cfg, 3, 64, device="cpu", dtype=torch.float32)
    assert tuple(cache.recurrent[0].shape) == (3, 24, 8) and tuple(cache.conv[0].shape) == (3, 2, 24) and cache.kv[0] is None
    assert tuple(cache.kv[1].shape) == (2, cache.num_pages, 2, 16, 16) and cache.recurrent[1] is None and cache.shift is None
    assert len(cache.state_tensors()) == 2 and cache.layer_state(1).pool_pages == cache.num_pages and not cache.layer_state(0).k_pool
    att = cfg.layers[1].mixer
    assert head_layout(att, torch.bfloat16) == (64, True) and head_layout(att, torch.float32) == (16, False)
    assert head_layout(GroupedAttention(1, 1, 65, 8, 1.0), torch.bfloat16) == (128, True)
    assert head_layout(GroupedAttention(1, 1, 8, 257, 1.0), torch.bfloat16) == (264, False)
    assert head_layout(GroupedAttention(1, 1, 8, 8, -1.0), torch.float16) == (8, False)


def test_rotation_frequencies_match_the_definition():
    for rot in (Rotary(6, 100.0), YARN, Rotary(16, 1e5, YarnScaling(32.0, 4096, 32.0, 1.0)), Rotary(2, 7.0, YarnScaling(2.0, 8, 1.0, 1.0))):
        raw = {"dims": rot.dims, "base": rot.base, **({"scaling": vars(rot.scaling)} if rot.scaling else {})}
        f, amp = oracle.rotation_frequencies(raw)
        torch.testing.assert_close(rot.frequencies(), f, rtol=1e-12, atol=0)
        cos, _ = rot.tables(5, "cpu")
        torch.testing.assert_close(cos[3].double(), torch.cos(3 * f) * amp, rtol=1e-6, atol=1e-7)


def test_oracle_is_causal_and_respects_its_chunks():
    cfg = small_config()
    w = all_weights(cfg)
    ids = torch.randint(0, 50, (13,), generator=torch.Generator().manual_seed(0))
    full = oracle.forward(cfg.to_zulopel(), w, ids)
    assert full.shape == (13, 50)
    for n in (1, 2, 7):
        torch.testing.assert_close(oracle.forward(cfg.to_zulopel(), w, ids[:n]), full[:n], rtol=1e-9, atol=1e-9)
    assert [oracle.first_visible(i, 4) for i in (0, 3, 4, 7, 8)] == [0, 0, 4, 4, 8]


def test_example_configuration_is_checked():
    import importlib.util
    from pathlib import Path
    root = Path(__file__).resolve().parents[1]
    spec = importlib.util.spec_from_file_location("zulopel_example", root / "examples" / "zulopel.py")
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    cfg = mod.load_config(root / "examples" / "configs" / "zulopel.toml")
    assert cfg["model"]["checkpoint"] == "models/zulopel" and cfg["generation"]["slots"] == 2


def test_groups_exclude_experts_even_when_every_choice_score_is_negative():
    s, corr = torch.tensor([0.4, 0.1, 0.3, 0.2]), torch.tensor([-1.0, -0.5, -2.0, -0.1])       # choice scores -0.6 -0.4 | -1.7 0.1
    assert oracle.choose(s, corr, 2, {"count": 2, "keep": 1}) == [3, 2]
    assert oracle.choose(s, corr, 2, {"count": 2, "keep": 2}) == [3, 1]
    assert oracle.choose(s, corr, 3, None) == [3, 1, 0]
