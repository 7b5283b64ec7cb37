"""Vabarax without a GPU: configuration reader, registry, cache bookkeeping, scheduler policy, command line."""
import io
import json

import pytest
import torch

import _vabarax_oracle as oracle
from rhinoforge_b200.api.errors import RPUBackendError, UnsupportedModelError
from rhinoforge_b200.models.mixed import DenseMLP, HGRN2, LatentAttention, MixedConfig, MixedLayer, random_weights, weight_shapes
from rhinoforge_b200.runtime.mixed_cache import MixedCache


def small_config(**kw) -> MixedConfig:
    base = dict(name="vabarax", vocab_size=50, hidden_size=24, rms_eps=1e-5, side_dim=5, layers=(
        MixedLayer(HGRN2(2, 6, 10), DenseMLP(20)), MixedLayer(LatentAttention(3, 8, 12, 9, 0.4, 4))))
    return MixedConfig(**{**base, **kw})


def test_config_round_trip_and_refusals():
    cfg = small_config()
    raw = cfg.to_vabarax()
    assert MixedConfig.from_vabarax(json.loads(json.dumps(raw))) == cfg
    for path, value in ((("layers", 0, "type"), "mamba"), (("layers", 0, "mlp", "kind"), "moe"), (("layers", 1, "mixer", "heads"), 0),
                        (("layers", 1, "mixer", "rope"), True), (("vocab",), "x"), (("layers",), [])):
        bad = json.loads(json.dumps(raw))
        d = bad
        for k in path[:-1]:
            d = d[k]
        d[path[-1]] = value
        with pytest.raises(UnsupportedModelError):
            MixedConfig.from_vabarax(bad)


def test_architecture_resolves_through_the_registry(tmp_path):
    from rhinoforge_b200.api._loading import local_native_config
    from rhinoforge_b200.api.causal_lm import RPUModelForCausalLM
    from rhinoforge_b200.runtime.registry import get_adapter
    raw = small_config().to_vabarax()
    (tmp_path / "config.json").write_text(json.dumps(raw))
    got = local_native_config(str(tmp_path))
    assert got == raw
    adapter = get_adapter(got["architecture"])
    cfg = adapter.config_from_dict(got)
    assert cfg.vocab_size == 50 and cfg.num_hidden_layers == 2 and cfg._mixed == small_config()
    with pytest.raises(UnsupportedModelError, match="device='rpu'"):
        RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=torch.bfloat16)
    (tmp_path / "config.json").write_text(json.dumps({**raw, "architecture": "NoSuchDesign"}))
    with pytest.raises(UnsupportedModelError, match="NoSuchDesign"):
        RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=torch.bfloat16, device="rpu")


def test_checkpoint_with_a_wrong_shape_is_refused(tmp_path):
    from safetensors.torch import save_file

    from rhinoforge_b200.api._loading import checkpoint_tensor_getter
    from rhinoforge_b200.adapters.vabarax import VabaraxAdapter
    from rhinoforge_b200.api.errors import WeightShapeMismatchError
    cfg = small_config()
    get = random_weights(cfg)
    w = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    adapter = VabaraxAdapter(None, config=VabaraxAdapter.config_from_dict(cfg.to_vabarax()), get_weight=get)
    save_file(w, str(tmp_path / "model.safetensors"))
    adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))
    w["l1.mix.uk"] = w["l1.mix.uk"][:, :-1].contiguous()
    save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(WeightShapeMismatchError, match="l1.mix.uk"):
        adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))
    w.pop("l0.shift")
    save_file(w, str(tmp_path / "model.safetensors"))
    with pytest.raises(WeightShapeMismatchError, match="l0.shift"):
        adapter._validate_shapes(cfg, checkpoint_tensor_getter(str(tmp_path)))


def test_oracle_runs_and_is_causal():
    cfg = small_config()
    get = random_weights(cfg, dtype=torch.float32)
    w = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    ids = torch.randint(0, 50, (11,), generator=torch.Generator().manual_seed(0))
    full = oracle.forward(cfg.to_vabarax(), w, ids)
    assert full.shape == (11, 50)
    for n in (1, 2, 7):
        torch.testing.assert_close(oracle.forward(cfg.to_vabarax(), w, ids[:n]), full[:n], rtol=1e-9, atol=1e-9)


def test_cache_shapes_follow_the_layers_and_pages_are_reused():
    cfg = small_config()
    cache = MixedCache(cfg, 3, 64, device="cpu", dtype=torch.float32)
    assert cache.latent[0] is None and tuple(cache.latent[1].shape) == (cache.num_pages, 16, 16)
    assert tuple(cache.recurrent[0].shape) == (3, 2, 8, 16) and cache.recurrent[1] is None
    assert tuple(cache.shift.shape) == (2, 3, 24)
    if cache._pool is not None:
        cache.ensure(0, 33)
        cache.ensure(1, 16)
        assert cache.owned_pages(0) == 3 and cache.owned_pages(1) == 1 and cache.free_pages() == cache.num_pages - 4
        first = cache._pt_host[0, :3].tolist()
        cache.release(0)
        cache.ensure(2, 48)
        assert sorted(cache._pt_host[2, :3].tolist()) == sorted(first)
    assert len(cache.state_tensors()) == 2


class _FakeEngine:
    """Records the steps a scheduler asks for; the "next token" of an entry is its last token plus one."""

    def __init__(self, slots=2, pages=64, max_seq_len=64, max_tokens=8):
        class Cache:
            pass
        import numpy as np
        self.cache = Cache()
        self.cache.batch_size, self.cache.max_seq_len, self.cache.num_pages = slots, max_seq_len, pages
        self.cache.lengths = np.zeros(slots, dtype=np.int64)
        self.released = []
        self.cache.release = lambda s: (self.released.append(s), self.cache.lengths.__setitem__(s, 0))
        self.max_tokens, self.steps = max_tokens, []

    def run_step(self, tokens, slots, want):
        self.steps.append([(s, int(t.numel())) for s, t in zip(slots, tokens)])
        assert len(set(slots)) == len(slots) and sum(int(t.numel()) for t in tokens) <= self.max_tokens
        for s, t in zip(slots, tokens):
            self.cache.lengths[s] += int(t.numel())
        return torch.tensor([int(t[-1]) + 1 for t in tokens], dtype=torch.int32), [None] * len(tokens)

    def check_status(self):
        pass


def test_scheduler_mixes_portions_with_decoded_tokens_and_reuses_slots():
    from rhinoforge_b200.runtime.scheduler import RequestScheduler
    eng = _FakeEngine()
    out = RequestScheduler(eng).generate([torch.tensor([10] * 5), torch.tensor([20] * 12), torch.tensor([30])], 3)
    assert out == [[11, 12, 13], [21, 22, 23], [31, 32, 33]]
    assert any(len({n for _, n in st}) > 1 and 1 in {n for _, n in st} for st in eng.steps)      # a portion beside a decoded token
    assert max(len(st) for st in eng.steps) == 2                                                 # never more than the slots


def test_scheduler_admits_within_the_page_pool_and_refuses_the_impossible():
    from rhinoforge_b200.runtime.scheduler import RequestScheduler
    eng = _FakeEngine(slots=4, pages=2, max_tokens=64)
    out = RequestScheduler(eng).generate([torch.tensor([1] * 20), torch.tensor([5] * 20)], 4)
    assert [len(o) for o in out] == [4, 4] and max(len(st) for st in eng.steps) == 1             # two pages each: one at a time
    with pytest.raises(RPUBackendError, match="cached tokens"):
        RequestScheduler(eng).generate([torch.tensor([1] * 40)], 4)
    sched = RequestScheduler(eng, token_budget=4)
    with pytest.raises(RPUBackendError, match="not live"):
        sched.finish("x")
    for r in "abcd":
        sched.admit(r)
    with pytest.raises(RPUBackendError, match="slots are taken"):
        sched.admit("e")


def test_eos_ends_a_request_early():
    from rhinoforge_b200.runtime.scheduler import RequestScheduler
    out = RequestScheduler(_FakeEngine()).generate([torch.tensor([3]), torch.tensor([6])], 5, eos_token_id=7)
    assert out == [[4, 5, 6, 7], [7]]


def test_trace_command_line_is_documented():
    from rhinoforge_b200.runtime.trace import parse_args
    a = parse_args(["--model", "m", "--dtype", "float32", "--out", "o", "--max-tokens", "64"])
    assert (a.model, a.dtype, a.out, a.max_tokens) == ("m", "float32", "o", 64)
    with pytest.raises(SystemExit):
        parse_args(["--model", "m", "--out", "o", "--max-tokens", "64", "--dtype", "int8"])


def test_trace_replay_writes_logits_in_entry_order(tmp_path, monkeypatch, capsys):
    """The replay loop over a fake model: output files, 'done' lines, release after 'end'."""
    import numpy as np

    from rhinoforge_b200.api import causal_lm
    from rhinoforge_b200.runtime import trace

    class Engine(_FakeEngine):
        def run_step(self, tokens, slots, want):
            nxt, _ = super().run_step(tokens, slots, want)
            return nxt, [torch.stack([torch.full((3,), float(t[i])) for i in w]) if w else torch.empty(0, 3)
                         for t, w in zip(tokens, want)]

    class Model:
        engine = Engine(slots=4)

        def bind_cache(self, **kw):
            self.kw = kw

        def close(self):
            pass
    model = Model()
    monkeypatch.setattr(causal_lm.RPUModelForCausalLM, "from_pretrained", classmethod(lambda cls, *a, **kw: model))
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}, {"id": "b", "tokens": [9], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [4], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": [8], "want": [0]}, {"id": "c", "tokens": [2, 3], "want": [1]}], "end": ["b", "c"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(x) for x in lines) + "\n"))
    model.engine.released.clear()
    assert trace.main(["--model", "m", "--out", str(tmp_path), "--max-tokens", "100"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x] == ["done 0", "done 1", "done 2"]
    read = lambda n: np.fromfile(tmp_path / f"{n}.f32", dtype="<f4").reshape(-1, 3)[:, 0].tolist()
    assert read(0) == [5.0, 7.0] and not (tmp_path / "1.f32").exists() and read(2) == [8.0, 3.0]
    assert model.kw == {"batch_size": 4, "max_seq_len": 112, "pool_tokens": 112}


def test_native_argument_blocks_have_the_same_size_on_both_sides():
    import ctypes as C

    from rhinoforge_b200 import _native as N
    if not N.available():
        pytest.skip("native library is not built")
    sizes = (C.c_int32 * 18)()
    N.lib().rf_mixed_struct_sizes(sizes)
    ours = (N.RfMixedConfig, N.RfMixedLayer, N.RfMixedForward, N.RfRows, N.RfStreamNorm, N.RfLatentAttn, N.RfHgrn2, N.RfHeadLinear,
            N.RfMixedState, N.RfAttn, N.RfQkvInsert, N.RfConvSilu, N.RfMamba1, N.RfMoeRouter, N.RfMoeExperts, N.RfLatentInsert,
            N.RfHeadRotate, N.RfDelta)
    assert list(sizes) == [C.sizeof(x) for x in ours]


def test_example_configuration_is_checked(tmp_path):
    import importlib.util
    from pathlib import Path
    root = Path(__file__).resolve().parents[1]
    spec = importlib.util.spec_from_file_location("vabarax_example", root / "examples" / "vabarax.py")
    mod = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(mod)
    good = (root / "examples" / "configs" / "vabarax.toml").read_text()
    assert mod.load_config(root / "examples" / "configs" / "vabarax.toml")["generation"]["max_new_tokens"] == 16
    for old, new in (("prompt_tokens = [[9", "prompt_tokens = [[], [9"), ("slots = 2", "slots = 0"), ('"bfloat16"', '"int8"'),
                     ("max_new_tokens = 16", "max_new_tokens = true")):
        assert old in good
        f = tmp_path / "c.toml"
        f.write_text(good.replace(old, new, 1))
        with pytest.raises(ValueError):
            mod.load_config(f)


def test_weight_table_names_every_tensor_once():
    cfg = small_config()
    names = [n for n, _, _ in weight_shapes(cfg)]
    assert len(names) == len(set(names))
    assert {"embed", "side.embed", "final.norm", "l0.mix.lower", "l0.mlp.up", "l1.mix.dkv.norm", "l1.side.norm"} <= set(names)
    assert not any(n.startswith("l1.mlp") or n == "l1.norm2" for n in names)
