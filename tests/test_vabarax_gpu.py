"""Vabarax served end to end against the plain oracle: prefill, decode, portions, batches, reuse, generation."""
import json

import pytest
import torch

import _vabarax_oracle as oracle
from rhinoforge_b200.models.mixed import DenseMLP, HGRN2, LatentAttention, MixedConfig, MixedLayer, random_weights, weight_shapes

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16

# sizes that are no multiples of the kernels' tiles, different in every layer; large score scales make the softmax peaked, so
# that one wrong key shows
CONFIGS = {
    "ragged": MixedConfig("ragged", 211, 76, 1e-5, (
        MixedLayer(HGRN2(3, 20, 12), DenseMLP(36)),
        MixedLayer(LatentAttention(5, 24, 40, 20, 0.9, 5), DenseMLP(52)),
        MixedLayer(LatentAttention(1, 96, 8, 72, 0.5, 37)),
        MixedLayer(HGRN2(1, 136, 160), DenseMLP(100))), 12),
    "wide": MixedConfig("wide", 1000, 256, 1e-6, (
        MixedLayer(LatentAttention(20, 128, 64, 200, 0.25, 130), DenseMLP(512)),
        MixedLayer(HGRN2(2, 128, 128)),
        MixedLayer(LatentAttention(2, 64, 64, 64, 0.6, 16), DenseMLP(256))), 32),
    "ones": MixedConfig("ones", 33, 40, 1e-4, (
        MixedLayer(LatentAttention(1, 1, 1, 1, 1.0, 1), DenseMLP(1)),
        MixedLayer(HGRN2(1, 1, 1), DenseMLP(3)),
        MixedLayer(LatentAttention(2, 3, 5, 7, 1.5, 2))), 1),
    "big-heads": MixedConfig("big-heads", 120, 64, 1e-6, (
        MixedLayer(LatentAttention(2, 264, 40, 48, 0.3, 9), DenseMLP(64)),
        MixedLayer(HGRN2(2, 264, 16))), 8),
    "linear-only": MixedConfig("linear-only", 64, 48, 1e-6, (MixedLayer(HGRN2(2, 24, 24), DenseMLP(40)), MixedLayer(HGRN2(1, 8, 96))), 8),
    "no-window": MixedConfig("no-window", 90, 64, 1e-6, (
        MixedLayer(LatentAttention(3, 32, 32, 48, 0.5), DenseMLP(64)),
        MixedLayer(LatentAttention(2, 64, 16, 32, 0.4, 700))), 8),
}
_engines, _weights = {}, {}


def weights(name):
    if name not in _weights:
        cfg = CONFIGS[name]
        get = random_weights(cfg, seed=7)
        _weights[name] = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    return _weights[name]


def engine(name, dtype):
    """One engine per configuration and dtype, reset for every test: 4 slots, a pool smaller than 4 full requests."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    if (name, dtype) not in _engines:
        w = weights(name)
        _engines[name, dtype] = MixedDecoderEngine(CONFIGS[name], lambda n: w[n], dtype=dtype, max_batch=4, max_seq_len=640,
                                                   max_prefill_tokens=512, kv_pool_tokens=1280)
    eng = _engines[name, dtype]
    eng.reset()
    return eng


def tokens(name, n, seed=0):
    return torch.randint(0, CONFIGS[name].vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).to(torch.int32)


_ref = {}


def reference(name, n, seed=0):
    """Oracle logits of ``tokens(name, n, seed)``: every shorter prompt of the same seed is a prefix of a longer one only when
    the generator says so, hence one entry per length."""
    if (name, n, seed) not in _ref:
        _ref[name, n, seed] = oracle.forward(CONFIGS[name].to_vabarax(), weights(name), tokens(name, n, seed))
    return _ref[name, n, seed]


def check(got, want, dtype, what="", loose=False):
    """Root mean square error of every position's logits.  ``loose``: heads of one value are sign functions under their norm,
    so in 16 bits single positions may differ more."""
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    if loose and dtype != F32:
        assert float(err.quantile(0.95)) < 4e-2 and float(err.max()) < 1.0, what
        return
    most, rest = (5e-5, 5e-5) if dtype == F32 else (6e-2, 2.5e-2)      # single positions are more sensitive to rounding than most
    assert float(err.max()) < most, f"{what}: relative error {float(err.max()):.2e} at row {int(err.argmax())}"
    if err.numel() >= 32:
        assert float(err.quantile(0.97)) < rest, f"{what}: 97 % of the rows within {float(err.quantile(0.97)):.2e}"


def run(eng, toks, cuts, slot=0, decode_tail=0):
    """Feed ``toks`` to one slot in portions of the given sizes (cycled), the last ``decode_tail`` one by one; all logits."""
    out, at, i, n = [], 0, 0, int(toks.numel())
    while at < n:
        step = min(cuts[i % len(cuts)], n - decode_tail - at) if at < n - decode_tail else 1
        _, lg = eng.run_step([toks[at:at + step]], [slot], [list(range(step))])
        out.append(lg[0])
        at, i = at + step, i + 1
    eng.check_status()
    return torch.cat(out)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", CONFIGS)
def test_prefill_matches_the_oracle_at_every_position(name, dtype):
    check(run(engine(name, dtype), tokens(name, 300), [300]), reference(name, 300), dtype, loose=name == "ones")


@pytest.mark.parametrize("name", ["ragged", "wide"])
def test_residual_stream_after_every_layer(name):
    taps = []
    oracle.forward(CONFIGS[name].to_vabarax(), weights(name), tokens(name, 60), taps)
    got = engine(name, F32).residual_taps(tokens(name, 60)).double().cpu()
    for layer, want in enumerate(taps):
        check(got[layer], want, F32, f"layer {layer}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", CONFIGS)
def test_token_by_token_equals_the_whole_prompt(name, dtype):
    """From the very first token on, over page borders and past every window."""
    check(run(engine(name, dtype), tokens(name, 150), [1]), reference(name, 150), dtype, loose=name == "ones")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[2], [3, 2], [15, 16, 17], [64, 2, 1, 30], [16], [129, 5]])
@pytest.mark.parametrize("name", ["ragged", "wide"])
def test_portions_of_any_size(name, dtype, cuts):
    check(run(engine(name, dtype), tokens(name, 300), cuts, slot=2, decode_tail=20), reference(name, 300), dtype, str(cuts))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["ragged", "wide"])
def test_mixed_batches_equal_each_request_alone(name, dtype):
    """Unequal requests advance together, portions beside single tokens, some left out of a step; slots and pages of finished
    requests go to new ones."""
    from rhinoforge_b200.runtime.scheduler import RequestScheduler
    eng = engine(name, dtype)
    sched = RequestScheduler(eng)
    lens = {"a": 300, "b": 150, "c": 1, "d": 60, "e": 150, "f": 60, "g": 300}
    seeds = {"a": 0, "b": 1, "c": 2, "d": 3, "e": 4, "f": 5, "g": 0}
    toks = {r: tokens(name, n, seeds[r]) for r, n in lens.items()}
    at, got = {r: 0 for r in lens}, {r: [] for r in lens}
    g = torch.Generator().manual_seed(11)
    pick = lambda n: int(torch.randint(0, n, (1,), generator=g))
    waiting, live, used = list(lens), [], set()
    while waiting or live:
        while waiting and len(live) < 4 and sum(lens[r] for r in live) + lens[waiting[0]] <= 1100:
            live.append(waiting.pop(0))
        entries = []
        for r in live:
            if len(live) > 1 and pick(5) == 0:
                continue                                        # left out of this step
            size = min([1, 1, 2, 3, 16, 29, 64, 120][pick(8)], lens[r] - at[r])
            entries.append((r, toks[r][at[r]:at[r] + size], list(range(size))))
        if not entries:
            continue
        _, lg = sched.step(entries)
        for (r, t, _), x in zip(entries, lg):
            got[r].append(x.clone())
            at[r] += int(t.numel())
            used.add((r, sched.slots[r]))
            if at[r] == lens[r]:
                sched.finish(r)
                live.remove(r)
    eng.check_status()
    assert len(used) == len(lens) and len({s for _, s in used}) <= 4      # seven requests in four slots
    for r, n in lens.items():
        check(torch.cat(got[r]), reference(name, n, seeds[r]), dtype, r)
    assert eng.cache.free_pages() == eng.cache.num_pages


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_what_a_finished_request_left_behind_is_not_seen(dtype):
    """Slots and pages full of another request's state: the next request starts from nothing."""
    eng = engine("ragged", dtype)
    for seed in (1, 2, 3):
        run(eng, tokens("ragged", 150, seed), [40], slot=1)
        eng.cache.release(1)
    check(run(eng, tokens("ragged", 150), [3, 50], slot=1), reference("ragged", 150), dtype)
    for n in (1, 2):
        eng.cache.release(1)
        check(run(eng, tokens("ragged", n, 9), [1], slot=1), reference("ragged", n, 9), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """Hundreds of single-token steps behind a short prompt: windows slide many times, states accumulate."""
    check(run(engine("wide", dtype), tokens("wide", 420), [7], decode_tail=413)[::7], reference("wide", 420)[::7], dtype)


@pytest.mark.parametrize("path", ["prompt", "decode", "portion"])
@pytest.mark.parametrize("window", [1, 16, 33, 64, 65])
def test_window_edges_show_in_the_logits(window, path):
    """One attention layer without token shift: the last logits depend on the token ``window - 1`` back and on nothing before."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    cfg = MixedConfig("edge", 64, 64, 1e-6, (MixedLayer(LatentAttention(2, 16, 16, 32, 0.05, window)),), 8)
    get = random_weights(cfg, seed=3)
    w = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    w["l0.shift"] = torch.zeros_like(w["l0.shift"])
    n = 150
    base = torch.randint(0, 64, (n,), generator=torch.Generator().manual_seed(1)).to(torch.int32)
    for dtype in (F32, BF16):
        eng = MixedDecoderEngine(cfg, lambda k: w[k], dtype=dtype, max_batch=1, max_seq_len=160, max_prefill_tokens=160)

        def last(t):
            eng.reset()
            cuts = {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 40, 40]}[path]
            return run(eng, t, cuts)[-1].double().cpu()
        ref = last(base)
        for back, visible in ((window - 1, True), (window, False)):
            other = base.clone()
            other[n - 1 - back] = (other[n - 1 - back] + 17) % 64
            diff = float((last(other) - ref).abs().max())
            assert (diff > 1e-3) == visible, (dtype, back, diff)
        eng.close()


def test_a_larger_cache_can_be_bound_later():
    """Engines are built small and get their cache at the first request: attention without a window then needs more room."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    w = weights("no-window")
    eng = MixedDecoderEngine(CONFIGS["no-window"], lambda n: w[n], dtype=BF16, max_batch=2, max_seq_len=16, max_prefill_tokens=64)
    eng.bind_cache(eng.make_cache(2, 320))
    check(run(eng, tokens("no-window", 300), [64, 40, 3], slot=1), reference("no-window", 300), BF16)
    eng.close()


def test_checkpoint_folder_generates_through_the_public_entry_points(tmp_path):
    """from_pretrained -> generate (graph path), generate_batch (scheduler, fewer slots than prompts), sampling through the
    Hugging Face loop; greedy tokens against the oracle up to near-ties."""
    from safetensors.torch import save_file

    from rhinoforge_b200.api.cache import RPUCache
    from rhinoforge_b200.api.causal_lm import RPUModelForCausalLM
    from rhinoforge_b200.runtime import live_handle
    cfg = CONFIGS["ragged"]
    (tmp_path / "config.json").write_text(json.dumps(cfg.to_vabarax()))
    save_file(weights("ragged"), str(tmp_path / "model.safetensors"))
    live_handle.release()
    model = RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=F32, device="rpu", max_batch=4)
    prompts = [tokens("ragged", n, 20 + n) for n in (40, 3, 1, 90, 17, 64)]

    def greedy_ok(prompt, new):
        logits = oracle.forward(cfg.to_vabarax(), weights("ragged"), torch.cat((prompt, torch.tensor(new[:-1], dtype=torch.int32))))
        top = logits[len(prompt) - 1:]
        for t, row in zip(new, top):
            assert float(row.max() - row[t]) < 1e-3, (t, int(row.argmax()))
    out = model.generate_batch(prompts, 12, slots=2, token_budget=32)
    assert [len(o) for o in out] == [12] * 6
    for p, o in zip(prompts, out):
        greedy_ok(p, o)
    ids = prompts[0][None].long()
    cache = RPUCache.from_model(model, input_ids=ids, max_new_tokens=12)
    got = model.generate(ids, past_key_values=cache, max_new_tokens=12, do_sample=False)
    assert got[0, :40].tolist() == prompts[0].tolist() and got[0, 40:].tolist() == out[0]
    torch.manual_seed(0)
    sampled = model.generate(ids, max_new_tokens=5, do_sample=True, top_k=3)
    assert sampled.shape == (1, 45)
    both = model.generate(torch.stack((prompts[0][:17], prompts[4])).long(), max_new_tokens=6)
    greedy_ok(prompts[4], both[1, 17:].tolist())
    with pytest.raises(ValueError, match="cannot rewind"):
        cache.reset_to_position(3)
    model.close()
    live_handle.release()


def test_one_scheduler_serves_the_dense_decoders_too():
    """Mixed steps over arbitrary slots on a plain K/V decoder: the same tokens as its static batch."""
    from rhinoforge_b200.models.decoder import random_state_dict, tiny_config
    from rhinoforge_b200.runtime.engine import DecoderEngine
    from rhinoforge_b200.runtime.scheduler import RequestScheduler
    cfg = tiny_config(num_layers=2)
    sd = random_state_dict(cfg, seed=0, dtype=torch.float16, norm_jitter=0.05)
    eng = DecoderEngine(cfg, lambda n: sd[n] if n in sd else sd["model.embed_tokens.weight"], dtype=torch.float16, max_batch=3, max_seq_len=128)
    gen = torch.Generator().manual_seed(5)
    prompts = [torch.randint(0, cfg.vocab_size, (n,), generator=gen) for n in (24, 9, 33)]
    alone = []
    for p in prompts:
        lg = eng.prefill([p], return_logits=True)[1]
        alone.append(lg[0].float())
    eng.reset()
    sched = RequestScheduler(eng)
    sched.step([("x", prompts[0][:10], [])])
    sched.step([("y", prompts[1], []), ("x", prompts[0][10:11], [])])
    _, lg = sched.step([("z", prompts[2], [32]), ("x", prompts[0][11:], [12])])
    assert torch.allclose(lg[0][0].float(), alone[2], atol=2e-2) and torch.allclose(lg[1][0].float(), alone[0], atol=2e-2)
    sched.finish("y")
    _, lg = sched.step([("w", prompts[1], [8])])
    assert torch.allclose(lg[0][0].float(), alone[1], atol=2e-2)
    eng.check_status()
    eng.close()
