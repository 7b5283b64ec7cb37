"""Zulopel served end to end against the plain oracle: prefill, decode, portions, batches, reuse, generation."""
import json

import pytest
import torch

import _zulopel_oracle as oracle
from rhinoforge_b200.models.mixed import (GroupedAttention, Mamba1, MixedConfig, MixedLayer, MoE, Rotary, YarnScaling, random_weights,
                                          weight_shapes)

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16
YARN = Rotary(10, 1000.0, YarnScaling(4.0, 64, 8.0, 0.5))

# sizes that are no multiples of the kernels' tiles, different in every layer; score scales that make the softmax peaked, so that
# one wrong key shows
CONFIGS = {
    "ragged": MixedConfig.zulopel("ragged", 211, 76, 1e-5, (
        MixedLayer(Mamba1(52, 5, 3, 3), MoE(6, 2, 20, 3, 2, 12)),
        MixedLayer(GroupedAttention(6, 2, 24, 40, 0.6, 37, YARN, True), MoE(5, 5, 9)),
        MixedLayer(GroupedAttention(2, 2, 8, 40, 0.9, 5, Rotary(8, 50.0), True), MoE(12, 3, 36, 2, 1, 100)),
        MixedLayer(Mamba1(40, 17, 40, 5))), 3.5),
    "wide": MixedConfig.zulopel("wide", 1000, 256, 1e-6, (
        MixedLayer(GroupedAttention(20, 1, 128, 64, 0.25, 130, Rotary(128, 1e4, YarnScaling(16.0, 48, 6.0, 1.0))), MoE(16, 4, 256, 4, 2, 512)),
        MixedLayer(Mamba1(512, 16, 16, 4), MoE(8, 1, 128, 8, 1, 64)),
        MixedLayer(GroupedAttention(4, 2, 64, 64, 0.4, None, None, True)),
        MixedLayer(GroupedAttention(4, 2, 200, 64, 0.2, 16, Rotary(32, 1e4), True), MoE(4, 2, 200)))),
    "ones": MixedConfig.zulopel("ones", 33, 40, 1e-4, (
        MixedLayer(Mamba1(1, 1, 1, 1), MoE(1, 1, 1)),
        MixedLayer(GroupedAttention(1, 1, 2, 1, 1.0, 1, Rotary(2, 10.0)), MoE(2, 1, 1, 2, 1, 1)),
        MixedLayer(GroupedAttention(2, 1, 3, 5, 1.5, 2, None, True)),
        MixedLayer(Mamba1(3, 2, 1, 2), MoE(3, 2, 3)))),
    "big-heads": MixedConfig.zulopel("big-heads", 120, 64, 1e-6, (
        MixedLayer(GroupedAttention(2, 1, 264, 40, 0.15, 9, Rotary(264, 1e4)), MoE(4, 2, 64)),
        MixedLayer(GroupedAttention(2, 1, 40, 300, -0.4, 50, Rotary(20, 1e4)), MoE(4, 2, 24, 2, 1)))),
    "scan-only": MixedConfig.zulopel("scan-only", 64, 48, 1e-6, (
        MixedLayer(Mamba1(96, 100, 8, 2), MoE(6, 2, 40)), MixedLayer(Mamba1(24, 256, 2, 9), MoE(9, 2, 16, 3, 2, 16))), 0.5),
    "attention-only": MixedConfig.zulopel("attention-only", 90, 64, 1e-6, (
        MixedLayer(GroupedAttention(32, 1, 32, 32, 0.5, 64, Rotary(16, 1e5))),
        MixedLayer(GroupedAttention(4, 4, 64, 16, 0.4, 700, YARN), MoE(4, 1, 32, 2, 2)))),
}
_engines, _weights, _ref = {}, {}, {}


def weights(name):
    if name not in _weights:
        get = random_weights(CONFIGS[name], seed=7)
        _weights[name] = {n: get(n) for n, _, _ in weight_shapes(CONFIGS[name])}
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


def reference(name, n, seed=0):
    if (name, n, seed) not in _ref:
        _ref[name, n, seed] = oracle.forward(CONFIGS[name].to_zulopel(), weights(name), tokens(name, n, seed))
    return _ref[name, n, seed]


def check(got, want, dtype, what="", loose=False):
    """Root mean square error of every position's logits.  In 16 bits a token whose experts are a close call may get others than
    in fp64; such tokens are few.  ``loose``: heads of one or two values are sign functions under their norm."""
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    worst = f"{what}: relative error {float(err.max()):.2e} at row {int(err.argmax())}"
    if dtype == F32:
        assert float(err.max()) < 1e-4, worst
        return
    assert float(err.max()) < 1.5 and float(err.median()) < 2e-2, worst
    if err.numel() >= 32:
        assert float(err.quantile(0.7 if loose else 0.85)) < 6e-2, f"{what}: 85 % of the rows within {float(err.quantile(0.85)):.2e}"


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


@pytest.mark.parametrize("name", CONFIGS)
def test_residual_stream_after_every_layer(name):
    taps = []
    oracle.forward(CONFIGS[name].to_zulopel(), weights(name), tokens(name, 60), taps)
    got = engine(name, F32).residual_taps(tokens(name, 60)).double().cpu()
    for layer, want in enumerate(taps):
        check(got[layer], want, F32, f"layer {layer}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", CONFIGS)
def test_token_by_token_equals_the_whole_prompt(name, dtype):
    """From the very first token on, over page borders and past every chunk."""
    check(run(engine(name, dtype), tokens(name, 150), [1]), reference(name, 150), dtype,
          loose=name == "ones")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[2], [3, 2], [15, 16, 17], [64, 2, 1, 30], [16], [129, 5]])
@pytest.mark.parametrize("name", ["ragged", "wide"])
def test_portions_of_any_size(name, dtype, cuts):
    check(run(engine(name, dtype), tokens(name, 300), cuts, slot=2, decode_tail=20), reference(name, 300), dtype, str(cuts))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["ragged", "wide", "scan-only"])
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
        check(run(eng, tokens("ragged", n, 9), [1], slot=1), reference("ragged", n, 9), dtype, loose=True)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding(dtype):
    """Hundreds of single-token steps behind a short prompt: chunks begin many times, states accumulate."""
    check(run(engine("wide", dtype), tokens("wide", 420), [7], decode_tail=413)[::7], reference("wide", 420)[::7], dtype)


@pytest.mark.parametrize("rows", [200, 256, 257, 300, 512])
def test_both_forms_of_the_experts_agree(rows):
    """Small batches stream the experts' weights past the rows, larger ones sort the rows by expert."""
    check(run(engine("wide", BF16), tokens("wide", 512)[:rows], [rows]), reference("wide", 512)[:rows], BF16)


@pytest.mark.parametrize("path", ["prompt", "decode", "portion"])
@pytest.mark.parametrize("chunk", [1, 16, 33, 64, 65, 100])
def test_chunk_edges_show_in_the_logits(chunk, path):
    """One attention layer alone: the logits of a position depend on the first token of its chunk and not on the one before."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    cfg = MixedConfig.zulopel("edge", 64, 64, 1e-6, (MixedLayer(GroupedAttention(2, 1, 16, 32, 0.02, chunk, Rotary(8, 100.0))),))
    get = random_weights(cfg, seed=3)
    w = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    n = 150
    base = torch.randint(0, 64, (n,), generator=torch.Generator().manual_seed(1)).to(torch.int32)
    first = (n - 1) // chunk * chunk
    for dtype in (F32, BF16):
        eng = MixedDecoderEngine(cfg, lambda k: w[k], dtype=dtype, max_batch=1, max_seq_len=160, max_prefill_tokens=160)

        def last(t):
            eng.reset()
            cuts = {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 40, 40]}[path]
            return run(eng, t, cuts)[-1].double().cpu()
        ref = last(base)
        for at, visible in ((first, True), (first - 1, False)):
            other = base.clone()
            other[at] = (other[at] + 17) % 64
            diff = float((last(other) - ref).abs().max())
            assert (diff > 1e-3) == visible, (dtype, at, diff)
        eng.close()


def test_a_larger_cache_can_be_bound_later():
    """Engines are built small and get their cache at the first request: the rotation tables then cover more positions."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    w = weights("wide")
    eng = MixedDecoderEngine(CONFIGS["wide"], lambda n: w[n], dtype=BF16, max_batch=2, max_seq_len=16, max_prefill_tokens=64)
    eng.bind_cache(eng.make_cache(2, 320))
    check(run(eng, tokens("wide", 300), [64, 40, 3], slot=1), reference("wide", 300), BF16)
    eng.close()


def test_checkpoint_folder_generates_through_the_public_entry_points(tmp_path):
    """from_pretrained -> generate (graph path), generate_batch (scheduler, fewer slots than prompts), sampling through the
    Hugging Face loop; greedy tokens against the oracle up to near-ties."""
    from safetensors.torch import save_file

    from rhinoforge_b200.api.cache import RPUCache
    from rhinoforge_b200.api.causal_lm import RPUModelForCausalLM
    from rhinoforge_b200.runtime import live_handle
    cfg = CONFIGS["ragged"]
    (tmp_path / "config.json").write_text(json.dumps(cfg.to_zulopel()))
    save_file(weights("ragged"), str(tmp_path / "model.safetensors"))
    live_handle.release()
    model = RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=F32, device="rpu", max_batch=4)
    prompts = [tokens("ragged", n, 20 + n) for n in (40, 3, 1, 90, 17, 64)]

    def greedy_ok(prompt, new):
        logits = oracle.forward(cfg.to_zulopel(), weights("ragged"), torch.cat((prompt, torch.tensor(new[:-1], dtype=torch.int32))))
        for t, row in zip(new, logits[len(prompt) - 1:]):
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
