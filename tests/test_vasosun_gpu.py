"""Vasosun served end to end against the plain oracle: prefill, decode, portions, batches, reuse, generation."""
import json

import pytest
import torch

import _vasosun_oracle as oracle
from rhinoforge_b200.models.mixed import (DeltaRule, GatedMLP, GroupedAttention, LatentAttention, MixedConfig, MixedLayer, MoE, Rotary, TokenPairs,
                                          YarnScaling, random_weights, weight_shapes)

pytestmark = pytest.mark.gpu
F32, BF16 = torch.float32, torch.bfloat16


def window(heads, kv, dim, vdim, scale, size, growth=0.0, every=0):
    return GroupedAttention(heads, kv, dim, vdim, scale, qk_norm=False, sink=False, gate=False, log_bias=True, window=size, growth=growth, growth_every=every)


def latent(heads, dim, vdim, rank, q_rank, rot, scale, of=None):
    return LatentAttention(heads, dim, vdim, rank, scale, q_rank=q_rank, rot=rot, kv_from=of)


def moe(experts, identity, top, ff):
    return MoE(experts, top, ff, gated=False, identity=identity, renormalise=False)


SLOW, FAST = Rotary(14, 1000.0, YarnScaling(4.0, 60, 8.0, 1.0)), Rotary(32, 1e5)
# sizes that are no multiples of the kernels' tiles, different in every layer; score scales that make the softmax peaked, so that
# one wrong key shows
CONFIGS = {
    "ragged": MixedConfig.vasosun("ragged", 211, 76, 1e-5, (
        MixedLayer(latent(5, 20, 36, 41, 27, SLOW, 0.25), moe(6, 2, 3, 20)),
        MixedLayer(DeltaRule(6, 2, 24, 40, 3), GatedMLP(52)),
        MixedLayer(window(6, 3, 20, 36, 0.3, 29, 0.4, 20)),
        MixedLayer(latent(3, 44, 12, 41, 50, SLOW, 0.2, 0), moe(5, 5, 2, 36)),
        MixedLayer(latent(4, 8, 20, 150, 33, FAST, 0.3), GatedMLP(40)),
        MixedLayer(DeltaRule(3, 3, 70, 24, 5)),
        MixedLayer(latent(7, 60, 8, 150, 24, FAST, 0.15, 4))), input_taps=3, pairs=TokenPairs(97, 31, 5), logit_softcap=9.0),
    "wide": MixedConfig.vasosun("wide", 1000, 256, 1e-6, (
        MixedLayer(DeltaRule(8, 4, 64, 64, 4), GatedMLP(640)),
        MixedLayer(window(20, 1, 128, 64, 0.2, 130, 0.5, 100), moe(16, 8, 4, 256)),
        MixedLayer(latent(16, 64, 128, 512, 192, Rotary(64, 1e6, YarnScaling(8.0, 128, 32.0, 1.0)), 0.1), moe(4, 2, 2, 200)),
        MixedLayer(DeltaRule(2, 1, 128, 96, 2), moe(8, 1, 1, 128)),
        MixedLayer(latent(20, 128, 64, 512, 96, Rotary(64, 1e6, YarnScaling(8.0, 128, 32.0, 1.0)), 0.08, 2))), input_taps=4, pairs=TokenPairs(501, 17, 29),
        logit_softcap=20.0),
    "ones": MixedConfig.vasosun("ones", 33, 40, 1e-4, (
        MixedLayer(DeltaRule(1, 1, 1, 1, 1), moe(1, 1, 1, 1)),
        MixedLayer(window(1, 1, 3, 5, 1.0, 1, 1.0, 1), GatedMLP(1)),
        MixedLayer(latent(1, 1, 1, 1, 1, Rotary(2, 10.0), 1.0), moe(2, 0, 1, 1)),
        MixedLayer(window(2, 1, 3, 5, 0.8, 2), moe(3, 3, 6, 3)),
        MixedLayer(latent(2, 3, 2, 1, 2, Rotary(2, 10.0), 0.7, 2))), input_taps=1, pairs=TokenPairs(1, 1, 1)),
    "big-heads": MixedConfig.vasosun("big-heads", 120, 64, 1e-6, (
        MixedLayer(latent(2, 240, 40, 64, 40, Rotary(32, 1e4), 0.1), moe(4, 2, 2, 64)),
        MixedLayer(DeltaRule(2, 1, 200, 300, 4), GatedMLP(100)),
        MixedLayer(window(2, 1, 40, 300, 0.4, 50))), input_taps=7, logit_softcap=6.0),
    "open": MixedConfig.vasosun("open", 90, 64, 1e-6, (
        MixedLayer(window(32, 1, 32, 32, 0.4, None)),
        MixedLayer(latent(4, 16, 16, 32, 16, Rotary(16, 1e5), 0.5)))),
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
        _ref[name, n, seed] = oracle.forward(CONFIGS[name].to_vasosun(), weights(name), tokens(name, n, seed))
    return _ref[name, n, seed]


def check(got, want, dtype, what="", loose=False):
    """Root mean square error of every position's logits.  In 16 bits a token whose experts are a close call may get others than
    in fp64; such tokens are few.  ``loose``: latents and heads of one value are sign functions under their norm."""
    got, want = got.double().cpu(), want.double()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()
    worst = f"{what}: relative error {float(err.max()):.2e} at row {int(err.argmax())}"
    if dtype == F32:
        assert float(err.max()) < 1e-4, worst
        return
    assert float(err.max()) < 1.5 and float(err.median()) < 4e-2, worst
    if err.numel() >= 32:
        assert float(err.quantile(0.7 if loose else 0.85)) < 1e-1, f"{what}: 85 % of the rows within {float(err.quantile(0.85)):.2e}"


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
    oracle.forward(CONFIGS[name].to_vasosun(), weights(name), tokens(name, 60), taps)
    got = engine(name, F32).residual_taps(tokens(name, 60)).double().cpu()
    for layer, want in enumerate(taps):
        check(got[layer], want, F32, f"layer {layer}")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", CONFIGS)
def test_token_by_token_equals_the_whole_prompt(name, dtype):
    """From the very first token on, over page borders, and past every window."""
    check(run(engine(name, dtype), tokens(name, 150), [1]), reference(name, 150), dtype, loose=name == "ones")


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[2], [3, 2], [15, 16, 17], [64, 2, 1, 30], [16], [129, 5]])
@pytest.mark.parametrize("name", ["ragged", "wide"])
def test_portions_of_any_size(name, dtype, cuts):
    check(run(engine(name, dtype), tokens(name, 300), cuts, slot=2, decode_tail=20), reference(name, 300), dtype, str(cuts))


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["ragged", "wide", "open"])
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
    """Hundreds of single-token steps behind a short prompt: every window passes over decoded tokens."""
    check(run(engine("wide", dtype), tokens("wide", 420), [7], decode_tail=413)[::7], reference("wide", 420)[::7], dtype)


@pytest.mark.parametrize("rows", [200, 256, 257, 300, 512])
def test_both_forms_of_the_experts_agree(rows):
    """Small batches stream the experts' weights past the rows, larger ones sort the rows by expert."""
    check(run(engine("wide", BF16), tokens("wide", 512)[:rows], [rows]), reference("wide", 512)[:rows], BF16)


def edge_engine(layer, dtype, taps=0):
    """One layer alone, token pairs off: a position's logits depend on exactly the tokens that its mixer and its convolution see."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    cfg = MixedConfig.vasosun("edge", 64, 64, 1e-6, (MixedLayer(layer),), input_taps=taps)
    get = random_weights(cfg, seed=3)
    w = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    return MixedDecoderEngine(cfg, lambda k: w[k], dtype=dtype, max_batch=1, max_seq_len=192, max_prefill_tokens=192)


def changes(eng, base, cuts, places):
    """Largest change of the last position's logits when the token at each place is another one."""
    def last(t):
        eng.reset()
        return run(eng, t, cuts)[-1].double().cpu()
    ref = last(base)
    out = {}
    for at in places:
        other = base.clone()
        other[at] = (other[at] + 17) % 64
        out[at] = float((last(other) - ref).abs().max())
    return out


@pytest.mark.parametrize("path", ["prompt", "decode", "portion"])
@pytest.mark.parametrize("size", [1, 7, 16, 33, 64, 65, 100])
def test_window_edges_show_in_the_logits(size, path):
    """Just inside and just outside the window."""
    n = 150
    base = torch.randint(0, 64, (n,), generator=torch.Generator().manual_seed(1)).to(torch.int32)
    cuts = {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 40, 40]}[path]
    for dtype in (F32, BF16):
        eng = edge_engine(window(16, 2, 16, 32, 0.02, size), dtype)
        for at, diff in changes(eng, base, cuts, (n - size, n - size - 1)).items():
            assert (diff > 1e-3) == (n - 1 - at < size), (dtype, at, diff)
        eng.close()


@pytest.mark.parametrize("path", ["prompt", "decode", "portion"])
def test_latent_attention_and_the_delta_rule_see_the_first_token(path):
    n = 150
    base = torch.randint(0, 64, (n,), generator=torch.Generator().manual_seed(2)).to(torch.int32)
    cuts = {"prompt": [n], "decode": [n - 1, 1], "portion": [n - 40, 40]}[path]
    for mixer in (latent(4, 16, 32, 24, 20, Rotary(8, 100.0), 0.02), DeltaRule(4, 2, 16, 32, 2)):
        eng = edge_engine(mixer, F32)
        assert all(diff > 1e-6 for diff in changes(eng, base, cuts, (0, 1, 15, 16, n - 2)).values())
        eng.close()


@pytest.mark.parametrize("cut", [1, 2, 3, 15, 16, 17, 40, 88, 89])
@pytest.mark.parametrize("taps", [2, 4, 6])
def test_input_convolution_reaches_back_over_a_portion_s_start(cut, taps):
    """Window of one position: the last logits depend on the last ``taps`` tokens and on no other."""
    n = 90
    base = torch.randint(0, 64, (n,), generator=torch.Generator().manual_seed(4)).to(torch.int32)
    for dtype in (F32, BF16):
        eng = edge_engine(window(2, 1, 16, 32, 0.5, 1), dtype, taps)
        for at, diff in changes(eng, base, [n - cut, cut], range(n - taps - 2, n)).items():
            assert (diff > 1e-3) == (n - 1 - at < taps), (dtype, at, diff)
        eng.close()


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("cuts", [[200], [1], [70, 130], [16, 17, 1]])
def test_a_far_key_that_stands_out_is_found_by_its_rotation(dtype, cuts):
    """Queries and keys whose rotated parts alone decide: the same token far away and near differ by their distance only, in a layer
    with its own cache and in one that attends over it."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    rot = Rotary(8, 300.0, YarnScaling(4.0, 100, 4.0, 1.0))
    cfg = MixedConfig.vasosun("far", 64, 64, 1e-6, (MixedLayer(latent(4, 16, 32, 24, 32, rot, 1.5)), MixedLayer(latent(2, 8, 16, 24, 16, rot, 1.5, 0))))
    get = random_weights(cfg, seed=5)
    w = {n: get(n) for n, _, _ in weight_shapes(cfg)}
    for p, dim in (("l0.mix.uq", 16), ("l1.mix.uq", 8)):
        w[p] = w[p].clone()
        w[p].view(-1, dim + 8, w[p].shape[1])[:, :dim] *= 0.1
    w["l0.mix.dkv"][24:] *= 2.0
    toks = torch.randint(0, 64, (200,), generator=torch.Generator().manual_seed(6)).to(torch.int32)
    eng = MixedDecoderEngine(cfg, lambda k: w[k], dtype=dtype, max_batch=1, max_seq_len=208, max_prefill_tokens=208)
    check(run(eng, toks, cuts), oracle.forward(cfg.to_vasosun(), w, toks), dtype)
    eng.close()


@pytest.mark.parametrize("cuts", [[1], [2], [40, 1], [17, 16, 1, 56], [90]])
def test_the_previous_token_reaches_over_portions(cuts):
    """Token pairs alone: a layer that sees one position, so the last logits depend on the last two tokens."""
    from rhinoforge_b200.runtime.mixed_engine import MixedDecoderEngine
    n = 90
    cfg = MixedConfig.vasosun("pairs", 64, 64, 1e-6, (MixedLayer(window(2, 1, 16, 32, 0.5, 1)),), pairs=TokenPairs(4099, 64, 1))
    get = random_weights(cfg, seed=3)
    w = {k: get(k) for k, _, _ in weight_shapes(cfg)}
    base = torch.randint(0, 47, (n,), generator=torch.Generator().manual_seed(5)).to(torch.int32)
    want = oracle.forward(cfg.to_vasosun(), w, base)
    for dtype in (F32, BF16):
        eng = MixedDecoderEngine(cfg, lambda k: w[k], dtype=dtype, max_batch=1, max_seq_len=96, max_prefill_tokens=96)
        check(run(eng, base, cuts), want, dtype)
        eng.reset()
        for at, diff in changes(eng, base, cuts, (n - 3, n - 2, n - 1)).items():
            assert (diff > 1e-3) == (at > n - 3), (dtype, at, diff)
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
    (tmp_path / "config.json").write_text(json.dumps(cfg.to_vasosun()))
    save_file(weights("ragged"), str(tmp_path / "model.safetensors"))
    live_handle.release()
    model = RPUModelForCausalLM.from_pretrained(str(tmp_path), dtype=F32, device="rpu", max_batch=4)
    prompts = [tokens("ragged", n, 20 + n) for n in (40, 3, 1, 90, 17, 64)]

    def greedy_ok(prompt, new):
        logits = oracle.forward(cfg.to_vasosun(), weights("ragged"), torch.cat((prompt, torch.tensor(new[:-1], dtype=torch.int32))))
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
