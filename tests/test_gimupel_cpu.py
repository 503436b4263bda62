"""Gimupel on the CPU: the package's host side (configuration, model description with looped layers, weights, state slots
per pass, step packing, scheduler, entry point) with the plain operation table, against the plain implementation on
whole sequences."""
import copy

import numpy as np
import pytest
import torch

import plain_gimupel as plain
from gimupel_util import CONFIGS, GIP_MIX, GIP_ODD, GIP_TC, drawn_config, make_dir, plain_logits, tokens_for
from pepilix_util import rel_rms, run_cut, run_mixed
from plain_ops import PlainOpsSpace
from fusezap_core_b200 import LLMEngine, SamplingParams
from fusezap_core_b200.cache import CacheManager, KVNeed
from fusezap_core_b200.config import describe
from fusezap_core_b200.config.gimupel import GimupelConfig
from fusezap_core_b200.engine import Portion, StepRunner, load_model

F = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("gimupel")
    return {name: make_dir(name, tmp) for name in CONFIGS}


def engine_parts(d, page=4, pages=48, slots=3, max_len=160):
    model = load_model(d, "float32", "cpu", max_len=max_len, ops=PlainOpsSpace(torch.float32))
    cache = CacheManager(model.cache_needs(), model.state_needs(), page, pages, slots, max_len, torch.float32, "cpu")
    return model, cache, StepRunner(model, cache, max_rows=max_len, max_wanted=max_len, max_segments=slots)


# ------------------------------------------------------------------------------------- the oracle's own mechanisms
def test_the_two_plain_recurrences_agree_and_follow_the_equations_for_one_channel():
    g = torch.Generator().manual_seed(2)
    x, B, C = (torch.randn(9, *s, generator=g, dtype=F) for s in ((4, 3), (2, 5), (2, 5)))
    dt, a, D = torch.rand(9, 4, generator=g, dtype=F), torch.randn(4, generator=g, dtype=F), torch.randn(4, generator=g, dtype=F)
    y, S = plain.ssd_recurrence(x, B, C, dt, a, D)
    y2, S2 = plain.ssd_recurrence_fast(x, B, C, dt, a, D)
    assert (y - y2).abs().max() < 1e-12 and (S - S2).abs().max() < 1e-12
    s = 0.0
    for t in range(9):      # head 3 reads the second group; state row 4, channel 1
        s = float(torch.exp(-torch.exp(a[3]) * dt[t, 3])) * s + float(dt[t, 3] * B[t, 1, 4] * x[t, 3, 1])
    assert abs(s - float(S[3, 4, 1])) < 1e-12


def test_the_two_plain_attentions_agree():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(23, 2, 6, generator=g, dtype=F) for _ in range(3))
    slow = plain.masked_attention(q, k, v, 0.4, lambda i, j: 0 <= i - j < 5)
    assert (slow - plain.masked_attention_fast(q, k, v, 0.4, plain.window_mask(23, 5))).abs().max() < 1e-12


def test_the_plain_router_on_a_hand_made_case():
    """Four groups of two; the correction moves the choice and not the weights; struck groups cannot win even where all
    choice scores are negative; a group counts its two best."""
    logit = lambda p: float(np.log(p / (1 - p)))
    s = [0.9, 0.1, 0.6, 0.6, 0.8, 0.3, 0.5, 0.5]
    z = torch.tensor([[logit(p) for p in s]], dtype=F)
    idx, w = plain.route(z, torch.zeros(8, dtype=F), 2, 4, 1, 2.0)
    assert idx[0].tolist() == [2, 3] and torch.allclose(w[0], torch.tensor([1.0, 1.0], dtype=F))      # 1.2 beats 1.0, 1.1 and 1.0
    c = torch.full((8,), -1.0, dtype=F)
    c[7] = -0.2
    idx, w = plain.route(z, c, 3, 4, 2, 1.0)         # choice scores: group 3 has 0.3 - 0.5, group 1 has -0.8
    assert idx[0].tolist() == [7, 2, 3]
    assert torch.allclose(w[0], torch.tensor([0.5, 0.6, 0.6], dtype=F) / 1.7)


def test_the_order_of_layers():
    assert plain.order_of_layers(GIP_MIX) == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert plain.order_of_layers(GIP_TC) == [(0, False), (1, False), (2, False)]


# ------------------------------------------------------------------------------------- configuration and description
def test_config_reads_every_size_and_round_trips():
    for cfg in (GIP_MIX, GIP_ODD, GIP_TC):
        typed = GimupelConfig.from_json(cfg)
        back = typed.to_json()
        assert GimupelConfig.from_json(back) == typed and back == cfg
    typed, spec = describe(GIP_MIX)
    assert spec.tie_embeddings and spec.embed_scale == 1.7 and spec.lm_head_name is None and spec.positions == {}
    assert [L.mixer.kind for L in spec.layers] == ["mamba2", "sink_attention", "mamba2", "sink_attention"]
    assert [(e.layer, e.cache, e.add_embedding) for e in spec.schedule] == [
        (0, 0, False), (1, 1, False), (2, 2, False), (1, 3, True), (2, 4, False), (1, 5, True), (2, 6, False), (3, 7, False)]
    p = spec.layers[1].mixer.params
    assert (p["window"], p["sink"], p["rotated"], p["qk_norm"], p["norm_weight"]) == (9, False, 0, True, False)
    f = spec.layers[1].ffn.params
    assert (f["scoring"], f["group_score"], f["weight_scale"], f["limit"], f["alpha"], f["up_shift"], f["sum_eps"]) == \
           ("sigmoid", "top2", 1.5, 0.7, 1.702, 1.0, 1e-20)
    assert spec.layers[0].ffn.kind == "swiglu" and spec.layers[3].ffn is None
    for loop in (None, {"start": 0, "stop": 1, "times": 1}):
        order = [(e.layer, e.add_embedding) for e in describe(dict(GIP_MIX, loop=loop))[1].schedule]
        assert order == [(i, False) for i in range(4)]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "not supported"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gelu"), "not supported"),
    (lambda c: c["layers"][0]["mixer"].update(groups=4), "multiple of groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=5), "multiple of norm_groups"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "lacks"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "groups"),
    (lambda c: c["layers"][1]["mlp"]["expert"].pop("limit"), "lacks"),
    (lambda c: c["layers"][1]["mlp"]["router"].pop("scale"), "lacks"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["embedding"].pop("scale"), "lacks"),
    (lambda c: c.pop("norm"), "lacks"),
])
def test_config_refusals(change, message):
    cfg = copy.deepcopy(GIP_MIX)
    change(cfg)
    with pytest.raises((ValueError, NotImplementedError), match=message):
        describe(cfg)


def test_random_weights_name_every_tensor(dirs):
    d, cfg, w = dirs["mix"]
    names = set(w)
    assert {"embed", "final.norm", "l0.norm1", "l0.norm2", "l0.mix.in", "l0.mix.conv", "l0.mix.conv.b", "l0.mix.dt_bias",
            "l0.mix.A_log", "l0.mix.D", "l0.mix.norm", "l0.mix.o", "l0.mlp.gate", "l0.mlp.up", "l0.mlp.down", "l1.mix.q",
            "l1.mix.k", "l1.mix.v", "l1.mix.o", "l1.mlp.router", "l1.mlp.correction", "l1.mlp.e5.gate", "l1.mlp.e0.down",
            "l3.mix.q", "l3.norm1"} <= names
    assert not any(k.startswith("l3.mlp") or "q.norm" in k or k == "head" for k in names)
    assert w["l0.mix.in"].shape == (72 + 72 + 2 * 60 + 6, 64) and w["l0.mix.conv"].shape == (192, 4) and w["l0.mix.norm"].shape == (72,)
    assert w["l1.mlp.correction"].shape == (6,) and w["l3.mix.v"].shape == (36, 64)


def test_state_and_caches_are_declared_per_pass(dirs):
    d, cfg, w = dirs["mix"]
    model, cache, runner = engine_parts(d, slots=2)
    needs = model.state_needs()
    assert sorted(needs) == [(n, x) for n in (0, 2, 4, 6) for x in ("S", "conv")]
    assert needs[(0, "conv")] == (3, 192) and needs[(4, "conv")] == (2, 112) and needs[(6, "S")] == needs[(2, "S")] == (4, 24, 16)
    caches = model.cache_needs()
    assert sorted(caches) == [1, 3, 5, 7] and caches[3] == KVNeed(2, 16, 9, value_dim=8) and caches[7] == KVNeed(3, 24, 20, value_dim=12)
    assert model.graph_safe() and "portions" in runner.needs
    assert engine_parts(dirs["odd"][0])[0].state_needs().get((1, "conv")) is None      # one tap keeps no inputs


# ------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_of_every_size_against_the_whole_sequence(dirs, name):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d)
    toks = tokens_for(cfg, (50,), seed=11)[0]
    ref = plain_logits(cfg, w, toks)
    for cuts in ((50,), (1,), (2,), (5, 3, 1, 7, 2, 19)):
        assert rel_rms(run_cut(runner, cache, "r", toks, cuts), ref) < 2e-5, (name, cuts)
        cache.check()


@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(dirs, name):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d, page=4, pages=30, slots=3, max_len=64)
    reqs = dict(zip("abcde", tokens_for(cfg, (41, 9, 23, 2, 30), seed=5)))
    plan = [[("a", 17), ("b", 2)], [("a", 1), ("b", 7), ("c", 20)], [("a", 20), ("c", 1)], [("a", 1), ("c", 1), ("d", 2)],
            [("a", 2), ("c", 1), ("e", 5)], [("e", 1)], [("e", 24)]]
    got = run_mixed(runner, cache, reqs, plan)
    cache.check()
    assert cache.live_requests() == [] and cache.states.num_free == 3
    for r, toks in reqs.items():
        assert rel_rms(got[r], plain_logits(cfg, w, toks)) < 2e-5, (name, r)


def test_a_requests_state_survives_steps_of_other_requests(dirs):
    d, cfg, w = dirs["one"]
    model, cache, runner = engine_parts(d, slots=2)
    a, b = tokens_for(cfg, (9, 7), seed=3)
    runner.run([Portion("a", a[:4], [])])
    runner.run([Portion("b", b[:6], [])])
    got_a = runner.run([Portion("a", a[4:], list(range(5)))]).numpy().copy()
    got_b = runner.run([Portion("b", b[6:], [0])]).numpy()
    assert rel_rms(got_a, plain_logits(cfg, w, a)[4:]) < 2e-5 and rel_rms(got_b, plain_logits(cfg, w, b)[6:]) < 2e-5


def test_the_embedding_is_added_again_once_per_later_pass(dirs):
    """Against itself with the loop's additions taken out in the oracle: the difference is large, so a missing or a second
    addition would show."""
    d, cfg, w = dirs["mix"]
    toks = tokens_for(cfg, (20,), seed=1)[0]
    ref = plain_logits(cfg, w, toks)
    order = plain.order_of_layers
    try:
        plain.order_of_layers = lambda c: [(i, False) for i, _ in order(c)]
        without = plain_logits(cfg, w, toks)
    finally:
        plain.order_of_layers = order
    assert rel_rms(without, ref) > 0.05


def test_a_pending_sum_resolves_to_its_other_stream():
    """What a norm that cannot take both streams in its own pass does with them."""
    from fusezap_core_b200.parts import PendingSum

    class Ctx:
        ops = PlainOpsSpace(torch.float32)
    x, delta, extra = (torch.randn(3, 4) for _ in range(3))
    want = x + delta
    got = PendingSum(delta, extra).resolve(Ctx, x)
    assert got is extra and torch.allclose(x, want)
    assert PendingSum(None, extra).resolve(Ctx, x) is extra and torch.allclose(x, want)


def test_greedy_generation_through_the_entry_point(dirs):
    """Through `LLMEngine` and its scheduler: portions of prompts beside decoding requests, more requests than state
    slots, a pool that does not hold all of them at once."""
    d, cfg, w = dirs["odd"]
    eng = LLMEngine.from_pretrained(d, dtype="float32", device="cpu", ops=PlainOpsSpace(torch.float32), max_model_len=64,
                                    num_blocks=14, block_size=8, max_num_seqs=2, max_prefill_tokens=8, cuda_graphs=False)
    P = tokens_for(cfg, (7, 19, 2, 30), seed=2)
    out = eng.generate(P, SamplingParams(max_tokens=5, ignore_eos=True))
    for prompt, new in zip(P, out):
        lg = plain_logits(cfg, w, list(prompt) + new)
        for i, t in enumerate(new):
            row = lg[len(prompt) - 1 + i]
            assert int(row.argmax()) == t or row.max() - row[t] < 1e-3


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    """The host side reads every size and constant from the configuration: drawn ones (the GPU tests' own) against the
    plain model, whole, in portions and token by token."""
    cfg = drawn_config(seed)
    d, cfg, w = make_dir(f"drawn{seed}", tmp_path, cfg, seed)
    model, cache, runner = engine_parts(d, page=4, pages=30, slots=2, max_len=64)
    toks = tokens_for(cfg, (40,), seed=seed)[0]
    ref = plain_logits(cfg, w, toks)
    for cuts in ((40,), (1,), (6, 2, 1, 17)):
        assert rel_rms(run_cut(runner, cache, "r", toks, cuts), ref) < 2e-5, (seed, cuts)
