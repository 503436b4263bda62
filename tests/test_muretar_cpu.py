"""Muretar on the CPU: the package's host side (configuration, model description with shared layers, weights, state slots and
caches per layer run, step packing, scheduler, entry point) with the plain operation table, against the plain implementation
on whole sequences."""
import copy

import numpy as np
import pytest
import torch

import plain_muretar as plain
from muretar_util import CONFIGS, MUR_MIX, MUR_ODD, MUR_ONE, MUR_TC, Oracle, drawn_config, make_dir, other_rank, plain_logits, tokens_for
from pepilix_util import rel_rms, run_cut, run_mixed
from plain_ops import PlainOpsSandwich
from fusezap_core_b200 import LLMEngine, SamplingParams
from fusezap_core_b200.cache import CacheManager, KVNeed
from fusezap_core_b200.config import describe
from fusezap_core_b200.config.muretar import MuretarConfig
from fusezap_core_b200.engine import Portion, StepRunner, load_model

F = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("muretar")
    return {name: make_dir(name, tmp) for name in CONFIGS}


def engine_parts(d, page=4, pages=48, slots=3, max_len=160):
    model = load_model(d, "float32", "cpu", max_len=max_len, ops=PlainOpsSandwich(torch.float32))
    cache = CacheManager(model.cache_needs(), model.state_needs(), page, pages, slots, max_len, torch.float32, "cpu")
    return model, cache, StepRunner(model, cache, max_rows=max_len, max_wanted=max_len, max_segments=slots)


# ------------------------------------------------------------------------------------- the oracle's own mechanisms
def test_the_two_plain_delta_recurrences_agree():
    g = torch.Generator().manual_seed(2)
    q, k = (plain.unit(torch.randn(9, 3, 5, generator=g, dtype=F)) for _ in range(2))
    v, d, b = torch.randn(9, 3, 4, generator=g, dtype=F), torch.rand(9, 3, generator=g, dtype=F), torch.rand(9, 3, generator=g, dtype=F)
    for a, c in zip(plain.delta_recurrence(q, k, v, d, b), plain.delta_recurrence_fast(q, k, v, d, b)):
        assert (a - c).abs().max() < 1e-12
    # with beta 1 and no decay the state returns the last value written under a key
    o, S = plain.delta_recurrence(k, k, v, torch.ones(9, 3, dtype=F), torch.ones(9, 3, dtype=F))
    assert (o - v).abs().max() < 1e-5


def test_the_two_plain_linear_attentions_agree_and_follow_the_equation_for_one_channel():
    g = torch.Generator().manual_seed(3)
    q, k, z = (torch.randn(9, 2, 5, generator=g, dtype=F) for _ in range(3))
    v, a = torch.randn(9, 2, 4, generator=g, dtype=F), plain.channel_decay(z, 3.0)
    for x, y in zip(plain.gla_recurrence(q, k, v, a), plain.gla_recurrence_fast(q, k, v, a)):
        assert (x - y).abs().max() < 1e-12
    s = 0.0
    for t in range(9):      # head 1, key channel 4, value channel 2
        s = float(torch.sigmoid(z[t, 1, 4])) ** (1 / 3.0) * s + float(k[t, 1, 4] * v[t, 1, 2])
    assert abs(s - float(plain.gla_recurrence(q, k, v, a)[1][1, 4, 2])) < 1e-12


def test_the_two_plain_attentions_agree():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(23, 2, 6, generator=g, dtype=F) for _ in range(3))
    assert (plain.causal_attention(q, k, v, 0.4) - plain.causal_attention_fast(q, k, v, 0.4)).abs().max() < 1e-12


def test_the_plain_rotation_turns_neighbours_and_keeps_relative_angles():
    g = torch.Generator().manual_seed(4)
    x = torch.randn(7, 1, 6, generator=g, dtype=F)
    y = plain.rotate(x, 4, 50.0, 2.0)
    assert torch.equal(y[..., 4:], x[..., 4:]) and torch.equal(y[0], x[0])
    a = 3 * 50.0 ** (-2 / 4) / 2.0
    u, v = float(x[3, 0, 2]), float(x[3, 0, 3])
    assert abs(float(y[3, 0, 2]) - (u * np.cos(a) - v * np.sin(a))) < 1e-12 and abs(float(y[3, 0, 3]) - (v * np.cos(a) + u * np.sin(a))) < 1e-12
    same = plain.rotate(x[:1].expand(7, 1, 6).clone(), 6, 50.0, 2.0)[:, 0]
    assert abs(float(same[1] @ same[4]) - float(same[3] @ same[6])) < 1e-12


def test_the_plain_router_on_a_hand_made_case():
    """The correction moves the choice and not the weights; weights are relative to the chosen scores, whatever the others have."""
    z = torch.log(torch.tensor([[0.4, 0.3, 0.2, 0.1]], dtype=F))
    idx, w = plain.route(z, torch.zeros(4, dtype=F), 2)
    assert idx[0].tolist() == [0, 1] and torch.allclose(w[0], torch.tensor([4 / 7, 3 / 7], dtype=F))
    idx, w = plain.route(z, torch.tensor([0.0, 0.0, -1.0, 0.5], dtype=F), 3)
    assert idx[0].tolist() == [3, 0, 1] and torch.allclose(w[0], torch.tensor([0.1, 0.4, 0.3], dtype=F) / 0.8)


def test_an_expert_that_hands_its_input_on():
    w = {"router": torch.zeros(3, 4, dtype=F), "correction": torch.tensor([0.0, 0.0, 5.0], dtype=F),
         **{f"e{e}.{n}": torch.full((4, 4), 9.0, dtype=F) for e in (0, 1) for n in ("up", "down")}}
    h = torch.randn(3, 4, generator=torch.Generator().manual_seed(0), dtype=F)
    mlp = {"router": {"experts": 2, "identity": 1, "top": 1}}
    assert torch.allclose(plain.mixture(w, "", mlp, h), h)


def test_layers_that_share_weights():
    assert [plain.owner(MUR_ODD, i) for i in range(7)] == [0, 1, 2, 0, 2, 2, 6]
    assert [plain.owner(MUR_ONE, i) for i in range(4)] == [2, 1, 2, 3]


# ------------------------------------------------------------------------------------- configuration and description
def test_config_reads_every_size_and_round_trips():
    for cfg in (MUR_MIX, MUR_ODD, MUR_ONE, MUR_TC):
        typed = MuretarConfig.from_json(cfg)
        back = typed.to_json()
        assert MuretarConfig.from_json(back) == typed
        for a, b in zip(back["layers"], cfg["layers"]):
            assert a["type"] == b["type"] and a.get("weights_of") == b.get("weights_of")
    typed, spec = describe(MUR_MIX)
    assert not spec.tie_embeddings and spec.lm_head_name == "head" and spec.embed_scale is None
    assert [(L.prefix, L.mixer.kind) for L in spec.layers] == [("l0.", "parallel_mixers"), ("l1.", "gated_linear_attention"),
                                                               ("l2.", "differential_attention"), ("l5.", "parallel_mixers")]
    assert [(e.layer, e.cache) for e in spec.schedule] == [(0, 0), (1, 1), (2, 2), (1, 3), (2, 4), (3, 5)]
    (_, a, wa), (_, b, wb) = spec.layers[0].mixer.params["mixers"]
    assert (wa, wb) == (0.5, 0.5) and spec.layers[0].mixer.params["norm_eps"] == 1e-5
    assert (a.params["rotated"], a.params["scale"], a.params["sink"], a.params["bias"]) == (12, 0.4, False, ("q", "k", "v", "out"))
    assert (b.params["taps"], b.params["head_decay"], b.params["gate"], b.params["query_scale"]) == (3, True, "silu", 10 ** -0.5)
    g, f = spec.layers[1].mixer.params, spec.layers[0].ffn.params
    assert (g["decay_root"], g["query_scale"], g["eps"]) == (16.0, 12 ** -0.5, 1e-5)
    assert (f["num_experts"], f["identity"], f["top"], f["shared_size"], f["activation"], f["sum_eps"]) == (5, 2, 3, 40, "relu2", 1e-20)
    assert spec.layers[1].ffn.kind == "swiglu" and spec.layers[3].ffn is None
    d = spec.layers[2].mixer.params
    assert (d["map_dim"], d["value_dim"], d["start"], d["bias"]) == (9, 16, 0.6, ("q", "k", "v"))
    factors = sorted(p.params["factor"] for p in spec.positions.values())
    assert factors == [1.0, 4.0] and all(p.params["precise"] for p in spec.positions.values())
    assert [(e.layer, e.cache) for e in describe(MUR_ONE)[1].schedule] == [(1, 0), (0, 1), (1, 2), (2, 3)]


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "not supported"),
    (lambda c: c["layers"][1]["mlp"].update(kind="gelu"), "not supported"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(scaling={}), "lacks"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(scaling={"factor": 0}), "positive"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(conv=0), "tap"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("vdim"), "lacks"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "lacks"),
    (lambda c: c["layers"][1]["mixer"].update(tau=0), "tau"),
    (lambda c: c["layers"][2]["mixer"].pop("diff"), "lacks"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "top"),
    (lambda c: c["layers"][0]["mlp"].pop("expert"), "lacks"),
    (lambda c: c["layers"][3].update(weights_of=9), "weights_of"),
    (lambda c: c["layers"][3].update(weights_of=3), "circle"),
    (lambda c: c["layers"][3]["mixer"].update(tau=4.0), "differs"),
    (lambda c: c["norm"].update(eps=0.0), "eps"),
    (lambda c: c.pop("norm"), "lacks"),
])
def test_config_refusals(change, message):
    cfg = copy.deepcopy(MUR_MIX)
    change(cfg)
    with pytest.raises((ValueError, NotImplementedError), match=message):
        describe(cfg)


def test_random_weights_name_every_tensor(dirs):
    d, cfg, w = dirs["mix"]
    names = set(w)
    assert {"embed", "head", "final.norm", "final.norm.b", "l0.norm1", "l0.norm1.b", "l0.norm1b", "l0.norm1b.b", "l0.norm2b.b",
            "l0.mix.left.q", "l0.mix.left.q.b", "l0.mix.left.o.b", "l0.mix.left.out", "l0.mix.right.out", "l0.mix.right.q.conv",
            "l0.mix.right.b", "l0.mix.right.a", "l0.mix.right.A_log", "l0.mix.right.dt_bias", "l0.mix.right.norm", "l0.mix.right.g",
            "l0.mix.right.o", "l1.mix.a1", "l1.mix.a2", "l1.mix.a2.b", "l1.mix.norm", "l1.mlp.gate", "l2.mix.lq1", "l2.mix.lk2",
            "l2.mix.v.b", "l0.mlp.router", "l0.mlp.correction", "l0.mlp.e4.up", "l0.mlp.shared.down", "l5.norm1b"} <= names
    assert not any(k.startswith(("l3.", "l4.", "l5.mlp", "l5.norm2")) or "e0.gate" in k or "shared.gate" in k or k == "l2.mix.o.b" for k in names)
    assert w["l0.mlp.router"].shape == (7, 64) and w["l0.mlp.correction"].shape == (7,) and w["l2.mix.q"].shape == (4 * 2 * 9, 64)
    assert w["l2.mix.k"].shape == (2 * 2 * 9, 64) and w["l0.mix.right.a"].shape == (4, 64) and w["l0.mix.right.g"].shape == (56, 64)


def test_state_and_caches_are_declared_per_layer_run(dirs):
    d, cfg, w = dirs["mix"]
    model, cache, runner = engine_parts(d, slots=2)
    needs = model.state_needs()
    assert needs == {(0, "right.S"): (4, 10, 14), (0, "right.conv"): (2, 2 * 2 * 10 + 56), (1, "S"): (3, 12, 20), (3, "S"): (3, 12, 20),
                     (5, "right.S"): (3, 24, 8)}          # one tap keeps no inputs
    caches = model.cache_needs()
    assert sorted(caches) == [0, 2, 4, 5] and caches[2] == caches[4] == KVNeed(2, 18, 0, value_dim=16)
    assert caches[0] == KVNeed(2, 16, 0, value_dim=12)
    assert model.graph_safe() and "portions" in runner.needs


# ------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_of_every_size_against_the_whole_sequence(dirs, name):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d)
    toks = tokens_for(cfg, (50,), seed=11)[0]
    ref = plain_logits(cfg, w, toks)
    for cuts in ((50,), (1,), (2,), (5, 3, 1, 7, 2, 19)):
        assert rel_rms(run_cut(runner, cache, "r", toks, cuts), ref) < 5e-5, (name, cuts)
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
        assert rel_rms(got[r], plain_logits(cfg, w, toks)) < 5e-5, (name, r)


def test_a_requests_state_survives_steps_of_other_requests(dirs):
    d, cfg, w = dirs["one"]
    model, cache, runner = engine_parts(d, slots=2)
    a, b = tokens_for(cfg, (9, 7), seed=3)
    runner.run([Portion("a", a[:4], [])])
    runner.run([Portion("b", b[:6], [])])
    got_a = runner.run([Portion("a", a[4:], list(range(5)))]).numpy().copy()
    got_b = runner.run([Portion("b", b[6:], [0])]).numpy()
    assert rel_rms(got_a, plain_logits(cfg, w, a)[4:]) < 5e-5 and rel_rms(got_b, plain_logits(cfg, w, b)[6:]) < 5e-5


def test_a_pending_norm_resolves_to_the_normed_term():
    """What a norm that cannot take both in its own pass does with a pending term that is normed first."""
    from fusezap_core_b200.engine.step import StepContext, Workspace
    from fusezap_core_b200.parts import PendingNorm
    from fusezap_core_b200.parts.norm import LayerNorm, RMSNorm
    ops, g = PlainOpsSandwich(torch.float32), torch.Generator().manual_seed(0)
    post, norm = LayerNorm(8, 1e-5, name="w", bias="b"), RMSNorm(8, 1e-5)
    post.bind({"w": torch.randn(8, generator=g), "w.b": torch.randn(8, generator=g)}, ops)
    norm.bind({"weight": torch.ones(8)}, ops)
    ctx = StepContext(ops, Workspace(torch.device("cpu"), 4), None, {}, None)
    x, delta = torch.randn(4, 8, generator=g), torch.randn(4, 8, generator=g)
    want = x + plain.layer_norm(delta, post.weight, post.bias, 1e-5)
    h = norm.forward(ctx, x, PendingNorm(delta, post))
    assert torch.allclose(x, want, atol=1e-6) and torch.allclose(h, plain.rms(want, 1e-5), atol=1e-5)


def test_greedy_generation_through_the_entry_point(dirs):
    """Through `LLMEngine` and its scheduler: portions of prompts beside decoding requests, more requests than state
    slots, a pool that does not hold all of them at once."""
    d, cfg, w = dirs["odd"]
    eng = LLMEngine.from_pretrained(d, dtype="float32", device="cpu", ops=PlainOpsSandwich(torch.float32), max_model_len=64,
                                    num_blocks=14, block_size=8, max_num_seqs=2, max_prefill_tokens=8, cuda_graphs=False)
    P = tokens_for(cfg, (7, 19, 2, 30), seed=2)
    out = eng.generate(P, SamplingParams(max_tokens=5, ignore_eos=True))
    for prompt, new in zip(P, out):
        lg = plain_logits(cfg, w, list(prompt) + new)
        for i, t in enumerate(new):
            row = lg[len(prompt) - 1 + i]
            assert int(row.argmax()) == t or row.max() - row[t] < 1e-3


def test_the_decay_projections_inner_size_is_the_checkpoints(tmp_path):
    """Whatever it is: five, which no product's tile divides, and more than the width."""
    for rank in (5, 80):
        d, cfg, w = make_dir(f"rank{rank}", tmp_path, MUR_MIX, 3, change=lambda t: other_rank(t, rank))
        assert w["l1.mix.a1"].shape[0] == rank
        model, cache, runner = engine_parts(d)
        toks = tokens_for(cfg, (40,), seed=rank)[0]
        Oracle(cfg, w, toks, "float32").check(run_cut(runner, cache, "r", toks, (11, 2, 1)), rank)


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    """The host side reads every size and constant from the configuration: drawn ones (the GPU tests' own) against the
    plain model, whole, in portions and token by token."""
    cfg = drawn_config(seed)
    d, cfg, w = make_dir(f"drawn{seed}", tmp_path, cfg, seed)
    model, cache, runner = engine_parts(d, page=4, pages=30, slots=2, max_len=64)
    toks = tokens_for(cfg, (40,), seed=seed)[0]
    ref = Oracle(cfg, w, toks, "float32")
    for cuts in ((40,), (1,), (6, 2, 1, 17)):
        ref.check(run_cut(runner, cache, "r", toks, cuts), (seed, cuts))
