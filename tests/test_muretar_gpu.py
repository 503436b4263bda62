"""Muretar on the GPU: every new or extended kernel alone against its plain function, then the model in both dtypes (portions
down to two tokens, unequal batches with pages and slots used again, long decoding across page borders, generation through
the entry point and the command line, drawn configurations)."""
import json
import math

import numpy as np
import pytest
import torch

import plain_muretar as plain
from gimupel_util import check_all
from muretar_util import CONFIGS, Oracle, corrections_apart, drawn_config, make_dir, plain_logits, rounded, tokens_for
from pepilix_util import run_cut, run_mixed
from test_gizulorn_gpu import Meta, close, paged, scan_portions, shuffled_tables
from fusezap_core_b200 import LLMEngine, SamplingParams
from fusezap_core_b200.cache import CacheManager, KVNeed
from fusezap_core_b200.engine import StepRunner, load_model
from fusezap_core_b200.engine.step import StepContext, Workspace
from fusezap_core_b200.kernels import cuda_ops

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("muretar")
    return {name: make_dir(name, tmp) for name in CONFIGS}


def engine_parts(d, dtype, page=4, pages=48, slots=3, max_len=192):
    model = load_model(d, dtype, DEV, max_len=max_len)
    cache = CacheManager(model.cache_needs(), model.state_needs(), page, pages, slots, max_len, model.ops.dtype, DEV)
    return model, cache, StepRunner(model, cache, max_rows=max_len, max_wanted=max_len, max_segments=slots)


def raw(w, dtype):
    return w if dtype == "float32" else rounded(w)


# ---------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_portions_of_every_size_against_the_whole_sequence(dirs, name, dtype):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d, dtype)
    toks = tokens_for(cfg, (150,), seed=11)[0]
    ref = Oracle(cfg, w, toks, dtype)
    first = None
    for cuts in ((150,), (1,), (2,), (5, 3, 1, 7, 2, 19), (100, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1), (64, 65, 2), (16, 17, 63)):
        got = run_cut(runner, cache, "r", toks, cuts)
        model.ops.check_errors()
        ref.check(got, (name, cuts))
        cache.check()
        if dtype == "float32":      # every sum's order is a function of the row alone: the cuttings agree bit for bit
            first = got if first is None else first
            assert np.array_equal(got, first), (name, cuts)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_requests_in_one_batch_with_pages_and_slots_used_again(dirs, name, dtype):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d, dtype, page=4, pages=64, slots=3, max_len=160)
    reqs = dict(zip("abcde", tokens_for(cfg, (61, 9, 33, 2, 130), seed=5)))
    plan = [[("a", 17), ("b", 2)], [("a", 1), ("b", 7), ("c", 30)], [("a", 20), ("c", 1)], [("a", 1), ("c", 1), ("d", 2)],
            [("a", 22), ("c", 1), ("e", 5)], [("e", 1)], [("e", 90)], [("e", 1)], [("e", 33)]]
    got = run_mixed(runner, cache, reqs, plan)
    model.ops.check_errors()
    cache.check()
    assert cache.live_requests() == [] and cache.states.num_free == 3
    check_all([(Oracle(cfg, w, toks, dtype), got[r]) for r, toks in reqs.items()], name)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "tc"])
def test_long_decoding_across_page_borders(dirs, name, dtype):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d, dtype, page=8, pages=48, slots=2, max_len=384)
    toks = tokens_for(cfg, (340,), seed=23)[0]
    got = run_cut(runner, cache, "long", toks, (21,) + (1,) * 319)
    model.ops.check_errors()
    Oracle(cfg, w, toks, dtype).check(got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_of_a_sequence(dirs, dtype):
    """Requests of one to six tokens, each alone and all in one step: the convolution's zeros, the empty states, a softmax
    over one key (the difference of the two maps is then one multiple of the value)."""
    for name in CONFIGS:
        d, cfg, w = dirs[name]
        model, cache, runner = engine_parts(d, dtype, slots=6)
        P = tokens_for(cfg, (1, 2, 3, 4, 5, 6), seed=9)
        refs = [Oracle(cfg, w, t, dtype) for t in P]
        alone = [run_cut(runner, cache, f"r{i}", t, (len(t),)) for i, t in enumerate(P)]
        both = run_mixed(runner, cache, {f"b{i}": t for i, t in enumerate(P)}, [[(f"b{i}", len(t)) for i, t in enumerate(P)]])
        check_all([(r, g) for i, r in enumerate(refs) for g in (alone[i], both[f"b{i}"])], name)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_mechanism_left_out_would_show(dirs, dtype):
    """What the oracle gives with one mechanism taken out or changed differs from the engine by far more than the limit, for
    every mechanism: so none of them is missing in the engine."""
    d, cfg, w = dirs["mix"]
    model, cache, runner = engine_parts(d, dtype)
    toks = tokens_for(cfg, (90,), seed=2)[0]
    got = run_cut(runner, cache, "r", toks, (40, 2, 1, 1, 16))
    wr = raw(w, dtype)
    ref = Oracle(cfg, w, toks, dtype)
    ref.check(got)
    typical = np.quantile(ref.errors(got), 0.9)
    keep = {k: getattr(plain, k) for k in ("layer_norm", "rotate", "mixing_number", "combine_maps", "route", "expert", "channel_decay",
                                           "unit", "causal_conv", "delta_recurrence_fast", "gla_recurrence_fast", "mixture")}

    def without_input(v, p, mlp, h):
        r = mlp["router"]
        y, idx, wt = keep["mixture"](v, p, mlp, h), *keep["route"](h @ v[p + "router"].T, v[p + "correction"], r["top"])
        return y - (wt * (idx >= r["experts"])).sum(-1, keepdim=True) * h

    def one_map(a1, a2, lam, diff, eps):
        return keep["combine_maps"](a1, 0 * a2, lam, diff, eps)
    broken = {
        "layer_norm": lambda x, v, b, eps: keep["layer_norm"](x, v, 0 * b, eps),
        "rotate": lambda x, dims, base, f: keep["rotate"](x, dims, base, 1.0),
        "mixing_number": lambda a, b, c, e, diff: torch.as_tensor(diff),
        "combine_maps": one_map,
        "route": lambda z, c, top: keep["route"](z, c * 0, top),
        "expert": lambda v, p, h: torch.relu(h @ v[p + "up"].T) @ v[p + "down"].T,
        "channel_decay": lambda z, tau: keep["channel_decay"](z, 1.0),
        "unit": lambda x: x,
        "causal_conv": lambda x, v: x * v[:, -1],
        "delta_recurrence_fast": lambda q, k, v, g, b: keep["delta_recurrence_fast"](q, k, v, torch.ones_like(g), b),
        "gla_recurrence_fast": lambda q, k, v, a: keep["gla_recurrence_fast"](q, k, v, torch.ones_like(a)),
        "mixture": without_input,
    }
    for name, fn in broken.items():
        try:
            setattr(plain, name, fn)
            ref.logits = plain_logits(cfg, wr, toks)
            assert np.quantile(ref.errors(got), 0.9) > 2.5 * typical + 1e-3, (name, typical)
        finally:
            setattr(plain, name, keep[name])


# ---------------------------------------------------------------------------------------- the scans alone
def gla_reference(proj, z, H, dk, dv, root, scale):
    T, x = proj.shape[0], proj.to(F)
    q, k = x[:, :H * dk].view(T, H, dk) * scale, x[:, H * dk: 2 * H * dk].reshape(T, H, dk)
    v = x[:, 2 * H * dk: 2 * H * dk + H * dv].reshape(T, H, dv)
    y, S = plain.gla_recurrence_fast(q, k, v, plain.channel_decay(z.to(F), root).view(T, H, dk))
    return y.reshape(T, H * dv), S


def run_gla(ops, inputs, T, H, dk, dv, root, steps, pad=1):
    """Two sequences through `channel_decay_scan` in the given steps; slots 1 and 3 of four, slot 2 must stay as it is."""
    state = torch.zeros(4, *ops.recurrent_state_shape(H, dk, dv), device=DEV)
    state[2] = 3.0
    got = [torch.zeros(T, H * dv) for _ in range(2)]
    for step in steps:
        meta = Meta([(n, at, (1, 3)[r]) for r, at, n in step], pad=pad)
        meta.max_portion = max(n for _, _, n in step)
        rows = lambda k: torch.cat([inputs[r][k][at: at + n] for r, at, n in step] + [torch.zeros(pad, inputs[0][k].shape[1])]).to(DEV)
        out = torch.full((meta.n_rows, H * dv), 7.0, device=DEV)
        ops.channel_decay_scan(rows(0), H, dk, dv, rows(1), root, dk ** -0.5, state, meta, out)
        ops.check_errors()
        k = 0
        for r, at, n in step:
            got[r][at: at + n] = out[k: k + n].cpu()
            k += n
    assert float(state[2].min()) == 3.0 == float(state[2].max()) and float(state[0].abs().max()) == 0.0
    return got, state


def near_exact(got, ref, dtype, what):
    """32-bit sums in both dtypes; in bfloat16 mode long portions take the operands of their products as two bfloat16 numbers
    each, 2^-17 off per term."""
    if dtype == "float32":
        return close(got, ref, "float32", what)
    err = (got.to(F) - ref).abs()
    assert not (err > 3e-5 * (ref.abs() + ref.abs().max())).any(), (what, float((err / ref.abs().max()).max()))


GLA_SIZES = [(3, 12, 20, 16.0), (1, 40, 16, 0.5), (5, 30, 6, 2.0), (2, 64, 32, 12.0), (2, 128, 128, 16.0), (1, 9, 7, 1.0), (3, 48, 64, 14.0),
             (3, 16, 16, 4.0), (1, 200, 40, 3.0), (2, 96, 300, 8.0), (1, 256, 16, 1.0), (4, 80, 48, 0.8)]


def gla_inputs(T, H, dk, dv, seed, spread=3.0):
    """Decay inputs from channels that hardly forget to channels that forget at once."""
    g = torch.Generator().manual_seed(seed)
    proj = torch.randn(T, H * (2 * dk + dv) + 8, generator=g)
    z = torch.randn(T, H * dk, generator=g) * spread + torch.linspace(-6, 8, H * dk)
    return proj, z


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dk,dv,root", GLA_SIZES)
def test_linear_attention_scan_carries_its_state_across_portions(dtype, H, dk, dv, root):
    """Portions down to one token, interleaved, a row of padding, a slot nobody uses."""
    ops, T = cuda_ops(dtype), 70
    inputs = [gla_inputs(T, H, dk, dv, seed=dk + r) for r in range(2)]
    got, state = run_gla(ops, inputs, T, H, dk, dv, root, scan_portions(T, seed=dv))
    for r in range(2):
        ref, S = gla_reference(*inputs[r], H, dk, dv, root, dk ** -0.5)
        near_exact(got[r], ref, dtype, f"request {r}")
        have = state[(1, 3)[r]][:, :, :dk].transpose(1, 2).cpu().to(F)
        assert (have - S).abs().max() < 3e-5 * (1 + S.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,dk,dv,root", GLA_SIZES)
def test_linear_attention_scan_of_long_portions(dtype, H, dk, dv, root):
    """Portions of hundreds of tokens around multiples of 16 and 64, two requests beside each other, then single tokens from
    the state they left, decays from none to total within one chunk; 32-bit close to the plain recurrence in both dtypes."""
    ops, T = cuda_ops(dtype), 421
    inputs = [gla_inputs(T, H, dk, dv, seed=3 * dk + r) for r in range(2)]
    steps = [[(0, 0, 200), (1, 0, 64)], [(0, 200, 1), (1, 64, 129)], [(1, 193, 63)], [(0, 201, 220), (1, 256, 2)], [(1, 258, 163)]]
    got, state = run_gla(ops, inputs, T, H, dk, dv, root, steps, pad=3)
    for r in range(2):
        ref, S = gla_reference(*inputs[r], H, dk, dv, root, dk ** -0.5)
        err = (got[r].to(F) - ref).abs()
        assert not (err > 4e-5 * (ref.abs() + ref.abs().max())).any(), (r, float((err / ref.abs().max()).max()))
        have = state[(1, 3)[r]][:, :, :dk].transpose(1, 2).cpu().to(F)
        assert (have - S).abs().max() < 4e-5 * (1 + S.abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_single_token_is_remembered_for_hundreds_of_tokens_and_decays_as_it_should(dtype):
    """Keys are zero except at one token (the first, at a chunk's border, in the middle): every later output is that token's
    value times the product of the decays, channel by channel, in one portion, in portions, and token by token at the end.
    A lost or doubled state at any border would show at once."""
    ops, T, H, dk, dv, root = cuda_ops(dtype), 700, 1, 32, 16, 4.0
    z = torch.linspace(-2.0, 9.0, dk).expand(T, dk).contiguous()
    log_a = torch.nn.functional.logsigmoid(z[0].to(F)) / root
    for j in (0, 63, 64, 300):
        proj = torch.zeros(T, 2 * dk + dv)
        proj[:, :dk] = torch.linspace(0.5, 1.5, dk)
        proj[j, dk: 2 * dk] = torch.linspace(-1.0, 2.0, dk)
        proj[:, 2 * dk:] = 0.7
        ages = torch.arange(T, dtype=F)[:, None] - j
        each = torch.where(ages >= 0, torch.exp(log_a * ages.clamp(min=0)), torch.zeros((), dtype=F))
        want = (each * proj[0, :dk].to(F) * dk ** -0.5 * proj[j, dk: 2 * dk].to(F)).sum(-1) * 0.7
        for steps in ([[(0, 0, T)]], [[(0, at, min(100, T - at))] for at in range(0, T, 100)],
                      [[(0, 0, 310)]] + [[(0, at, 1)] for at in range(310, 330)] + [[(0, 330, 370)]]):
            got, _ = run_gla(ops, [(proj, z)] * 2, T, H, dk, dv, root, steps)
            assert ((got[0].to(F) - want[:, None]).abs() <= 3e-4 * want[:, None].abs() + 2e-6).all(), (j, len(steps))


DELTA_SIZES = [(4, 2, 8, 16), (2, 1, 20, 12), (3, 3, 12, 8), (2, 2, 128, 40), (6, 3, 48, 260), (2, 1, 9, 7), (1, 1, 136, 10), (4, 2, 64, 64), (2, 1, 128, 128),
               (2, 2, 32, 96)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("long", [False, True])
@pytest.mark.parametrize("H,Hk,dk,dv", DELTA_SIZES)
def test_delta_rule_with_one_decay_per_head(dtype, long, H, Hk, dk, dv):
    """The decay inputs and beta as columns of one wide product; heads that hardly forget and heads that forget at once;
    portions down to one token, or of hundreds beside short ones."""
    ops, g, dt = cuda_ops(dtype), torch.Generator().manual_seed(dk + dv), DT[dtype]
    T = 300 if long else 60
    C, width, off = 2 * Hk * dk + H * dv, H + H + 9, 5
    qkv = [torch.randn(T, C, generator=g).to(dt) for _ in range(2)]
    rows = [torch.randn(T, width, generator=g) * 2 for _ in range(2)]
    a_log = torch.linspace(-6.0, 1.5, H) if H > 1 else torch.tensor([-2.0])
    dt_bias = torch.randn(H, generator=g)
    state = torch.zeros(3, *ops.recurrent_state_shape(H, dk, dv), device=DEV)
    slots, got = (2, 0), [torch.zeros(T, H * dv), torch.zeros(T, H * dv)]
    steps = [[(0, 0, 130), (1, 0, 64)], [(0, 130, 1), (1, 64, 65)], [(0, 131, 169), (1, 129, 2)], [(1, 131, 169)]] if long else scan_portions(T, seed=dk)
    for step in steps:
        meta = Meta([(n, p0, slots[r]) for r, p0, n in step], pad=2)
        meta.max_portion = max(n for _, _, n in step)
        cat = lambda xs, w, d: torch.cat([xs[r][p0: p0 + n] for r, p0, n in step] + [torch.zeros(2, w, dtype=d)]).to(DEV)
        out = torch.full((meta.n_rows, H * dv), 9.0, device=DEV)
        wide = cat(rows, width, torch.float32)
        ops.gated_delta_scan(cat(qkv, C, dt), H, Hk, dk, dv, wide, wide, a_log.to(DEV), dt_bias.to(DEV), 1e-6, dk ** -0.5, state, meta, out,
                             head_decay=True, high_offset=off, beta_offset=off + H + 2)
        at = 0
        for r, p0, n in step:
            got[r][p0: p0 + n] = out[at: at + n].cpu()
            at += n
    ops.check_errors()
    for r in (0, 1):
        x, y = qkv[r].to(F), rows[r].to(F)
        rep = H // Hk
        q = (plain.unit(x[:, :Hk * dk].view(T, Hk, dk)) * dk ** -0.5).repeat_interleave(rep, 1)
        k = plain.unit(x[:, Hk * dk: 2 * Hk * dk].view(T, Hk, dk)).repeat_interleave(rep, 1)
        decay = torch.exp(-torch.exp(a_log.to(F)) * plain.softplus(y[:, off: off + H] + dt_bias.to(F)))
        ref, S = plain.delta_recurrence_fast(q, k, x[:, 2 * Hk * dk:].view(T, H, dv), decay, torch.sigmoid(y[:, off + H + 2: off + 2 * H + 2]))
        if long:
            err = (got[r].view(T, H, dv).to(F) - ref).abs()
            assert not (err > 6e-5 * (ref.abs() + ref.abs().max())).any(), (r, float((err / ref.abs().max()).max()))
        else:
            near_exact(got[r].view(T, H, dv), ref, dtype, f"request {r}")
        have = state[slots[r]][:, :, :dk].transpose(1, 2).cpu().to(F)
        assert (have - S).abs().max() < (1e-4 if long else 3e-5) * (1 + S.abs().max())
    assert float(state[1].abs().max()) == 0.0


# ---------------------------------------------------------------------------------------- differential attention
def diff_rows(dtype, H, G, d, dv, T, portions, page, seed, loud=None, scale=0.3, lam=0.37, eps=1e-5, mult=0.4, side_by_side=False):
    """One sequence of T tokens in shuffled pages; `portions` ((rows, first position) each) are asked for in one step. loud
    (key position, map): that map's key there and every query of that map point one way, so that its score stands out."""
    ops, g, dt = cuda_ops(dtype), torch.Generator().manual_seed(seed), DT[dtype]
    q, k = torch.randn(T, H, 2, d, generator=g), torch.randn(T, G, 2, d, generator=g)
    v = torch.randn(T, G, dv, generator=g)
    if loud is not None:
        j, m = loud
        way = torch.nn.functional.normalize(torch.randn(d, generator=g), dim=0)
        k[j, :, m] = way * 12.0
        q[:, :, m] = q[:, :, m] * 0.05 + way * 6.0
    pages = -(-T // page)
    table = shuffled_tables(1, pages, pages + 5, seed)
    cache = paged(KVNeed(G, 2 * d, 0, value_dim=0 if dv == 2 * d and not side_by_side else dv), page, pages + 5, dtype)
    qkv = torch.cat([q.view(T, -1), k.view(T, -1), v.view(T, -1)], 1).float().to(DEV)
    qn = torch.empty(T, H * 2 * d, dtype=dt, device=DEV)
    ops.rotate_kv_write(qkv, None, None, 0, 0, Meta([(T, 0, 0)], table), cache, qn, H, G, 2 * d, dv)
    meta = Meta([(n, p0, 0) for n, p0 in portions], table.repeat(len(portions), 1), pad=1)
    meta.max_portion = max(n for n, _ in portions)
    rows = [p for n, p0 in portions for p in range(p0, p0 + n)]
    qs = torch.cat([qn[rows], torch.zeros(1, H * 2 * d, dtype=dt, device=DEV)]).contiguous()
    out = torch.full((len(rows) + 1, H * dv), 7.0, dtype=dt, device=DEV)
    ops.check_differential_attention(H, G, d, dv)
    ops.differential_attention(qs, cache, meta, out, H, G, d, dv, scale, torch.tensor([lam], device=DEV), eps, mult)
    ops.check_errors()
    assert float(out[-1].float().abs().max()) == 0.0
    q, k, v = (t.to(dt).to(F) for t in (q, k, v))
    rep = H // G
    a = [plain.causal_attention_fast(q[:, :, m], k[:, :, m].repeat_interleave(rep, 1), v.repeat_interleave(rep, 1), scale) for m in (0, 1)]
    ref = plain.combine_maps(a[0], a[1], torch.tensor(lam, dtype=F), mult_to_diff(mult), eps)
    return out[:-1].view(len(rows), H, dv), ref[rows], v, a


def mult_to_diff(mult):
    return 1.0 - mult


def near(got, ref, dtype, what=None):
    err = (got.detach().cpu().to(F) - ref).abs()
    tol = 2e-5 if dtype == "float32" else 2.0 ** -5
    assert not (err > tol * (ref.abs() + ref.abs().mean() + 1e-3)).any(), (what, float(err.max()))


DIFF_SIZES = [(4, 2, 9, 16), (6, 3, 20, 12), (1, 1, 33, 17), (2, 1, 4, 8), (6, 3, 32, 64), (2, 2, 64, 128), (4, 1, 64, 64), (3, 3, 32, 128),
              (6, 2, 64, 128), (16, 2, 16, 40), (40, 1, 8, 24), (2, 1, 128, 256)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv", DIFF_SIZES)
def test_differential_attention_of_portions_and_single_tokens(dtype, H, G, d, dv):
    portions = [(70, 0), (2, 80), (1, 97), (1, 199), (1, 5), (90, 100), (1, 0)]
    got, ref, _, _ = diff_rows(dtype, H, G, d, dv, 200, portions, page=4, seed=H * d)
    near(got, ref, dtype)
    got, ref, _, _ = diff_rows(dtype, H, G, d, dv, 200, [(1, p) for p in (0, 1, 31, 32, 63, 64, 150, 199)], page=4, seed=H + d)
    near(got, ref, dtype, "single tokens")
    if dv == 2 * d:      # the cache's other layout, which the general kernels take
        got, ref, _, _ = diff_rows(dtype, H, G, d, dv, 200, [(1, p) for p in (0, 1, 31, 150, 199)], page=8, seed=d, side_by_side=True)
        near(got, ref, dtype, "keys and values side by side")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("as_portion", [True, False])
@pytest.mark.parametrize("d,dv", [(9, 16), (32, 64), (64, 128), (20, 12)])
def test_a_loud_key_of_either_map_is_found_however_far_away_it_is(dtype, as_portion, d, dv):
    """One key's score in one map exceeds all others by far, so that map's result is that key's value: keys at position 0, at
    page borders and in the middle, rows just after the key and far behind it, in prompt portions and as single tokens."""
    page, T = 8, 700
    for m in (0, 1):
        for j in (0, 7, 8, 127, 128, 300):
            rows = sorted({p for p in (j, j + 1, j + 31, j + 64, T - 1) if j <= p < T})
            portions = [(r - max(0, r - 69) + 1, max(0, r - 69)) for r in rows] if as_portion else [(1, p) for p in rows]
            got, ref, v, a = diff_rows(dtype, 2, 1, d, dv, T, portions, page, seed=j + m, loud=(j, m), scale=1.0)
            near(got, ref, dtype, f"key {j} of map {m}")
            for p in rows:
                assert (a[m][p] - v[j]).abs().max() < 0.05          # (the oracle's map does return that key's value)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,d,dv", [(4, 2, 16, 12), (6, 1, 64, 32), (3, 3, 128, 64), (2, 1, 64, 128), (8, 2, 48, 64)])
def test_causal_attention_with_keys_and_values_of_unequal_size(dtype, H, G, d, dv):
    """The attention beside the delta rule: no window, no sink, key and value sizes apart (with tensor-core kernels and without)."""
    ops, g, dt, T, page = cuda_ops(dtype), torch.Generator().manual_seed(d), DT[dtype], 300, 16
    q, k, v = (torch.randn(T, h, n, generator=g) for h, n in ((H, d), (G, d), (G, dv)))
    k[3] *= 6.0
    pages = -(-T // page)
    table = shuffled_tables(1, pages, pages + 5, d)
    cache = paged(KVNeed(G, d, 0, value_dim=dv), page, pages + 5, dtype)
    qkv = torch.cat([q.view(T, -1), k.view(T, -1), v.view(T, -1)], 1).float().to(DEV)
    qn = torch.empty(T, H * d, dtype=dt, device=DEV)
    ops.check_sink_attention(H, G, d, dv)
    ops.rotate_kv_write(qkv, None, None, 0, 0, Meta([(T, 0, 0)], table), cache, qn, H, G, d, dv)
    q, k, v = (t.to(dt).to(F) for t in (q, k, v))
    ref = plain.causal_attention_fast(q, k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1), 0.3)
    for portions in ([(150, 0), (130, 170), (1, 160)], [(1, p) for p in (0, 15, 16, 31, 32, 299)]):
        meta = Meta([(n, p0, 0) for n, p0 in portions], table.repeat(len(portions), 1), pad=1)
        meta.max_portion = max(n for n, _ in portions)
        rows = [p for n, p0 in portions for p in range(p0, p0 + n)]
        qs = torch.cat([qn[rows], torch.zeros(1, H * d, dtype=dt, device=DEV)]).contiguous()
        out = torch.full((len(rows) + 1, H * dv), 7.0, dtype=dt, device=DEV)
        ops.sink_attention(qs, cache, meta, out, H, G, d, dv, 0.3, 0, 0, None)
        ops.check_errors()
        assert float(out[-1].float().abs().max()) == 0.0
        near(out[:-1].view(len(rows), H, dv), ref[rows], dtype)


# ---------------------------------------------------------------------------------------- norms and sums of rows
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D", [64, 200, 1030, 7, 2048, 4096, 9000])
def test_layer_norm_with_a_bias_and_a_pending_term_that_is_normed_first(dtype, D):
    """In one pass: the pending term's own layer norm (rows with a mean far above their spread among them), its addition to
    the stream, the norm of the sum with a bias; selected rows."""
    from fusezap_core_b200.parts import PendingNorm
    from fusezap_core_b200.parts.norm import LayerNorm
    ops, g = cuda_ops(dtype), torch.Generator().manual_seed(D)
    made = []
    for i in range(2):
        n = LayerNorm(D, (1e-5, 1e-3)[i], name="w", bias="b")
        t = {"w": torch.randn(D, generator=g), "w.b": torch.randn(D, generator=g)}
        n.bind({k: v.to(DEV) for k, v in t.items()}, ops)
        made.append((n, t["w"].to(F), t["w.b"].to(F)))
    (norm, w, b), (post, pw, pb) = made
    x, delta = torch.randn(9, D, generator=g), torch.randn(9, D, generator=g)
    delta[2] += 100.0
    delta[5] *= 1e-3
    ctx = StepContext(ops, Workspace(torch.device(DEV), 9), Meta([(9, 0, -1)]), {}, None)
    xd = x.to(DEV)
    h = norm.forward(ctx, xd, PendingNorm(delta.to(DEV), post))
    full = x.to(F) + plain.layer_norm(delta.to(F), pw, pb, 1e-3)
    lim = torch.full((9, 1), 5e-6, dtype=F)
    lim[2] = 2e-4             # (100 in 32-bit leaves an absolute error of 1e-5 in every deviation)
    assert ((xd.cpu().to(F) - full).abs() <= lim * (1 + full.abs())).all()
    ref = plain.layer_norm(full, w, b, 1e-5)
    if dtype == "bfloat16":
        lim = lim + 2.0 ** -8
    assert ((h.cpu().to(F) - ref).abs() <= 2 * lim * (1 + ref.abs())).all()
    rows = torch.tensor([7, -1, 0], dtype=torch.int32, device=DEV)
    xd = x.to(DEV)
    h = norm.forward(ctx, xd, PendingNorm(delta.to(DEV), post), rows=rows)
    assert torch.equal(xd.cpu(), x) and float(h[1].float().abs().max()) == 0.0
    close(h[[0, 2]], ref[[7, 0]], dtype)
    h = norm.forward(ctx, x.to(DEV), delta.to(DEV))
    close(h[[0, 1, 3, 4]], plain.layer_norm((x + delta).to(F), w, b, 1e-5)[[0, 1, 3, 4]], dtype)
    out = torch.empty(9, D, device=DEV)
    post.forward_into(ctx, delta.to(DEV), out)
    close(out[[0, 1, 3, 4]], plain.layer_norm(delta.to(F), pw, pb, 1e-3)[[0, 1, 3, 4]], "float32")


@pytest.mark.parametrize("D", [64, 200, 1030, 7, 2048, 4096, 9000])
@pytest.mark.parametrize("terms", [1, 2, 3])
def test_sum_of_normed_terms(D, terms):
    ops, g = cuda_ops("float32"), torch.Generator().manual_seed(D)
    t = [torch.randn(6, D, generator=g) * 10.0 ** i for i in range(terms)]
    w = [torch.randn(D, generator=g) for _ in range(terms)]
    s = [0.5, 0.25, -2.0][:terms]
    out = torch.empty(6, D, device=DEV)
    ops.normed_sum([x.to(DEV) for x in t], [x.to(DEV) for x in w], s, 1e-5, out)
    close(out, sum(a * plain.rms(x.to(F), 1e-5) * y.to(F) for a, x, y in zip(s, t, w)), "float32")


# ---------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D,E,identity,top,I,shared,n", [(64, 5, 2, 3, 24, 40, 40), (64, 1, 4, 2, 40, 0, 7), (64, 8, 4, 12, 8, 8, 300), (64, 10, 0, 3, 80, 32, 1),
                                                         (128, 4, 1, 1, 64, 192, 130), (40, 3, 3, 6, 12, 20, 19), (256, 16, 2, 4, 128, 256, 260)])
def test_ungated_experts_beside_experts_that_hand_their_input_on(dtype, D, E, identity, top, I, shared, n):
    from fusezap_core_b200.parts.routed_moe import RoutedMoE
    ops, g, dt = cuda_ops(dtype), torch.Generator().manual_seed(E * I), DT[dtype]
    names = {"router": "router", "correction": "correction", "expert": "e{}", "up": "up", "down": "down", "shared": "shared"}
    ff = RoutedMoE(D, I, E, top, renormalize=True, correction=True, sum_eps=1e-20, shared_size=shared, shared_gate=False, identity=identity,
                   activation="relu2", names=names)
    w = {k: torch.randn(p.shape, generator=g) * (0.3 if p.role == "vector" else 2.0 / D ** 0.5) for k, p in ff.tensors().items()}
    w = {k: v.to(dt).float() if v.dim() >= 2 else v for k, v in w.items()}
    ff.bind({k: (v.to(dt) if v.dim() >= 2 else v).to(DEV) for k, v in w.items()}, ops)
    h = torch.randn(n + 1, D, generator=g).to(dt)
    ctx = StepContext(ops, Workspace(torch.device(DEV), n + 1), Meta([(n, 0, -1)], pad=1), {}, None)
    ctx.ws.get("moe_terms", ((n + 1) * top, D), torch.float32).fill_(float("nan"))      # (what no expert writes must not be read)
    out = ff.forward(ctx, h.to(DEV))
    ops.check_errors()
    mlp = {"router": {"experts": E, "identity": identity, "top": top}, "shared": {"ff": shared} if shared else None}
    wf = {k: v.to(F) for k, v in w.items()}
    ref = plain.mixture(wf, "", mlp, h[:n].to(F))
    err = (out[:n].cpu().to(F) - ref).abs().max(-1).values / ref.abs().max()
    # (a row whose choice scores nearly tie may choose otherwise)
    assert float(err.median()) < (1e-5 if dtype == "float32" else 1e-2) and float((err > 0.1).float().mean()) < 0.05
    assert float(out[n].abs().max()) == 0.0
    if identity:
        idx, _ = plain.route(h[:n].to(F) @ wf["router"].T, wf["correction"], top)
        assert n < 5 or (idx >= E).any()


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (8, 512, 1024), (17, 200, 320), (64, 128, 4096), (130, 384, 256), (300, 1024, 2048), (2048, 512, 512),
                                   (5, 33, 40), (260, 2048, 4096)])
def test_product_with_a_squared_relu(M, N, K):
    """Every form of the product (few rows with K cut and not, rows by the hundred, pairs of SMs): the same as the product
    followed by the activation, in bfloat16 and float32."""
    ops, g = cuda_ops("bfloat16"), torch.Generator().manual_seed(M)
    a, w, b = torch.randn(M, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) / K ** 0.5).bfloat16(), torch.randn(N, generator=g)
    ref = torch.clamp(a.double() @ w.double().T + b.double(), min=0.0) ** 2
    for dt in (torch.bfloat16, torch.float32):
        out = torch.full((M, N), 7.0, dtype=dt, device=DEV)
        assert ops.linear_act(a.to(DEV), w.to(DEV), b.to(DEV), out, "relu2")
        ops.check_errors()
        err = (out.cpu().double() - ref).abs()
        assert (err <= (2.0 ** -8 if dt == torch.bfloat16 else 2e-5) * (1 + ref)).all(), (dt, float(err.max()))


# ------------------------------------------------------------------------------------------------ the model, further
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "tc"])
def test_greedy_generation_through_the_entry_point(dirs, dtype, name, tmp_path):
    """Through `LLMEngine` and its scheduler (portions of prompts beside decoding requests, more requests than state
    slots, a pool that does not hold all requests at once, captured decode steps): every generated token is the plain
    model's choice, or within rounding of it (in bfloat16 with experts whose choice does not hang on rounding)."""
    d, cfg, w = dirs[name] if dtype == "float32" else make_dir(name, tmp_path, change=corrections_apart)
    eng = LLMEngine.from_pretrained(d, dtype=dtype, device=DEV, max_model_len=96, num_blocks=20, block_size=8,
                                    max_num_seqs=3, max_prefill_tokens=16)
    P = tokens_for(cfg, (7, 23, 2, 41, 12), seed=2)
    out = eng.generate(P, SamplingParams(max_tokens=14, ignore_eos=True))
    assert eng.stats["graph_replays"] > 0
    gaps = []
    for prompt, new in zip(P, out):
        lg = plain_logits(cfg, raw(w, dtype), list(prompt) + new)
        for i, t in enumerate(new):
            row = lg[len(prompt) - 1 + i]
            gaps.append((row.max() - row[t]) / lg.std())
    assert np.quantile(gaps, 0.95) < (1e-4 if dtype == "float32" else 0.15) and max(gaps) < (1e-3 if dtype == "float32" else 1.0), (max(gaps), name)


def test_command_line_generates_from_a_preset_with_random_weights(capsys):
    from fusezap_core_b200.cli import main
    assert main(["generate", "--random", "tiny-muretar", "--prompt-lens", "5,40,1", "--max-tokens", "6", "--ignore-eos",
                 "--max-model-len", "128", "--num-blocks", "32", "--max-num-seqs", "2"]) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert [o["num_prompt_tokens"] for o in lines] == [5, 40, 1]
    assert all(len(o["token_ids"]) == 6 and o["finish_reason"] == "length" for o in lines)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("rank", [5, 80])
def test_the_decay_projections_inner_size_is_the_checkpoints(dtype, rank, tmp_path):
    from muretar_util import MUR_MIX, other_rank
    d, cfg, w = make_dir(f"rank{rank}", tmp_path, MUR_MIX, 3, change=lambda t: other_rank(t, rank))
    model, cache, runner = engine_parts(d, dtype)
    toks = tokens_for(cfg, (90,), seed=rank)[0]
    Oracle(cfg, w, toks, dtype).check(run_cut(runner, cache, "r", toks, (50, 2, 1, 1)), rank)
    model.ops.check_errors()


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Every size and constant comes from the configuration: drawn ones in float32 against the plain model (whole, in
    portions, token by token), and in bfloat16; a long prompt first, so that prompt portions reach every kernel."""
    cfg = drawn_config(seed)
    d, cfg, w = make_dir(f"drawn{seed}", tmp_path, cfg, seed)
    toks = tokens_for(cfg, (150,), seed=seed)[0]
    for dtype in ("float32", "bfloat16"):
        model, cache, runner = engine_parts(d, dtype, page=16, pages=12, slots=2, max_len=160)
        ref = Oracle(cfg, w, toks, dtype)
        for cuts in ((150,), (130, 1), (70, 2, 1, 17)):
            got = run_cut(runner, cache, "r", toks, cuts)
            model.ops.check_errors()
            ref.check(got, (seed, dtype, cuts, json.dumps(cfg)[:900]))


@pytest.mark.parametrize("seed", range(5))
def test_configurations_of_a_small_models_size(seed, tmp_path):
    """Widths of a few hundred, head sizes up to 128, prompts of hundreds of tokens in a pool that holds the live requests
    only: whole, with a decoded tail, in portions down to two tokens, and beside other requests, in both dtypes."""
    cfg = drawn_config(seed, small=False)
    d, cfg, w = make_dir(f"model{seed}", tmp_path, cfg, seed)
    L = (421, 700, 333, 1000, 512)[seed]
    toks, *others = tokens_for(cfg, (L, 1, 23, 97), seed=seed)
    for dtype in ("float32", "bfloat16"):
        need = sum(-(-len(t) // 64) * 64 for t in [toks] + others)
        model, cache, runner = engine_parts(d, dtype, page=16, pages=need // 16, slots=4, max_len=1024)
        refs = [Oracle(cfg, w, t, dtype) for t in [toks] + others]
        what = (seed, dtype, json.dumps(cfg)[:900])
        for cuts in ((L,), (L - 40,) + (1,) * 40, (5, 64, 2, 33, 128, 7, 1, 1, 100, 2, 16, 17)):
            got = run_cut(runner, cache, "r", toks, cuts)
            model.ops.check_errors()
            refs[0].check(got, (*what, cuts))
        reqs = dict(zip("abcd", [toks] + others))
        plan = [[("a", 100), ("b", 1)], [("a", 2), ("c", 23)], [("a", 64), ("d", 50)], [("a", 1), ("d", 2)]] + \
               [[("a", 200), ("d", 1)]] * 50
        got = run_mixed(runner, cache, reqs, plan)
        model.ops.check_errors()
        check_all([(ref, got[r]) for r, ref in zip("abcd", refs)], (*what, "mixed"))
