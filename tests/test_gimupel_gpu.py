"""Gimupel on the GPU: every new or extended kernel alone against its plain function, then the model in both dtypes (portions
down to two tokens, unequal batches with pages and slots used again, long decoding across window and page borders,
generation through the entry point and the command line, drawn configurations)."""
import json
import math

import numpy as np
import pytest
import torch

import plain_gimupel as plain
from gimupel_util import CONFIGS, Oracle, check_all, drawn_config, make_dir, plain_logits, rounded, tokens_for
from pepilix_util import run_cut, run_mixed
from test_gizulorn_gpu import Meta, close, paged, scan_portions, shuffled_tables
from fusezap_core_b200 import LLMEngine, SamplingParams
from fusezap_core_b200.cache import CacheManager, KVNeed
from fusezap_core_b200.engine import StepRunner, load_model
from fusezap_core_b200.kernels import cuda_ops

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}
F = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    tmp = tmp_path_factory.mktemp("gimupel")
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
def test_long_decoding_across_window_and_page_borders(dirs, name, dtype):
    d, cfg, w = dirs[name]
    model, cache, runner = engine_parts(d, dtype, page=8, pages=48, slots=2, max_len=384)
    toks = tokens_for(cfg, (340,), seed=23)[0]
    got = run_cut(runner, cache, "long", toks, (21,) + (1,) * 319)
    model.ops.check_errors()
    Oracle(cfg, w, toks, dtype).check(got)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_first_tokens_of_a_sequence(dirs, dtype):
    """Requests of one to six tokens, each alone and all in one step: the convolution's zeros, the empty state, windows that
    are not yet full."""
    for name in CONFIGS:
        d, cfg, w = dirs[name]
        model, cache, runner = engine_parts(d, dtype, slots=6)
        P = tokens_for(cfg, (1, 2, 3, 4, 5, 6), seed=9)
        refs = [plain_logits(cfg, raw(w, dtype), t) for t in P]
        scale = np.sqrt(np.mean([((r - r.mean(-1, keepdims=True)) ** 2).mean() for r in refs]))
        alone = [run_cut(runner, cache, f"r{i}", t, (len(t),)) for i, t in enumerate(P)]
        both = run_mixed(runner, cache, {f"b{i}": t for i, t in enumerate(P)}, [[(f"b{i}", len(t)) for i, t in enumerate(P)]])
        errs = []
        for i, ref in enumerate(refs):
            for got in (alone[i], both[f"b{i}"]):
                e = got - ref
                errs += list(np.sqrt(((e - e.mean(-1, keepdims=True)) ** 2).mean(-1)) / scale)
        assert np.median(errs) < (2e-5 if dtype == "float32" else 3e-2) and max(errs) < (2e-4 if dtype == "float32" else 1.0), (name, max(errs))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_missing_pass_state_or_embedding_would_show(dirs, dtype):
    """What the oracle gives with one mechanism taken out differs from the engine by far more than the limit, for every
    mechanism: so none of them is missing in the engine."""
    d, cfg, w = dirs["mix"]
    model, cache, runner = engine_parts(d, dtype)
    toks = tokens_for(cfg, (90,), seed=2)[0]
    got = run_cut(runner, cache, "r", toks, (40, 2, 1, 1, 16))
    wr = raw(w, dtype)
    ref = Oracle(cfg, w, toks, dtype)
    ref.check(got)
    typical = np.quantile(ref.errors(got), 0.9)
    keep = {k: getattr(plain, k) for k in ("order_of_layers", "rms", "window_mask", "route", "layer_norm", "gated_norm", "expert")}
    broken = {
        "order_of_layers": lambda c: [(i, False) for i, _ in keep["order_of_layers"](c)],
        "window_mask": lambda T, s: keep["window_mask"](T, s + 1),
        "route": lambda z, c, *a: keep["route"](z, c * 0, *a),
        "layer_norm": lambda x, v, eps: plain.rms(x, eps) * v,
        "gated_norm": lambda y, z, g, eps, v: keep["gated_norm"](y, z, 1, eps, v),
        "expert": lambda v, p, h, limit: keep["expert"](v, p, h, 1e9),
    }
    for name, fn in broken.items():
        try:
            setattr(plain, name, fn)
            ref.logits = plain_logits(cfg, wr, toks)
            assert np.quantile(ref.errors(got), 0.9) > 2.5 * typical + 1e-3, (name, typical)
        finally:
            setattr(plain, name, keep[name])


# ---------------------------------------------------------------------------------------- the state-space scan alone
def ssd_inputs(T, H, G, P, N, dt, seed):
    g = torch.Generator().manual_seed(seed)
    xbc = torch.randn(T, H * P + 2 * G * N, generator=g).to(dt)
    proj = torch.randn(T, H + 7, generator=g) * 1.5
    bias, a_log, skip = torch.randn(H, generator=g) - 1.0, torch.linspace(-6.0, 2.0, H) if H > 1 else torch.tensor([-1.0]), torch.randn(H, generator=g)
    return xbc, proj, bias, a_log, skip


def ssd_reference(xbc, proj, off, H, G, P, N, bias, a_log, skip):
    T, v = xbc.shape[0], xbc.to(F)
    x, B, C = v[:, :H * P].reshape(T, H, P), v[:, H * P: H * P + G * N].reshape(T, G, N), v[:, H * P + G * N:].reshape(T, G, N)
    d = plain.softplus(proj[:, off: off + H].to(F) + bias.to(F))
    y, S = plain.ssd_recurrence_fast(x, B, C, d, a_log.to(F), skip.to(F))
    return y.reshape(T, H * P), S


def run_scan(ops, inputs, T, H, G, P, N, steps, off, pad=1):
    """Two sequences through `ssd_scan` in the given steps; slots 1 and 3 of four, slot 2 must stay as it is."""
    state = torch.zeros(4, *ops.recurrent_state_shape(H, N, P), device=DEV)
    state[2] = 3.0
    got = [torch.zeros(T, H * P) for _ in range(2)]
    _, _, bias, a_log, skip = inputs[0]
    for step in steps:
        meta = Meta([(n, at, (1, 3)[r]) for r, at, n in step], pad=pad)
        meta.max_portion = max(n for _, _, n in step)
        rows = lambda k: torch.cat([inputs[r][k][at: at + n] for r, at, n in step] + [torch.zeros(pad, *inputs[0][k].shape[1:], dtype=inputs[0][k].dtype)]).to(DEV)
        out = torch.full((meta.n_rows, H * P), 7.0, device=DEV)
        ops.ssd_scan(rows(0), H, G, N, P, rows(1), off, bias.to(DEV), a_log.to(DEV), skip.to(DEV), state, meta, out)
        ops.check_errors()
        k = 0
        for r, at, n in step:
            got[r][at: at + n] = out[k: k + n].cpu()
            k += n
    assert float(state[2].min()) == 3.0 == float(state[2].max()) and float(state[0].abs().max()) == 0.0
    return got, state


SSD_SIZES = [(6, 3, 12, 20), (3, 1, 20, 9), (8, 4, 5, 40), (5, 5, 8, 130), (2, 1, 64, 128), (4, 2, 64, 64), (1, 1, 7, 256), (2, 2, 48, 32),
             (3, 1, 16, 16), (2, 1, 80, 48), (2, 1, 128, 96), (1, 1, 32, 240)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,P,N", SSD_SIZES)
def test_scan_carries_its_state_across_portions(dtype, H, G, P, N):
    """Portions down to one token, interleaved, heads that hardly forget and heads that forget at once, a row of padding, a
    slot nobody uses; blocks of few and of many threads leave the same bits."""
    import fusezap_core_b200.kernels.table as table
    ops, T = cuda_ops(dtype), 70
    inputs = []
    for r in range(2):
        one = ssd_inputs(T, H, G, P, N, DT[dtype], seed=H * N + r)
        inputs.append(one if not inputs else (*one[:2], *inputs[0][2:]))
    steps = scan_portions(T, seed=H + N)
    refs = [ssd_reference(*i[:2], 4, H, G, P, N, *i[2:]) for i in inputs]
    outs = []
    keep = table.SSD_SPREAD_ROWS
    try:
        for rows in (1, 1 << 30):
            table.SSD_SPREAD_ROWS = rows
            got, state = run_scan(ops, inputs, T, H, G, P, N, steps, 4)
            outs.append(got)
            for r in range(2):
                close(got[r], refs[r][0], "float32" if dtype == "float32" else "bfloat16", f"request {r}")
                S = state[(1, 3)[r]][:, :, :N].transpose(1, 2).cpu().to(F)
                assert (S - refs[r][1]).abs().max() < 3e-5 * (1 + refs[r][1].abs().max())
    finally:
        table.SSD_SPREAD_ROWS = keep
    if not (dtype == "bfloat16"):
        assert all(torch.equal(a, b) for a, b in zip(*outs))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("H,G,P,N", SSD_SIZES)
def test_scan_of_long_portions(dtype, H, G, P, N):
    """Portions of hundreds of tokens around multiples of 64, two requests beside each other, then single tokens from the
    state they left; a result 32-bit close to the plain recurrence although x, B and C are 16-bit in bfloat16."""
    ops, T = cuda_ops(dtype), 421
    inputs = []
    for r in range(2):
        one = ssd_inputs(T, H, G, P, N, DT[dtype], seed=3 * H + N + r)
        inputs.append(one if not inputs else (*one[:2], *inputs[0][2:]))
    steps = [[(0, 0, 200), (1, 0, 64)], [(0, 200, 1), (1, 64, 129)], [(1, 193, 63)], [(0, 201, 220), (1, 256, 2)], [(1, 258, 163)]]
    refs = [ssd_reference(*i[:2], 2, H, G, P, N, *i[2:]) for i in inputs]
    got, state = run_scan(ops, inputs, T, H, G, P, N, steps, 2, pad=3)
    if dtype == "bfloat16":      # without the tensor-core kernel the same within rounding
        ops.ssd_tensor_cores = False
        try:
            slow, _ = run_scan(ops, inputs, T, H, G, P, N, steps, 2, pad=3)
        finally:
            ops.ssd_tensor_cores = True
        assert max(float((a - b).abs().max() / b.abs().max()) for a, b in zip(got, slow)) < 3e-5
        if N % 16 == 0 and P % 16 == 0:
            assert not torch.equal(got[0], slow[0])      # (two kernels did run)
    for r in range(2):
        ref = refs[r][0]
        err = (got[r].to(F) - ref).abs()
        assert not (err > 3e-5 * (ref.abs() + ref.abs().max())).any(), (r, float((err / ref.abs().max()).max()))
        S = state[(1, 3)[r]][:, :, :N].transpose(1, 2).cpu().to(F)
        assert (S - refs[r][1]).abs().max() < 3e-5 * (1 + refs[r][1].abs().max())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_single_token_is_remembered_for_hundreds_of_tokens_and_decays_as_it_should(dtype):
    """x is zero except at one token (the first, one at a chunk's border, one in the middle): every later output is that
    token's value times the product of the decays, for a slow, a medium and a fast head, in one portion, in portions, and
    token by token at the end. A lost or doubled state at any border would show at once."""
    ops, T, H, G, P, N = cuda_ops(dtype), 700, 3, 1, 16, 32
    g = torch.Generator().manual_seed(0)
    b = torch.randn(N, generator=g).to(DT[dtype])
    proj = torch.full((T, H), -4.0)
    bias, a_log, skip = torch.zeros(H), torch.tensor([-4.0, -1.5, 3.0]), torch.zeros(H)
    d = math.log1p(math.exp(-4.0))
    for j in (0, 63, 64, 300):
        xbc = torch.zeros(T, H * P + 2 * N, dtype=DT[dtype])
        xbc[j, :H * P] = 2.0
        xbc[:, H * P: H * P + N] = b
        xbc[:, H * P + N:] = b
        dot = float((b.to(F) ** 2).sum())
        ages = torch.arange(T, dtype=F) - j
        want = torch.stack([torch.where(ages >= 0, torch.exp(-math.exp(float(a)) * d * ages) * d * dot * 2.0, torch.zeros((), dtype=F)) for a in a_log], 1)
        for steps in ([[(0, 0, T)]], [[(0, at, min(100, T - at))] for at in range(0, T, 100)],
                      [[(0, 0, 310)]] + [[(0, at, 1)] for at in range(310, 330)] + [[(0, 330, 370)]]):
            got, _ = run_scan(ops, [(xbc, proj, bias, a_log, skip)] * 2, T, H, G, P, N, steps, 0)
            y = got[0].view(T, H, P).to(F)
            assert ((y - want[:, :, None]).abs() <= 2e-4 * want[:, :, None] + 1e-6 * dot).all(), (j, len(steps))


# ---------------------------------------------------------------------------------------- its convolution and norm
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("C,taps,off,width", [(48, 4, 24, 80), (40, 2, 8, 48), (7, 5, 3, 13), (256, 3, 0, 256), (33, 1, 5, 40), (64, 8, 64, 136), (24, 7, 16, 41)])
def test_convolution_over_columns_of_a_wider_product(dtype, C, taps, off, width):
    """Portions and single tokens, interleaved; with the state moved on in the convolution's own launch where the step has
    single tokens only, the same bits as with the launch of its own."""
    ops, g, T, dt = cuda_ops(dtype), torch.Generator().manual_seed(C), 40, DT[dtype]
    x = [torch.randn(T, width, generator=g) for _ in range(2)]
    w, b = torch.randn(C, taps, generator=g).to(dt), torch.randn(C, generator=g)
    outs = []
    for inline in (False, True):
        state = torch.zeros(3, taps - 1, C, device=DEV) if taps > 1 else None
        got = [torch.zeros(T, C, dtype=dt) for _ in range(2)]
        steps = scan_portions(24, seed=taps) + [[(0, t, 1), (1, t, 1)] for t in range(24, T)]
        for step in steps:
            meta = Meta([(n, at, (2, 0)[r]) for r, at, n in step], pad=1)
            meta.portion_tiles = max(n for _, _, n in step) if inline else 0
            rows = torch.cat([x[r][at: at + n] for r, at, n in step] + [torch.zeros(1, width)]).to(DEV)
            out = torch.full((meta.n_rows, C), 7.0, dtype=dt, device=DEV)
            ops.short_conv(rows, w.to(DEV), state, meta, out, False, "silu", bias=b.to(DEV), offset=off)
            assert float(out[-1].float().abs().max()) == 0.0
            k = 0
            for r, at, n in step:
                got[r][at: at + n] = out[k: k + n].cpu()
                k += n
        outs.append(got)
        for r in range(2):
            ref = plain.silu(plain.causal_conv(x[r][:, off: off + C].to(F), w.to(F), b.to(F)))
            close(got[r], ref, dtype, f"request {r}")
            if taps > 1:
                assert torch.equal(state[(2, 0)[r]].cpu(), x[r][T - taps + 1:, off: off + C])
    assert all(torch.equal(a, b) for a, b in zip(*outs))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("wide", [True, False])
@pytest.mark.parametrize("taps", [2, 3, 4])
def test_convolution_of_steps_of_hundreds_of_rows(dtype, wide, taps):
    """Portions whose borders fall anywhere among the rows that one thread takes, with single tokens and padding between
    them: the same bits as the rows of small steps."""
    ops, g, dt, C, T = cuda_ops(dtype), torch.Generator().manual_seed(taps), DT[dtype], 72, 330
    width = 96 if wide else C
    off = 16 if wide else None
    tin = torch.float32 if wide else dt
    x = [torch.randn(T, width, generator=g).to(tin) for _ in range(3)]
    w, b = torch.randn(C, taps, generator=g).to(dt), torch.randn(C, generator=g)
    outs = []
    for steps in ([[(0, 0, 201), (1, 0, 1), (2, 0, 102)], [(0, 201, 129), (1, 1, 3), (2, 102, 228)], [(1, 4, 326)]],
                  [[(r, at, min(50, T - at)) for r in range(3)] for at in range(0, T, 50)]):
        state = torch.zeros(5, taps - 1, C, device=DEV)
        got = [torch.zeros(T, C, dtype=dt) for _ in range(3)]
        for step in steps:
            meta = Meta([(n, at, (2, 0, 4)[r]) for r, at, n in step], pad=3)
            rows = torch.cat([x[r][at: at + n] for r, at, n in step] + [torch.zeros(3, width, dtype=tin)]).to(DEV)
            out = torch.full((meta.n_rows, C), 7.0, dtype=dt, device=DEV)
            kw = {"offset": off} if wide else {}
            ops.short_conv(rows, w.to(DEV), state, meta, out, not wide, "silu", bias=b.to(DEV), **kw)
            assert float(out[-3:].float().abs().max()) == 0.0
            k = 0
            for r, at, n in step:
                got[r][at: at + n] = out[k: k + n].cpu()
                k += n
        outs.append(got)
    for r in range(3):
        xr = (x[r][:, off: off + C] if wide else x[r]).to(F)
        close(outs[0][r], plain.silu(plain.causal_conv(xr, w.to(F), b.to(F)) + (0 if wide else xr)), dtype, f"request {r}")
        assert torch.equal(outs[0][r], outs[1][r])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("parts,size,off,extra", [(4, 20, 0, 0), (1, 384, 8, 24), (3, 7, 2, 5), (2, 2048, 0, 64), (1, 4500, 4, 4), (5, 1, 0, 3), (1, 20000, 0, 0), (8, 130, 0, 2)])
def test_norm_in_parts_with_the_gate_first(dtype, parts, size, off, extra):
    ops, g, n = cuda_ops(dtype), torch.Generator().manual_seed(size), 9
    width = parts * size
    y = torch.randn(n, width, generator=g) * torch.rand(n, 1, generator=g) * 3
    y[:, : size] *= 30.0            # one part is much louder than the others: its norm must not touch theirs
    gate = torch.randn(n, off + width + extra, generator=g) * 2
    w = torch.rand(width, generator=g) + 0.5
    ops._meta_rows = torch.tensor([0] * (n - 1) + [-1], dtype=torch.int32, device=DEV)
    out = torch.full((n, width), 7.0, dtype=DT[dtype], device=DEV)
    ops.head_norm_gate(y.to(DEV), parts, size, w.to(DEV), 1e-5, gate.to(DEV), off, "silu", out, gate_first=True)
    ref = plain.gated_norm(y.to(F), gate[:, off: off + width].to(F), parts, 1e-5, w.to(F))
    close(out[: n - 1], ref[: n - 1], dtype)
    assert float(out[n - 1].float().abs().max()) == 0.0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("D", [64, 200, 1030, 7, 2048, 4096, 9000])
def test_layer_norm_with_the_pending_term_and_the_added_stream(dtype, D):
    """Rows with a mean far above their spread (a variance taken as a difference of squares would be lost), the pending
    term and the other stream joined in the same pass, selected rows."""
    from fusezap_core_b200.parts import PendingSum
    from fusezap_core_b200.parts.norm import LayerNorm
    from fusezap_core_b200.engine.step import StepContext, Workspace
    ops, g = cuda_ops(dtype), torch.Generator().manual_seed(D)
    norm = LayerNorm(D, 1e-5, name="w")
    w = torch.randn(D, generator=g)
    norm.bind({"w": w.to(DEV)}, ops)
    x, delta, extra = (torch.randn(9, D, generator=g) for _ in range(3))
    x[3] += 300.0
    x[4] *= 1e-3
    ctx = StepContext(ops, Workspace(torch.device(DEV), 9), Meta([(9, 0, -1)]), {}, None)
    for d, e in ((delta, extra), (delta, None), (None, extra), (None, None)):
        xd = x.to(DEV)
        up = lambda t: None if t is None else t.to(DEV)
        h = norm.forward(ctx, xd, PendingSum(up(d), up(e)) if e is not None else up(d))
        full = x + (d if d is not None else 0)
        full = full + (e if e is not None else 0)
        assert torch.equal(xd.cpu(), full)
        ref = plain.layer_norm(full.to(F), w.to(F), 1e-5)
        lim = torch.full((9, 1), 3e-6 if dtype == "float32" else 2.0 ** -8, dtype=F)
        lim[3] += 3e-4            # (300 in 32-bit leaves an absolute error of 3e-5 in every deviation)
        assert ((h.cpu().to(F) - ref).abs() <= lim * (1 + ref.abs())).all()
    rows = torch.tensor([7, -1, 0], dtype=torch.int32, device=DEV)
    xd = x.to(DEV)
    h = norm.forward(ctx, xd, delta.to(DEV), rows=rows)
    assert torch.equal(xd.cpu(), x) and float(h[1].float().abs().max()) == 0.0
    close(h[[0, 2]], plain.layer_norm((x + delta)[[7, 0]].to(F), w.to(F), 1e-5), dtype)


def test_the_gather_writes_its_copy():
    g = torch.Generator().manual_seed(0)
    for D, dt in ((64, torch.bfloat16), (36, torch.float32), (7, torch.bfloat16)):
        ops = cuda_ops("bfloat16")
        table = torch.randn(11, D, generator=g).to(dt).to(DEV)
        tok = torch.tensor([3, 0, 10, 3], dtype=torch.int32, device=DEV)
        x, c = torch.zeros(4, D, device=DEV), torch.zeros(4, D, device=DEV)
        ops.embed(table, tok, x, None, None, 1.7, copy=c)
        ops.check_errors()
        assert torch.equal(x, c) and torch.equal(x.cpu(), table[tok.long()].float().cpu() * torch.tensor(1.7))


# ---------------------------------------------------------------------------------------- attention
def windowed_rows(dtype, Hq, Hkv, dk, dv, window, T, portions, page, seed, loud=None, scale=0.8):
    """One sequence of T tokens in shuffled pages; `portions` ((rows, first position) each) are asked for in one step. The
    queries and keys go through the kernel that norms the heads. loud: (key position, share): that key and every query
    point one way, so that its score stands out however the vectors are scaled."""
    ops, g, dt = cuda_ops(dtype), torch.Generator().manual_seed(seed), DT[dtype]
    q, k = (torch.randn(T, h, dk, generator=g) * (0.1 + 5 * torch.rand(T, h, 1, generator=g)) for h in (Hq, Hkv))
    v = torch.randn(T, Hkv, dv, generator=g)
    if loud is not None:
        way = torch.nn.functional.normalize(torch.randn(dk, generator=g), dim=0)
        k[loud] = way * 3.0
        q = q * 0.05 + way * 2.0
    pages = -(-T // page)
    table = shuffled_tables(1, pages, pages + 5, seed)
    cache = paged(KVNeed(Hkv, dk, window, value_dim=dv), page, pages + 5, dtype)
    qkv = torch.cat([q.view(T, -1), k.view(T, -1), v.view(T, -1)], 1).float().to(DEV)
    ones, qn = torch.ones(dk, device=DEV), torch.empty(T, Hq * dk, dtype=dt, device=DEV)
    ops.rotate_kv_write(qkv, None, None, 0, 0, Meta([(T, 0, 0)], table), cache, qn, Hq, Hkv, dk, dv, q_norm=ones, k_norm=ones, norm_eps=1e-6)
    meta = Meta([(n, p0, 0) for n, p0 in portions], table.repeat(len(portions), 1), pad=1)
    meta.max_portion = max(n for n, _ in portions)
    rows = [p for n, p0 in portions for p in range(p0, p0 + n)]
    qs = torch.cat([qn[rows], torch.zeros(1, Hq * dk, dtype=dt, device=DEV)]).contiguous()
    out = torch.empty(len(rows) + 1, Hq * dv, dtype=dt, device=DEV)
    ops.sink_attention(qs, cache, meta, out, Hq, Hkv, dk, dv, scale, window, 0, None)
    ops.check_errors()
    assert float(out[-1].float().abs().max()) == 0.0
    rep = Hq // Hkv
    qf, kf = (plain.rms(t.to(F), 1e-6) for t in (q, k))
    assert (qn.view(T, Hq, dk).cpu().to(F) - qf).abs().max() < (1e-5 if dtype == "float32" else 0.05)
    if dtype == "bfloat16":      # the oracle starts from what the kernels hold: normed, rounded once
        qf, kf, v = qf.float().to(dt).to(F), kf.float().to(dt).to(F), v.to(dt)
    ref = plain.masked_attention_fast(qf, kf.repeat_interleave(rep, 1), v.to(F).repeat_interleave(rep, 1), scale, plain.window_mask(T, window))
    return out[:-1].view(len(rows), Hq, dv), ref[rows], v


def near(got, ref, dtype, what=None, largest_score=100.0):
    """(a score of some hundred has an error of some 1e-5 in 32-bit, and so have its exponential and the result)"""
    err, ref = (got.detach().cpu().to(F) - ref).abs(), ref.to(F)
    tol = 1e-7 * largest_score if dtype == "float32" else 2.0 ** -6
    assert not (err > tol * (ref.abs() + 2 * ref.abs().mean() + 1e-3)).any(), (what, float(err.max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("Hq,Hkv,dk,dv,window", [(4, 2, 16, 8, 9), (3, 3, 24, 40, 300), (8, 2, 80, 48, 88), (6, 3, 64, 64, 33),
                                                 (4, 4, 128, 128, 70), (2, 1, 128, 128, 64), (1, 1, 32, 16, 1), (6, 1, 64, 64, 100)])
def test_windowed_attention_of_normed_heads(dtype, Hq, Hkv, dk, dv, window):
    got, ref, _ = windowed_rows(dtype, Hq, Hkv, dk, dv, window, T=200, page=4, seed=Hq * dk + window,
                                portions=[(70, 0), (2, 80), (1, 97), (1, 199), (1, 5), (90, 100)])
    near(got, ref, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("as_portion", [True, False])
@pytest.mark.parametrize("dk,dv,window", [(16, 8, 12), (64, 64, 96), (80, 48, 33), (128, 128, 70), (64, 64, 64), (24, 24, 1)])
def test_a_loud_key_is_seen_exactly_inside_the_window(dtype, as_portion, dk, dv, window):
    """One key's score exceeds all others by far, so a row's output is that key's value if the row sees the key: keys at
    position 0, at page borders and in the middle; rows just inside and just outside the window, in prompt portions and
    as single tokens."""
    page, T = 8, 300
    for j in (0, 7, 8, 100, 127, 128):
        rows = sorted({p for p in (j, j + 1, j + window - 2, j + window - 1, j + window, j + window + 1, T - 1) if j <= p < T})
        portions = [(r - max(0, r - 69) + 1, max(0, r - 69)) for r in rows] if as_portion else [(1, p) for p in rows]
        got, ref, v = windowed_rows(dtype, 2, 1, dk, dv, window, T, portions, page, seed=j, loud=j, scale=4.0)
        near(got, ref, dtype, f"key {j}", 4.0 * max(dk, 25))
        at = 0
        for n, p0 in portions:
            for p in range(p0, p0 + n):
                if p in rows and p >= j:
                    same = bool((got[at].float().cpu() - v[j].float()).abs().max() < 0.1)
                    assert same == (p - j < window) or window == 1, (j, p)
                at += 1


# ---------------------------------------------------------------------------------------- the router and the experts
@pytest.mark.parametrize("E,top,groups,keep", [(8, 3, 4, 2), (6, 2, 3, 2), (7, 3, 7, 4), (1, 1, 1, 1), (12, 8, 3, 2), (16, 4, 1, 1), (256, 8, 8, 4),
                                               (64, 6, 64, 10), (5, 5, 1, 1), (96, 33, 4, 3), (1500, 2, 2, 1)])
def test_router_with_sigmoid_scores_groups_and_a_correction(E, top, groups, keep):
    """Choice scores on both sides of zero, corrections larger than the differences of the scores; against the plain rule
    row by row, and the softmax rule through the same kernel."""
    from test_gizulorn_gpu import Meta
    ops, g, n = cuda_ops("float32"), torch.Generator().manual_seed(E + top), 37
    z = torch.randn(n, E + 3, generator=g) * 2
    corr = torch.rand(E, generator=g) * 1.5 - 1.2
    meta = Meta([(n - 1, 0, -1)], pad=1)
    w = torch.full((n, top), 7.0, device=DEV)
    zd = z.to(DEV)
    ops.route_by_scores(zd, E, top, groups, keep, True, meta, w, 1, scoring="sigmoid", correction=corr.to(DEV), group_top=2, sum_eps=1e-20, scale=1.7)
    choice = ops._scratch_bufs["router choices"][: n * top].view(n, top).cpu()
    idx, wt = plain.route(z[: n - 1, :E].to(F), corr.to(F), top, groups, keep, 1.7)
    same = (choice[: n - 1] == idx).all(-1)
    assert same.float().mean() > 0.9            # (choice scores equal to the last 32-bit place may come out either way)
    assert (w[: n - 1].cpu().to(F) - wt)[same].abs().max() < 1e-5 and float(w[n - 1].abs().max()) == 0.0
    for row in choice[: n - 1].tolist():
        assert len(set(row)) == top and max(row) < E and min(row) >= 0
    ops.route_by_scores(zd, E, top, groups, keep, False, meta, w, 1)
    s = torch.softmax(z[: n - 1, :E].to(F), -1)
    gs = s.view(n - 1, groups, -1).max(-1).values
    allowed = torch.zeros_like(gs, dtype=torch.bool).scatter_(1, torch.sort(gs, dim=-1, descending=True, stable=True).indices[:, :keep], True)
    ref = torch.sort(s.masked_fill(~allowed.repeat_interleave(E // groups, 1), -1.0), dim=-1, descending=True, stable=True).values[:, :top]
    assert (w[: n - 1].cpu().to(F) - ref).abs().max() < 1e-6


def test_router_ties_go_to_the_lower_index():
    ops = cuda_ops("float32")
    z = torch.zeros(2, 8, device=DEV)
    meta, w = Meta([(2, 0, -1)]), torch.empty(2, 3, device=DEV)
    ops.route_by_scores(z, 8, 3, 4, 2, True, meta, w, 1, scoring="sigmoid", correction=torch.full((8,), -0.9, device=DEV), group_top=2, scale=3.0)
    assert ops._scratch_bufs["router choices"][:6].cpu().tolist() == [0, 1, 2] * 2
    assert torch.allclose(w.cpu(), torch.ones(2, 3))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("E,top,I,groups,keep,limit,n", [(6, 2, 24, 3, 2, 0.7, 40), (1, 1, 40, 1, 1, 7.0, 7), (8, 8, 8, 4, 4, 0.1, 300), (10, 3, 80, 5, 3, 1.0, 1),
                                                         (4, 1, 64, 2, 1, 2.5, 130)])
def test_experts_with_clamped_gates(dtype, E, top, I, groups, keep, limit, n):
    """A limit that most values exceed and one that few do; the product with u + 1; groups and correction."""
    from fusezap_core_b200.parts.routed_moe import RoutedMoE
    from fusezap_core_b200.engine.step import StepContext, Workspace
    ops, g, dt, D = cuda_ops(dtype), torch.Generator().manual_seed(E * I), DT[dtype], 64
    names = {"router": "router", "correction": "correction", "expert": "e{}", "gate": "gate", "up": "up", "down": "down"}
    ff = RoutedMoE(D, I, E, top, groups, keep, renormalize=True, scoring="sigmoid", correction=True, group_score="top2", sum_eps=1e-20,
                   weight_scale=1.3, alpha=1.702, limit=limit, up_shift=1.0, names=names)
    w = {k: torch.randn(p.shape, generator=g) * (0.4 if p.role == "vector" else 0.25) for k, p in ff.tensors().items()}
    w = {k: v.to(dt).float() if v.dim() >= 2 else v for k, v in w.items()}
    ff.bind({k: (v.to(dt) if v.dim() >= 2 else v).to(DEV) for k, v in w.items()}, ops)
    h = torch.randn(n + 1, D, generator=g).to(dt)
    ctx = StepContext(ops, Workspace(torch.device(DEV), n + 1), Meta([(n, 0, -1)], pad=1), {}, None)
    out = ff.forward(ctx, h.to(DEV))
    ops.check_errors()
    mlp = {"router": {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "scale": 1.3}, "expert": {"limit": limit}}
    ref = plain.mixture({k: v.to(F) for k, v in w.items()}, "", mlp, h[:n].to(F))
    err = (out[:n].cpu().to(F) - ref).abs().max(-1).values / ref.abs().max()
    # (a row whose choice scores nearly tie may choose otherwise in bfloat16)
    assert float(err.median()) < (1e-5 if dtype == "float32" else 2e-2) and float((err > 0.1).float().mean()) < 0.1
    assert float(out[n].abs().max()) == 0.0


# ------------------------------------------------------------------------------------------------ the model, further
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mix", "odd"])
def test_greedy_generation_through_the_entry_point(dirs, dtype, name):
    """Through `LLMEngine` and its scheduler (portions of prompts beside decoding requests, more requests than state
    slots, a pool that does not hold all requests at once, captured decode steps): every generated token is the plain
    model's choice, or within rounding of it."""
    d, cfg, w = dirs[name]
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
    assert main(["generate", "--random", "tiny-gimupel", "--prompt-lens", "5,40,1", "--max-tokens", "6", "--ignore-eos",
                 "--max-model-len", "128", "--num-blocks", "32", "--max-num-seqs", "2"]) == 0
    lines = [json.loads(x) for x in capsys.readouterr().out.splitlines() if x.startswith("{")]
    assert [o["num_prompt_tokens"] for o in lines] == [5, 40, 1]
    assert all(len(o["token_ids"]) == 6 and o["finish_reason"] == "length" for o in lines)


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
