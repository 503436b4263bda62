"""Muretar through the trace replay program on the GPU: a `bin/trace_run` process replays the same requests whole, with
their last 32 tokens one by one, in portions down to two tokens, and four at a time in a pool so small that pages and
state slots are used again; every position is compared with the plain model's logits of the whole request, and in
float32 the cuttings must agree with each other bit for bit (every sum's order is a function of the row alone).

The small configurations are those of `muretar_util`; the larger one has layer sizes of a few hundred that reach the
tensor-core products, the tensor-core attention and the long-portion scans, a bfloat16 checkpoint and requests of up to
1,300 tokens, replayed by a small scheduler in a pool that does not hold all requests."""
import numpy as np
import pytest
import torch

from gimupel_util import check_all
from muretar_util import CONFIGS, Oracle, att, dense, gla, layer, left, make_dir, model, moe, par, right, tokens_for
from test_replay_gpu import LENGTHS, POOL_TOKENS, build_trace
from util import TraceBuilder, run_trace

pytestmark = pytest.mark.gpu


def _compare(got: dict, ref_of, refs, what: str) -> None:
    """The rows of each cutting together (the ids' first letters)."""
    kinds: dict = {}
    for rid, rows in sorted(got.items()):
        ref = refs[ref_of(rid)]
        assert sorted(rows) == list(range(len(ref.logits))), f"{what} {rid}: positions {sorted(rows)[:5]}..."
        kinds.setdefault(rid[0], []).append((ref, np.stack([rows[p] for p in range(len(ref.logits))])))
    for kind, pairs in kinds.items():
        check_all(pairs, (what, kind))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_replay_all_cuttings(name, dtype, tmp_path):
    d, cfg, w = make_dir(name, tmp_path)
    P = tokens_for(cfg, LENGTHS, seed=3)
    refs = [Oracle(cfg, w, ids, dtype) for ids in P]
    tb = build_trace(P)
    assert tb.most_live == 4 and max(len(s["entries"]) for s in tb.steps) == 4
    outs = run_trace(d, dtype, str(tmp_path / "out"), max_tokens=POOL_TOKENS, steps=tb.steps)
    got = tb.collect(outs, cfg["vocab"])
    assert {r[0] for r in got} == {"w", "d", "p", "m"}
    if dtype == "float32":
        for rid, rows in sorted(got.items()):
            if rid[0] == "w":
                continue
            whole = got["w" + rid[1:]]
            for p, row in rows.items():
                assert np.array_equal(row, whole[p]), (f"{name}: request {rid} position {p} differs from the whole "
                                                       f"request's row by {np.abs(row - whole[p]).max():.3e}")
    _compare(got, lambda rid: int(rid[1:]), refs, name)


LARGER = model(512, 384, 1e-5, [
    layer(par(left(6, 2, 64, 64, 0.1, 3e4, 48, 2.0), right(4, 2, 48, 80, 4)), moe(9, 3, 3, 96, 160)),
    layer(gla(4, 64, 96, 9.0), dense(448)),
    layer(att(6, 3, 32, 64, 0.15, 0.35), moe(6, 1, 2, 128, 64)),
    1,
    layer(att(3, 1, 64, 128, 0.1, 0.75), None),
    layer(par(left(4, 1, 128, 64, 0.08, 8e5, 128), right(3, 3, 64, 32, 2)), dense(200)),
    2,
])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_a_larger_model_with_long_requests_in_a_small_pool(dtype, tmp_path):
    d, cfg, w = make_dir("larger", tmp_path, LARGER, 11, dtype="bfloat16")
    assert w["embed"].dtype == torch.bfloat16
    lengths = (1300, 260, 1, 23, 333, 97)
    P = dict(zip("abcdef", tokens_for(cfg, lengths, seed=5)))
    refs = {r: Oracle(cfg, w, ids, dtype) for r, ids in P.items()}
    # a little scheduler: up to four live; portions of changing size, then each request's last tokens one by one
    rng = np.random.default_rng(8)
    tb, waiting, live, peak = TraceBuilder(), list(P), {}, 0
    single = {r: max(0, len(P[r]) - int(rng.integers(8, 140))) for r in P}
    while waiting or live:
        while waiting and len(live) < 4 and (not live or rng.random() < 0.7):
            live[waiting.pop(0)] = 0
        peak = max(peak, sum(-(-len(P[r]) // 64) * 64 for r in live))
        entries, ends = [], []
        for r in list(live):
            if rng.random() < 0.2 and len(live) > 1:
                continue
            at = live[r]
            n = 1 if at >= single[r] else min(int(rng.choice([2, 3, 5, 16, 17, 64, 100, 200])), single[r] - at)
            entries.append((r, P[r][at: at + n], "all"))
            live[r] = at + n
            if live[r] == len(P[r]):
                ends.append(r)
                del live[r]
        if entries:
            tb.step(entries, end=ends)
    assert max(len(s["entries"]) for s in tb.steps) == 4 and peak < sum(-(-n // 64) * 64 for n in lengths)
    outs = run_trace(d, dtype, str(tmp_path / "out"), max_tokens=peak, steps=tb.steps)
    _compare(tb.collect(outs, cfg["vocab"]), lambda rid: rid, refs, "larger")
