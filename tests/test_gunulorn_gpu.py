"""Gunulorn on the GPU against the plain restatement (f64, whole sequences): each mechanism, every way of cutting a sequence into
rounds, shared batches, pages and state slots used again, single keys, edges of windows and kept tokens, generation through the engine."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import gunulorn_models as M
import gunulorn_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = 1, 2
LAYERS = {"conv": M.conv(), "window": M.window(), "dense": M.window(mlp=M.dense())}


@pytest.fixture(autouse=True)
def default_tuning(L):
    yield
    for k, v in (("stack_pdl", 1), ("stack_fork", 1), ("stack_tc", 1), ("tc_block", 256), ("tc_cluster", 1)):
        L.set_tuning(k, v)


def check(got, want, dt, what="", tol=None):
    e, tol = M.rel_err(got, want), tol or M.TOL[dt]
    assert e <= tol, f"{what}: error {e:.3g} > {tol:.3g}"
    return e


def every_cut(L, raw, w, toks, dt, cuts, want=None, **kw):
    """Whole and in portions of the given sizes, against the restatement."""
    want = M.reference(raw, w, toks) if want is None else want
    tol = M.tolerance(dt, raw, w, toks, want)
    _, ctx = M.load(L, raw, w, dt, **kw)
    r = M.Runner(ctx)
    for c in (None, *cuts):
        check(r.whole(toks, c), want, dt, f"portions {c}", tol)
    assert ctx.device_status() == 0 and ctx.pages_free == ctx.pages_total
    ctx.close()
    return want


def differs(raw, w, toks, want, by=1e-2):
    assert M.rel_err(M.reference(raw, w, toks), want) > by, "the mechanism does not show"


# ------------------------------------------------------------------ mechanisms alone

ALONE = [(kind, off) for kind in ("conv", "window", "dense") for off in ((), ("ff",), ("mixer",))] + [(kind, ("mixer", "experts")) for kind in ("conv", "window")]


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("kind,off", ALONE)
def test_mechanism_alone(L, dt, kind, off):
    raw = M.config([LAYERS[kind]])
    w = M.silence(M.weights(raw, 1), raw, *off)
    toks = M.random_tokens(raw, 70, 2)
    want, stream = M.reference(raw, w, toks, True)
    tol = M.tolerance(dt, raw, w, toks, want)
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    got = r.whole(toks)
    x = ctx.hidden(70).cpu().double()
    assert float((x - stream[-1]).abs().max()) / float(stream[-1].abs().max()) <= (2e-5 if dt == F32 else 3e-2)
    check(got, want, dt, off, tol)
    check(r.whole(toks, [1]), want, dt, f"{off}, decoded", tol)
    ctx.close()


def test_eps_matters_and_is_read(L):
    raw = M.config([M.window(mlp=M.dense()), M.conv()], eps=0.3)
    w = M.weights(raw, 6)
    toks = M.random_tokens(raw, 30, 7)
    want = every_cut(L, raw, w, toks, F32, [[1]])
    differs(dict(raw, norm={"eps": 1e-5}), w, toks, want)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("scale,cap", [(1.0, 1.0), (0.25, 30.0), (7.0, 3.0), (1.0, 100.0)])
def test_scaled_and_capped_logits(L, dt, scale, cap):
    """Rounds of one, a few and many tokens take different kernels for the head."""
    raw = M.config([M.conv(mlp=None)], scale=scale, cap=cap)
    w = M.weights(raw, 8)
    toks = M.random_tokens(raw, 90, 9)
    want = every_cut(L, raw, w, toks, dt, [[1], [2], [3], [4], [5], [20, 40]])
    if dt == F32:
        differs(dict(raw, logit_softcap=2 * cap), w, toks, want, 1e-5)


@pytest.mark.parametrize("rot,vdim", [(2, 2), (6, 10), (14, 30), (20, 64), (0, 28)])
def test_rotations(L, rot, vdim):
    """Rotated parts of every width (none among them), values of every size: pairs that end inside a group of four."""
    raw = M.config([M.window(200, 0, rot=rot, vdim=vdim, base=30.0, scale=0.5, mlp=None)])
    w = M.weights(raw, 8)
    toks = M.random_tokens(raw, 90, 9)
    for dt in (F32, BF16):
        want = every_cut(L, raw, w, toks, dt, [[1], [40, 7]])
    differs(M.config([M.window(200, 0, rot=rot, vdim=vdim, base=900.0, scale=0.5, mlp=None)]), w, toks, want, 1e-3 if vdim > 2 else -1)


@pytest.mark.parametrize("part", ["values", "outputs"])
def test_rotated_values_show(L, part):
    """The restatement without the turn of the values, or without the turn back, comes out differently."""
    raw = M.config([M.window(50, 4, mlp=None)])
    w = M.weights(raw, 10)
    toks = M.random_tokens(raw, 60, 11)
    want = every_cut(L, raw, w, toks, F32, [[1]])
    real = R.turn
    vd = raw["layers"][0]["mixer"]["vdim"]
    R.turn = lambda x, dims, base, sign=1: x if dims == vd and (sign < 0) == (part == "outputs") else real(x, dims, base, sign)
    try:
        differs(raw, w, toks, want)
    finally:
        R.turn = real


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_convolution_taps(L, taps):
    raw = M.config([M.conv(taps, mlp=None), M.conv(taps + 1, kv_from=0, mlp=None)])
    w = M.weights(raw, 10)
    toks = M.random_tokens(raw, 40, 11)
    for dt in (F32, BF16):
        every_cut(L, raw, w, toks, dt, [[1], [2], [3, 1], [8, 7], [4, 9, 1, 1], [16], [17, 2]])


def test_sinks_and_factors_per_head_show(L):
    """The first tokens without the sink of either kind, and without the factors, come out differently; the sink takes no factor."""
    for layer in (M.conv(mlp=None), M.window(mlp=None)):
        raw = M.config([layer])
        w = M.weights(raw, 24)
        if "l0.mix.sink" in w:
            w["l0.mix.sink"] = w["l0.mix.sink"] + 1
        toks = M.random_tokens(raw, 6, 25)
        want = every_cut(L, raw, w, toks, F32, [[1], [2]])
        every_cut(L, raw, w, toks, BF16, [[1], [2]], want)
        real = R.softmax_attention
        try:
            R.softmax_attention = lambda q, k, v, scale, sink, *a: real(q, k, v, scale, sink - 1e9, *a)
            differs(raw, w, toks, want)
            if "l0.mix.sink" in w:
                R.softmax_attention = lambda q, k, v, scale, sink, *a: real(q, k, v, scale, sink * w["l0.mix.temp"], *a)
                differs(raw, w, toks, want, 1e-3)
        finally:
            R.softmax_attention = real
        if "l0.mix.temp" in w:
            differs(raw, dict(w, **{"l0.mix.temp": torch.ones_like(w["l0.mix.temp"])}), toks, want, 1e-3)


def test_scores_far_above_and_below_the_sink(L):
    """Sinks that take everything or nothing, scores of both signs far from zero: nothing overflows."""
    for sink, scale in ((60.0, 1.0), (-60.0, 1.0), (0.5, 60.0)):
        raw = M.config([M.conv(heads=4, kv_heads=4, scale=scale, mlp=None), M.window(heads=2, kv_heads=2, rot=2, scale=scale, mlp=None)])
        w = M.weights(raw, 28)
        w["l0.mix.sink"] = torch.full_like(w["l0.mix.sink"], sink)
        for i in (0, 1):
            for end in ("", ".conv") if i == 0 else ("",):
                w[f"l{i}.mix.k{end}"] = (1 if end else -1) * w[f"l{i}.mix.q{end}"].clone()
        for dt in (F32, BF16):
            assert torch.isfinite(every_cut(L, raw, w, [7] * 20, dt, [[1], [6]])).all()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("ff", [1, 50, 64, 513, 700, 4200, 16500])
def test_normed_powers(L, dt, ff):
    """Every width of the activation kernel; each of the four numbers shows."""
    raw = M.config([M.window(mlp=M.dense(ff))], width=40)
    w = M.weights(raw, 16)
    toks = M.random_tokens(raw, 12, 17)
    want = every_cut(L, raw, w, toks, dt, [[1], [5]])
    for i in range(4):
        act = w["l0.mlp.act"].clone()
        act[i] = -act[i]
        differs(raw, dict(w, **{"l0.mlp.act": act}), toks, want, 1e-3)
    for name in ("up.b", "down.b"):
        differs(raw, dict(w, **{"l0.mlp." + name: torch.zeros_like(w["l0.mlp." + name])}), toks, want, 1e-3)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n", [40, 300])
@pytest.mark.parametrize("mlp", [M.moe(30, 5, 2, 2), M.moe(30, 1, 1, 0), M.moe(64, 2, 2, 0), M.moe(9, 12, 3, 5), M.moe(130, 3, 1, 1), M.moe(16, 34, 7, 8), M.moe(20, 1, 2, 3),
                                 M.moe(20, 3, 5, 2)])
def test_experts(L, dt, n, mlp):
    """One expert to forty, some or all of them, none that return their input to many more than the others; small rounds and large."""
    raw = M.config([M.conv(mlp=mlp), M.window(mlp=mlp)], width=176)
    w = M.weights(raw, 18)
    toks = M.random_tokens(raw, n, 19)
    want = every_cut(L, raw, w, toks, dt, [[1, n - 6, 5], [33], [64], [65]])
    differs(raw, M.silence(w, raw, "experts"), toks, want, 5e-3)


def test_tokens_that_use_no_matrices_at_all(L):
    """Corrections send every token to the experts that return their input, then to the others only."""
    raw = M.config([M.window(mlp=M.moe(30, 3, 2, 4)), M.conv(mlp=M.moe(30, 3, 2, 4))])
    for sign in (3, -3):
        w = M.weights(raw, 20)
        for i in (0, 1):
            c = torch.zeros(7)
            c[3:] = sign
            w[f"l{i}.mlp.correction"] = c.to(torch.bfloat16)
        for dt in (F32, BF16):
            toks = M.random_tokens(raw, 100, 21)
            want = every_cut(L, raw, w, toks, dt, [[1], [70]])
        same = M.rel_err(M.reference(raw, M.silence(w, raw, "experts"), toks), want)
        assert same == 0 if sign > 0 else same > 1e-2


def test_routing_by_random_routers(L):
    """Routers and corrections as they come (32-bit arithmetic: no rounding swaps two experts)."""
    raw = M.config([M.conv(mlp=M.moe(30, 30, 5, 7)), M.window(mlp=M.moe(30, 70, 2, 3)), M.window(mlp=M.moe(30, 3, 2, 1))])
    w = M.weights(raw, 20, steady=False)
    toks = M.random_tokens(raw, 120, 21)
    want = every_cut(L, raw, w, toks, F32, [[1], [50]])
    differs(raw, {k: torch.zeros_like(v) if k.endswith("correction") else v for k, v in w.items()}, toks, want, 1e-3)


@pytest.mark.parametrize("dt", [F32, BF16])
def test_borrowed_keys(L, dt):
    """Two layers read one layer's cache with queries, convolutions, sinks, factors, scales and head ratios of their own."""
    raw = M.config([M.window(mlp=None), M.conv(3, mlp=None), M.conv(5, kv_from=1, scale=0.6, mlp=None), M.window(mlp=None), M.conv(2, heads=2, kv_from=1, mlp=None), M.conv(mlp=None)])
    w = M.weights(raw, 22)
    toks = M.random_tokens(raw, 160, 23)
    every_cut(L, raw, w, toks, dt, [[1], [64], [100, 1, 2]])


# ------------------------------------------------------------------ sizes

SIZES = {
    "ones": M.config([M.conv(1, 1, 1, 1, 1, 1.0, mlp=M.moe(1, 1, 1, 1)), M.window(1, 1, 1, 1, 2, 2, 2, 10.0, 1.0, mlp=M.dense(1))], width=8, vocab=7, scale=1.0, cap=1.0),
    "large_heads": M.config([M.conv(4, 3, 1, 256, 200, 0.06), M.window(40, 17, 2, 2, 130, 256, 64, 1e4, 0.1), M.window(100, 9, 3, 1, 256, 130, 256, 1e4, 0.06, mlp=M.dense(300))],
                            width=136, vocab=150),
    "wide_groups": M.config([M.conv(3, 40, 1, 16, 16, 0.5), M.window(33, 70, 66, 1, 12, 8, 4, 1e3, 0.5), M.window(20, 5, 34, 2, 16, 16, 16, 1e3, 0.5)], width=96, vocab=64),
    "many_key_heads": M.config([M.conv(4, 12, 12, 64, 128, 0.2), M.window(64, 64, 16, 16, 64, 64, 64, 1e4, 0.2)], width=128, vocab=96),
    "usual": M.config([M.window(100, 16, 8, 2, 128, 128, 64, 5e5, 128 ** -0.5, mlp=M.dense(900)), M.conv(4, 8, 2, 128, 128, 128 ** -0.5, mlp=M.moe(300, 8, 2, 2)),
                       M.window(100, 16, 8, 2, 128, 128, 64, 5e5, 128 ** -0.5, mlp=M.moe(300, 8, 2, 2))], width=200, vocab=333),
    "wide": M.config([M.conv(mlp=M.moe(700, 4, 2, 1)), M.window(mlp=M.dense(1500))], width=1032, vocab=333),
    "wider": M.config([M.window(heads=2, mlp=M.dense(90))], width=4200, vocab=33),
    "windows_only": M.config([M.window(50), M.window(7, 3, mlp=None)]),
    "first_without_feed_forward": M.config([M.conv(mlp=None), M.window(), M.conv(mlp=None)]),
    "mixed": M.MIXED,
}


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(L, name, dt):
    raw = SIZES[name]
    w = M.weights(raw, 11)
    every_cut(L, raw, w, M.random_tokens(raw, 150, 12), dt, [[120] + [1] * 30, [2, 64, 3, 17]])


# ------------------------------------------------------------------ schedules

@pytest.fixture(scope="module")
def mixed():
    raw = M.MIXED
    w = M.weights(raw, 21)
    toks = M.random_tokens(raw, 200, 22)
    want = M.reference(raw, w, toks)
    return raw, w, toks, want, {dt: M.tolerance(dt, raw, w, toks, want) for dt in (F32, BF16)}


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("page_tokens", [64, 8, 128])
def test_portions(L, mixed, dt, page_tokens):
    raw, w, toks, want, tol = mixed
    _, ctx = M.load(L, raw, w, dt, page_tokens=page_tokens)
    r = M.Runner(ctx)
    for cuts in ([1], [2], [3, 1, 2], [7, 64, 2], [8], [9, 15], [16], [17, 31], [64], [65, 63], [100, 2, 2], [199, 1]):
        check(r.whole(toks, cuts), want, dt, f"portions {cuts}, pages of {page_tokens}", tol[dt])
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_first_tokens(L, mixed, dt):
    raw, w, toks, want, tol = mixed
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    for n in (1, 2, 3, 4, 5, 7, 8, 9, 15, 16, 17, 31, 33):
        for cuts in (None, [1], [2, 1]):
            check(r.whole(toks[:n], cuts), want[:n], dt, f"{n} tokens, portions {cuts}", 1.5 * tol[dt])
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_mixed_batches_equal_each_request_alone(L, mixed, dt):
    raw, w = mixed[:2]
    lens = {"a": 190, "b": 3, "c": 77, "d": 130, "e": 1, "f": 64}
    toks = {k: M.random_tokens(raw, n, 40 + n) for k, n in lens.items()}
    want = {k: M.reference(raw, w, t) for k, t in toks.items()}
    # the pool holds just the live requests, so pages and slots change hands
    _, ctx = M.load(L, raw, w, dt, tokens=512)
    r = M.Runner(ctx)
    rng = np.random.default_rng(5)
    left, waiting, live = {k: list(t) for k, t in toks.items()}, list(lens), []
    while waiting or live:
        while waiting and len(live) < 4 and sum((lens[k] + 63) // 64 for k in live + [waiting[0]]) <= 8:
            live.append(waiting.pop(0))
        entries = []
        for k in live:
            if len(live) > 1 and rng.random() < 0.2:
                continue  # left out of this round
            n = int(rng.choice([1, 1, 2, 5, 33, 64, 100]))
            entries.append((k, left[k][:n]))
            left[k] = left[k][n:]
        if not entries:
            continue
        done = [k for k, _ in entries if not left[k]]
        r.step(entries, end=done)
        live = [k for k in live if k not in done]
    for k in lens:
        check(r.logits(k), want[k], dt, k, M.tolerance(dt, raw, w, toks[k], want[k]))
    assert ctx.pages_free == ctx.pages_total
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_many_requests_in_a_round(L, dt):
    """More requests than a warp has lanes, of unequal portions, then decoded together."""
    raw = M.config([M.window(12, 2), M.conv(heads=6, kv_heads=1), M.window(mlp=M.dense())])
    w = M.weights(raw, 33)
    toks = {i: M.random_tokens(raw, 3 + (7 * i) % 31, 300 + i) for i in range(70)}
    want = {i: M.reference(raw, w, t) for i, t in toks.items()}
    _, ctx = M.load(L, raw, w, dt, tokens=8192, max_tokens=2048, max_seqs=70)
    r = M.Runner(ctx)
    r.step([(i, t[:-2]) for i, t in toks.items()])
    r.step([(i, t[-2:-1]) for i, t in toks.items()])  # more tokens than a small round of experts has
    some = [i for i in toks if i % 2]
    r.step([(i, toks[i][-1:]) for i in some], end=some)
    rest = [i for i in toks if not i % 2]
    r.step([(i, toks[i][-1:]) for i in rest], end=rest)
    for i in toks:
        check(r.logits(i), want[i], dt, i, M.tolerance(dt, raw, w, toks[i], want[i]))
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_slots_and_pages_carry_nothing_over(L, mixed, dt):
    """A short request after a long one in the same pages and state slot, several times over."""
    raw, w = mixed[:2]
    _, ctx = M.load(L, raw, w, dt, tokens=128, max_seqs=1, max_tokens=128)
    r = M.Runner(ctx)
    for i, n in enumerate((128, 1, 2, 127, 3, 65, 1)):
        toks = M.random_tokens(raw, n, 60 + i)
        want = M.reference(raw, w, toks)
        check(r.whole(toks, [[n], [1, 2], [5]][i % 3]), want, dt, f"request {i} of {n} tokens", M.tolerance(dt, raw, w, toks, want))
    ctx.close()


@pytest.mark.parametrize("key,value", [("stack_pdl", 0), ("stack_fork", 0), ("stack_tc", 0), ("stack_tc", 2), ("tc_block", 64), ("tc_cluster", 0), ("tc_cluster", 2)])
def test_every_form_of_a_round(L, key, value):
    """The alternatives behind the tuning keys compute the same: prompts, then one to four requests decode together."""
    raw = M.config([M.window(50, 20, heads=20, kv_heads=5, mlp=M.dense(200)), M.conv(heads=20, kv_heads=5), M.window(100, 5), M.conv(heads=20, kv_heads=5, kv_from=1, mlp=None)])
    w = M.weights(raw, 65)
    toks = {k: M.random_tokens(raw, n, 66 + n) for k, n in (("a", 290), ("b", 150), ("c", 60), ("d", 45))}
    _, ctx = M.load(L, raw, w, BF16, tokens=640)
    L.set_tuning(key, value, ctx)
    r = M.Runner(ctx)
    at = {"a": 200, "b": 120, "c": 40, "d": 35}
    r.step([(k, toks[k][:n]) for k, n in at.items()])
    for i in range(90):
        r.step([(k, toks[k][n + i:n + i + 1]) for k, n in at.items() if n + i < len(toks[k])])
    for k in toks:
        want = M.reference(raw, w, toks[k])
        check(r.logits(k), want, BF16, k, M.tolerance(BF16, raw, w, toks[k], want))
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_long_decoding(L, mixed, dt):
    raw, w = mixed[:2]
    toks = M.random_tokens(raw, 400, 62)
    want = M.reference(raw, w, toks)
    _, ctx = M.load(L, raw, w, dt)
    check(M.Runner(ctx).whole(toks, [5] + [1] * 400), want, dt, "", M.tolerance(dt, raw, w, toks, want))
    ctx.close()


# ------------------------------------------------------------------ single keys that show

KEY, QUERY = 5, 9


def planted_model(kind, heads, kv_heads, size=0, keep=0):
    first = M.conv(3, heads, kv_heads, 32, 32, 0.3, mlp=None) if kind == "conv" else M.window(size, keep, heads, kv_heads, 32, 32, 16, 1e4, 0.3, mlp=None)
    raw = M.config([first, M.window(mlp=M.dense())])
    return raw, M.plant_key(raw, M.weights(raw, 71), KEY, QUERY)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("heads,kv_heads", [(4, 4), (6, 2)])
def test_one_far_key(L, dt, heads, kv_heads):
    """The last token's first-layer attention falls on ONE earlier key, at every kind of place (first token, page and tile borders,
    next to the query); the restatement without that key differs by far more than the tolerance."""
    raw, w = planted_model("conv", heads, kv_heads)
    _, ctx = M.load(L, raw, w, dt, tokens=320)
    r = M.Runner(ctx)
    n = 260
    base = M.random_tokens(raw, n, 72, avoid=(KEY, QUERY))
    base[-1] = QUERY
    lost = M.reference(raw, w, base)[-1:]
    for p in (0, 1, 15, 16, 62, 63, 64, 65, 127, 128, 191, 192, 255, 256, 258):
        toks = list(base)
        toks[p] = KEY
        want = M.reference(raw, w, toks)[-1:]
        assert M.rel_err(lost, want) > 0.1, "the planted key does not show"
        for cuts in (None, [n - 1, 1], [n - 2, 2], [100]):
            check(r.whole(toks, cuts)[-1:], want, dt, f"key at {p}, portions {cuts}", 2 * M.TOL[dt])
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("size,keep", [(1, 0), (2, 1), (16, 20), (40, 64), (63, 65), (64, 3), (65, 130), (100, 16)])
def test_edges_of_a_window_and_of_the_kept_tokens(L, dt, size, keep):
    """A key just inside the window counts, the one just outside does not, but the first tokens always do: in prompts, in the last
    tokens of a portion, decoded."""
    raw, w = planted_model("window", 6, 2, size, keep)
    _, ctx = M.load(L, raw, w, dt, tokens=320)
    r = M.Runner(ctx)
    for at in (size, 64, 127, 130, 250):
        base = M.random_tokens(raw, at + 3, 80 + at, avoid=(KEY, QUERY))
        base[at] = QUERY
        lost = M.reference(raw, w, base)[at:at + 1]
        for p in sorted({at - size + 1, at - size, at - size - 1, 0, keep - 1, keep, keep + 1, keep // 2}):
            if not 0 <= p < at:
                continue
            toks = list(base)
            toks[p] = KEY
            want = M.reference(raw, w, toks)[at:at + 1]
            shows = at - p < size or p < keep
            assert (M.rel_err(lost, want) > 0.1) == shows or not shows, "the planted key does not show"
            for cuts in (None, [at, 1, 1, 1], [at - 1, 2, 2] if at > 1 else [1], [max(at - 5, 1), 8]):
                check(r.whole(toks, cuts)[at:at + 1], want, dt, f"key at {p} before {at}, portions {cuts}", 2 * M.TOL[dt])
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("kind", ["conv", "window"])
def test_the_next_token_is_not_seen(L, dt, kind):
    """The key right AFTER the query (same portion, tile border included) must not count, not even among the kept tokens."""
    raw, w = planted_model(kind, 6, 2, 30, 70)
    _, ctx = M.load(L, raw, w, dt, tokens=256)
    r = M.Runner(ctx)
    for at in (0, 1, 7, 15, 62, 63, 64, 126, 127):
        toks = M.random_tokens(raw, 140, 80 + at, avoid=(KEY, QUERY))
        toks[at], toks[at + 1] = QUERY, KEY
        want = M.reference(raw, w, toks)
        for cuts in (None, [at + 2], [at + 1, 2]):
            check(r.whole(toks, cuts)[:at + 1], want[:at + 1], dt, f"query at {at}, portions {cuts}", 3 * M.TOL[dt])
    ctx.close()


@pytest.mark.parametrize("kind,size,keep", [("conv", 0, 0), ("window", 900, 0), ("window", 700, 500)])
def test_splits_of_a_long_context(L, kind, size, keep):
    """A planted key in every split of a decoded token's context, with pages that are not in order."""
    raw, w = planted_model(kind, 4, 2, size, keep)
    _, ctx = M.load(L, raw, w, BF16, tokens=2048)
    r = M.Runner(ctx)
    base = M.random_tokens(raw, 1500, 75, avoid=(KEY, QUERY))
    base[-1] = QUERY
    r.step([("x", base[:70]), ("y", base[:300])])
    r.step([("x", base[:1])], end=["y"])  # the next request's pages come from the middle of the pool
    for p in (3, 330, 499, 500, 599, 600, 777, 799, 800, 1100, 1498):
        toks = list(base)
        toks[p] = KEY
        want = M.reference(raw, w, toks)[-1:]
        check(r.whole(toks, [700, 799, 1])[-1:], want, BF16, f"key at {p}", 2 * M.TOL[BF16])
    ctx.close()


def test_the_convolution_reaches_across_rounds(L):
    """What a token a few places back changes, in whichever round it came; borrowed keys have it too."""
    raw = M.config([M.conv(4, mlp=None), M.conv(3, kv_from=0, mlp=None)])
    w = M.weights(raw, 91)
    for name in w:
        if name.endswith(".conv"):
            w[name] = w[name].flip(-1).contiguous() + 1  # every tap counts
    toks = M.random_tokens(raw, 24, 92)
    want = every_cut(L, raw, w, toks, F32, [[1], [2], [3], [5, 1], [20, 1], [1, 7]])
    real = R.causal_conv

    def cut(x, c):  # a state that is lost at token 20
        return torch.cat([real(x[:20], c), real(x[20:], c)])
    R.causal_conv = cut
    try:
        assert M.rel_err(M.reference(raw, w, toks)[20:], want[20:]) > 0.05
    finally:
        R.causal_conv = real


# ------------------------------------------------------------------ engine

def greedy(raw, w, prompt, steps):
    toks = list(prompt)
    margins = []
    for _ in range(steps):
        lg = M.reference(raw, w, toks)[-1]
        top = torch.topk(lg, 2).values
        margins.append(float(top[0] - top[1]) / float(lg.std()))
        toks.append(int(lg.argmax()))
    return toks[len(prompt):], margins


@pytest.mark.parametrize("graph", [True, False])
@pytest.mark.parametrize("dt", [F32, BF16])
def test_greedy_generation(L, dt, graph):
    raw = M.config([M.window(8, 2, mlp=M.dense()), M.conv(), M.window(20, 5, mlp=None), M.conv(kv_from=1)])
    w = M.weights(raw, 101)
    prompts = [M.random_tokens(raw, n, 110 + n) for n in (5, 70, 1, 33)]
    want = [greedy(raw, w, p, 10) for p in prompts]
    # a bf16 run may take the other of two tokens whose logits rounding can swap
    near = [4 * M.tolerance(dt, raw, w, p + ids) if dt == BF16 else 0 for p, (ids, _) in zip(prompts, want)]
    _, ctx = M.load(L, raw, w, dt, tokens=1024, max_seqs=8)
    ctx.set_cuda_graph(graph)

    def compare(got):
        for g, (ids, margins), limit in zip(got, want, near):
            for a, b, m in zip(g, ids, margins):
                if a != b:
                    assert m < limit, (g, ids, m, limit)
                    break
    for _ in range(3):  # rounds that follow one another without a pause
        compare(L.generate(ctx, [np.array(p, np.uint32) for p in prompts], 10))
        compare(L.generate_continuous(ctx, [np.array(p, np.uint32) for p in prompts], 10, max_round_tokens=24, prefill_chunk=16))
    assert ctx.pages_free == ctx.pages_total and ctx.device_status() == 0
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_seeded_sampling_replays(L, dt):
    raw = M.config([M.conv(), M.window(mlp=M.dense())], vocab=102)
    w = M.weights(raw, 121)
    _, ctx = M.load(L, raw, w, dt, tokens=1024, max_seqs=8)
    prompts = [np.array(M.random_tokens(raw, n, 130 + n), np.uint32) for n in (4, 20)]
    args = L.SampleArgs.new(0.8, 0.9, 40)
    a = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7)
    c = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=8)
    assert a == L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7) and a != c
    assert all(0 <= t < raw["vocab"] for s in a + c for t in s)
    ctx.close()


def test_convolution_inputs_limit_what_can_be_resumed(L):
    """A state goes on where it ends; without convolutions of two taps and more any position of the cache does."""
    out = torch.zeros(4, 2, dtype=torch.int32, device="cuda")
    for layers, stateful in (([M.conv(2, mlp=None)], True), ([M.conv(1, mlp=None), M.window(mlp=None)], False)):
        raw = M.config(layers)
        _, ctx = M.load(L, raw, M.weights(raw, 141), F32, tokens=512, max_seqs=2)
        a, b, c = (ctx.seq_create() for _ in range(3))
        ctx.step([(a, 0, 5)], [1, 2, 3, 4, 5], out)
        assert [ctx.seq_resumable(a, n) for n in (3, 5)] == ([0, 5] if stateful else [3, 5])
        if stateful:
            with pytest.raises(L.LcuError) as e:
                ctx.step([(a, 4, 1)], [6], out)
            assert e.value.code == L.ERR_STATE
            ctx.step([(b, 0, 1)], [1], out)
            with pytest.raises(L.LcuError) as e:  # both state slots are taken
                ctx.step([(c, 0, 1)], [1], out)
            assert e.value.code == L.ERR_NO_PAGES
            ctx.seq_free(b)
        ctx.step([(c, 0, 1), (a, 5, 1)], [1, 6], out)
        ctx.close()


def test_parked_conversations_resume_where_their_state_is(L):
    raw = M.config([M.conv(), M.window(8, 3, mlp=None), M.window(mlp=M.dense())])
    w = M.weights(raw, 151)
    _, ctx = M.load(L, raw, w, F32, tokens=512, max_seqs=4)
    svc = L.Service(ctx)
    prompt = M.random_tokens(raw, 20, 152)
    with torch.cuda.stream(svc.stream):
        s = svc.new_session()
        svc.start(s, prompt, 4)
        ids = []
        while True:
            r, out = svc.step()
            if out is None:
                break
            svc.stream.synchronize()
            ids += list(svc.decode(r, out).values())
        assert ids == greedy(raw, w, prompt, 4)[0]
        history = prompt + ids[:-1]  # what the cache has seen
        svc.park(s, history)
        more = history + [ids[-1], 17, 18]
        t, reused = svc.send(more, max_steps=1)
        assert reused == len(history)
        r, out = svc.step()
        svc.stream.synchronize()
        assert svc.decode(r, out)[t.id] == greedy(raw, w, more, 1)[0][0]
        svc.stop(t.id)
        svc.park(t, more)
        fork = more[:10] + [3, 4, 5]  # a shorter common prefix: the state cannot go back, the cache restarts
        u, reused = svc.send(fork, max_steps=1)
        assert reused == 0
        r, out = svc.step()
        svc.stream.synchronize()
        assert svc.decode(r, out)[u.id] == greedy(raw, w, fork, 1)[0][0]
    ctx.close()


def test_graph_rounds_keep_the_state_in_step(L):
    """Captured decode rounds alternate the halves of the double-buffered state through the descriptor, not through the graph."""
    raw = M.config([M.conv(4), M.window(6, 2), M.conv(2, kv_from=0)])
    w = M.weights(raw, 161)
    toks = M.random_tokens(raw, 40, 162)
    want = M.reference(raw, w, toks)
    _, ctx = M.load(L, raw, w, F32)
    st = torch.cuda.Stream()
    out = torch.zeros(4, 2, dtype=torch.int32, device="cuda")
    with torch.cuda.stream(st):
        s = ctx.seq_create()
        ctx.step([(s, 0, 3)], toks[:3], out, stream=st)
        for i in range(3, 40):
            ctx.step([(s, i, 1)], toks[i:i + 1], out, stream=st)
            st.synchronize()
            check(ctx.logits(1).cpu(), want[i:i + 1], F32, f"token {i}")
            assert int(out[0, 0]) == int(want[i].argmax())
    ctx.close()


def test_descriptions_that_make_no_sense_are_refused(L):
    cfg = M.cfg_of(M.MIXED)
    for layer, field, value in ((0, "keep_first", -1), (0, "window", 0), (0, "sink", 3), (0, "rot_adjacent", 0), (0, "v_dim", 27), (0, "rot_base", 0.0), (0, "logit_cap", -1.0),
                                (0, "ff_act", 5), (0, "identity", 1), (1, "conv", 65), (1, "conv", -1), (1, "bias", 1), (1, "qk_norm", 3), (1, "mixer", L.MIX_ATTENTION | L.MIX_DELTA),
                                (1, "top", 8), (1, "top", 0), (1, "identity", -1), (1, "route_softmax", 0), (1, "ff_bias", 1), (1, "post_norm", 1), (1, "shared_ff", 16),
                                (3, "rot_values", 1), (3, "kv_heads", 3), (3, "kv_from", 4), (0, "pair_buckets", 5)):
        d = cfg.layer_descs()
        setattr(d[layer], field, value)
        with pytest.raises(L.LcuError) as e:
            L.Context(cfg.desc(), layers=d)
        assert e.value.code == L.ERR_INVALID, (layer, field, value)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_run_replays_a_schedule(L, tmp_path, dtype):
    raw = M.MIXED
    w = M.weights(raw, 171)
    M.write_model(tmp_path / "m", raw, w)
    a, b = M.random_tokens(raw, 70, 172), M.random_tokens(raw, 12, 173)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [0, 65]}, {"id": "b", "tokens": b[:2], "want": [1]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:12], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[66:], "want": [3]}, {"id": "c", "tokens": b[:12], "want": [11]}], "end": ["a", "c"]}]
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    wa, wb = M.reference(raw, w, a), M.reference(raw, w, b)
    got = {i: torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", "<f4")).view(-1, raw["vocab"]) for i in (0, 2)}
    dt = F32 if dtype == "float32" else BF16
    tol = 1.5 * M.tolerance(dt, raw, w, a, wa)
    check(got[0], torch.stack([wa[0], wa[65], wb[1]]), dt, "", tol)
    check(got[2], torch.stack([wa[69], wb[11]]), dt, "", tol)
    assert not os.path.exists(tmp_path / "1.f32")
