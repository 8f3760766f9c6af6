"""Mupuvik on the GPU against the plain restatement (f64, whole sequences): each mechanism, every way of cutting a sequence into
rounds, shared batches, pages and state slots used again, single keys, window edges and lost state, generation through the engine."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import mupuvik_models as M
import mupuvik_ref as R

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = 1, 2
LAYERS = {"ssd": M.ssd(), "window": M.window(), "both": M.both()}


@pytest.fixture(autouse=True)
def default_tuning(L):
    yield
    for k, v in (("stack_pdl", 1), ("stack_tc", 1), ("tc_block", 256), ("tc_cluster", 1)):
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


# ------------------------------------------------------------------ mechanisms alone

ALONE = [(kind, off) for kind in ("ssd", "window", "both") for off in ((), ("ff",), ("mixer",), ("ff", "pairs"))] + [
    ("both", off) for off in (("mixer", "experts"), ("mixer", "shared"), ("ff", "left"), ("ff", "right"))]


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
    raw = M.config(list(LAYERS.values()), eps=0.3)
    w = M.weights(raw, 6)
    toks = M.random_tokens(raw, 30, 7)
    want = every_cut(L, raw, w, toks, F32, [[1]])
    assert M.rel_err(M.reference(dict(raw, norm={"eps": 1e-5}), w, toks), want) > 1e-2


def test_embedding_scale_and_pairs(L):
    """Factors larger than the table, a table of one bucket, scale one; the previous token crosses portions and rounds."""
    for scale, buckets, mul in ((1.0, 97, (1000, 98)), (0.3, 1, (3, 4)), (20.0, 2, (1, 1)), (3.0, 65521, (31, 17))):
        raw = M.config([M.both(mlp=None)], scale=scale, buckets=buckets, mul=mul)
        w = M.silence(M.weights(raw, 8), raw, "mixer")
        toks = M.random_tokens(raw, 40, 9)
        want = every_cut(L, raw, w, toks, F32, [[1], [2], [3, 1, 5]])
        assert M.rel_err(M.reference(raw, M.silence(w, raw, "pairs"), toks), want) > 0.02


@pytest.mark.parametrize("rot", [2, 6, 14, 20])
def test_rotations(L, rot):
    """Rotated parts of every width, an odd number of pairs and whole heads among them."""
    raw = M.config([M.both(rot=rot, base=30.0, scale=0.5)])
    w = M.silence(M.weights(raw, 8), raw, "right")
    toks = M.random_tokens(raw, 90, 9)
    want = every_cut(L, raw, w, toks, F32, [[1], [40, 7]])
    other = M.both(rot=rot, base=900.0, scale=0.5) if rot > 2 else M.both(rot=4, base=30.0, scale=0.5)
    assert M.rel_err(M.reference(M.config([other]), w, toks), want) > 1e-3


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_convolution_taps(L, taps):
    raw = M.config([M.ssd(conv=taps, mlp=None)])
    w = M.weights(raw, 10)
    toks = M.random_tokens(raw, 40, 11)
    for dt in (F32, BF16):
        every_cut(L, raw, w, toks, dt, [[1], [2], [3, 1], [8, 7], [4, 9, 1, 1], [16], [17, 2]])


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("heads,groups,vdim,parts", [(4, 1, 12, 1), (4, 4, 12, 4), (6, 3, 20, 2), (6, 2, 5, 10), (2, 1, 9, 18), (8, 2, 16, 32)])
def test_norm_parts_and_groups(L, dt, heads, groups, vdim, parts):
    """Parts that hold several heads, one, a piece of one, borders inside heads; heads of sizes that four does not divide."""
    raw = M.config([M.ssd(heads=heads, groups=groups, vdim=vdim, parts=parts, mlp=None)])
    w = M.weights(raw, 12)
    toks = M.random_tokens(raw, 50, 13)
    want = every_cut(L, raw, w, toks, dt, [[1], [20, 3]])
    if parts > 1:
        assert M.rel_err(M.reference(M.config([M.ssd(heads=heads, groups=groups, vdim=vdim, parts=1, mlp=None)]), w, toks), want) > 1e-2


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("rank,tau,bias", [(1, 1.0, 0.0), (5, 16.0, 3.0), (16, 1.0, -30.0), (33, 0.5, 8.0), (70, 16.0, -4.0)])
def test_decay_maps(L, dt, rank, tau, bias):
    """Inner sizes around the multiples of eight; decays from none to complete: products of decays vanish, nothing divides by them."""
    raw = M.config([M.both(rank=rank, tau=tau, mlp=None)])
    w = M.silence(M.weights(raw, 14), raw, "left")
    w["l0.mix.right.a2.b"] = (w["l0.mix.right.a2.b"].float() + bias).to(torch.bfloat16)
    every_cut(L, raw, w, M.random_tokens(raw, 80, 15), dt, [[1], [30], [16, 2, 15]])


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("rate", [-9.0, 0.0, 3.0])
def test_state_space_decays_from_none_to_complete(L, dt, rate):
    raw = M.config([M.ssd(mlp=None), M.ssd(state=64, vdim=32, parts=1, mlp=None)])
    w = M.weights(raw, 16)
    for k in w:
        if k.endswith("A_log"):
            w[k] = torch.full_like(w[k], rate)
        if k.endswith("dt_bias"):
            w[k] = w[k] + 2
    every_cut(L, raw, w, M.random_tokens(raw, 90, 17), dt, [[1], [30]])


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n", [40, 300])
@pytest.mark.parametrize("mlp", [M.moe(30, 5, 2), M.moe(30, 1, 1, 0.4, 0), M.moe(64, 2, 2, 1.0, 0), M.moe(9, 12, 3, 0.2, 100, 3.0), M.moe(130, 3, 1, 5.0, 7, 0.05),
                                 M.moe(16, 40, 7, 1.0, 16, 1.0)])
def test_experts(L, dt, n, mlp):
    """One to forty experts, all of them or one, tiles of 64 to 256 rows, limits that clip much or nothing; small rounds and large."""
    raw = M.config([M.ssd(mlp=mlp), M.window(mlp=mlp)], width=176)
    w = M.weights(raw, 18)
    toks = M.random_tokens(raw, n, 19)
    want = every_cut(L, raw, w, toks, dt, [[1, n - 6, 5], [33], [64], [65]])
    for part in ("experts", "shared") if mlp.get("shared") else ("experts",):
        assert M.rel_err(M.reference(raw, M.silence(w, raw, part), toks), want) > 5e-3


def test_routing_by_random_routers(L):
    """Routers as they come (32-bit arithmetic: no rounding swaps two experts)."""
    raw = M.config([M.ssd(mlp=M.moe(30, 37, 5)), M.window(mlp=M.moe(30, 70, 2)), M.both(mlp=M.moe(30, 3, 2))])
    w = M.weights(raw, 20, steady=False)
    every_cut(L, raw, w, M.random_tokens(raw, 120, 21), F32, [[1], [50]])


@pytest.mark.parametrize("dt", [F32, BF16])
def test_borrowed_keys_with_windows_of_their_own(L, dt):
    """Two layers read one layer's cache, one through a wider window, one through a narrower one."""
    raw = M.config([M.ssd(mlp=None), M.window(20, mlp=None), M.window(70, kv_from=1, mlp=None), M.ssd(mlp=None), M.window(3, kv_from=1, scale=0.6, mlp=None)])
    w = M.weights(raw, 22)
    toks = M.random_tokens(raw, 160, 23)
    want = every_cut(L, raw, w, toks, dt, [[1], [64], [100, 1, 2]])
    same = M.config([M.ssd(mlp=None), M.window(20, mlp=None), M.window(20, kv_from=1, mlp=None), M.ssd(mlp=None), M.window(20, kv_from=1, scale=0.6, mlp=None)])
    assert M.rel_err(M.reference(same, w, toks), want) > 1e-2


def test_sink_and_norm_weights_show(L):
    """The first tokens without the sink, and without the weights of the query and key norms, come out differently."""
    raw = M.config([M.both(mlp=None)])
    w = M.silence(M.weights(raw, 24), raw, "right")
    toks = M.random_tokens(raw, 5, 25)
    want = every_cut(L, raw, w, toks, F32, [[1], [2]])
    real = R.softmax_attention
    R.softmax_attention = lambda *a, sink=False, **k: real(*a, **k)
    try:
        assert M.rel_err(M.reference(raw, w, toks), want) > 1e-2
    finally:
        R.softmax_attention = real
    for kind, raw in (("both", raw), ("window", M.config([M.window(mlp=None)]))):
        w = M.weights(raw, 26)
        if kind == "both":
            w = M.silence(w, raw, "right")
        plain = {k: torch.ones_like(v) if k.endswith((".q.norm", ".k.norm")) else v for k, v in w.items()}
        toks = M.random_tokens(raw, 30, 27)
        want = every_cut(L, raw, w, toks, F32, [[1]])
        assert M.rel_err(M.reference(raw, plain, toks), want) > 1e-3


def test_scores_far_below_the_sink(L):
    """Queries against keys of the opposite sign: the sink takes nearly everything, nothing overflows."""
    raw = M.config([M.both(rot=2, scale=60.0, mlp=None)])
    w = M.silence(M.weights(raw, 28), raw, "right")
    w["l0.mix.left.k"] = -w["l0.mix.left.q"][:40].clone()
    for dt in (F32, BF16):
        got = every_cut(L, raw, w, [7] * 20, dt, [[1], [6]])
        assert torch.isfinite(got).all()


# ------------------------------------------------------------------ sizes

SIZES = {
    "ones": M.config([M.ssd(1, 1, 1, 1, 1, 1, mlp=M.moe(1, 1, 1, 1.0, 1)), M.window(1, 1, 1, 1, 1, 1.0, mlp=None), M.both(1, 1, 2, 1, 2, 10.0, 1.0, 1, 1, 1, 1.0, 1, (1.0, 1.0), mlp=None)],
                     width=8, vocab=7, buckets=3),
    "large_heads": M.config([M.ssd(2, 1, 256, 200, 4, 2), M.window(40, 3, 1, 256, 200, 0.06), M.both(2, 2, 130, 256, 64, 1e4, 0.1, 2, 256, 160, 16.0, 16),
                             M.ssd(3, 3, 160, 256, 4, 1)], width=136, vocab=150),
    "wide_groups": M.config([M.ssd(40, 2, 24, 8, 4, 8), M.window(33, 40, 1, 16, 16, 0.5), M.both(66, 1, 12, 8, 4, 1e3, 0.5, 17, 8, 40)], width=96, vocab=64),
    "many_key_heads": M.config([M.ssd(16, 16, 128, 64, 4, 16), M.window(64, 12, 12, 64, 128, 0.2), M.both(16, 16, 64, 64, 64, 1e4, 0.2, 16, 64, 64)], width=128, vocab=96),
    "usual": M.config([M.ssd(16, 2, 128, 64, 4, 2, mlp=M.moe(300, 8, 2, 2.0, 200, 2.0)), M.window(100, 8, 2, 128, 128, 128 ** -0.5),
                       M.both(8, 2, 128, 128, 128, 5e5, 128 ** -0.5, 4, 128, 256, 16.0, 16, mlp=M.moe(300, 8, 2, 2.0, 200, 2.0))], width=200, vocab=333),
    "wide": M.config([M.ssd(mlp=M.moe(700, 4, 2, 1.0, 130, 1.0))], width=1032, vocab=333),
    "attention_only": M.config([M.window(50), M.window(7, kv_from=0)]),
    "state_only": M.config([M.ssd(), M.ssd(mlp=None)]),
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
    raw = M.config([M.ssd(), M.window(12), M.both(heads=6, kv_heads=1)])
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


@pytest.mark.parametrize("key,value", [("stack_pdl", 0), ("stack_tc", 0), ("stack_tc", 2), ("tc_block", 64), ("tc_cluster", 0), ("tc_cluster", 2)])
def test_every_form_of_a_round(L, key, value):
    """The alternatives behind the tuning keys compute the same: prompts, then one to four requests decode together."""
    raw = M.config([M.ssd(state=64, vdim=64, parts=2), M.window(50, heads=20, kv_heads=5), M.both(g_dim=64, g_vdim=64), M.window(100, heads=20, kv_heads=5, kv_from=1, mlp=None)])
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


def planted_model(kind, heads, kv_heads, size=0, mlp=None):
    first = M.both(heads, kv_heads, 32, 32, 16, 1e4, 1.2, mlp=mlp) if kind == "both" else M.window(size, heads, kv_heads, 32, 32, 1.2, mlp=mlp)
    raw = M.config([first, M.ssd(mlp=None)])
    return raw, M.plant_key(raw, M.silence(M.weights(raw, 71), raw, "right"), KEY, QUERY)


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("heads,kv_heads", [(4, 4), (6, 2)])
def test_one_far_key(L, dt, heads, kv_heads):
    """The last token's first-layer attention falls on ONE earlier key, at every kind of place (first token, page and tile borders,
    next to the query); the restatement without that key differs by far more than the tolerance."""
    raw, w = planted_model("both", heads, kv_heads)
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
@pytest.mark.parametrize("size", [1, 2, 16, 40, 63, 64, 65, 100])
def test_edges_of_a_window(L, dt, size):
    """A key just inside the window counts, the one just outside does not: in prompts, in the last tokens of a portion, decoded."""
    raw, w = planted_model("window", 6, 2, size)
    _, ctx = M.load(L, raw, w, dt, tokens=320)
    r = M.Runner(ctx)
    for at in (size, 63, 64, 127, 130, 200):
        if at < size:
            continue
        base = M.random_tokens(raw, at + 3, 80 + at, avoid=(KEY, QUERY))
        base[at] = QUERY
        lost = M.reference(raw, w, base)[at:at + 1]
        for back, shows in ((size - 1, True), (size, False), (size + 1, False), (0, False)):
            if back == 0 or back > at:
                continue
            toks = list(base)
            toks[at - back] = KEY
            want = M.reference(raw, w, toks)[at:at + 1]
            if shows:
                assert M.rel_err(lost, want) > 0.1, "the planted key does not show"
            for cuts in (None, [at, 1, 1, 1], [at - 1, 2, 2] if at > 1 else [1], [max(at - 5, 1), 8]):
                check(r.whole(toks, cuts)[at:at + 1], want, dt, f"key {back} before {at}, portions {cuts}", 2 * M.TOL[dt])
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("kind", ["both", "window"])
def test_the_next_token_is_not_seen(L, dt, kind):
    """The key right AFTER the query (same portion, tile border included) must not count."""
    raw, w = planted_model(kind, 6, 2, 90)
    _, ctx = M.load(L, raw, w, dt, tokens=256)
    r = M.Runner(ctx)
    for at in (0, 1, 7, 15, 62, 63, 64, 126, 127):
        toks = M.random_tokens(raw, 140, 80 + at, avoid=(KEY, QUERY))
        toks[at], toks[at + 1] = QUERY, KEY
        want = M.reference(raw, w, toks)
        for cuts in (None, [at + 2], [at + 1, 2]):
            check(r.whole(toks, cuts)[:at + 1], want[:at + 1], dt, f"query at {at}, portions {cuts}", 3 * M.TOL[dt])
    ctx.close()


@pytest.mark.parametrize("kind,size", [("both", 0), ("window", 900)])
def test_splits_of_a_long_context(L, kind, size):
    """A planted key in every split of a decoded token's context, with pages that are not in order."""
    raw, w = planted_model(kind, 4, 2, size)
    _, ctx = M.load(L, raw, w, BF16, tokens=2048)
    r = M.Runner(ctx)
    base = M.random_tokens(raw, 1500, 75, avoid=(KEY, QUERY))
    base[-1] = QUERY
    r.step([("x", base[:70]), ("y", base[:300])])
    r.step([("x", base[:1])], end=["y"])  # the next request's pages come from the middle of the pool
    for p in (3, 330, 599, 600, 777, 1100, 1498):
        toks = list(base)
        toks[p] = KEY
        want = M.reference(raw, w, toks)[-1:]
        check(r.whole(toks, [700, 799, 1])[-1:], want, BF16, f"key at {p}", 2 * M.TOL[BF16])
    ctx.close()


# ------------------------------------------------------------------ recurrent state

@pytest.mark.parametrize("kind", ["ssd", "gla"])
def test_the_state_reaches_back_to_the_first_token(L, kind):
    """Decays near one: what the first token left behind still shows hundreds of tokens later."""
    raw = M.config([M.ssd(state=64, vdim=40, parts=1, mlp=None) if kind == "ssd" else M.both(g_dim=64, g_vdim=40, mlp=None)])
    w = M.silence(M.weights(raw, 91), raw, "left", "pairs")
    if kind == "ssd":
        w["l0.mix.A_log"] = torch.full_like(w["l0.mix.A_log"], -7.0)
    else:
        w["l0.mix.right.a2.b"] = torch.full_like(w["l0.mix.right.a2.b"], 9.0)
    toks = M.random_tokens(raw, 120, 92)
    want = every_cut(L, raw, w, toks, F32, [[1], [2], [3, 8, 5], [60], [119, 1], [7, 1]])
    other = M.reference(raw, w, [(toks[0] + 1) % raw["vocab"]] + toks[1:])
    assert M.rel_err(other[-1:], want[-1:]) > 1e-3
    every_cut(L, raw, w, toks, BF16, [[1], [60], [7, 1]], want)


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
    """Fed-back tokens stay on the device: the pairs they make with the tokens before them, and all state, must follow."""
    raw = M.config([M.ssd(), M.window(8), M.both(mlp=None), M.window(20, kv_from=1)])
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
    raw = M.config([M.ssd(), M.both(mlp=None)], vocab=102)
    w = M.weights(raw, 121)
    _, ctx = M.load(L, raw, w, dt, tokens=1024, max_seqs=8)
    prompts = [np.array(M.random_tokens(raw, n, 130 + n), np.uint32) for n in (4, 20)]
    args = L.SampleArgs.new(0.8, 0.9, 40)
    a = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7)
    c = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=8)
    assert a == L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7) and a != c
    assert all(0 <= t < raw["vocab"] for s in a + c for t in s)
    ctx.close()


@pytest.mark.parametrize("layers", [[M.ssd(mlp=None)], [M.window(mlp=None)]])
def test_recurrent_state_limits_what_can_be_resumed(L, layers):
    """A model without recurrent layers keeps the previous token: a state too."""
    raw = M.config(layers)
    w = M.weights(raw, 141)
    _, ctx = M.load(L, raw, w, F32, tokens=512, max_seqs=2)
    out = torch.zeros(4, 2, dtype=torch.int32, device="cuda")
    a, b, c = (ctx.seq_create() for _ in range(3))
    ctx.step([(a, 0, 5)], [1, 2, 3, 4, 5], out)
    assert [ctx.seq_resumable(a, n) for n in (3, 5, 9)] == [0, 5, 5]
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
    raw = M.config([M.ssd(), M.window(8, mlp=None), M.both()])
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
    raw = M.config([M.ssd(), M.window(6), M.both()])
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
    for layer, field, value in ((0, "norm_parts", 7), (0, "norm_parts", 0), (0, "delta_kv_heads", 3), (0, "delta_conv", 0), (0, "mixer", L.MIX_SSD | L.MIX_GLA), (0, "top", 6),
                                (0, "top", 0), (0, "glu_limit", 0.0), (0, "shared_limit", 0.0), (0, "post_norm", 0), (0, "pair_prev", 53), (1, "window", -1), (1, "qk_norm", 4),
                                (1, "kv_from", 2), (1, "kv_from", 1), (4, "kv_heads", 3), (4, "dim", 24), (3, "gate_rank", 0), (3, "gate_tau", 0.0), (3, "delta_kv_heads", 1),
                                (3, "mixer", L.MIX_ATTENTION | L.MIX_DELTA)):
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
