"""Galarax on the GPU against the plain restatement (f64, whole sequences): each mechanism, every way of cutting a sequence into
rounds, shared batches, pages and state slots used again, single keys and lost state, generation through the engine."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import galarax_models as M
import galarax_ref as G

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = 1, 2


@pytest.fixture(autouse=True)
def default_tuning(L):
    yield
    for k, v in (("stack_pdl", 1), ("stack_fuse", 1), ("stack_tc", 1), ("delta_tc", 1), ("tc_block", 256)):
        L.set_tuning(k, v)


def check(got, want, dt, what="", tol=None):
    e, tol = M.rel_err(got, want), tol or M.TOL[dt]
    assert e <= tol, f"{what}: error {e:.3g} > {tol:.3g}"
    return e


def whole(L, raw, w, toks, dt, cuts=None, **kw):
    _, ctx = M.load(L, raw, w, dt, **kw)
    got = M.Runner(ctx).whole(toks, cuts)
    assert ctx.device_status() == 0 and ctx.pages_free == ctx.pages_total
    ctx.close()
    return got


# ------------------------------------------------------------------ mechanisms alone

@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("off", [("right", "ff"), ("left", "ff"), ("left", "right"), ("ff",), ()])
def test_mechanism_alone(L, dt, off):
    raw = M.config([M.layer()])
    w = M.silence(M.weights(raw, 1), raw, *off)
    toks = M.random_tokens(raw, 70, 2)
    want, stream = M.reference(raw, w, toks, True)
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    got = r.whole(toks)
    x = ctx.hidden(70).cpu().double()
    assert float((x - stream[-1]).abs().max()) / float(stream[-1].abs().max()) <= (2e-5 if dt == F32 else 2e-2)
    check(got, want, dt, off)
    check(r.whole(toks, [1]), want, dt, f"{off}, decoded")
    ctx.close()


def single_mixer_model(L, which, w):
    """The layers' weights of a Galarax model with ONE of its two mixers (no gain on its output)."""
    from llama_cu_b200 import galarax, layered as Y
    raw = M.config([M.layer()])
    full = galarax.read_config(raw)
    m = full.layers[0].mixer
    mixer = m.left if which == "left" else m.right
    layers = (Y.LayerConfig(mixer, 50, False, act=L.ACT_RELU2, pre_norm=True),)
    cfg = Y.LayeredConfig("single", full.d, full.vocab, layers, full.eps, nctx=512)
    t = lambda n: w["l0.mix." + which + "." + n]
    rows = Y.attention_rows(mixer, cfg.d, *map(t, "qkv")) if which == "left" else Y.delta_rows(mixer, cfg.d, *map(t, "qkvgba"))
    parts = [(L.W_MIX_IN, torch.cat(rows))]
    if which == "left":
        parts += Y.pack_attention(mixer, cfg.d, t("o"), [t(n + ".b") for n in "qkv"])
    else:
        parts += Y.pack_delta(mixer, cfg.d, *(t(n) for n in ("q.conv", "k.conv", "v.conv", "A_log", "dt_bias", "norm", "o")))
    parts += Y.pack_pre_norm_block(cfg.d, 50, 1 + w["l0.norm1"].float(), 1 + w["l0.norm2"].float(), w["l0.mlp.up"], w["l0.mlp.down"])
    weights = Y.pack_common(cfg.d, w["embed"], 1 + w["final.norm"].float(), w["head"]) + [((0, k), v) for k, v in parts]
    return raw, cfg, weights


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("which", ["left", "right"])
def test_a_layer_with_one_of_the_mixers(L, dt, which):
    """The mixers serve alone as well: attention without a recurrent state, a delta rule without cached rows."""
    from dataclasses import replace
    w = M.weights(M.config([M.layer()]), 3)
    raw, cfg, weights = single_mixer_model(L, which, w)
    toks = M.random_tokens(raw, 50, 4)
    f = {k: v.double() for k, v in w.items()}
    x, m, eps = f["embed"][toks], raw["layers"][0]["mixer"][which], raw["norm"]["eps"]
    x = x + getattr(G, which)(G.centred_norm(x, f["l0.norm1"], eps), f, f"l0.mix.{which}.", m, eps)
    x = x + G.feed_forward(G.centred_norm(x, f["l0.norm2"], eps), f, "l0.mlp.")
    want = G.centred_norm(x, f["final.norm"], eps) @ f["head"].T
    cfg = replace(cfg, act_dtype=dt)
    ctx = L.load_model(cfg, weights, kv_bytes=max(512 * cfg.kv_bytes_per_token(), 1 << 20), max_tokens=512, max_seqs=4)
    r = M.Runner(ctx)
    for cuts in (None, [1], [20, 2, 1]):
        check(r.whole(toks, cuts), want, dt, f"{which}, portions {cuts}")
    ctx.close()


def test_eps_matters_and_is_read(L):
    raw = M.config([M.layer()], eps=0.3)
    w = M.weights(raw, 6)
    toks = M.random_tokens(raw, 30, 7)
    got = whole(L, raw, w, toks, F32)
    check(got, M.reference(raw, w, toks), F32)
    assert M.rel_err(got, M.reference(dict(raw, norm={"eps": 1e-5}), w, toks)) > 1e-2


@pytest.mark.parametrize("rot", [M.rotary(2, 10.0, 0), M.rotary(6, 1e4, 8.0, 64, 32.0, 1.0), M.rotary(20, 7.0, 1.5, 20, 2.0, 1.0), M.rotary(10, 1e6, 32.0, 100000, 4.0, 0.5),
                                 M.rotary(16, 500.0, 2.0, 30, 0.1, 0.05)])
def test_rotations(L, rot):
    """Rotated parts of every width (pairs that four-wide loads cannot take, whole heads), with and without scaling; without
    the scaling the result is another one."""
    raw = M.config([M.layer(rot=rot, scale=0.5)])
    w = M.silence(M.weights(raw, 8), raw, "right")
    toks = M.random_tokens(raw, 90, 9)
    got = whole(L, raw, w, toks, F32)
    check(got, M.reference(raw, w, toks), F32)
    if "scaling" in rot:
        assert M.rel_err(got, M.reference(M.config([M.layer(rot=M.rotary(rot["dims"], rot["base"], 0), scale=0.5)]), w, toks)) > 1e-3


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 5, 9])
def test_convolution_taps(L, taps):
    raw = M.config([M.layer(conv=taps, ff=0)])
    w = M.silence(M.weights(raw, 10), raw, "left")
    toks = M.random_tokens(raw, 40, 11)
    want = M.reference(raw, w, toks)
    for dt in (F32, BF16):
        _, ctx = M.load(L, raw, w, dt)
        r = M.Runner(ctx)
        for cuts in (None, [1], [2], [3, 1], [8, 7], [4, 9, 1, 1]):
            check(r.whole(toks, cuts), want, dt, f"{taps} taps, portions {cuts}")
        ctx.close()


# ------------------------------------------------------------------ sizes

SIZES = {
    "ones": M.config([M.layer(heads=1, kv_heads=1, dim=2, vdim=1, rot=M.rotary(2, 10.0), scale=1.0, d_heads=1, d_kv_heads=1, d_dim=1, d_vdim=1, conv=1, ff=1)], width=8, vocab=7),
    "large_heads": M.config([M.layer(heads=3, kv_heads=1, dim=256, vdim=200, rot=M.rotary(64, 1e4), scale=0.06, d_heads=2, d_kv_heads=2, d_dim=256, d_vdim=256, ff=96),
                             M.layer(heads=2, kv_heads=2, dim=130, vdim=256, scale=0.1, d_heads=4, d_kv_heads=2, d_dim=160, d_vdim=96)], width=136, vocab=150),
    "wide_groups": M.config([M.layer(heads=40, kv_heads=1, dim=16, vdim=16, scale=0.5, d_heads=12, d_kv_heads=1, d_dim=24, d_vdim=24),
                             M.layer(heads=66, kv_heads=1, dim=12, vdim=8, scale=0.5, d_heads=20, d_kv_heads=2, d_dim=8, d_vdim=40)], width=96, vocab=64),
    "many_key_heads": M.config([M.layer(heads=12, kv_heads=12, dim=64, vdim=128, scale=0.2, d_heads=16, d_kv_heads=16, d_dim=128, d_vdim=128, ff=64)], width=128, vocab=96),
    "usual": M.config([M.layer(heads=8, kv_heads=2, dim=128, vdim=128, rot=M.rotary(64, 5e5, 4.0, 256), scale=128 ** -0.5, d_heads=8, d_kv_heads=4, d_dim=128, d_vdim=128, ff=300)],
                      width=200, vocab=333),
    "wide": M.config([M.layer(ff=700)], width=1032, vocab=333),
    "mixed": M.MIXED,
    "looped_whole": M.config([M.layer(), M.layer(conv=3)], loop=(0, 2, 2)),
    "looped_once": M.config([M.layer(), M.layer()], loop=(1, 2, 1)),
    "looped_last": M.config([M.layer(), M.layer(ff=0)], loop=(1, 2, 4)),
}


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(L, name, dt):
    raw = SIZES[name]
    w = M.weights(raw, 11)
    toks = M.random_tokens(raw, 150, 12)
    want = M.reference(raw, w, toks)
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    tol = M.tolerance(dt, raw, w, toks, want)
    check(r.whole(toks), want, dt, "whole", tol)
    check(r.whole(toks, [120] + [1] * 30), want, dt, "decoded", tol)
    check(r.whole(toks, [2, 64, 3, 17]), want, dt, "portions", tol)
    assert ctx.device_status() == 0 and ctx.pages_free == ctx.pages_total
    ctx.close()


# ------------------------------------------------------------------ schedules

@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("page_tokens", [64, 8, 128])
def test_portions(L, dt, page_tokens):
    raw = M.MIXED
    w = M.weights(raw, 21)
    toks = M.random_tokens(raw, 200, 22)
    want = M.reference(raw, w, toks)
    _, ctx = M.load(L, raw, w, dt, page_tokens=page_tokens)
    r = M.Runner(ctx)
    for cuts in ([1], [2], [3, 1, 2], [7, 64, 2], [8], [9, 15], [64], [65, 63], [100, 2, 2], [199, 1]):
        check(r.whole(toks, cuts), want, dt, f"portions {cuts}, pages of {page_tokens}")
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("n", [1, 2, 3, 4, 5, 7, 8, 9, 16, 17])
def test_first_tokens(L, dt, n):
    raw = M.MIXED
    w = M.weights(raw, 23)
    toks = M.random_tokens(raw, n, 24 + n)
    want = M.reference(raw, w, toks)
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    for cuts in (None, [1], [2, 1]):
        check(r.whole(toks, cuts), want, dt, f"{n} tokens, portions {cuts}")
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_mixed_batches_equal_each_request_alone(L, dt):
    raw = M.MIXED
    w = M.weights(raw, 31)
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
        check(r.logits(k), want[k], dt, k)
    assert ctx.pages_free == ctx.pages_total
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_many_requests_in_a_round(L, dt):
    """More requests than a warp has lanes, of unequal portions, then decoded together."""
    raw = M.config([M.layer(), M.layer(heads=6, kv_heads=1)])
    w = M.weights(raw, 33)
    toks = {i: M.random_tokens(raw, 3 + (7 * i) % 31, 300 + i) for i in range(40)}
    _, ctx = M.load(L, raw, w, dt, tokens=4096, max_tokens=1024, max_seqs=40)
    r = M.Runner(ctx)
    r.step([(i, t[:-2]) for i, t in toks.items()])
    r.step([(i, t[-2:-1]) for i, t in toks.items()])
    r.step([(i, t[-1:]) for i, t in toks.items()], end=list(toks))
    for i, t in toks.items():
        check(r.logits(i), M.reference(raw, w, t), dt, i)
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_slots_and_pages_carry_nothing_over(L, dt):
    """A short request after a long one in the same pages and state slot, several times over."""
    raw = M.MIXED
    w = M.weights(raw, 51)
    _, ctx = M.load(L, raw, w, dt, tokens=128, max_seqs=1, max_tokens=128)
    r = M.Runner(ctx)
    for i, n in enumerate((128, 1, 2, 127, 3, 65, 1)):
        toks = M.random_tokens(raw, n, 60 + i)
        check(r.whole(toks, [[n], [1, 2], [5]][i % 3]), M.reference(raw, w, toks), dt, f"request {i} of {n} tokens")
    ctx.close()


@pytest.mark.parametrize("key,value", [("stack_pdl", 0), ("stack_fuse", 0), ("stack_fuse", 2), ("stack_tc", 0), ("stack_tc", 2), ("tc_block", 64), ("delta_tc", 0)])
def test_every_form_of_a_round(L, key, value):
    """The alternatives behind the tuning keys compute the same: prompts, then one to four requests decode together."""
    raw = M.config([M.layer(heads=20, kv_heads=5, d_dim=64, d_vdim=64), M.layer(ff=0), M.layer()], loop=(0, 2, 2))
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
        check(r.logits(k), M.reference(raw, w, toks[k]), BF16, k)
    ctx.close()


def test_long_decoding(L):
    raw = M.MIXED
    w = M.weights(raw, 61)
    toks = M.random_tokens(raw, 400, 62)
    want = M.reference(raw, w, toks)
    for dt in (F32, BF16):
        check(whole(L, raw, w, toks, dt, [5] + [1] * 400), want, dt)


# ------------------------------------------------------------------ single keys that show

@pytest.fixture(scope="module")
def planted():
    key, query = 5, 9
    out = []
    for heads, kv_heads in ((4, 4), (6, 2)):
        raw = M.config([M.layer(heads=heads, kv_heads=kv_heads, dim=32, vdim=32, rot=M.rotary(16, 1e4), scale=1.5), M.layer()])
        w = M.silence(M.weights(raw, 71), raw, "right")
        out.append((raw, M.plant_key(raw, w, key, query), key, query))
    return out


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("case", [0, 1])
def test_one_far_key(L, planted, dt, case):
    """The last token's first-layer attention falls on ONE earlier key, at every kind of place (first token, page and tile borders,
    next to the query); the restatement without that key differs by far more than the tolerance."""
    raw, w, key, query = planted[case]
    _, ctx = M.load(L, raw, w, dt, tokens=320)
    r = M.Runner(ctx)
    n = 260
    base = M.random_tokens(raw, n, 72, avoid=(key, query))
    base[-1] = query
    lost = M.reference(raw, w, base)[-1:]
    for p in (0, 1, 15, 16, 62, 63, 64, 65, 127, 128, 191, 192, 255, 256, 258):
        toks = list(base)
        toks[p] = key
        want = M.reference(raw, w, toks)[-1:]
        assert M.rel_err(lost, want) > 0.1, "the planted key does not show"
        for cuts in (None, [n - 1, 1], [n - 2, 2], [100]):
            check(r.whole(toks, cuts)[-1:], want, dt, f"key at {p}, portions {cuts}")
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_the_next_token_is_not_seen(L, planted, dt):
    """The key right AFTER the query (same portion, tile border included) must not count."""
    raw, w, key, query = planted[1]
    _, ctx = M.load(L, raw, w, dt, tokens=256)
    r = M.Runner(ctx)
    for at in (0, 1, 7, 15, 62, 63, 64, 126, 127):
        toks = M.random_tokens(raw, 140, 80 + at, avoid=(key, query))
        toks[at], toks[at + 1] = query, key
        want = M.reference(raw, w, toks)
        for cuts in (None, [at + 2], [at + 1, 2]):
            check(r.whole(toks, cuts)[:at + 1], want[:at + 1], dt, f"query at {at}, portions {cuts}")
    ctx.close()


def test_splits_of_a_long_context(L):
    """A planted key in every split of a decoded token's context, with pages that are not in order."""
    raw = M.config([M.layer(heads=4, kv_heads=2, dim=32, vdim=32, rot=M.rotary(16, 1e4), scale=1.5, ff=0)])
    key, query = 5, 9
    w = M.plant_key(raw, M.silence(M.weights(raw, 74), raw, "right"), key, query)
    _, ctx = M.load(L, raw, w, BF16, tokens=2048)
    r = M.Runner(ctx)
    base = M.random_tokens(raw, 1500, 75, avoid=(key, query))
    base[-1] = query
    r.step([("x", base[:70]), ("y", base[:300])])
    r.step([("x", base[:1])], end=["y"])  # the next request's pages come from the middle of the pool
    for p in (3, 330, 777, 1100, 1498):
        toks = list(base)
        toks[p] = key
        want = M.reference(raw, w, toks)[-1:]
        check(r.whole(toks, [700, 799, 1])[-1:], want, BF16, f"key at {p}")
    ctx.close()


# ------------------------------------------------------------------ recurrent state

def slow_decay(raw, seed):
    """The delta rule alone, with decays near one: what the first token left behind still shows hundreds of tokens later."""
    w = M.silence(M.weights(raw, seed), raw, "left", "ff")
    for k in w:
        if k.endswith("A_log"):
            w[k] = torch.full_like(w[k], -7.0)
        if k.endswith("right.b"):  # small steps: later tokens do not overwrite the first
            w[k] = torch.zeros_like(w[k])
    return w


@pytest.mark.parametrize("dt", [F32])
def test_the_state_reaches_back_to_the_first_token(L, dt):
    raw = M.config([M.layer(d_heads=4, d_kv_heads=2, d_dim=64, d_vdim=40)])
    w = slow_decay(raw, 91)
    toks = M.random_tokens(raw, 120, 92)
    want = M.reference(raw, w, toks)
    other = M.reference(raw, w, [(toks[0] + 1) % raw["vocab"]] + toks[1:])
    assert M.rel_err(other[-1:], want[-1:]) > 1e-3
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    for cuts in (None, [1], [2], [3, 8, 5], [60], [119, 1], [7, 1]):
        check(r.whole(toks, cuts), want, dt, f"portions {cuts}")
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("decay", [-9.0, 0.0, 3.0])
def test_decays_from_none_to_complete(L, dt, decay):
    """Decay rates from nothing to e^-20 a token and more: products of decays vanish, nothing divides by them."""
    raw = M.config([M.layer(d_dim=32, d_vdim=32), M.layer(d_heads=2, d_kv_heads=1)])
    w = M.silence(M.weights(raw, 93), raw, "left")
    for k in w:
        if k.endswith("A_log"):
            w[k] = torch.full_like(w[k], decay)
    toks = M.random_tokens(raw, 90, 94)
    want = M.reference(raw, w, toks)
    tol = M.tolerance(dt, raw, w, toks, want)
    for cuts in (None, [1], [30]):
        got = whole(L, raw, w, toks, dt, cuts)
        assert torch.isfinite(got).all()
        check(got, want, dt, f"decay {decay}, portions {cuts}", tol)


def test_repeated_keys_with_full_steps(L):
    """The same token over and over with steps near one: the triangle of a block is far from the identity."""
    raw = M.config([M.layer(ff=0)])
    w = M.silence(M.weights(raw, 95), raw, "left")
    for k in w:
        if k.endswith("right.b"):
            w[k] = (w[k].float() * 12).to(torch.bfloat16)
    toks = [7] * 30 + [7, 8] * 10 + [9] * 20
    want = M.reference(raw, w, toks)
    for cuts in (None, [1], [5]):
        check(whole(L, raw, w, toks, F32, cuts), want, F32, f"portions {cuts}")


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
    raw = M.config([M.layer(), M.layer(heads=6, kv_heads=2, dim=36, conv=3, ff=0), M.layer(d_heads=3, d_kv_heads=1)], loop=(1, 3, 2))
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
    raw = M.config([M.layer(), M.layer(ff=0)], vocab=102)
    w = M.weights(raw, 121)
    _, ctx = M.load(L, raw, w, dt, tokens=1024, max_seqs=8)
    prompts = [np.array(M.random_tokens(raw, n, 130 + n), np.uint32) for n in (4, 20)]
    args = L.SampleArgs.new(0.8, 0.9, 40)
    a = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7)
    c = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=8)
    assert a == L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7) and a != c
    assert all(0 <= t < raw["vocab"] for s in a + c for t in s)
    ctx.close()


def test_recurrent_state_limits_what_can_be_resumed(L):
    raw = M.MIXED
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
    raw = M.MIXED
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
    """Captured decode rounds alternate the halves of the convolutions' state through the descriptor, not through the graph."""
    raw = M.config([M.layer(), M.layer()])
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
    check(got[0], torch.stack([wa[0], wa[65], wb[1]]), dt)
    check(got[2], torch.stack([wa[69], wb[11]]), dt)
    assert not os.path.exists(tmp_path / "1.f32")
