"""Zefedra on the GPU against the plain restatement (f64, whole sequences): each mechanism, every way of cutting a sequence
into rounds, shared batches, pages and state slots used again, keys far away, generation through the engine."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import zefedra_models as M
import zefedra_ref as Z

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BF16, F32 = 1, 2


@pytest.fixture(autouse=True)
def default_tuning(L):
    yield
    for k, v in (("expand_min", 0), ("stack_pdl", 1), ("stack_fuse", 1), ("latent_tc", 1), ("tc_block", 256)):
        L.set_tuning(k, v)


def check(got, want, dt, what=""):
    e = M.rel_err(got, want)
    assert e <= M.TOL[dt], f"{what}: error {e:.3g} > {M.TOL[dt]}"
    return e


# ------------------------------------------------------------------ mechanisms alone

def only(w, raw, keep):
    """Weights with everything but one mechanism of layer 0 switched off."""
    w = dict(w)
    if keep != "shift":
        w["l0.shift"] = torch.zeros_like(w["l0.shift"])
    if keep == "ff":
        w["l0.mix.o"] = torch.zeros_like(w["l0.mix.o"])
    return w


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("keep,layer", [("ff", M.layer()), ("mixer", M.layer(ff=0)), ("gate", M.layer(True, ff=0)), ("shift", M.layer(ff=0))])
def test_mechanism_alone(L, dt, keep, layer):
    raw = M.config([layer])
    w = only(M.weights(raw, 1), raw, keep)
    if keep == "ff":  # both branches of the activation, large and small
        w["l0.mlp.up"] = (w["l0.mlp.up"].float() * 2).to(torch.bfloat16)
    toks = M.random_tokens(raw, 70, 2)
    want, stream = M.reference(raw, w, toks, True)
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    got = r.whole(toks)
    x = ctx.hidden(70).cpu().double()
    scale = float(stream[-1].abs().max())
    assert float((x - stream[-1]).abs().max()) / scale <= (2e-5 if dt == F32 else 2e-2)
    check(got, want, dt, keep)
    ctx.close()


@pytest.mark.parametrize("p,q", [(-30.0, 25.0), (25.0, -30.0), (0.0, 0.0)])
def test_activation_parameters_far_from_zero(L, p, q):
    raw = M.config([M.layer()])
    w = M.weights(raw, 4)
    w["l0.mlp.act"] = torch.tensor([p, q], dtype=torch.bfloat16)
    toks = M.random_tokens(raw, 20, 5)
    _, ctx = M.load(L, raw, w, F32)
    check(M.Runner(ctx).whole(toks), M.reference(raw, w, toks), F32)
    ctx.close()


def test_eps_matters_and_is_read(L):
    raw = M.config([M.layer(), M.layer(True)], eps=0.3)
    w = M.weights(raw, 6)
    toks = M.random_tokens(raw, 30, 7)
    _, ctx = M.load(L, raw, w, F32)
    got = M.Runner(ctx).whole(toks)
    check(got, M.reference(raw, w, toks), F32)
    assert M.rel_err(got, M.reference(dict(raw, norm={"eps": 1e-5}), w, toks)) > 1e-2
    ctx.close()


# ------------------------------------------------------------------ sizes

SIZES = {
    "one_head_ones": M.config([M.layer(heads=1, dim=1, vdim=1, q_rank=1, kv_rank=1, ff=1)], width=8, vocab=7),
    "many_heads": M.config([M.layer(True, heads=37, dim=8, vdim=8, q_rank=24, kv_rank=64, ff=64)], width=64, vocab=64),
    "seventeen_heads": M.config([M.layer(True, heads=17, dim=16, vdim=32, q_rank=64, kv_rank=200, ff=64)], width=128, vocab=96),
    "wide_latent": M.config([M.layer(heads=4, dim=64, vdim=128, q_rank=96, kv_rank=512, ff=96), M.layer(True, heads=6, dim=192, vdim=64, q_rank=100, kv_rank=320, ff=0)], width=160, vocab=150),
    "unexpandable": M.config([M.layer(heads=2, dim=256, vdim=160, q_rank=64, kv_rank=96, ff=64)], width=96, vocab=80),
    "mixed": M.MIXED,
    "wide": M.config([M.layer(heads=5, dim=48, vdim=40, q_rank=130, kv_rank=90, ff=700)], width=1032, vocab=333),
    "shared_twice": M.config([M.layer(True), M.layer(True, weights_of=0), M.layer(True, weights_of=1), M.layer()]),
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
    for expand in ((0,) if dt == F32 else (2, -1)):
        L.set_tuning("expand_min", expand, ctx)
        check(r.whole(toks), want, dt, f"whole, expand_min {expand}")
        check(r.whole(toks, [120] + [1] * 30), want, dt, f"decoded, expand_min {expand}")
    assert ctx.device_status() == 0 and ctx.pages_free == ctx.pages_total
    ctx.close()


# ------------------------------------------------------------------ schedules

@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("page_tokens", [64, 16, 128])
def test_portions(L, dt, page_tokens):
    raw = M.MIXED
    w = M.weights(raw, 21)
    toks = M.random_tokens(raw, 200, 22)
    want = M.reference(raw, w, toks)
    _, ctx = M.load(L, raw, w, dt, page_tokens=page_tokens)
    r = M.Runner(ctx)
    for expand in ((0,) if dt == F32 else (0, 2, -1)):
        L.set_tuning("expand_min", expand, ctx)
        for cuts in ([1], [2], [3, 1, 2], [7, 64, 2], [64], [65, 63], [100, 2, 2], [199, 1]):
            check(r.whole(toks, cuts), want, dt, f"portions {cuts}, expand_min {expand}, pages of {page_tokens}")
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


@pytest.mark.parametrize("key", ["latent_tc", "stack_fuse", "stack_pdl", "tc_block"])
def test_every_form_of_a_decode_round(L, key):
    """The alternatives behind the tuning keys compute the same: two requests decode together, then one alone."""
    raw = M.config([M.layer(True, heads=20, dim=32, vdim=16, q_rank=48, kv_rank=128, ff=64), M.layer(heads=3)])
    w = M.weights(raw, 65)
    a, b = M.random_tokens(raw, 290, 66), M.random_tokens(raw, 150, 67)
    want = {"a": M.reference(raw, w, a), "b": M.reference(raw, w, b)}
    _, ctx = M.load(L, raw, w, BF16)
    L.set_tuning(key, 64 if key == "tc_block" else 0, ctx)
    r = M.Runner(ctx)
    r.step([("a", a[:200]), ("b", b[:120])])
    for i in range(90):
        r.step([("a", a[200 + i:201 + i])] + ([("b", b[120 + i:121 + i])] if i < 30 else []))
    for k in want:
        check(r.logits(k), want[k], BF16, k)
    ctx.close()


def test_long_decoding(L):
    raw = M.MIXED
    w = M.weights(raw, 61)
    toks = M.random_tokens(raw, 400, 62)
    want = M.reference(raw, w, toks)
    for dt in (F32, BF16):
        _, ctx = M.load(L, raw, w, dt)
        check(M.Runner(ctx).whole(toks, [5] + [1] * 400), want, dt)
        ctx.close()


# ------------------------------------------------------------------ single keys that show

@pytest.fixture(scope="module")
def planted():
    raw = M.config([M.layer(heads=4, dim=32, vdim=32, q_rank=48, kv_rank=64), M.layer(True)])
    w = M.weights(raw, 71)
    w["l0.shift"] = torch.zeros_like(w["l0.shift"])
    key, query = 5, 9
    return raw, M.plant_key(raw, w, 0, key, query, 14.0), key, query


@pytest.mark.parametrize("dt", [F32, BF16])
@pytest.mark.parametrize("expand", [2, -1])
def test_one_far_key(L, planted, dt, expand):
    """The last token's first-layer attention falls on ONE earlier key, at every kind of place (first token, page borders,
    next to the query); the restatement without that key differs by far more than the tolerance."""
    raw, w, key, query = planted
    _, ctx = M.load(L, raw, w, dt, tokens=320)
    L.set_tuning("expand_min", expand, ctx)
    r = M.Runner(ctx)
    n = 260
    base = M.random_tokens(raw, n, 72, avoid=(key, query))
    base[-1] = query
    lost = M.reference(raw, w, base)[-1:]
    for p in (0, 1, 62, 63, 64, 65, 127, 128, 191, 192, 255, 256, 258):
        toks = list(base)
        toks[p] = key
        want = M.reference(raw, w, toks)[-1:]
        assert M.rel_err(lost, want) > 0.2, "the planted key does not show"
        for cuts in (None, [n - 1, 1], [n - 2, 2], [100]):
            check(r.whole(toks, cuts)[-1:], want, dt, f"key at {p}, portions {cuts}")
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_the_next_token_is_not_seen(L, planted, dt):
    """The key right AFTER the query (same portion, tile border included) must not count."""
    raw, w, key, query = planted
    _, ctx = M.load(L, raw, w, dt, tokens=256)
    r = M.Runner(ctx)
    for at in (0, 1, 62, 63, 64, 126, 127):
        toks = M.random_tokens(raw, 140, 80 + at, avoid=(key, query))
        toks[at], toks[at + 1] = query, key
        want = M.reference(raw, w, toks)
        for expand in (2, -1):
            L.set_tuning("expand_min", expand, ctx)
            check(r.whole(toks)[:at + 1], want[:at + 1], dt, f"query at {at}, expand_min {expand}")
    ctx.close()


def test_running_maximum_grows_tile_by_tile(L, planted):
    """Several planted keys whose scores grow along the sequence: the online softmax rescales at every tile."""
    raw, w, key, query = planted
    w = dict(w)
    e = w["embed"].clone()
    for i, t in enumerate((11, 12, 13, 14)):  # directions ever closer to the planted key's
        mix = 0.5 + 0.12 * i
        e[t] = (mix * e[key].float() + (1 - mix) * e[t].float()).to(torch.bfloat16)
    w["embed"] = e
    toks = M.random_tokens(raw, 300, 90, avoid=(key, query, 11, 12, 13, 14))
    for i, t in enumerate((11, 12, 13, 14, key)):
        toks[10 + 64 * i:14 + 64 * i] = [t] * 4
    toks[-1] = query
    want = M.reference(raw, w, toks)
    for dt in (F32, BF16):
        _, ctx = M.load(L, raw, w, dt, tokens=320)
        r = M.Runner(ctx)
        for expand in (2, -1):
            L.set_tuning("expand_min", expand, ctx)
            check(r.whole(toks)[-1:], want[-1:], dt)
            check(r.whole(toks, [299, 1])[-1:], want[-1:], dt)
        ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_token_shift_across_portions(L, dt):
    """With shift weights near one a token's mixer reads the PREVIOUS token: a lost, stale or doubled state shows."""
    raw = M.config([M.layer(), M.layer(True)])
    w = M.weights(raw, 91)
    for k in ("l0.shift", "l1.shift"):
        w[k] = torch.full_like(w[k], 0.96875)
    toks = M.random_tokens(raw, 24, 92)
    want = M.reference(raw, w, toks)
    zero = dict(w, **{k: torch.zeros_like(w[k]) for k in ("l0.shift", "l1.shift")})
    assert M.rel_err(M.reference(raw, zero, toks), want) > 0.3
    _, ctx = M.load(L, raw, w, dt)
    r = M.Runner(ctx)
    for cuts in (None, [1], [2], [3], [1, 2, 4]):
        check(r.whole(toks, cuts), want, dt, f"portions {cuts}")
    ctx.close()


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
    raw = M.MIXED
    w = M.weights(raw, 101)
    prompts = [M.random_tokens(raw, n, 110 + n) for n in (5, 70, 1, 33)]
    want = [greedy(raw, w, p, 10) for p in prompts]
    _, ctx = M.load(L, raw, w, dt, tokens=1024, max_seqs=8)
    ctx.set_cuda_graph(graph)

    def compare(got):
        for g, (ids, margins) in zip(got, want):
            for a, b, m in zip(g, ids, margins):
                if a != b:
                    assert dt == BF16 and m < 0.1, (g, ids, m)
                    break
    compare(L.generate(ctx, [np.array(p, np.uint32) for p in prompts], 10))
    compare(L.generate_continuous(ctx, [np.array(p, np.uint32) for p in prompts], 10, max_round_tokens=24, prefill_chunk=16))
    assert ctx.pages_free == ctx.pages_total and ctx.device_status() == 0
    ctx.close()


@pytest.mark.parametrize("dt", [F32, BF16])
def test_seeded_sampling_replays(L, dt):
    raw = M.config([M.layer(), M.layer(True)], vocab=102)
    w = M.weights(raw, 121)
    _, ctx = M.load(L, raw, w, dt, tokens=1024, max_seqs=8)
    prompts = [np.array(M.random_tokens(raw, n, 130 + n), np.uint32) for n in (4, 20)]
    args = L.SampleArgs.new(0.8, 0.9, 40)
    a = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7)
    b = L.generate_continuous(ctx, prompts, 12, max_round_tokens=8, sample_args=args, seed=7)
    c = L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=8)
    assert a == L.generate_continuous(ctx, prompts, 12, sample_args=args, seed=7) and a != c
    assert dt == BF16 or a == b
    assert all(0 <= t < raw["vocab"] for s in a + b + c for t in s)
    ctx.close()


def test_recurrent_state_limits_what_can_be_resumed(L):
    raw = M.MIXED
    w = M.weights(raw, 141)
    _, ctx = M.load(L, raw, w, F32, tokens=512, max_seqs=2)
    out = torch.zeros(4, 2, dtype=torch.int32, device="cuda")
    a, b, c = (ctx.seq_create() for _ in range(3))
    ctx.step([(a, 0, 5)], [1, 2, 3, 4, 5], out)
    assert [ctx.seq_resumable(a, n) for n in (3, 5, 9)] == [0, 5, 5]
    for pos in (4, 6):
        with pytest.raises(L.LcuError) as e:
            ctx.step([(a, pos, 1)], [6], out)
        assert e.value.code == L.ERR_STATE
    ctx.step([(b, 0, 1)], [1], out)
    with pytest.raises(L.LcuError) as e:  # both state slots are taken
        ctx.step([(c, 0, 1)], [1], out)
    assert e.value.code == L.ERR_NO_PAGES
    ctx.seq_free(b)
    ctx.step([(c, 0, 1), (a, 5, 1)], [1, 6], out)
    ctx.step([(a, 0, 2)], [1, 2], out)  # starting again is always possible
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
    """Captured decode rounds alternate the halves of the state buffer through the descriptor, not through the graph."""
    raw = M.config([M.layer(), M.layer(True)])
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


def test_logits_of_llama_rounds(L):
    """lcu_step_logits on a LLaMA context: the asked rows equal the head of rounds that end there."""
    cfg = L.CONFIGS["tiny"]
    ctx = L.load_model(cfg, L.synth_weights_numpy(cfg, 0))
    toks = np.arange(3, 19, dtype=np.uint32)
    s = ctx.seq_create()
    rows = ctx.step_logits([(s, 0, 16)], toks, [4, 15]).cpu()
    out = torch.zeros(2, 2, dtype=torch.int32, device="cuda")
    for n, row in ((5, rows[0]), (16, rows[1])):
        t = ctx.seq_create()
        ctx.step([(t, 0, n)], toks[:n], out)
        assert float((ctx.logits(1)[0].float().cpu() - row).abs().max()) < 5e-3
        ctx.seq_free(t)
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
