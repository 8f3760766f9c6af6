"""Gunulorn without a GPU: configuration, packing, and the restatement's mechanisms."""
import math

import pytest
import torch

import gunulorn_models as M
import gunulorn_ref as R

F64 = torch.float64


def test_configuration_is_read_from_the_file(L):
    from llama_cu_b200 import layered as Y
    cfg = M.cfg_of(M.MIXED)
    assert (cfg.d, cfg.vocab, cfg.eps, cfg.arch, cfg.logit_scale, cfg.logit_cap) == (72, 101, 1e-5, "Gunulorn", 1.5, 5.0)
    a, b, c, d = (cfg.layers[i].mixer for i in range(4))
    assert (a.heads, a.kv_heads, a.dim, a.v_dim, a.scale, a.window, a.keep_first, a.sink, a.rot_values, a.conv, a.kv_from) == (4, 2, 20, 28, 0.25, 9, 3, 1, True, 0, -1)
    assert a.rot == Y.Rotary(8, 300.0, adjacent=True) and not a.bias and a.qk_norm == 0 and not a.head_temp and not a.out_gate
    assert (b.heads, b.kv_heads, b.dim, b.v_dim, b.scale, b.window, b.keep_first, b.sink, b.rot, b.conv, b.head_temp, b.kv_from) == (6, 2, 20, 12, 0.3, 0, 0, 2, None, 3, True, -1)
    assert (c.window, c.keep_first, c.rot.dims) == (30, 70, 36) and (d.conv, d.kv_from) == (2, 1)
    assert cfg.layers[0].ff == Y.PolyNormFf(50) and cfg.layers[3].ff == 0
    assert cfg.layers[1].ff == Y.GluFf(30, math.inf, 1.0, 0.0, 5, 2, softmax=True, identity=2)
    o = cfg.layer_descs()
    assert all(x.mixer == L.MIX_ATTENTION and x.pre_norm and not x.post_norm for x in o)
    assert [x.parallel_ff for x in o] == [1, 1, 1, 0, 1, 1, 1, 0] and [x.kv_from for x in o] == [0, 0, 0, 2, 0, 0, 2, 0]
    assert [x.window for x in o] == [9, 0, 30, 0, 70, 0, 0, 1] and [x.keep_first for x in o] == [3, 0, 70, 0, 0, 0, 0, 5]
    assert [x.sink for x in o] == [1, 2, 1, 2, 1, 2, 2, 1] and [x.conv for x in o] == [0, 3, 0, 2, 0, 4, 1, 0] and [x.head_temp for x in o] == [0, 1, 0, 1, 0, 1, 1, 0]
    assert [x.rot_values for x in o] == [1, 0, 1, 0, 1, 0, 0, 1] and (o[0].rot_dims, o[0].rot_base, o[0].rot_adjacent) == (8, 300.0, 1)
    assert (o[0].ff, o[0].ff_act, o[0].ff_bias, o[0].experts) == (50, L.ACT_POLYNORM, 1, 0)
    assert (o[1].ff, o[1].ff_act, o[1].experts, o[1].top, o[1].identity, o[1].route_softmax, o[1].shared_ff, o[1].glu_limit) == (30, L.ACT_GLU, 5, 2, 2, 1, 0, math.inf)
    assert (o[0].logit_scale, o[0].logit_cap, o[0].embed_scale, o[0].pair_buckets) == (1.5, 5.0, 1.0, 0)


@pytest.mark.parametrize("bad", [{"type": "latent_attention"}, {"mlp": {"kind": "shared"}}])
def test_unknown_parts_are_refused(L, bad):
    with pytest.raises(ValueError):
        M.cfg_of(M.config([dict(M.conv(), **bad)]))


@pytest.mark.parametrize("layers", [[M.conv(kv_from=0)], [M.window(), M.conv(kv_from=0)], [M.conv(), M.conv(kv_from=0), M.conv(kv_from=1)], [M.conv(kv_from=1), M.conv()]])
def test_keys_come_from_an_earlier_layer_of_the_same_kind_with_its_own(L, layers):
    with pytest.raises(ValueError):
        M.cfg_of(M.config(layers))


def test_missing_and_misshapen_tensors_are_named(L):
    from llama_cu_b200 import gunulorn, layered
    cfg, w = M.cfg_of(M.MIXED), M.weights(M.MIXED)
    for name, change in (("l1.mix.sink", lambda t: None), ("l1.mix.k.conv", lambda t: t[:, 1:]), ("head", lambda t: t[:-1]), ("l1.mlp.e2.down", lambda t: None),
                         ("l1.mlp.correction", lambda t: t[:-2]), ("l0.mlp.act", lambda t: t[:3]), ("l0.mlp.down.b", lambda t: None)):
        bad = dict(w)
        t = change(bad.pop(name))
        if t is not None:
            bad[name] = t
        with pytest.raises(ValueError, match=name):
            list(gunulorn.pack(cfg, layered.Tensors(bad)))


def test_tensor_names(L):
    from llama_cu_b200 import gunulorn
    names = set(gunulorn.tensor_shapes(M.cfg_of(M.MIXED)))
    assert {"l3.mix.q", "l3.mix.q.conv", "l3.mix.temp", "l3.mix.sink", "l3.mix.o", "head", "l0.mlp.up.b", "l2.mlp.router"} <= names
    assert not {"l3.mix.k", "l3.mix.k.conv", "l3.mix.v", "l3.mix.v.conv", "l3.norm2", "l0.mix.sink", "l0.mix.q.conv", "l1.mlp.e5.up", "l2.mlp.up"} & names


def test_packing_pads_with_zeros_and_keeps_every_number(L):
    from llama_cu_b200 import gunulorn, layered
    cfg, w = M.cfg_of(M.MIXED), M.weights(M.MIXED, steady=False)
    p = dict(gunulorn.pack(cfg, layered.Tensors(w)))
    # q 6 x 32 | k 2 x 32 | v 2 x 16
    x, c = p[(1, L.W_MIX_IN)], p[(1, L.W_ATT_CONV)]
    assert x.shape == (192 + 64 + 32, 128) and torch.equal(x[224:244, :72], w["l1.mix.k"][20:40]) and torch.equal(x[272:284, :72], w["l1.mix.v"][12:24])
    assert c.shape == (3, 288) and torch.equal(c[:, 32:52], w["l1.mix.q.conv"][20:40].float().T) and torch.equal(c[:, 272:284], w["l1.mix.v.conv"][12:24].float().T)
    assert float(c.abs().sum()) == pytest.approx(sum(float(w[f"l1.mix.{n}.conv"].float().abs().sum()) for n in "qkv"), rel=1e-5)
    assert torch.equal(p[(1, L.W_SINK)], w["l1.mix.sink"].float()) and torch.equal(p[(1, L.W_HEAD_TEMP)], w["l1.mix.temp"].float())
    assert p[(3, L.W_MIX_IN)].shape == (192, 128) and p[(3, L.W_ATT_CONV)].shape == (2, 192)
    assert p[(0, L.W_MIX_IN)].shape == (4 * 32 + 2 * 32 + 2 * 32, 128) and (0, L.W_ATT_CONV) not in p and (0, L.W_SINK) not in p
    o = p[(0, L.W_ATT_OUT)]
    assert o.shape == (128, 128) and torch.equal(o[:72, 32:60], w["l0.mix.o"][:, 28:56]) and not o[:, 28:32].any() and not o[72:].any()
    # the dense feed-forward
    assert p[(0, L.W_UP)].shape == (64, 128) and torch.equal(p[(0, L.W_UP)][:50, :72], w["l0.mlp.up"]) and torch.equal(p[(0, L.W_UP_BIAS)][:50], w["l0.mlp.up.b"].float())
    assert torch.equal(p[(0, L.W_DOWN_BIAS)][:72], w["l0.mlp.down.b"].float()) and not p[(0, L.W_DOWN_BIAS)][72:].any() and torch.equal(p[(0, L.W_ACT)], w["l0.mlp.act"].float())
    # experts: gate and up rows in turn; the router has rows for those without matrices
    u = p[(1, L.W_UP)]
    assert u.shape == (5, 128, 128) and torch.equal(u[3, 0:60:2, :72], w["l1.mlp.e3.gate"]) and torch.equal(u[3, 1:61:2, :72], w["l1.mlp.e3.up"]) and not u[3, 60:].any()
    assert p[(1, L.W_ROUTER)].shape == (8, 128) and torch.equal(p[(1, L.W_ROUTER)][:7, :72], w["l1.mlp.router"]) and torch.equal(p[(1, L.W_CORRECTION)][:7], w["l1.mlp.correction"].float())
    assert torch.equal(p[(1, L.W_NORM1)][:72], w["l1.norm1"].float()) and torch.equal(p[(1, L.W_NORM2)][:72], w["l1.norm2"].float())
    assert not any((3, k) in p for k in (L.W_NORM2, L.W_UP, L.W_ROUTER)) and (1, L.W_POST1) not in p
    assert torch.equal(p[(-1, L.W_LM_HEAD)][:101, :72], w["head"]) and torch.equal(p[(-1, L.W_OUT_NORM)][:72], w["final.norm"].float())


def test_pages_hold_the_keys_of_layers_that_have_their_own(L):
    assert M.cfg_of(M.MIXED).kv_bytes_per_token() == 2 * (2 * (32 + 32) + 2 * (32 + 16) + (48 + 16) + 4 * (16 + 32) + (48 + 32) + 2 * (32 + 32))


# ---- the restatement against closed forms

def test_reference_convolution():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    assert R.causal_conv(x, torch.tensor([[3.0, 2.0]], dtype=F64))[:, 0].tolist() == [2.0, 23.0, 230.0]
    assert R.causal_conv(x, torch.tensor([[2.0]], dtype=F64))[:, 0].tolist() == [2.0, 20.0, 200.0]


def test_reference_turns_neighbours_and_back():
    x = torch.zeros(3, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 5] = 1.0, 1.0, 7.0
    y = R.turn(x, 4, 100.0)
    a, b = 2.0, 2.0 * 100.0 ** -0.5
    assert torch.allclose(y[2, 0], torch.tensor([math.cos(a), math.sin(a), -math.sin(b), math.cos(b), 0.0, 7.0], dtype=F64))
    assert torch.allclose(R.turn(y, 4, 100.0, -1), x)


def test_reference_window_and_kept_tokens():
    assert R.visible(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]] and R.visible(2).int().tolist() == [[1, 0], [1, 1]]
    assert R.visible(5, 2, 1).int().tolist() == [[1, 0, 0, 0, 0], [1, 1, 0, 0, 0], [1, 1, 1, 0, 0], [1, 0, 1, 1, 0], [1, 0, 0, 1, 1]]
    assert torch.equal(R.visible(6, 2, 9), R.visible(6))


def test_reference_sinks():
    q = torch.zeros(2, 2, 1, dtype=F64)
    v = torch.tensor([[[3.0]], [[9.0]]], dtype=F64)
    got = R.softmax_attention(q, q[:, :1], v, torch.ones(2, dtype=F64), torch.tensor([0.0, math.log(2.0)], dtype=F64))
    assert got[:, 0, 0].tolist() == pytest.approx([1.5, 4.0]) and got[:, 1, 0].tolist() == pytest.approx([1.0, 3.0])
    far = R.softmax_attention(q, q[:, :1], v, torch.ones(2, dtype=F64), torch.full((2,), -1e9, dtype=F64))
    assert far[:, 0, 0].tolist() == [3.0, 6.0]


def test_reference_normed_powers():
    z = torch.tensor([[1.0, -2.0]], dtype=F64)
    got = R.poly_norm(z, torch.tensor([1.0, 10.0, 100.0, 7.0], dtype=F64), 0.0)
    want = [s * 1 / 2.5 ** 0.5 + 10 * q / 8.5 ** 0.5 + 100 * c / 32.5 ** 0.5 + 7 for s, q, c in ((1, 1, 1), (-2, 4, -8))]
    assert got[0].tolist() == pytest.approx(want)


def test_reference_routing():
    r = {"router": torch.tensor([[0.0], [2.0], [1.0]], dtype=F64), "correction": torch.tensor([5.0, 0.0, 0.0], dtype=F64)}
    e, s = R.route(torch.ones(1, 1, dtype=F64), r, "", 2)
    assert e.tolist() == [[0, 1]] and s.tolist()[0] == pytest.approx([1 / (1 + math.exp(2)), math.exp(2) / (1 + math.exp(2))])


def test_reference_experts_that_return_their_input():
    one = torch.ones(1, 1, dtype=F64)
    w = {"router": torch.zeros(2, 1, dtype=F64), "correction": torch.zeros(2, dtype=F64), "e0.gate": 2 * one, "e0.up": 3 * one, "e0.down": 5 * one}
    m = {"router": {"experts": 1, "identity": 1, "top": 2}}
    assert float(R.experts(one, w, "", m)) == pytest.approx(0.5 * (5 * 2 / (1 + math.exp(-2)) * 3) + 0.5)


def test_reference_soft_cap():
    assert R.soft_cap(torch.tensor([0.0, 1e9, 3.0], dtype=F64), 2.0).tolist() == pytest.approx([0.0, 2.0, 2 * math.tanh(1.5)])


def test_reference_is_causal():
    raw = M.MIXED
    w = M.weights(raw)
    a, b = M.random_tokens(raw, 12, 1), M.random_tokens(raw, 12, 2)
    ya, yb = M.reference(raw, w, a), M.reference(raw, w, a[:7] + b[7:])
    assert torch.allclose(ya[:7], yb[:7]) and not torch.allclose(ya[7], yb[7])


def test_reference_sublayers_read_the_same_input():
    raw = M.config([M.window(mlp=M.dense())])
    w = M.weights(raw, 3)
    toks = M.random_tokens(raw, 9, 4)
    x = w["embed"].double()[toks]
    parts = [M.reference(raw, M.silence(w, raw, off), toks, True)[1][0] - x for off in ("mixer", "ff")]
    assert torch.allclose(M.reference(raw, w, toks, True)[1][0] - x, parts[0] + parts[1])


def test_steady_routes_use_every_expert_but_those_that_are_never_chosen():
    raw = M.config([M.window(), M.conv(mlp=M.moe(6, 8, 3, 4)), M.conv(mlp=M.moe(6, 2, 1, 0))])
    w = M.weights(raw, 3)
    used, real = set(), R.route

    def spy(h, w, pre, top):
        e, s = real(h, w, pre, top)
        used.update((pre, int(x)) for x in e.flatten())
        return e, s
    R.route = spy
    try:
        M.reference(raw, w, M.random_tokens(raw, 90, 4))
    finally:
        R.route = real
    assert len(used) == 6 + 11 + 1
