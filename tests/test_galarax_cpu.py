"""Galarax without a GPU: configuration, the loop, packing, the library's own checks, and the restatement's mechanisms."""
import math

import pytest
import torch

import galarax_models as M
import galarax_ref as G


def cfg_of(raw):
    from llama_cu_b200 import galarax
    return galarax.read_config(raw)


def test_configuration_is_read_from_the_file(L):
    cfg = cfg_of(M.MIXED)
    assert (cfg.d, cfg.vocab, cfg.eps, cfg.arch) == (72, 101, 1e-5, "Galarax")
    a, b = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert (a.left.heads, a.left.kv_heads, a.left.dim, a.left.v_dim, a.left.scale) == (4, 2, 20, 12, 0.3)
    assert (a.left.rot.dims, a.left.rot.base, a.left.rot.factor, a.left.rot.original, a.left.rot.fast, a.left.rot.slow) == (8, 3e4, 3.0, 40, 16.0, 1.5)
    assert (b.right.heads, b.right.kv_heads, b.right.dim, b.right.v_dim, b.right.conv, cfg.layers[1].ff) == (3, 1, 40, 8, 3, 0)
    assert cfg.layers[2].mixer.left.rot.factor == 0
    o = cfg.layer_descs()
    assert o[0].mixer == L.MIX_ATTENTION | L.MIX_DELTA and o[0].pre_norm == 1 and o[0].token_shift == 0 and o[0].ff_act == L.ACT_RELU2
    assert (o[1].delta_heads, o[1].delta_dim, o[1].delta_conv, o[1].kv_heads, o[1].rot_base) == (3, 40, 3, 2, 1e3)


def test_the_loop_is_unrolled(L):
    runs = cfg_of(M.MIXED).layers
    assert [l.file_layer for l in runs] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [l.weights_of for l in runs] == [-1, -1, -1, 1, 2, 1, 2, -1]
    assert [l.step for l in runs] == [-1, 0, -1, 1, -1, 2, -1, -1]
    assert [l.add_embed for l in runs] == [False, False, False, True, False, True, False, False]
    assert [(i, t) for i, t in G.schedule(M.MIXED)] == [(l.file_layer, l.step if l.step >= 0 else None) for l in runs]
    whole = cfg_of(M.config([M.layer(), M.layer()], loop=(0, 2, 2))).layers
    assert [(l.weights_of, l.step, l.add_embed) for l in whole] == [(-1, 0, False), (-1, -1, False), (0, 1, True), (1, -1, False)]
    once = cfg_of(M.config([M.layer(), M.layer()], loop=(1, 2, 1))).layers
    assert [(l.weights_of, l.step, l.add_embed) for l in once] == [(-1, -1, False), (-1, 0, False)]
    assert [(l.step, l.add_embed) for l in cfg_of(M.config([M.layer()])).layers] == [(-1, False)]
    for bad in ((0, 3, 2), (1, 1, 2), (0, 1, 0)):
        with pytest.raises(ValueError):
            cfg_of(M.config([M.layer(), M.layer()], loop=bad))


@pytest.mark.parametrize("bad", [{"type": "latent_attention"}, {"mlp": {"kind": "experts", "ff": 8}}])
def test_unknown_parts_are_refused(L, bad):
    with pytest.raises(ValueError):
        cfg_of(M.config([dict(M.layer(), **bad)]))


def test_missing_and_misshapen_tensors_are_named(L):
    from llama_cu_b200 import galarax, layered
    cfg, w = cfg_of(M.MIXED), M.weights(M.MIXED)
    for name, change in (("l1.mix.right.A_log", lambda t: None), ("l2.mix.left.k.b", lambda t: t[:-1]), ("loop.step", lambda t: t[:2])):
        bad = dict(w)
        t = change(bad.pop(name))
        if t is not None:
            bad[name] = t
        with pytest.raises(ValueError, match=name):
            list(galarax.pack(cfg, layered.Tensors(bad)))


def test_packing_pads_with_zeros_and_keeps_every_number(L):
    from llama_cu_b200 import galarax, layered
    cfg, w = cfg_of(M.MIXED), M.weights(M.MIXED)
    p = {k: v for k, v in galarax.pack(cfg, layered.Tensors(w))}
    x, lt, rt = p[(0, L.W_MIX_IN)], "l0.mix.left.", "l0.mix.right."
    # q 4 x 32 | k 2 x 32 | v 2 x 16 | q 2 x 32 | k 2 x 32 | v 4 x 32 | g 4 x 32 | b 8 | a 8
    assert x.shape == (224 + 128 + 256 + 16, 128)
    assert torch.equal(x[32:52, :72], w[lt + "q"][20:40]) and torch.equal(x[160:180, :72], w[lt + "k"][20:40]) and torch.equal(x[208:220, :72], w[lt + "v"][12:24])
    assert torch.equal(x[256:268, :72], w[rt + "q"][12:24]) and torch.equal(x[288:300, :72], w[rt + "k"][:12]) and torch.equal(x[384:404, :72], w[rt + "v"][20:40])
    assert torch.equal(x[480:500, :72], w[rt + "g"][:20]) and torch.equal(x[608:612, :72], w[rt + "b"]) and torch.equal(x[616:620, :72], w[rt + "a"])
    names = [lt + n for n in "qkv"] + [rt + n for n in "qkvgba"]
    assert float(x.float().abs().sum()) == pytest.approx(sum(float(w[n].float().abs().sum()) for n in names), rel=1e-5)
    b = p[(0, L.W_MIX_BIAS)]
    assert b.shape == (224,) and torch.equal(b[32:52], w[lt + "q.b"][20:40].float()) and torch.equal(b[192:204], w[lt + "v.b"][:12].float()) and not b[204:208].any()
    c = p[(0, L.W_CONV)]
    assert c.shape == (4, 256) and torch.equal(c[:, 32:44], w[rt + "q.conv"][12:24].float().T) and torch.equal(c[:, 128:148], w[rt + "v.conv"][:20].float().T)
    o = p[(0, L.W_ATT_OUT)]
    assert o.shape == (128, 64) and torch.equal(o[:72, 16:28], w[lt + "o"][:, 12:24]) and not o[:, 12:16].any()
    o = p[(0, L.W_DELTA_OUT)]
    assert o.shape == (128, 128) and torch.equal(o[:72, 32:52], w[rt + "o"][:, 20:40])
    assert torch.equal(p[(0, L.W_DELTA_DECAY)][0, :4], w[rt + "A_log"].float()) and torch.equal(p[(0, L.W_DELTA_DECAY)][1, :4], w[rt + "dt_bias"].float())
    assert torch.equal(p[(0, L.W_NORM1)][:72], 1 + w["l0.norm1"].float()) and not p[(0, L.W_NORM1)][72:].any()
    assert torch.equal(p[(0, L.W_BRANCH_NORM)][1, :72], w["l0.mix.right.out"].float() / 2)
    assert torch.equal(p[(-1, L.W_OUT_NORM)][:72], 1 + w["final.norm"].float())
    assert torch.equal(p[(3, L.W_STEP)][:72], w["loop.step"][1].float()) and (3, L.W_MIX_IN) not in p and (1, L.W_UP) not in p


def test_pages_and_bytes(L):
    from dataclasses import replace
    cfg = cfg_of(M.MIXED)
    rows = [2 * (32 + 16), 2 * (48 + 32), 3 * (16 + 32), 80 + 80]
    assert cfg.kv_bytes_per_token() == 2 * (rows[0] + 3 * rows[1] + 3 * rows[2] + rows[3])
    assert replace(cfg, act_dtype=L.F32).kv_bytes_per_token() == 2 * cfg.kv_bytes_per_token()
    assert cfg.state_bytes_per_sequence() == 4 * (4 * 32 * 32 + 3 * 3 * 16 * 64 + 3 * 5 * 32 * 64 + 8 * 48 * 64)


def test_contexts_need_a_gpu_and_sane_descriptions(L):
    cfg = cfg_of(M.MIXED)
    for field, value in (("kv_heads", 3), ("dim", 300), ("mixer", 9), ("mixer", 3), ("rot_dims", 7), ("rot_dims", 40), ("delta_heads", 5), ("delta_v_dim", 257),
                         ("delta_conv", 0), ("ff_act", 1), ("token_shift", 1), ("pre_norm", 0), ("rot_slow", 0.0)):
        d = cfg.layer_descs()
        setattr(d[0], field, value)
        with pytest.raises(L.LcuError):
            L.Context(cfg.desc(), layers=d)
    if not torch.cuda.is_available():
        with pytest.raises(L.LcuError) as e:
            L.Context(cfg.desc(), layers=cfg.layer_descs())
        assert e.value.code == L.ERR_CUDA


# ---- the restatement against closed forms
def test_reference_rotation():
    rot = {"dims": 4, "base": 100.0}
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 5] = 1.0, 1.0, 7.0
    y = G.rotate(x, rot)[2, 0]
    a, b = 2.0, 2.0 * 100.0 ** -0.5
    assert torch.allclose(y, torch.tensor([math.cos(a), -math.sin(b), math.sin(a), math.cos(b), 0.0, 7.0], dtype=torch.float64))


def test_reference_frequency_scaling():
    rot = M.rotary(64, 1e4, 4.0, 2048, 32.0, 1.0)
    f, gain = G.yarn_frequencies(rot)
    plain = [1e4 ** (-2 * i / 64) for i in range(32)]
    turns = [2048 * p / (2 * math.pi) for p in plain]
    for i in range(32):  # many turns: as it was; less than one turn: divided; otherwise in between
        if turns[i] > 64:
            assert f[i] == pytest.approx(plain[i])
        elif turns[i] < 0.5:
            assert f[i] == pytest.approx(plain[i] / 4)
        assert plain[i] / 4 * (1 - 1e-9) <= f[i] <= plain[i] * (1 + 1e-9)
    assert gain == pytest.approx(1 + 0.1 * math.log(4.0)) and any(plain[i] / 4 < f[i] * 0.999 and f[i] < plain[i] * 0.999 for i in range(32))


def test_reference_delta_rule_replaces_what_a_key_holds():
    k = torch.tensor([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0]], dtype=torch.float64)[:, None]
    v = torch.tensor([[2.0], [5.0], [3.0]], dtype=torch.float64)[:, None]
    one = torch.ones(3, 1, dtype=torch.float64)
    o = G.delta_rule(k, k, v, one, one)[:, 0, 0]
    assert o.tolist() == [2.0, 5.0, 3.0]  # the third token overwrites the first
    o = G.delta_rule(k, k, v, one * 0.5, one)[:, 0, 0]
    assert o.tolist() == [2.0, 5.0, 3.0]
    q = torch.tensor([[1.0, 0.0]] * 3, dtype=torch.float64)[:, None]
    o = G.delta_rule(q, k, v, one * 0.5, one * 0.5)[:, 0, 0]
    assert o.tolist() == [1.0, 0.5, 0.25 + 0.5 * (3 - 0.25)]


def test_reference_convolution_and_causality():
    x = torch.tensor([[1.0], [2.0], [4.0]], dtype=torch.float64)
    assert G.causal_conv(x, torch.tensor([[10.0, 1.0]], dtype=torch.float64))[:, 0].tolist() == [1.0, 12.0, 24.0]
    raw = M.MIXED
    w = M.weights(raw)
    a, b = M.random_tokens(raw, 12, 1), M.random_tokens(raw, 12, 2)
    ya, yb = M.reference(raw, w, a), M.reference(raw, w, a[:7] + b[7:])
    assert torch.allclose(ya[:7], yb[:7]) and not torch.allclose(ya[7], yb[7])


def test_reference_passes_add_the_embedding_and_their_vector():
    raw = M.config([M.layer()], loop=(0, 1, 2))
    w = M.silence(M.weights(raw), raw, "left", "right", "ff")
    toks = [3, 9]
    _, x = M.reference(raw, w, toks, True)
    e, s = w["embed"][toks].double(), w["loop.step"].double()
    assert torch.allclose(x[0], e + s[0]) and torch.allclose(x[1], 2 * e + s[0] + s[1])
