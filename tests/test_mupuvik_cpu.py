"""Mupuvik without a GPU: configuration, packing, and the restatement's mechanisms."""
import math

import pytest
import torch

import mupuvik_models as M
import mupuvik_ref as R


def test_configuration_is_read_from_the_file(L):
    from llama_cu_b200 import layered as Y
    cfg = M.cfg_of(M.MIXED)
    assert (cfg.d, cfg.vocab, cfg.eps, cfg.arch, cfg.embed_scale) == (72, 101, 1e-5, "Mupuvik", 7.0)
    assert cfg.pairs == Y.PairEmbedding(53, 60, 5)
    a, b, c, d, e = (cfg.layers[i].mixer for i in (0, 1, 2, 3, 4))
    assert a == Y.SsdMixer(4, 2, 20, 12, 4, 3) and c == Y.SsdMixer(3, 1, 40, 17, 3, 1)
    assert (b.heads, b.kv_heads, b.dim, b.v_dim, b.scale, b.window, b.kv_from, b.rot, b.bias, b.qk_norm, b.sink, b.out_gate) == (6, 2, 20, 12, 0.3, 9, -1, None, True, 3, False, True)
    assert (e.window, e.kv_from) == (30, 1)
    assert d.right == Y.GlaMixer(3, 12, 20, 4.0, 5) and d.scales == (1.3, 0.7)
    assert d.left.rot == Y.Rotary(8, 300.0, adjacent=True) and d.left.sink and d.left.out_gate and not d.left.bias and d.left.qk_norm == 2 and d.left.window == 0
    assert cfg.layers[0].ff == Y.GluFf(30, 0.8, 1.702, 1.0, 5, 2, 50, 1.1) and cfg.layers[2].ff == 0
    assert cfg.layers[4].ff == Y.GluFf(70, 2.0, 1.702, 1.0, 3, 1, 0, 0.0)
    o = cfg.layer_descs()
    assert [x.mixer for x in o] == [L.MIX_SSD, L.MIX_ATTENTION, L.MIX_SSD, L.MIX_ATTENTION | L.MIX_GLA, L.MIX_ATTENTION, L.MIX_ATTENTION | L.MIX_GLA, L.MIX_ATTENTION]
    assert all(x.pre_norm and x.post_norm for x in o) and [x.kv_from for x in o] == [0, 0, 0, 0, 2, 0, 0] and [x.window for x in o] == [0, 9, 0, 0, 30, 0, 70]
    assert (o[0].delta_heads, o[0].delta_kv_heads, o[0].delta_dim, o[0].delta_v_dim, o[0].delta_conv, o[0].norm_parts) == (4, 2, 20, 12, 4, 3)
    assert (o[3].delta_heads, o[3].delta_kv_heads, o[3].gate_rank, o[3].gate_tau, o[3].rot_adjacent, o[3].sink) == (3, 3, 5, 4.0, 1, 1)
    assert o[3].out_scale == pytest.approx(1.3) and o[3].out_scale2 == pytest.approx(0.7)
    assert (o[0].ff, o[0].ff_act, o[0].experts, o[0].top, o[0].shared_ff) == (30, L.ACT_GLU, 5, 2, 50) and o[0].shared_limit == pytest.approx(1.1)
    assert (o[0].embed_scale, o[0].pair_buckets, o[0].pair_prev, o[0].pair_cur) == (7.0, 53, 7, 5)  # 60 mod 53


@pytest.mark.parametrize("bad", [{"type": "latent_attention"}, {"mlp": {"kind": "dense", "ff": 8}}])
def test_unknown_parts_are_refused(L, bad):
    with pytest.raises(ValueError):
        M.cfg_of(M.config([dict(M.window(), **bad)]))


@pytest.mark.parametrize("layers", [[M.window(kv_from=0)], [M.ssd(), M.window(kv_from=0)], [M.window(), M.window(kv_from=0), M.window(kv_from=1)], [M.window(kv_from=1), M.window()]])
def test_keys_come_from_an_earlier_attention_layer_with_its_own(L, layers):
    with pytest.raises(ValueError):
        M.cfg_of(M.config(layers))


def test_missing_and_misshapen_tensors_are_named(L):
    from llama_cu_b200 import layered, mupuvik
    cfg, w = M.cfg_of(M.MIXED), M.weights(M.MIXED)
    for name, change in (("l0.mix.A_log", lambda t: None), ("l1.mix.k.b", lambda t: t[:-1]), ("bigram", lambda t: t[:-1]), ("l4.mlp.e2.down", lambda t: None),
                         ("l3.mix.right.a2", lambda t: t[:, 1:])):
        bad = dict(w)
        t = change(bad.pop(name))
        if t is not None:
            bad[name] = t
        with pytest.raises(ValueError, match=name):
            list(mupuvik.pack(cfg, layered.Tensors(bad)))


def test_tensor_names(L):
    from llama_cu_b200 import mupuvik
    names = set(mupuvik.tensor_shapes(M.cfg_of(M.MIXED)))
    assert {"l4.mix.q", "l4.mix.q.b", "l4.mix.q.norm", "l4.mix.g", "l4.mix.o"} <= names
    assert not {"l4.mix.k", "l4.mix.k.b", "l4.mix.k.norm", "l4.mix.v", "l4.mix.v.b", "l2.norm2", "l2.mlp.router", "l4.mlp.shared.up", "head"} & names


def test_packing_pads_with_zeros_and_keeps_every_number(L):
    from llama_cu_b200 import layered, mupuvik
    cfg, w = M.cfg_of(M.MIXED), M.weights(M.MIXED, steady=False)
    p = {k: v for k, v in mupuvik.pack(cfg, layered.Tensors(w))}
    # C 2 x 32 | B 2 x 32 | x 4 x 16 | z 4 x 16 | dt 8; the file: z 48 | x 48 | B 40 | C 40 | dt 4
    x, f = p[(0, L.W_MIX_IN)], w["l0.mix.in"]
    assert x.shape == (64 + 64 + 64 + 64 + 8, 128)
    assert torch.equal(x[32:52, :72], f[156:176]) and torch.equal(x[64:84, :72], f[96:116]) and torch.equal(x[144:156, :72], f[60:72])
    assert torch.equal(x[192:204, :72], f[:12]) and torch.equal(x[256:260, :72], f[176:180])
    assert float(x.float().abs().sum()) == pytest.approx(float(f.float().abs().sum()), rel=1e-5)
    c, b = p[(0, L.W_CONV)], p[(0, L.W_CONV_BIAS)]
    assert c.shape == (4, 192) and torch.equal(c[:, 32:52], w["l0.mix.conv"][108:128].float().T) and torch.equal(b[144:156], w["l0.mix.conv.b"][12:24].float())
    assert torch.equal(p[(0, L.W_DELTA_DECAY)][:, :4], torch.stack([w["l0.mix." + n].float() for n in ("A_log", "dt_bias", "D")]))
    assert torch.equal(p[(0, L.W_DELTA_NORM)][16:28], w["l0.mix.norm"][12:24].float())
    o = p[(0, L.W_DELTA_OUT)]
    assert o.shape == (128, 64) and torch.equal(o[:72, 16:28], w["l0.mix.o"][:, 12:24]) and not o[:, 12:16].any()
    # window attention: q 6 x 32 | k 2 x 32 | v 2 x 16 | gates 8
    x = p[(1, L.W_MIX_IN)]
    assert x.shape == (192 + 64 + 32 + 8, 128) and torch.equal(x[288:294, :72], w["l1.mix.g"]) and torch.equal(x[224:244, :72], w["l1.mix.k"][20:40])
    g = p[(1, L.W_QK_GAIN)]
    assert g.shape == (256,) and torch.equal(g[32:52], w["l1.mix.q.norm"][20:40].float()) and torch.equal(g[224:244], w["l1.mix.k.norm"][20:40].float())
    assert p[(4, L.W_MIX_IN)].shape == (192 + 8, 128) and p[(4, L.W_MIX_BIAS)].shape == (192,) and p[(4, L.W_QK_GAIN)].shape == (192,)
    # both mixers: q 4 x 32 | k 2 x 32 | v 2 x 16 | gates 8 | q 3 x 32 | k 3 x 32 | v 3 x 32 | g 3 x 32 | first map 8
    x = p[(3, L.W_MIX_IN)]
    assert x.shape == (128 + 64 + 32 + 8 + 4 * 96 + 8, 128)
    assert torch.equal(x[232 + 32:232 + 44, :72], w["l3.mix.right.q"][12:24]) and torch.equal(x[616:621, :72], w["l3.mix.right.a1"]) and not x[621:].any()
    assert p[(3, L.W_QK_GAIN)].shape == (64,) and torch.equal(p[(3, L.W_QK_GAIN)][32:52], w["l3.mix.left.k.norm"].float())
    m = p[(3, L.W_GATE_MAP)]
    assert m.shape == (6, 96) and torch.equal(m[:5, 32:44], w["l3.mix.right.a2"][12:24].float().T) and torch.equal(m[5, 64:76], w["l3.mix.right.a2.b"][24:].float())
    # experts: gate and up rows in turn
    u, d = p[(0, L.W_UP)], p[(0, L.W_FF_DOWN)]
    assert u.shape == (5, 128, 128) and torch.equal(u[3, 0:60:2, :72], w["l0.mlp.e3.gate"]) and torch.equal(u[3, 1:61:2, :72], w["l0.mlp.e3.up"]) and not u[3, 60:].any()
    assert d.shape == (5, 128, 64) and torch.equal(d[4, :72, :30], w["l0.mlp.e4.down"])
    assert p[(0, L.W_ROUTER)].shape == (8, 128) and p[(0, L.W_SHARED_UP)].shape == (128, 128) and torch.equal(p[(0, L.W_SHARED_DOWN)][:72, :50], w["l0.mlp.shared.down"])
    assert torch.equal(p[(0, L.W_POST1)][:72], 1 + w["l0.norm1b"].float()) and torch.equal(p[(0, L.W_POST2)][:72], 1 + w["l0.norm2b"].float())
    assert (2, L.W_NORM2) not in p and (2, L.W_POST2) not in p and (2, L.W_UP) not in p and (4, L.W_SHARED_UP) not in p
    assert torch.equal(p[(-1, L.W_LM_HEAD)][:101, :72], w["embed"]) and torch.equal(p[(-1, L.W_PAIR_EMBD)][:, :72], w["bigram"])


def test_pages_and_bytes(L):
    cfg = M.cfg_of(M.MIXED)
    assert cfg.kv_bytes_per_token() == 2 * (2 * (32 + 16) + 2 * (32 + 16) + (48 + 32) + 4 * (16 + 32))
    assert cfg.state_bytes_per_sequence() == 4 * (4 * 16 * 32 + 3 * 32 * 64 + 3 * 32 * 32 + 2 * 16 * 64)


# ---- the restatement against closed forms

def test_reference_pairs():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 4}
    assert R.bigram_rows([5, 2, 7], b) == [10, (15 + 8) % 10, (6 + 28) % 10]


def test_reference_rotation_of_neighbours():
    x = torch.zeros(3, 1, 6, dtype=torch.float64)
    x[:, 0, 0], x[:, 0, 3], x[:, 0, 5] = 1.0, 1.0, 7.0
    y = R.rotate(x, {"dims": 4, "base": 100.0})[2, 0]
    a, b = 2.0, 2.0 * 100.0 ** -0.5
    assert torch.allclose(y, torch.tensor([math.cos(a), math.sin(a), -math.sin(b), math.cos(b), 0.0, 7.0], dtype=torch.float64))


def test_reference_window_and_sink():
    assert R.visible(4, 2).int().tolist() == [[1, 0, 0, 0], [1, 1, 0, 0], [0, 1, 1, 0], [0, 0, 1, 1]] and R.visible(2, 0).int().tolist() == [[1, 0], [1, 1]]
    q = torch.zeros(2, 1, 1, dtype=torch.float64)
    v = torch.tensor([[[3.0]], [[9.0]]], dtype=torch.float64)
    assert R.softmax_attention(q, q, v, 1.0)[:, 0, 0].tolist() == [3.0, 6.0]
    assert R.softmax_attention(q, q, v, 1.0, sink=True)[:, 0, 0].tolist() == pytest.approx([1.5, 4.0])
    assert R.softmax_attention(q, q, v, 1.0, window=1)[:, 0, 0].tolist() == [3.0, 9.0]


def test_reference_recurrences():
    one = torch.ones(3, 1, dtype=torch.float64)
    x = torch.tensor([[[1.0]], [[10.0]], [[100.0]]], dtype=torch.float64)
    b = torch.ones(3, 1, 1, dtype=torch.float64)
    assert R.ssd(x, b, b, 2 * one, torch.zeros(1, dtype=torch.float64))[:, 0, 0].tolist() == [2.0, 22.0, 222.0]
    half = R.ssd(x, b, b, one, torch.tensor([math.log(2.0)], dtype=torch.float64))[:, 0, 0]
    assert half.tolist() == pytest.approx([1.0, 10.5, 105.25])
    k = torch.tensor([[[1.0, 1.0]]] * 3, dtype=torch.float64)
    d = torch.tensor([[[0.5, 1.0]]] * 3, dtype=torch.float64)
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]], [[0.0, 1.0]]], dtype=torch.float64)
    assert R.gla(q, k, x, d)[:, 0, 0].tolist() == [1.0, 10.5, 111.0]


def test_reference_norm_in_parts_and_gate():
    y = R.gated_norm(torch.tensor([[3.0, 4.0, 1.0, 1.0]], dtype=torch.float64), torch.full((1, 4), 50.0, dtype=torch.float64), torch.ones(4, dtype=torch.float64), 2, 0.0)
    assert torch.allclose(y, torch.tensor([[3 / 12.5 ** 0.5, 4 / 12.5 ** 0.5, 1.0, 1.0]], dtype=torch.float64))


def test_reference_experts():
    one = torch.ones(1, 1, dtype=torch.float64)
    w = {"e.gate": 4 * one, "e.up": -9 * one, "e.down": one}
    assert float(R.expert(one, w, "e.", 2.0)) == pytest.approx(2 / (1 + math.exp(-3.404)) * -1.0)
    assert float(R.expert(0.1 * one, w, "e.", 2.0)) == pytest.approx(0.4 / (1 + math.exp(-0.6808)) * 0.1)  # the weight scales the input
    r = {"router": torch.tensor([[1.0], [3.0], [-1.0]], dtype=torch.float64)}
    e, s = R.route(one, r, "", 2)
    assert e.tolist() == [[1, 0]] and s.tolist()[0] == pytest.approx([1 / (1 + math.exp(-3)), 1 / (1 + math.exp(-1))])


def test_reference_is_causal():
    raw = M.MIXED
    w = M.weights(raw)
    a, b = M.random_tokens(raw, 12, 1), M.random_tokens(raw, 12, 2)
    ya, yb = M.reference(raw, w, a), M.reference(raw, w, a[:7] + b[7:])
    assert torch.allclose(ya[:7], yb[:7]) and not torch.allclose(ya[7], yb[7])


def test_steady_routes_use_every_expert():
    raw = M.MIXED
    w = M.weights(raw, 3)
    used = set()
    real = R.route

    def spy(h, w, pre, top):
        e, s = real(h, w, pre, top)
        used.update((pre, int(x)) for x in e.flatten())
        return e, s
    R.route = spy
    try:
        M.reference(raw, w, M.random_tokens(raw, 60, 4))
    finally:
        R.route = real
    assert len(used) == sum(e["mlp"]["router"]["experts"] for e in raw["layers"] if e["mlp"])
