"""Zefedra without a GPU: configuration, file reading, packing, the library's own checks, and the restatement's mechanisms."""
import math

import pytest
import torch

import zefedra_models as M
import zefedra_ref as Z


def cfg_of(raw):
    from llama_cu_b200 import zefedra
    return zefedra.read_config(raw)


def test_configuration_is_read_from_the_file(L):
    cfg = cfg_of(M.MIXED)
    assert (cfg.d, cfg.vocab, cfg.eps, cfg.n_layers) == (72, 101, 1e-5, 4)
    a, b, c, d = cfg.layers
    assert (a.mixer.heads, a.mixer.dim, a.mixer.v_dim, a.mixer.q_rank, a.mixer.kv_rank, a.ff) == (3, 20, 12, 24, 40, 50)
    assert not a.mixer.out_gate and b.mixer.out_gate and b.ff == 0
    assert (a.weights_of, c.weights_of) == (-1, 0) and c.mixer == a.mixer
    o = cfg.layer_descs()
    assert (o[3].heads, o[3].v_dim, o[3].out_gate, o[3].token_shift) == (2, 40, 1, 1) and abs(o[3].scale - 36 ** -0.5) < 1e-7


@pytest.mark.parametrize("bad", [{"type": "window_attention"}, {"mlp": {"kind": "experts", "ff": 8}}])
def test_unknown_parts_are_refused(L, bad):
    with pytest.raises(ValueError):
        cfg_of(M.config([dict(M.layer(), **bad)]))


def test_file_round_trip(L, tmp_path):
    from llama_cu_b200 import layered
    w = M.weights(M.MIXED, 3)
    M.write_model(tmp_path / "m", M.MIXED, w)
    got = layered.read_safetensors(str(tmp_path / "m" / "model.safetensors"))
    assert got.keys() == w.keys() and all(torch.equal(got[k], w[k]) for k in w)
    assert got["l0.norm1"].shape == () and not any(k.startswith("l2.") for k in got)


def test_missing_and_misshapen_tensors_are_named(L):
    from llama_cu_b200 import layered, zefedra
    cfg, w = cfg_of(M.MIXED), M.weights(M.MIXED)
    for name, change in (("l1.mix.g", lambda t: None), ("l3.mlp.up", lambda t: t[:-1])):
        bad = {k: v for k, v in w.items()}
        t = change(bad.pop(name))
        if t is not None:
            bad[name] = t
        with pytest.raises(ValueError, match=name):
            list(zefedra.pack(cfg, layered.Tensors(bad)))


def test_unknown_architecture(L, tmp_path):
    M.write_model(tmp_path / "m", dict(M.MIXED, architecture="Other"), M.weights(M.MIXED))
    with pytest.raises(ValueError, match="Other"):
        L.load_pretrained(str(tmp_path / "m"))


def test_packing_pads_with_zeros_and_keeps_every_number(L):
    from llama_cu_b200 import layered, zefedra
    cfg, w = cfg_of(M.MIXED), M.weights(M.MIXED)
    p = {k: v for k, v in zefedra.pack(cfg, layered.Tensors(w))}
    assert p[(-1, L.W_EMBD)].shape == (101, 128) and p[(-1, L.W_LM_HEAD)].shape == (104, 128)
    x = p[(3, L.W_LAT_IN)]
    assert x.shape == (128 + 192 + 8, 128)
    assert torch.equal(x[:70, :72], w["l3.mix.dq"]) and torch.equal(x[128:258, :72], w["l3.mix.dkv"]) and torch.equal(x[320:322, :72], w["l3.mix.g"])
    assert float(x.float().abs().sum()) == pytest.approx(sum(float(w["l3.mix." + n].float().abs().sum()) for n in ("dq", "dkv", "g")), rel=1e-5)
    ukt, ukv = p[(0, L.W_UKT)], p[(0, L.W_UKV)]
    uk = w["l0.mix.uk"].view(3, 20, 40)
    assert ukt.shape == (3, 64, 32) and torch.equal(ukt[1, :40, :20], uk[1].T)
    assert ukv.shape == (3 * 32 + 3 * 16, 64) and torch.equal(ukv[96 + 16:96 + 28, :40], w["l0.mix.uv"][12:24])
    o = p[(0, L.W_LAT_OUT)]
    assert o.shape == (128, 64) and torch.equal(o[:72, 16:28], w["l0.mix.o"][:, 12:24]) and not o[:, 12:16].any()
    sc = p[(0, L.W_SCALARS)]
    assert sc.tolist() == [float(w["l0.norm1"]), float(w["l0.norm2"]), float(w["l0.mlp.act"][0]), float(w["l0.mlp.act"][1])]


def test_pages_and_bytes(L):
    from dataclasses import replace
    cfg = cfg_of(M.MIXED)
    assert cfg.kv_bytes_per_token() == (64 + 128 + 64 + 192) * 2
    assert replace(cfg, act_dtype=L.F32).kv_bytes_per_token() == (64 + 128 + 64 + 192) * 4


def test_layered_contexts_need_a_gpu_and_sane_descriptions(L):
    cfg = cfg_of(M.MIXED)
    for field, value in (("heads", 0), ("kv_rank", 600), ("mixer", 9), ("weights_of", 7), ("ff_act", 5)):
        d = cfg.layer_descs()
        setattr(d[0], field, value)
        with pytest.raises(L.LcuError):
            L.Context(cfg.desc(), layers=d)
    if not torch.cuda.is_available():
        with pytest.raises(L.LcuError) as e:
            L.Context(cfg.desc(), layers=cfg.layer_descs())
        assert e.value.code == L.ERR_CUDA


# ---- the restatement against closed forms
def test_reference_token_shift_and_norm():
    h = torch.tensor([[1.0, 2.0], [3.0, 6.0]], dtype=torch.float64)
    got = Z.token_shift(h, torch.tensor([0.25, 1.0], dtype=torch.float64))
    assert torch.allclose(got, torch.tensor([[0.75, 0.0], [2.5, 2.0]], dtype=torch.float64))
    assert torch.allclose(Z.scalar_norm(torch.tensor([[3.0, 4.0]], dtype=torch.float64), 2.0, 0.5), torch.tensor([[6.0, 8.0]], dtype=torch.float64) / math.sqrt(13.0))


def test_reference_xielu_is_smooth_at_zero_and_matches_its_branches():
    p, q = torch.tensor(0.3, dtype=torch.float64), torch.tensor(-0.7, dtype=torch.float64)
    z = torch.tensor([-2.0, -1e-6, 0.0, 1e-6, 1.5], dtype=torch.float64)
    y = Z.xielu(z, p, q)
    sp, sq = math.log1p(math.exp(0.3)), math.log1p(math.exp(-0.7))
    assert float(y[0]) == pytest.approx((0.5 + sq) * (math.exp(-2) + 1) - 1.0)
    assert float(y[4]) == pytest.approx(sp * 2.25 + 0.75)
    assert float((y[3] - y[1]) / 2e-6) == pytest.approx(0.5, abs=1e-4)


def test_reference_attention_is_causal_and_gated():
    raw = M.config([M.layer(True)])
    w = {k: v.double() for k, v in M.weights(raw).items()}
    h = torch.randn(9, 72, dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    y = Z.latent_attention(h, w, "l0.mix.", raw["layers"][0]["mixer"], 1e-5, True)
    h2 = h.clone()
    h2[6:] += 1.0
    y2 = Z.latent_attention(h2, w, "l0.mix.", raw["layers"][0]["mixer"], 1e-5, True)
    assert torch.allclose(y[:6], y2[:6]) and not torch.allclose(y[6], y2[6])
    assert not torch.allclose(y, Z.latent_attention(h, w, "l0.mix.", raw["layers"][0]["mixer"], 1e-5, False))
