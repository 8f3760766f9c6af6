"""Small random Galarax models for the tests: configurations, weights, and what is planted in them."""
import torch

import galarax_ref as G
from zefedra_models import Runner, random_tokens, rel_err, write_model  # noqa: F401  (common to the layered families)

TOL = {1: 2.5e-2, 2: 2e-5}  # bf16, f32


def rotary(dims=8, base=3e4, factor=3.0, original=40, fast=16.0, slow=1.5):
    r = {"dims": dims, "base": base}
    if factor:
        r["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return r


def layer(heads=4, kv_heads=2, dim=20, vdim=12, rot=None, scale=0.3, d_heads=4, d_kv_heads=2, d_dim=12, d_vdim=20, conv=4, ff=50):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot or rotary(), "scale": scale},
                      "right": {"heads": d_heads, "kv_heads": d_kv_heads, "dim": d_dim, "vdim": d_vdim, "conv": conv}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=101, eps=1e-5, loop=None):
    raw = {"architecture": "Galarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return raw


# every branch, sizes that need padding, values that differ from one another, a loop with layers ahead of it and behind it
MIXED = config([layer(), layer(heads=6, kv_heads=2, dim=36, vdim=24, rot=rotary(36, 1e3, 5.0, 25, 8.0, 1.0), scale=0.2, d_heads=3, d_kv_heads=1, d_dim=40,
                              d_vdim=8, conv=3, ff=0),
                layer(heads=3, kv_heads=3, dim=16, vdim=32, rot=rotary(6, 50.0, 0), d_heads=5, d_kv_heads=5, d_dim=33, d_vdim=17, conv=2, ff=90),
                layer(heads=5, kv_heads=1, dim=70, vdim=66, rot=rotary(14, 2e5, 2.0, 4096, 32.0, 1.0), scale=0.1, d_heads=8, d_kv_heads=4, d_dim=64, d_vdim=36,
                      conv=6, ff=40)], loop=(1, 3, 3))


def weights(raw, seed=0):
    """{name: bf16 tensor on the host}, as a file would hold them."""
    from llama_cu_b200 import galarax
    return dict(galarax.synth_tensors(galarax.read_config(raw), seed, "cpu"))


def load(L, raw, w, dt, tokens=512, max_seqs=4, max_tokens=None, **kw):
    """A context whose pool holds `tokens` tokens."""
    from dataclasses import replace
    from llama_cu_b200 import galarax, layered
    cfg = replace(galarax.read_config(raw), act_dtype=dt, nctx=tokens)
    ctx = L.load_model(cfg, galarax.pack(cfg, layered.Tensors(w)), kv_bytes=(tokens + 127) // 128 * 128 * cfg.kv_bytes_per_token(),
                       max_tokens=max_tokens or tokens, max_seqs=max_seqs, **kw)
    return cfg, ctx


def reference(raw, w, tokens, keep_layers=False):
    return G.forward(raw, w, list(tokens), torch.float64, keep_layers)


def tolerance(dt, raw, w, toks, want=None):
    """What a bf16 run may differ by: three times what rounding the inputs of the matrix products changes in the restatement."""
    if dt == 2:
        return TOL[dt]
    want = reference(raw, w, toks) if want is None else want
    return max(TOL[dt], 3 * rel_err(G.forward(raw, w, list(toks), torch.float64, operand=torch.bfloat16), want))


def silence(w, raw, *what):
    """Weights with mechanisms switched off in every layer: "left" or "right" (gain on that mixer's output), "ff"."""
    w = dict(w)
    for name in w:
        for part, end in (("left", "left.out"), ("right", "right.out"), ("ff", "mlp.down")):
            if part in what and name.endswith(end):
                w[name] = torch.zeros_like(w[name])
    return w


def plant_key(raw, w, token_key, token_query, strength=25.0):
    """Rank-one terms in layer 0's query and key maps so that `token_query` scores `token_key` far above anything else in every
    head, along the last dimension of a head (which must not be rotated)."""
    m, eps = raw["layers"][0]["mixer"]["left"], raw["norm"]["eps"]
    assert m["rot"]["dims"] < m["dim"]
    x = w["embed"][[token_key, token_query]].double()
    if raw.get("loop") and raw["loop"]["start"] == 0:
        x = x + w["loop.step"][0].double()
    h = G.centred_norm(x, w["l0.norm1"].double(), eps)
    out = dict(w)
    for name, heads, v in (("q", m["heads"], h[1]), ("k", m["kv_heads"], h[0])):
        t = w["l0.mix.left." + name].double().view(heads, m["dim"], -1).clone()
        t[:, -1] += strength * v / (v * v).sum()
        out["l0.mix.left." + name] = t.view(heads * m["dim"], -1).to(torch.bfloat16)
    return out
