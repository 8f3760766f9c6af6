"""Small random Gunulorn models for the tests: configurations, weights, and what is planted in them."""
import torch

import gunulorn_ref as R
from zefedra_models import Runner, random_tokens, rel_err, write_model  # noqa: F401  (common to the layered families)

TOL = {1: 2.5e-2, 2: 2e-5}  # bf16, f32


def dense(ff=50):
    return {"kind": "dense", "ff": ff}


def moe(ff=30, experts=5, top=2, identity=2):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}}


def conv(taps=3, heads=6, kv_heads=2, dim=20, vdim=12, scale=0.3, kv_from=None, mlp="usual"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": taps}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": moe() if mlp == "usual" else mlp}


def window(size=9, keep=3, heads=4, kv_heads=2, dim=20, vdim=28, rot=8, base=300.0, scale=0.25, mlp="usual"):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot, "base": base},
                                             "mask": {"size": size, "keep_first": keep}}, "mlp": moe() if mlp == "usual" else mlp}


def config(layers, width=72, vocab=101, eps=1e-5, scale=1.5, cap=5.0):
    return {"architecture": "Gunulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale, "logit_softcap": cap, "layers": layers}


# every branch, sizes that need padding, values that differ from one another
MIXED = config([window(9, 3, mlp=dense(50)), conv(3), window(30, 70, heads=3, kv_heads=1, dim=36, vdim=10, rot=36, mlp=moe(70, 3, 1, 1)), conv(2, kv_from=1, mlp=None),
                window(70, 0, heads=4, kv_heads=4, dim=16, vdim=32, rot=2, base=1e4, mlp=dense(130)), conv(4, heads=5, kv_heads=1, dim=36, vdim=24, mlp=moe(20, 4, 4, 0)),
                conv(1, heads=4, kv_heads=2, kv_from=1, scale=0.5, mlp=moe(9, 2, 3, 4)), window(1, 5, mlp=None)])


def cfg_of(raw):
    from llama_cu_b200 import gunulorn
    return gunulorn.read_config(raw)


def weights(raw, seed=0, steady=True):
    """{name: bf16 tensor on the host}, as a file would hold them.  steady: see steady_routes."""
    from llama_cu_b200 import gunulorn
    w = dict(gunulorn.synth_tensors(cfg_of(raw), seed, "cpu"))
    return steady_routes(raw, w, seed) if steady else w


def steady_routes(raw, w, seed):
    """Routers that read some coordinates of the residual stream which next to nothing but the embedding writes (experts that return
    their input see them 64 times smaller): a token's experts depend on the token alone and no rounding swaps two of them.
    Corrections of +-2 outweigh every score: one expert is always chosen, one never, where there is room."""
    ffs = [e["mlp"] for e in raw["layers"] if e["mlp"] and e["mlp"]["kind"] == "moe"]
    n = max([f["router"]["experts"] + f["router"]["identity"] for f in ffs] + [0])
    if not n or n > raw["width"] // 4:
        return w
    g = torch.Generator().manual_seed(seed + 1000)
    w = {k: v.clone() for k, v in w.items()}
    levels = torch.linspace(-2.5, 2.5, n)
    w["embed"][:, :n] = torch.stack([levels[torch.randperm(n, generator=g)] for _ in range(raw["vocab"])]).to(torch.bfloat16)
    for name in w:
        if name.endswith((".o", ".down", ".down.b")):
            w[name][:n] = 0
    for i, e in enumerate(raw["layers"]):
        if e["mlp"] not in ffs or not e["mlp"]:
            continue
        p, m = f"l{i}.", e["mlp"]["router"]
        total = m["experts"] + m["identity"]
        w[p + "norm2"][:n] = 2.0 ** -6
        r = torch.zeros(total, raw["width"])
        r[torch.arange(total), torch.randperm(n, generator=g)[:total]] = 1.5 * 2 ** 6
        w[p + "mlp.router"] = r.to(torch.bfloat16)
        c = torch.zeros(total)
        a, b = torch.randperm(total, generator=g)[:2].tolist() if total > 1 else (0, 0)
        if m["top"] > 1:
            c[a] = 2
        if total > m["top"]:
            c[b] = -2
        w[p + "mlp.correction"] = c.to(torch.bfloat16)
    return w


def load(L, raw, w, dt, tokens=512, max_seqs=4, max_tokens=None, **kw):
    """A context whose pool holds `tokens` tokens."""
    from dataclasses import replace
    from llama_cu_b200 import gunulorn, layered
    cfg = replace(cfg_of(raw), act_dtype=dt, nctx=tokens)
    page = kw.get("page_tokens") or 64
    ctx = L.load_model(cfg, gunulorn.pack(cfg, layered.Tensors(w)), kv_bytes=max((tokens + page - 1) // page * page * cfg.kv_bytes_per_token(), 1 << 16),
                       max_tokens=max_tokens or tokens, max_seqs=max_seqs, **kw)
    return cfg, ctx


def reference(raw, w, tokens, keep_layers=False):
    return R.forward(raw, w, list(tokens), torch.float64, keep_layers)


def tolerance(dt, raw, w, toks, want=None):
    """What a run may differ by: three times what rounding the inputs of the matrix products to bf16, or all of it to 32 bits, changes
    in the restatement."""
    want = reference(raw, w, toks) if want is None else want
    kw = dict(dtype=torch.float32) if dt == 2 else dict(operand=torch.bfloat16)
    return max(TOL[dt], 3 * rel_err(R.forward(raw, w, list(toks), **kw), want))


def silence(w, raw, *what):
    """Weights with parts switched off in every layer: "mixer" (its last matrix), "ff" (its input, its last matrix and bias), "experts"
    (their last matrices; those that return their input stay)."""
    w = dict(w)
    for name in w:
        last = name.split(".", 1)[-1]
        if (("mixer" in what and last == "mix.o") or ("ff" in what and last in ("norm2", "mlp.down", "mlp.down.b"))
                or ("experts" in what and last.startswith("mlp.e") and last.endswith(".down"))):
            w[name] = torch.zeros_like(w[name])
    return w


def plant_key(raw, w, token_key, token_query, strength=10.0):
    """Rank-one terms in layer 0's query and key maps so that `token_query` scores `token_key` far above anything else in every
    head, along the last dimension of a head (which must not be rotated); convolutions pass that dimension as it is."""
    m, eps = raw["layers"][0]["mixer"], raw["norm"]["eps"]
    assert "rot" not in m or m["rot"]["dims"] < m["dim"]
    out = dict(w)
    h = R.norm(w["embed"][[token_key, token_query]].double(), w["l0.norm1"].double(), eps)
    for name, heads, v in (("q", m["heads"], h[1]), ("k", m["kv_heads"], h[0])):
        name = "l0.mix." + name
        t = w[name].double().view(heads, m["dim"], -1).clone()
        t[:, -1] += strength * v / (v * v).sum()
        out[name] = t.view(heads * m["dim"], -1).to(torch.bfloat16)
        if "conv" in m:
            c = w[name + ".conv"].clone().view(heads, m["dim"], -1)
            c[:, -1] = 0
            c[:, -1, -1] = 1
            out[name + ".conv"] = c.view(heads * m["dim"], -1)
    if "conv" in m:
        out["l0.mix.temp"] = w["l0.mix.temp"].abs()
    return out
