"""Small random Mupuvik models for the tests: configurations, weights, and what is planted in them."""
import torch

import mupuvik_ref as R
from zefedra_models import Runner, random_tokens, rel_err, write_model  # noqa: F401  (common to the layered families)

TOL = {1: 2.5e-2, 2: 2e-5}  # bf16, f32


def moe(ff=30, experts=5, top=2, limit=0.8, shared=50, shared_limit=1.1):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def ssd(heads=4, groups=2, state=20, vdim=12, conv=4, parts=3, mlp="usual"):
    return {"type": "mamba2", "mixer": {"heads": heads, "groups": groups, "state": state, "vdim": vdim, "conv": conv, "norm_groups": parts},
            "mlp": moe() if mlp == "usual" else mlp}


def window(size=9, heads=6, kv_heads=2, dim=20, vdim=12, scale=0.3, kv_from=None, mlp="usual"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": moe() if mlp == "usual" else mlp}


def both(heads=4, kv_heads=2, dim=20, vdim=12, rot=8, base=300.0, scale=0.3, g_heads=3, g_dim=12, g_vdim=20, tau=4.0, rank=5, scales=(1.3, 0.7), mlp="usual"):
    """`rank` is no key of a configuration file: `shapes` gives it as a file's tensor would."""
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"dims": rot, "base": base}, "scale": scale},
                      "right": {"heads": g_heads, "dim": g_dim, "vdim": g_vdim, "tau": tau, "rank": rank}, "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": moe() if mlp == "usual" else mlp}


def config(layers, width=72, vocab=101, eps=1e-5, scale=7.0, buckets=53, mul=(60, 5)):
    return {"architecture": "Mupuvik", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": scale, "bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}}, "layers": layers}


# every branch, sizes that need padding, values that differ from one another
MIXED = config([ssd(), window(9), ssd(heads=3, groups=1, state=40, vdim=17, conv=3, parts=1, mlp=None), both(),
                window(30, kv_from=1, mlp=moe(70, 3, 1, 2.0, 0)), both(heads=5, kv_heads=1, dim=36, vdim=24, rot=36, g_heads=2, g_dim=40, g_vdim=8, tau=16.0, rank=9,
                                                                       scales=(0.5, 2.0), mlp=None),
                window(70, heads=4, kv_heads=4, dim=16, vdim=32, scale=0.25, mlp=moe(20, 4, 4, 0.5, 10, 0.3))])


def shapes(raw):
    return {f"l{i}.mix.right.a1": (e["mixer"]["right"]["rank"], raw["width"]) for i, e in enumerate(raw["layers"]) if e["type"] == "parallel"}


def cfg_of(raw):
    from llama_cu_b200 import mupuvik
    return mupuvik.read_config(raw, shapes(raw))


def weights(raw, seed=0, steady=True):
    """{name: bf16 tensor on the host}, as a file would hold them.  steady: see steady_routes."""
    from llama_cu_b200 import mupuvik
    w = dict(mupuvik.synth_tensors(cfg_of(raw), seed, "cpu"))
    for name in w:  # a token's query and key alike: else the norm of a first token's output may enlarge rounding alone
        if name.endswith("right.q"):
            w[name] = (0.6 * w[name].float() + 0.8 * w[name[:-1] + "k"].float()).to(torch.bfloat16)
    return steady_routes(raw, w, seed) if steady else w


def steady_routes(raw, w, seed):
    """Routers that read some coordinates of the residual stream which nothing but the embedding writes: a token's experts depend on
    the token alone and no rounding swaps two of them."""
    n = max([e["mlp"]["router"]["experts"] for e in raw["layers"] if e["mlp"]] + [0])
    if not n or n > raw["width"] // 4:
        return w
    g = torch.Generator().manual_seed(seed + 1000)
    w = {k: v.clone() for k, v in w.items()}
    levels = torch.linspace(-2.5, 2.5, n)
    codes = torch.stack([levels[torch.randperm(n, generator=g)] for _ in range(raw["vocab"])])
    w["embed"][:, :n] = (codes / raw["embedding"]["scale"]).to(torch.bfloat16)
    w["bigram"][:, :n] = 0
    for i, e in enumerate(raw["layers"]):
        p = f"l{i}."
        for name in ("norm1b", "norm2b") if e["mlp"] else ("norm1b",):
            w[p + name][:n] = -1
        if e["mlp"]:
            w[p + "norm2"][:n] = 0
            m = e["mlp"]["router"]["experts"]
            r = torch.zeros(m, raw["width"])
            r[torch.arange(m), torch.randperm(n, generator=g)[:m]] = 1.5
            w[p + "mlp.router"] = r.to(torch.bfloat16)
    return w


def load(L, raw, w, dt, tokens=512, max_seqs=4, max_tokens=None, **kw):
    """A context whose pool holds `tokens` tokens."""
    from dataclasses import replace
    from llama_cu_b200 import layered, mupuvik
    cfg = replace(cfg_of(raw), act_dtype=dt, nctx=tokens)
    page = kw.get("page_tokens") or 64
    ctx = L.load_model(cfg, mupuvik.pack(cfg, layered.Tensors(w)), kv_bytes=max((tokens + page - 1) // page * page * cfg.kv_bytes_per_token(), 1 << 16)
                       if cfg.kv_bytes_per_token() > 1 else 1 << 20, max_tokens=max_tokens or tokens, max_seqs=max_seqs, **kw)
    return cfg, ctx


def reference(raw, w, tokens, keep_layers=False):
    return R.forward(raw, w, list(tokens), torch.float64, keep_layers)


def tolerance(dt, raw, w, toks, want=None):
    """What a run may differ by: three times what rounding the inputs of the matrix products to bf16, or all of it to 32 bits, changes
    in the restatement (norms of small sums enlarge it at some tokens)."""
    want = reference(raw, w, toks) if want is None else want
    kw = dict(dtype=torch.float32) if dt == 2 else dict(operand=torch.bfloat16)
    return max(TOL[dt], 3 * rel_err(R.forward(raw, w, list(toks), **kw), want))


def silence(w, raw, *what):
    """Weights with parts switched off in every layer: "mixer" or "ff" (gain of the norm on its output), "left" or "right" (that
    mixer's output projection), "experts", "shared" (their last matrices), "pairs"."""
    w = dict(w)
    for name in w:
        if ("mixer" in what and name.endswith("norm1b")) or ("ff" in what and name.endswith("norm2b")):
            w[name] = torch.full_like(w[name], -1)
        for part, end in (("left", "left.o"), ("right", "right.o"), ("shared", "shared.down"), ("pairs", "bigram")):
            if part in what and name.endswith(end):
                w[name] = torch.zeros_like(w[name])
        if "experts" in what and ".mlp.e" in name and name.endswith(".down"):
            w[name] = torch.zeros_like(w[name])
    return w


def plant_key(raw, w, token_key, token_query, strength=40.0):
    """Rank-one terms in layer 0's query and key maps so that `token_query` scores `token_key` far above anything else in every
    head, along the last dimension of a head (which must not be rotated); the embedding of pairs is taken out."""
    e, eps = raw["layers"][0], raw["norm"]["eps"]
    m, p = (e["mixer"]["left"], "l0.mix.left.") if e["type"] == "parallel" else (e["mixer"], "l0.mix.")
    assert "rot" not in m or m["rot"]["dims"] < m["dim"]
    out = dict(w)
    out["bigram"] = torch.zeros_like(w["bigram"])
    h = R.centred_norm(w["embed"][[token_key, token_query]].double() * raw["embedding"]["scale"], w["l0.norm1"].double(), eps)
    for name, heads, v in (("q", m["heads"], h[1]), ("k", m["kv_heads"], h[0])):
        t = w[p + name].double().view(heads, m["dim"], -1).clone()
        t[:, -1] += strength * v / (v * v).sum()
        out[p + name] = t.view(heads * m["dim"], -1).to(torch.bfloat16)
        g = out[p + name + ".norm"].clone().view(-1, m["dim"])
        g[:, -1] = 1
        out[p + name + ".norm"] = g.view(-1)
    return out
