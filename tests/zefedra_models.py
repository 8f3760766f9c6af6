"""Small random Zefedra models for the tests: configurations, weights, files, and the comparison with the plain restatement."""
import json
import os
import struct

import numpy as np
import torch

import zefedra_ref as Z


def layer(gated=False, heads=3, dim=20, vdim=12, q_rank=24, kv_rank=40, ff=50, scale=None, weights_of=None):
    e = {"type": "latent_attention_2" if gated else "latent_attention",
         "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale or dim ** -0.5},
         "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        e["weights_of"] = weights_of
    return e


def config(layers, width=72, vocab=101, eps=1e-5):
    return {"architecture": "Zefedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# every branch, sizes that need padding, values that differ from one another
MIXED = config([layer(), layer(True, heads=5, dim=8, vdim=24, q_rank=40, kv_rank=72, ff=0), layer(weights_of=0),
                layer(True, heads=2, dim=36, vdim=40, q_rank=70, kv_rank=130, ff=90)])


def weights(raw, seed=0):
    """{name: bf16 tensor on the host}, as a file would hold them."""
    from llama_cu_b200 import zefedra
    return dict(zefedra.synth_tensors(zefedra.read_config(raw), seed, "cpu"))


def write_model(path, raw, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(raw, f)
    header, blobs, at = {"__metadata__": {"format": "pt"}}, [], 0
    for name, t in w.items():
        b = t.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(header).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return str(path)


def load(L, raw, w, dt, tokens=512, max_seqs=4, max_tokens=None, **kw):
    """A context whose pool holds `tokens` tokens."""
    from dataclasses import replace
    from llama_cu_b200 import layered, zefedra
    cfg = replace(zefedra.read_config(raw), act_dtype=dt, nctx=tokens)
    ctx = L.load_model(cfg, zefedra.pack(cfg, layered.Tensors(w)), kv_bytes=(tokens + 63) // 64 * 64 * cfg.kv_bytes_per_token(),
                       max_tokens=max_tokens or tokens, max_seqs=max_seqs, **kw)
    return cfg, ctx


def reference(raw, w, tokens, keep_layers=False):
    return Z.forward(raw, w, list(tokens), torch.float64, keep_layers)


def rel_err(got, want):
    """Largest over positions of rms(difference, mean taken off) / rms of the wanted logits over everything."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return float((d * d).mean(-1).sqrt().max() / want.double().pow(2).mean().sqrt())


TOL = {1: 2.5e-2, 2: 2e-5}  # bf16, f32


class Runner:
    """Feeds portions of sequences through `step_logits`, every token's logits kept."""

    def __init__(self, ctx):
        self.ctx, self.live, self.out = ctx, {}, {}
        self.stream = torch.cuda.Stream()

    def step(self, entries, end=()):
        """entries: [(id, tokens)]"""
        reqs, toks = [], []
        for i, t in entries:
            if i not in self.live:
                self.live[i] = [self.ctx.seq_create(), 0]
                self.out[i] = []
            reqs.append((self.live[i][0], self.live[i][1], len(t)))
            self.live[i][1] += len(t)
            toks += [int(x) for x in t]
        with torch.cuda.stream(self.stream):
            lg = self.ctx.step_logits(reqs, toks, list(range(len(toks))), stream=self.stream).cpu()
        at = 0
        for i, t in entries:
            self.out[i].append(lg[at:at + len(t)])
            at += len(t)
        for i in end:
            self.ctx.seq_free(self.live.pop(i)[0])

    def logits(self, i):
        return torch.cat(self.out[i])

    def whole(self, tokens, cuts=None):
        """One request alone, cut into portions of the sizes in `cuts` (cycled); frees it."""
        name, at, k = object(), 0, 0
        tokens = list(tokens)
        while at < len(tokens):
            n = cuts[k % len(cuts)] if cuts else len(tokens)
            k += 1
            part = tokens[at:at + n]
            at += len(part)
            self.step([(name, part)], end=[name] if at == len(tokens) else [])
        return self.logits(name)


def plant_key(raw, w, layer_index, token_key, token_query, beta):
    """Adds a rank-one term to the query map of layer 0 (whose mixer must read unshifted embeddings: shift 0) so that
    `token_query` scores `token_key` far above anything else in every head."""
    assert layer_index == 0
    f = {k: v.double() for k, v in w.items()}
    eps, m = raw["norm"]["eps"], raw["layers"][0]["mixer"]
    h = f["embed"][[token_key, token_query]]
    c_q, c = Z.latents(h, f["l0.mix.dq"], f["l0.mix.dq.norm"], f["l0.mix.dkv"], f["l0.mix.dkv.norm"], eps)
    k, u = (f["l0.mix.uk"] @ c[0]).view(m["heads"], -1), c_q[1]
    k = (k / (k * k).sum(-1, keepdim=True)).reshape(-1)  # a unit of score in every head
    out = dict(w)
    out["l0.mix.uq"] = (f["l0.mix.uq"] + beta / m["scale"] * k[:, None] * u[None] / (u * u).sum()).to(torch.bfloat16)
    return out


def random_tokens(raw, n, seed, avoid=()):
    rng = np.random.default_rng(seed)
    pool = np.array([t for t in range(raw["vocab"]) if t not in avoid])
    return [int(x) for x in rng.choice(pool, n)]
