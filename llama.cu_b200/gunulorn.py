"""Gunulorn: mixer and feed-forward side by side on one residual stream; softmax attention behind short convolutions, with a learned sink
and a factor per head, whose keys and values another layer may use; attention through a sliding window that keeps the first tokens, keys
and values with rotary positions; dense feed-forwards of normed powers, experts some of which return their input; capped logits.
Configuration keys and tensor names only; the mechanisms live in the library."""
import math

from .layered import (W_MIX_IN, AttentionMixer, GluFf, LayerConfig, LayeredConfig, PolyNormFf, Rotary, Tensors, attention_rows, pack_attention, pack_common,
                      pack_experts, pack_norms, pack_poly)


def conv_attention(heads, kv_heads, dim, v_dim, scale, conv, kv_from=-1):
    return AttentionMixer(heads, kv_heads, dim, v_dim, scale, None, bias=False, qk_norm=0, sink=2, kv_from=kv_from, conv=conv, head_temp=True)


def window_attention(heads, kv_heads, dim, v_dim, scale, rot_dims, base, window, keep_first):
    return AttentionMixer(heads, kv_heads, dim, v_dim, scale, Rotary(rot_dims, base, adjacent=True), bias=False, qk_norm=0, window=window, sink=1,
                          keep_first=keep_first, rot_values=True)


def expert_ff(ff, experts, top, identity):
    """SiLU-gated experts without limits."""
    return GluFf(ff, math.inf, experts=experts, top=top, softmax=True, identity=identity)


def read_mixer(i, e):
    m, kind = e["mixer"], e["type"]
    sizes = (m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"])
    if kind == "attention":
        j = m.get("kv_from")
        return conv_attention(*sizes, m["conv"], -1 if j is None else j)
    if kind == "attention_2":
        return window_attention(*sizes, m["rot"]["dims"], m["rot"]["base"], m["mask"]["size"], m["mask"]["keep_first"])
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def read_feed_forward(i, mlp):
    if mlp is None:
        return 0
    if mlp["kind"] == "dense":
        return PolyNormFf(mlp["ff"])
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    r = mlp["router"]
    return expert_ff(mlp["expert"]["ff"], r["experts"], r["top"], r["identity"])


def layer(i, mixer, ff):
    return LayerConfig(mixer, ff, False, pre_norm=True, parallel_ff=bool(ff), file_layer=i)


def read_config(raw, shapes=None):
    """LayeredConfig from the parsed config.json."""
    layers = tuple(layer(i, read_mixer(i, e), read_feed_forward(i, e.get("mlp"))) for i, e in enumerate(raw["layers"]))
    for i, l in enumerate(layers):
        j = l.mixer.kv_from
        if j >= 0 and not (j < i and layers[j].mixer.conv and layers[j].mixer.kv_from < 0):
            raise ValueError(f"layer {i}: keys and values of layer {j}")
    return LayeredConfig("gunulorn", raw["width"], raw["vocab"], layers, raw["norm"]["eps"], arch="Gunulorn", logit_scale=raw["logit_scale"],
                         logit_cap=raw["logit_softcap"])


def uniform(name, n_layers, d, heads, kv_heads, dim, window, keep_first, dense_ff, ff, experts, top, identity, vocab, conv=4, base=5e5, eps=1e-5, nctx=2048):
    """Three window layers, then one that sees everything (every second of those with borrowed keys); the first feed-forward is dense,
    and again every eighth."""
    def mixer(i):
        if i % 4 == 3:
            return conv_attention(heads, kv_heads, dim, dim, dim ** -0.5, conv, i - 4 if i % 8 == 7 else -1)
        return window_attention(heads, kv_heads, dim, dim, dim ** -0.5, dim // 2, base, window, keep_first)
    f = expert_ff(ff, experts, top, identity)
    layers = tuple(layer(i, mixer(i), PolyNormFf(dense_ff) if i % 8 == 0 else f) for i in range(n_layers))
    return LayeredConfig(name, d, vocab, layers, eps, nctx=nctx, arch="Gunulorn", logit_cap=30.0)


def tensor_shapes(cfg):
    """{name: shape} of the model file."""
    d = cfg.d
    out = {"embed": (cfg.vocab, d), "final.norm": (d,), "head": (cfg.vocab, d)}
    for i, l in enumerate(cfg.layers):
        m, f, p = l.mixer, l.ff, f"l{i}."
        out.update({p + n: (d,) for n in (("norm1", "norm2") if f else ("norm1",))})
        p += "mix."
        rows = {"q": m.heads * m.dim, "k": m.own_kv_heads * m.dim, "v": m.own_kv_heads * m.v_dim}
        for n, r in rows.items():
            if r:
                out[p + n] = (r, d)
                if m.conv:
                    out[p + n + ".conv"] = (r, m.conv)
        if m.conv:
            out.update({p + n: (m.heads,) for n in ("sink", "temp")})
        out[p + "o"] = (d, m.heads * m.v_dim)
        p = f"l{i}.mlp."
        if isinstance(f, PolyNormFf):
            out.update({p + "up": (f.ff, d), p + "up.b": (f.ff,), p + "down": (d, f.ff), p + "down.b": (d,), p + "act": (4,)})
        elif f:
            n = f.experts + f.identity
            out.update({p + "router": (n, d), p + "correction": (n,)})
            for e in range(f.experts):
                out.update({f"{p}e{e}.gate": (f.ff, d), f"{p}e{e}.up": (f.ff, d), f"{p}e{e}.down": (d, f.ff)})
    return out


def pack_mixer(m, d, t):
    """(rows of the fused input projection, [(kind, tensor)]); t(name) is a tensor of the mixer."""
    own = "qkv" if m.kv_from < 0 else "q"
    more = dict(conv=[t(n + ".conv") for n in own], sink=t("sink"), temp=t("temp")) if m.conv else {}
    return attention_rows(m, d, *map(t, own)), pack_attention(m, d, t("o"), **more)


def pack(cfg, tensors):
    """Yields ((layer, kind), tensor) in the library's layouts."""
    import torch
    shapes = tensor_shapes(cfg)

    def t(name):
        return tensors.take(name, *shapes[name])

    yield from pack_common(cfg.d, t("embed"), t("final.norm"), t("head"))
    for i, l in enumerate(cfg.layers):
        p, f = f"l{i}.", l.ff
        rows, parts = pack_mixer(l.mixer, cfg.d, lambda n: t(p + "mix." + n))
        parts = [(W_MIX_IN, torch.cat(rows))] + parts + pack_norms(cfg.d, t(p + "norm1"), norm2=t(p + "norm2") if f else None)
        p += "mlp."
        if isinstance(f, PolyNormFf):
            parts += pack_poly(f, cfg.d, *(t(p + n) for n in ("up", "up.b", "down", "down.b", "act")))
        elif f:
            parts += pack_experts(f, cfg.d, t(p + "router"), (tuple(t(f"{p}e{e}.{n}") for n in ("gate", "up", "down")) for e in range(f.experts)),
                                  correction=t(p + "correction"))
        for kind, w in parts:
            yield (i, kind), w


def synth_weights(cfg, seed=0, device="cuda:0"):
    """Seeded random weights in the library's layouts: yields ((layer, kind), tensor)."""
    return pack(cfg, synth_tensors(cfg, seed, device))


def synth_tensors(cfg, seed=0, device="cuda:0"):
    """Seeded random tensors of the model's shapes (a `Tensors` table), drawn on `device`: fan-in scaled matrices, small biases."""
    import torch
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    out = Tensors()
    for name, shape in tensor_shapes(cfg).items():
        w = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2", "temp"):
            w = 1.0 + 0.2 * w
        elif last == "b":
            w = 0.3 * w
        elif last == "act":
            w = 0.5 + 0.3 * w
        elif last == "correction":
            w = 0.05 * w
        elif last == "conv":
            w = w / shape[-1] ** 0.5 * 1.5
        elif name != "embed" and last != "sink":
            w = w / shape[-1] ** 0.5
        out[name] = w.to(torch.bfloat16)
    return out
