"""Mupuvik: layers of state space duality, sliding-window attention (whose keys and values another layer may lend), and softmax
attention beside gated linear attention; norms ahead of every sublayer and on its output, feed-forwards of experts, an embedding of
token pairs, a head that is the embedding table.  Configuration keys and tensor names only; the mechanisms live in the library."""
from .layered import (W_MIX_IN, W_PAIR_EMBD, AttentionMixer, GlaMixer, GluFf, LayerConfig, LayeredConfig, PairEmbedding, ParallelMixer, Rotary,
                      SsdMixer, Tensors, _pad, attention_rows, gla_rows, pack_attention, pack_common, pack_experts, pack_gla, pack_norms, pack_ssd,
                      pad_to, ssd_rows)

GLU_ALPHA, GLU_SHIFT = 1.702, 1.0  # of every expert's activation


def read_mixer(i, e, shapes):
    m, kind = e["mixer"], e["type"]
    if kind == "mamba2":
        return SsdMixer(m["heads"], m["groups"], m["state"], m["vdim"], m["conv"], m["norm_groups"])
    if kind == "attention":
        j = m.get("kv_from")
        return AttentionMixer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], None, bias=True, qk_norm=3, window=m["mask"]["size"], out_gate=True,
                              kv_from=-1 if j is None else j)
    if kind == "parallel":
        l, r = m["left"], m["right"]
        rank = (shapes or {}).get(f"l{i}.mix.right.a1", (16,))[0]  # the file's tensor gives it
        left = AttentionMixer(l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["scale"], Rotary(l["rot"]["dims"], l["rot"]["base"], adjacent=True), bias=False,
                              qk_norm=2, sink=True, out_gate=True)
        return ParallelMixer(left, GlaMixer(r["heads"], r["dim"], r["vdim"], r["tau"], rank), (m["left_scale"], m["right_scale"]))
    raise ValueError(f"layer {i}: unknown mixer type {kind!r}")


def read_feed_forward(i, mlp):
    if mlp is None:
        return 0
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    e, r, s = mlp["expert"], mlp["router"], mlp.get("shared")
    return GluFf(e["ff"], e["limit"], GLU_ALPHA, GLU_SHIFT, r["experts"], r["top"], s["ff"] if s else 0, s["limit"] if s else 0.0)


def read_config(raw, shapes=None):
    """LayeredConfig from the parsed config.json and the shapes of the file's tensors."""
    layers = tuple(LayerConfig(read_mixer(i, e, shapes), read_feed_forward(i, e.get("mlp")), False, pre_norm=True, post_norm=True, file_layer=i)
                   for i, e in enumerate(raw["layers"]))
    for i, l in enumerate(layers):
        j = getattr(l.mixer, "kv_from", -1)
        if j >= 0 and not (j < i and isinstance(layers[j].mixer, AttentionMixer) and layers[j].mixer.kv_from < 0):
            raise ValueError(f"layer {i}: keys and values of layer {j}")
    e = raw["embedding"]
    b = e.get("bigram")
    return LayeredConfig("mupuvik", raw["width"], raw["vocab"], layers, raw["norm"]["eps"], arch="Mupuvik", embed_scale=e["scale"],
                         pairs=PairEmbedding(b["buckets"], b["mul_prev"], b["mul_cur"]) if b else None)


def uniform(name, n_layers, d, heads, kv_heads, dim, window, s_heads, s_groups, s_dim, s_vdim, g_heads, g_dim, g_vdim, ff, experts, top, shared, vocab,
            conv=4, rank=16, base=5e5, eps=1e-5, nctx=2048):
    """Layers in turn: state space, window, state space, attention beside linear attention, and again with borrowed window keys."""
    ssd = SsdMixer(s_heads, s_groups, s_dim, s_vdim, conv, s_groups)
    both = ParallelMixer(AttentionMixer(heads, kv_heads, dim, dim, dim ** -0.5, Rotary(dim, base, adjacent=True), bias=False, qk_norm=2, sink=True, out_gate=True),
                         GlaMixer(g_heads, g_dim, g_vdim, 16.0, rank), (1.0, 1.0))

    def mixer(i):
        if i % 4 == 1:
            return AttentionMixer(heads, kv_heads, dim, dim, dim ** -0.5, None, qk_norm=3, window=window, out_gate=True, kv_from=i - 4 if i % 8 == 5 else -1)
        return both if i % 4 == 3 else ssd
    f = GluFf(ff, 7.0, GLU_ALPHA, GLU_SHIFT, experts, top, shared, 7.0)
    layers = tuple(LayerConfig(mixer(i), f, False, pre_norm=True, post_norm=True, file_layer=i) for i in range(n_layers))
    return LayeredConfig(name, d, vocab, layers, eps, nctx=nctx, arch="Mupuvik", embed_scale=d ** 0.5, pairs=PairEmbedding(65521, 31, 17))


def attention_shapes(m, p, d, bias):
    out = {}
    for n, rows in [("q", m.heads * m.dim)] + ([("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.v_dim)] if m.kv_from < 0 else []):
        out[p + n] = (rows, d)
        if bias:
            out[p + n + ".b"] = (rows,)
        if n != "v":
            out[p + n + ".norm"] = (m.dim if m.qk_norm == 2 else rows,)
    out.update({p + "g": (m.heads, d), p + "o": (d, m.heads * m.v_dim)})
    return out


def mixer_shapes(m, p, d):
    if isinstance(m, SsdMixer):
        inner, ch = m.heads * m.v_dim, m.heads * m.v_dim + 2 * m.groups * m.dim
        return {p + "in": (inner + ch + m.heads, d), p + "conv": (ch, m.conv), p + "conv.b": (ch,), p + "dt_bias": (m.heads,), p + "A_log": (m.heads,),
                p + "D": (m.heads,), p + "norm": (inner,), p + "o": (d, inner)}
    if isinstance(m, AttentionMixer):
        return attention_shapes(m, p, d, True)
    out, r, p = attention_shapes(m.left, p + "left.", d, False), m.right, p + "right."
    keys, values = r.heads * r.dim, r.heads * r.v_dim
    out.update({p + "q": (keys, d), p + "k": (keys, d), p + "v": (values, d), p + "g": (values, d), p + "o": (d, values), p + "norm": (r.v_dim,),
                p + "a1": (r.rank, d), p + "a2": (keys, r.rank), p + "a2.b": (keys,)})
    return out


def tensor_shapes(cfg):
    """{name: shape} of the model file."""
    out = {"embed": (cfg.vocab, cfg.d), "final.norm": (cfg.d,)}
    if cfg.pairs:
        out["bigram"] = (cfg.pairs.buckets + 1, cfg.d)
    for i, l in enumerate(cfg.layers):
        p, f = f"l{i}.", l.ff
        out.update({p + n: (cfg.d,) for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ())})
        out.update(mixer_shapes(l.mixer, p + "mix.", cfg.d))
        if not f:
            continue
        p += "mlp."
        out[p + "router"] = (f.experts, cfg.d)
        for name, ff in [(f"e{e}", f.ff) for e in range(f.experts)] + ([("shared", f.shared)] if f.shared else []):
            out.update({f"{p}{name}.gate": (ff, cfg.d), f"{p}{name}.up": (ff, cfg.d), f"{p}{name}.down": (cfg.d, ff)})
    return out


def pack_mixer(m, d, t):
    """(rows of the fused input projection, [(kind, tensor)]); t(name) is a tensor of the mixer."""
    if isinstance(m, SsdMixer):
        return ssd_rows(m, d, t("in")), pack_ssd(m, d, *map(t, ("conv", "conv.b", "A_log", "dt_bias", "D", "norm", "o")))
    if isinstance(m, AttentionMixer):
        own = "qkv" if m.kv_from < 0 else "q"
        return (attention_rows(m, d, *map(t, own), g=t("g")),
                pack_attention(m, d, t("o"), [t(n + ".b") for n in own] if m.bias else None, [t(n + ".norm") for n in own if n != "v"]))
    rows, parts = pack_mixer(m.left, d, lambda n: t("left." + n))
    r, rt = m.right, lambda n: t("right." + n)
    return rows + gla_rows(r, d, *map(rt, ("q", "k", "v", "g", "a1"))), parts + pack_gla(r, d, *map(rt, ("a2", "a2.b", "norm", "o")))


def pack(cfg, tensors):
    """Yields ((layer, kind), tensor) in the library's layouts."""
    import torch
    shapes = tensor_shapes(cfg)

    def t(name):
        return tensors.take(name, *shapes[name])

    yield from pack_common(cfg.d, t("embed"), 1 + t("final.norm").float(), t("embed"))
    if cfg.pairs:
        yield (-1, W_PAIR_EMBD), _pad(t("bigram"), cfg.pairs.buckets + 1, pad_to(cfg.d, 64))
    for i, l in enumerate(cfg.layers):
        p, f = f"l{i}.", l.ff
        rows, parts = pack_mixer(l.mixer, cfg.d, lambda n: t(p + "mix." + n))
        parts = [(W_MIX_IN, torch.cat(rows))] + parts
        parts += pack_norms(cfg.d, *(1 + t(p + n).float() for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f else ())))
        if f:
            def expert(e):
                return tuple(t(f"{p}mlp.{e}.{n}") for n in ("gate", "up", "down"))
            parts += pack_experts(f, cfg.d, t(p + "mlp.router"), (expert(f"e{e}") for e in range(f.experts)), expert("shared") if f.shared else None)
        for kind, w in parts:
            yield (i, kind), w


def synth_weights(cfg, seed=0, device="cuda:0"):
    """Seeded random weights in the library's layouts: yields ((layer, kind), tensor)."""
    return pack(cfg, synth_tensors(cfg, seed, device))


def synth_tensors(cfg, seed=0, device="cuda:0"):
    """Seeded random tensors of the model's shapes (a `Tensors` table), drawn on `device`: fan-in scaled matrices, small biases,
    decays spread between fast and slow."""
    import torch
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    out = Tensors()
    for name, shape in tensor_shapes(cfg).items():
        w = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm":
            w = 0.2 * w
        elif last in ("norm", "D"):
            w = 1.0 + 0.2 * w
        elif last == "b":
            w = 0.3 * w
        elif last == "A_log":
            w = w - 1.0
        elif last == "dt_bias":
            w = w - 1.5
        elif last == "conv":
            w = w / shape[-1] ** 0.5 * 1.5
        elif name == "embed":
            w = w / cfg.embed_scale
        elif name != "bigram":
            w = w / shape[-1] ** 0.5
        out[name] = w.to(torch.bfloat16)
    return out
