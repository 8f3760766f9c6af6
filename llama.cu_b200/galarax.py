"""Galarax: softmax attention and a gated delta rule side by side in every layer, pre-norm with weights around zero, squared-ReLU
feed-forwards, a range of layers that runs several times.  Configuration keys and tensor names only; the mechanisms live in the
library."""
from .layered import (ACT_RELU2, W_BRANCH_NORM, W_MIX_IN, W_STEP, AttentionMixer, DeltaMixer, LayerConfig, LayeredConfig, ParallelMixer,
                      Rotary, Tensors, _pad, attention_rows, delta_rows, pack_attention, pack_common, pack_delta, pack_pre_norm_block, pad_to)


def read_rotary(rot):
    sc = rot.get("scaling") or {}
    return Rotary(rot["dims"], rot["base"], sc.get("factor", 0.0), sc.get("original", 0.0), sc.get("fast", 0.0), sc.get("slow", 0.0))


def read_layer(i, e):
    if e["type"] != "parallel":
        raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
    l, r, mlp = e["mixer"]["left"], e["mixer"]["right"], e.get("mlp")
    if mlp is not None and mlp["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
    mixer = ParallelMixer(AttentionMixer(l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["scale"], read_rotary(l["rot"])),
                          DeltaMixer(r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]))
    return LayerConfig(mixer, mlp["ff"] if mlp is not None else 0, False, act=ACT_RELU2, pre_norm=True, file_layer=i)


def unroll(layers, loop):
    """The layers as they run: the looped range once per pass, later passes with the first one's weights; every pass starts with
    its own vector added to the residual stream, all but the first also with the embedding output."""
    from dataclasses import replace
    if not loop:
        return tuple(layers)
    a, b, times = loop["start"], loop["stop"], loop["times"]
    if not 0 <= a < b <= len(layers) or times < 1:
        raise ValueError(f"loop over layers {a} .. {b} of {len(layers)}, {times} times")
    out = list(layers[:a])
    for t in range(times):
        for i in range(a, b):
            l = layers[i]
            if i == a:
                l = replace(l, step=t, add_embed=t > 0)
            out.append(replace(l, weights_of=i) if t else l)
    return tuple(out + list(layers[b:]))


def read_config(raw, shapes=None):
    """LayeredConfig from the parsed config.json."""
    layers = unroll([read_layer(i, e) for i, e in enumerate(raw["layers"])], raw.get("loop"))
    return LayeredConfig("galarax", raw["width"], raw["vocab"], layers, raw["norm"]["eps"], arch="Galarax")


def uniform(name, n_layers, d, heads, kv_heads, dim, d_heads, d_kv_heads, d_dim, d_vdim, ff, vocab, conv=4, base=5e5, eps=1e-5, nctx=2048):
    """A model of equal layers that run once."""
    mixer = ParallelMixer(AttentionMixer(heads, kv_heads, dim, dim, dim ** -0.5, Rotary(dim // 2, base, 4.0, nctx, 32.0, 1.0)),
                          DeltaMixer(d_heads, d_kv_heads, d_dim, d_vdim, conv))
    layers = tuple(LayerConfig(mixer, ff, False, act=ACT_RELU2, pre_norm=True, file_layer=i) for i in range(n_layers))
    return LayeredConfig(name, d, vocab, layers, eps, nctx=nctx, arch="Galarax")


def tensor_shapes(cfg):
    """{name: shape} of the model file."""
    out = {"embed": (cfg.vocab, cfg.d)}
    steps = sum(l.step >= 0 for l in cfg.layers)
    if steps:
        out["loop.step"] = (steps, cfg.d)
    for l in cfg.layers:
        if l.weights_of >= 0:
            continue
        p, m, r = f"l{l.file_layer}.", l.mixer.left, l.mixer.right
        out[p + "norm1"] = (cfg.d,)
        if l.ff:
            out[p + "norm2"] = (cfg.d,)
        p += "mix."
        for n, rows in (("q", m.heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.kv_heads * m.v_dim)):
            out[p + "left." + n], out[p + "left." + n + ".b"] = (rows, cfg.d), (rows,)
        out[p + "left.o"] = (cfg.d, m.heads * m.v_dim)
        for n, rows in (("q", r.kv_heads * r.dim), ("k", r.kv_heads * r.dim), ("v", r.heads * r.v_dim)):
            out[p + "right." + n], out[p + "right." + n + ".conv"] = (rows, cfg.d), (rows, r.conv)
        out.update({p + "right.b": (r.heads, cfg.d), p + "right.A_log": (r.heads,), p + "right.norm": (r.v_dim,), p + "right.a": (r.heads, cfg.d),
                    p + "right.dt_bias": (r.heads,), p + "right.g": (r.heads * r.v_dim, cfg.d), p + "right.o": (cfg.d, r.heads * r.v_dim),
                    p + "left.out": (cfg.d,), p + "right.out": (cfg.d,)})
        if l.ff:
            p = f"l{l.file_layer}.mlp."
            out[p + "up"], out[p + "down"] = (l.ff, cfg.d), (cfg.d, l.ff)
    out["final.norm"], out["head"] = (cfg.d,), (cfg.vocab, cfg.d)
    return out


def pack(cfg, tensors):
    """Yields ((layer, kind), tensor) in the library's layouts."""
    import torch
    shapes, wp = tensor_shapes(cfg), pad_to(cfg.d, 64)

    def t(name):
        return tensors.take(name, *shapes[name])

    yield from pack_common(cfg.d, t("embed"), 1 + t("final.norm").float(), t("head"))
    for i, l in enumerate(cfg.layers):
        if l.step >= 0:
            yield (i, W_STEP), _pad(t("loop.step")[l.step].float(), wp)
        if l.weights_of >= 0:
            continue
        p, m, r = f"l{l.file_layer}.", l.mixer.left, l.mixer.right
        lt, rt = (lambda n: t(p + "mix.left." + n)), (lambda n: t(p + "mix.right." + n))
        rows = attention_rows(m, cfg.d, *map(lt, "qkv")) + delta_rows(r, cfg.d, *map(rt, "qkvgba"))
        parts = [(W_MIX_IN, torch.cat(rows))]
        parts += pack_attention(m, cfg.d, lt("o"), [lt(n + ".b") for n in "qkv"])
        parts += pack_delta(r, cfg.d, *(rt(n) for n in ("q.conv", "k.conv", "v.conv", "A_log", "dt_bias", "norm", "o")))
        # half the sum of the two normed outputs: the halves go into the gains
        parts.append((W_BRANCH_NORM, torch.stack([_pad(0.5 * t(p + "mix." + s + ".out").float(), wp) for s in ("left", "right")])))
        ff = dict(gain2=1 + t(p + "norm2").float(), up=t(p + "mlp.up"), down=t(p + "mlp.down")) if l.ff else {}
        for kind, w in parts + pack_pre_norm_block(cfg.d, l.ff, 1 + t(p + "norm1").float(), **ff):
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
        if name.endswith("right.norm") or last == "out":
            w = 1.0 + 0.1 * w
        elif last in ("norm1", "norm2", "norm", "step", "b") and len(shape) == 1 or last == "step":
            w = 0.2 * w
        elif last == "A_log":
            w = w - 1.0
        elif last == "dt_bias":
            w = w - 1.5
        elif last == "conv":
            w = w / shape[-1] ** 0.5 * 1.5
        elif name != "embed":
            w = w / shape[-1] ** 0.5
        out[name] = w.to(torch.bfloat16)
    return out
