"""Zefedra: latent attention without positions, token shift ahead of every mixer, scalar-gain norms on the sublayers'
outputs, xIELU feed-forwards, layers that may share another layer's tensors.  Configuration keys and tensor names only;
the mechanisms live in the library."""
from .layered import LatentMixer, LayerConfig, LayeredConfig, pack_block, pack_common, pack_latent

MIXERS = {"latent_attention": False, "latent_attention_2": True}  # -> per-head output gate


def read_config(raw, shapes=None):
    """LayeredConfig from the parsed config.json."""
    layers = []
    for i, e in enumerate(raw["layers"]):
        if e["type"] not in MIXERS:
            raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
        m, mlp = e["mixer"], e.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        mixer = LatentMixer(m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"], MIXERS[e["type"]])
        j = e.get("weights_of")
        layers.append(LayerConfig(mixer, mlp["ff"] if mlp is not None else 0, True, -1 if j is None else j))
    return LayeredConfig("zefedra", raw["width"], raw["vocab"], tuple(layers), raw["norm"]["eps"])


def uniform(name, n_layers, d, heads, dim, v_dim, q_rank, kv_rank, ff, vocab, gated=True, eps=1e-6, nctx=2048):
    """A model of equal layers, gated and plain mixers alternating (`gated`) or all plain."""
    def layer(i):
        return LayerConfig(LatentMixer(heads, dim, v_dim, q_rank, kv_rank, dim ** -0.5, gated and i % 2 == 1), ff)
    return LayeredConfig(name, d, vocab, tuple(layer(i) for i in range(n_layers)), eps, nctx=nctx)


def tensor_shapes(cfg):
    """{name: shape} of the model file."""
    out = {"embed": (cfg.vocab, cfg.d), "final.norm": (), "head": (cfg.vocab, cfg.d)}
    for i, l in enumerate(cfg.layers):
        if l.weights_of >= 0:
            continue
        m, p = l.mixer, f"l{i}."
        out.update({p + "norm1": (), p + "shift": (cfg.d,), p + "mix.dq": (m.q_rank, cfg.d), p + "mix.dq.norm": (m.q_rank,),
                    p + "mix.uq": (m.heads * m.dim, m.q_rank), p + "mix.dkv": (m.kv_rank, cfg.d), p + "mix.dkv.norm": (m.kv_rank,),
                    p + "mix.uk": (m.heads * m.dim, m.kv_rank), p + "mix.uv": (m.heads * m.v_dim, m.kv_rank),
                    p + "mix.o": (cfg.d, m.heads * m.v_dim)})
        if m.out_gate:
            out[p + "mix.g"] = (m.heads, cfg.d)
        if l.ff:
            out.update({p + "norm2": (), p + "mlp.up": (l.ff, cfg.d), p + "mlp.down": (cfg.d, l.ff), p + "mlp.act": (2,)})
    return out


def pack(cfg, tensors):
    """Yields ((layer, kind), tensor) in the library's layouts."""
    shapes = tensor_shapes(cfg)

    def t(name):
        return tensors.take(name, *shapes[name])

    yield from pack_common(cfg.d, t("embed"), t("final.norm"), t("head"))
    for i, l in enumerate(cfg.layers):
        if l.weights_of >= 0:
            continue
        p = f"l{i}."
        ff = {k: t(p + n) for k, n in (("norm2", "norm2"), ("up", "mlp.up"), ("down", "mlp.down"), ("act", "mlp.act"))} if l.ff else {}
        parts = pack_latent(l.mixer, cfg.d, *(t(p + "mix." + n) for n in ("dq", "dq.norm", "uq", "dkv", "dkv.norm", "uk", "uv", "o")),
                            g=t(p + "mix.g") if l.mixer.out_gate else None)
        for kind, w in parts + pack_block(cfg.d, l.ff, t(p + "norm1"), shift=t(p + "shift"), **ff):
            yield (i, kind), w


def synth_weights(cfg, seed=0, device="cuda:0"):
    """Seeded random weights in the library's layouts: yields ((layer, kind), tensor)."""
    return pack(cfg, synth_tensors(cfg, seed, device))


def synth_tensors(cfg, seed=0, device="cuda:0"):
    """Seeded random tensors of the model's shapes (a `Tensors` table), drawn on `device`: fan-in scaled matrices, gains
    around one."""
    import torch
    from .layered import Tensors
    g = torch.Generator(device=device)
    g.manual_seed(seed)
    out = Tensors()
    for name, shape in tensor_shapes(cfg).items():
        w = torch.randn(shape, generator=g, device=device, dtype=torch.float32)
        last = name.rsplit(".", 1)[-1]
        if last.startswith("norm"):
            w = 1.0 + 0.1 * w
        elif last == "shift":
            w = torch.sigmoid(w)
        elif last == "act":
            w = 0.5 * w
        elif name != "embed":
            w = w / shape[-1] ** 0.5
        out[name] = w.to(torch.bfloat16)
    return out
