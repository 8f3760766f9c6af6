"""Models described layer by layer: configuration, packing of weights into the library's padded layouts, and the registry
of architectures that a folder with config.json + model.safetensors can name.

A family's module turns config.json into a `LayeredConfig` and its tensors into a `Tensors` table; everything from there on
(packing, upload, cache, rounds, sampling) is common.
"""
import json
import os
import struct
from dataclasses import dataclass

import numpy as np

from . import (ACT_XIELU, BF16, F32, MIX_LATENT, W_EMBD, W_FF_DOWN, W_KV_NORM, W_LAT_IN, W_LAT_OUT, W_LM_HEAD, W_OUT_NORM,
               W_Q_NORM, W_SCALARS, W_SHIFT, W_UKT, W_UKV, W_UP, W_UQ, LayerDesc, ModelDesc)


def pad_to(v, m):
    return (v + m - 1) // m * m


@dataclass(frozen=True)
class LatentMixer:
    """Latent attention without positions; queries go through a latent of their own."""
    heads: int
    dim: int
    v_dim: int
    q_rank: int
    kv_rank: int
    scale: float
    out_gate: bool = False


@dataclass(frozen=True)
class LayerConfig:
    mixer: LatentMixer
    ff: int = 0  # 0: no feed-forward
    token_shift: bool = True
    weights_of: int = -1


@dataclass(frozen=True)
class LayeredConfig:
    name: str
    d: int
    vocab: int
    layers: tuple
    eps: float
    act_dtype: int = BF16  # or F32: everything in 32-bit arithmetic
    nctx: int = 2048
    arch: str = "Zefedra"  # key of `architectures()`

    @property
    def family(self):
        return architectures()[self.arch]

    @property
    def n_layers(self):
        return len(self.layers)

    @property
    def wdt(self):
        return BF16

    def desc(self, page_tokens=0, max_tokens=0, max_seqs=0, nctx=None):
        d = ModelDesc()
        d.n_layers, d.d, d.vocab, d.nctx, d.eps = self.n_layers, self.d, self.vocab, nctx or self.nctx, self.eps
        d.act_dtype, d.weight_dtype, d.norm_dtype = self.act_dtype, BF16, BF16
        d.page_tokens, d.max_tokens, d.max_seqs = page_tokens, max_tokens, max_seqs
        return d

    def layer_descs(self):
        out = (LayerDesc * self.n_layers)()
        for o, l in zip(out, self.layers):
            m = l.mixer
            o.mixer, o.heads, o.dim, o.v_dim, o.q_rank, o.kv_rank = MIX_LATENT, m.heads, m.dim, m.v_dim, m.q_rank, m.kv_rank
            o.out_gate, o.token_shift, o.ff, o.ff_act = int(m.out_gate), int(l.token_shift), l.ff, ACT_XIELU
            o.weights_of, o.scale = l.weights_of, m.scale
        return out

    def kv_bytes_per_token(self, tp=1):
        eb = 4 if self.act_dtype == F32 else 2
        return sum(pad_to(l.mixer.kv_rank, 64) for l in self.layers) * eb

    def weight_bytes_per_step(self, tp=1):
        total = self.vocab * self.d * 2.0
        for l in self.layers:
            m = l.mixer
            total += 2.0 * (self.d * (m.q_rank + m.kv_rank + (m.heads if m.out_gate else 0)) + m.heads * m.dim * m.q_rank
                            + m.heads * (m.dim + m.v_dim) * m.kv_rank + self.d * m.heads * m.v_dim + 2 * l.ff * self.d)
        return total


def _pad(t, *shape):
    """Zero-pads a tensor at the end of every dimension."""
    import torch
    if tuple(t.shape) == shape:
        return t.contiguous()
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def pack_latent(m, d, dq, dq_norm, uq, dkv, dkv_norm, uk, uv, o, g=None):
    """[(kind, tensor)] of a latent mixer in the library's layouts (see lcu_layer_weight_shape): one fused input projection,
    per-head sizes padded to 16, summed-over sizes to 64, the key map once more transposed per head for absorbed queries."""
    import torch
    dp, vp, qp, rp, wp = pad_to(m.dim, 16), pad_to(m.v_dim, 16), pad_to(m.q_rank, 64), pad_to(m.kv_rank, 64), pad_to(d, 64)
    parts = [_pad(dq, qp, wp), _pad(dkv, rp, wp)]
    if m.out_gate:
        parts.append(_pad(g, pad_to(m.heads, 8), wp))
    k = _pad(uk.reshape(m.heads, m.dim, m.kv_rank), m.heads, dp, rp)
    v = _pad(uv.reshape(m.heads, m.v_dim, m.kv_rank), m.heads, vp, rp)
    out = _pad(o.reshape(d, m.heads, m.v_dim), d, m.heads, vp).reshape(d, m.heads * vp)
    return [(W_LAT_IN, torch.cat(parts)), (W_Q_NORM, _pad(dq_norm, qp)), (W_KV_NORM, _pad(dkv_norm, rp)),
            (W_UQ, _pad(uq.reshape(m.heads, m.dim, m.q_rank), m.heads, dp, qp)), (W_UKT, k.transpose(1, 2).contiguous()),
            (W_UKV, torch.cat([k.reshape(-1, rp), v.reshape(-1, rp)])), (W_LAT_OUT, _pad(out, wp, pad_to(m.heads * vp, 64)))]


def pack_common(d, embed, final_gain, head):
    wp = pad_to(d, 64)
    return [((-1, W_EMBD), _pad(embed, embed.shape[0], wp)), ((-1, W_OUT_NORM), final_gain.float().reshape(1)),
            ((-1, W_LM_HEAD), _pad(head, pad_to(head.shape[0], 8), wp))]


def pack_block(d, ff, norm1, norm2=None, shift=None, up=None, down=None, act=None):
    """[(kind, tensor)] of what surrounds a mixer: norm gains, token shift, feed-forward."""
    import torch
    wp, fp = pad_to(d, 64), pad_to(ff, 64)
    sc = torch.zeros(4, dtype=torch.float32, device=norm1.device)
    sc[0] = norm1.float()
    out = []
    if ff:
        sc[1], sc[2:4] = norm2.float(), act.float()
        out += [(W_UP, _pad(up, fp, wp)), (W_FF_DOWN, _pad(down, wp, fp))]
    if shift is not None:
        out.append((W_SHIFT, _pad(shift, wp)))
    return out + [(W_SCALARS, sc)]


# ------------------------------------------------------------------ files

_ST_DTYPES = {"BF16": "bfloat16", "F16": "float16", "F32": "float32", "I32": "int32"}


def read_safetensors(path):
    """{name: torch tensor} of a safetensors file (host memory, mapped)."""
    import torch
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        header = json.loads(f.read(n))
    data = np.memmap(path, np.uint8, "c", offset=8 + n)
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        if e["dtype"] not in _ST_DTYPES:
            raise ValueError(f"{path}: tensor {name} has dtype {e['dtype']}")
        a, b = e["data_offsets"]
        dt = getattr(torch, _ST_DTYPES[e["dtype"]])
        out[name] = torch.from_numpy(np.array(data[a:b])).view(dt).reshape(e["shape"])
    return out


class Tensors(dict):
    """The tensors of a model file; reads are checked against the configuration."""

    def take(self, name, *shape):
        if name not in self:
            raise ValueError(f"tensor {name} is missing")
        t = self[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, the configuration says {shape}")
        import torch
        return t if t.dtype == torch.bfloat16 else t.to(torch.bfloat16)


def architectures():
    """config.json's "architecture" -> module with read_config(dict) and pack(cfg, Tensors)."""
    from . import zefedra
    return {"Zefedra": zefedra}


def load_pretrained(path, act_dtype=BF16, device=0, nctx=None, kv_tokens=None, page_tokens=0, max_tokens=0, max_seqs=0):
    """(config, Context) of the model in a folder with config.json and model.safetensors; the cache pool holds `kv_tokens`
    tokens (default: one full context)."""
    from dataclasses import replace
    from .model import load_model
    with open(os.path.join(path, "config.json")) as f:
        raw = json.load(f)
    arch = raw.get("architecture")
    known = architectures()
    if arch not in known:
        raise ValueError(f"{path}: architecture {arch!r} is not one of {sorted(known)}")
    cfg = replace(known[arch].read_config(raw), act_dtype=act_dtype)
    if nctx:
        cfg = replace(cfg, nctx=nctx)
    weights = known[arch].pack(cfg, Tensors(read_safetensors(os.path.join(path, "model.safetensors"))))
    tokens = kv_tokens or cfg.nctx
    pt = page_tokens or 64
    ctx = load_model(cfg, weights, device=device, kv_bytes=(tokens + pt - 1) // pt * pt * cfg.kv_bytes_per_token(), page_tokens=page_tokens,
                     max_tokens=max_tokens, max_seqs=max_seqs)
    return cfg, ctx
