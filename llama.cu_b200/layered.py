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

from . import (ACT_RELU2, ACT_XIELU, BF16, F32, MIX_ATTENTION, MIX_DELTA, MIX_LATENT, W_ATT_OUT, W_BRANCH_NORM, W_CONV, W_DELTA_DECAY,
               W_DELTA_NORM, W_DELTA_OUT, W_EMBD, W_FF_DOWN, W_KV_NORM, W_LAT_IN, W_LAT_OUT, W_LM_HEAD, W_MIX_BIAS, W_MIX_IN, W_NORM1,
               W_NORM2, W_OUT_NORM, W_Q_NORM, W_SCALARS, W_SHIFT, W_STEP, W_UKT, W_UKV, W_UP, W_UQ, LayerDesc, ModelDesc)


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

    def describe(self, o):
        o.mixer, o.heads, o.dim, o.v_dim, o.q_rank, o.kv_rank = MIX_LATENT, self.heads, self.dim, self.v_dim, self.q_rank, self.kv_rank
        o.out_gate, o.scale = int(self.out_gate), self.scale

    def cached_per_token(self):
        return pad_to(self.kv_rank, 64)

    def state_bytes(self):
        return 0

    def weights(self, d):
        return (d * (self.q_rank + self.kv_rank + (self.heads if self.out_gate else 0)) + self.heads * self.dim * self.q_rank
                + self.heads * (self.dim + self.v_dim) * self.kv_rank + d * self.heads * self.v_dim)


@dataclass(frozen=True)
class Rotary:
    """Frequencies base^(-2i / dims); factor > 0: scaled for longer contexts (YaRN)."""
    dims: int
    base: float
    factor: float = 0.0
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0


@dataclass(frozen=True)
class AttentionMixer:
    """Softmax attention with grouped heads, rotary positions, optionally biases and normalised queries and keys."""
    heads: int
    kv_heads: int
    dim: int
    v_dim: int
    scale: float
    rot: Rotary
    bias: bool = True
    qk_norm: bool = True

    def describe(self, o):
        o.mixer |= MIX_ATTENTION
        o.heads, o.kv_heads, o.dim, o.v_dim, o.scale = self.heads, self.kv_heads, self.dim, self.v_dim, self.scale
        o.bias, o.qk_norm, r = int(self.bias), int(self.qk_norm), self.rot
        if r is not None:
            o.rot_dims, o.rot_base, o.rot_factor, o.rot_original, o.rot_fast, o.rot_slow = r.dims, r.base, r.factor, r.original, r.fast, r.slow

    def cached_per_token(self):
        return self.kv_heads * (pad_to(self.dim, 16) + pad_to(self.v_dim, 16))

    def state_bytes(self):
        return 0

    def weights(self, d):
        return d * (self.heads + self.kv_heads) * (self.dim + self.v_dim)


@dataclass(frozen=True)
class DeltaMixer:
    """Gated delta rule behind short convolutions, its output normed and gated per head."""
    heads: int
    kv_heads: int
    dim: int
    v_dim: int
    conv: int

    def describe(self, o):
        o.mixer |= MIX_DELTA
        o.delta_heads, o.delta_kv_heads, o.delta_dim, o.delta_v_dim, o.delta_conv = self.heads, self.kv_heads, self.dim, self.v_dim, self.conv

    def cached_per_token(self):
        return 0

    def state_bytes(self):
        return 4 * self.heads * pad_to(self.v_dim, 16) * pad_to(self.dim, 32)

    def weights(self, d):
        return d * (2 * self.kv_heads * self.dim + 3 * self.heads * self.v_dim + 2 * self.heads)


@dataclass(frozen=True)
class ParallelMixer:
    """Two mixers on the same input, their outputs normed over the width and averaged."""
    left: AttentionMixer
    right: DeltaMixer

    def describe(self, o):
        self.left.describe(o)
        self.right.describe(o)

    def cached_per_token(self):
        return self.left.cached_per_token() + self.right.cached_per_token()

    def state_bytes(self):
        return self.left.state_bytes() + self.right.state_bytes()

    def weights(self, d):
        return self.left.weights(d) + self.right.weights(d)


@dataclass(frozen=True)
class LayerConfig:
    """One layer as it runs; a layer that runs several times is listed several times (`weights_of`)."""
    mixer: object
    ff: int = 0  # 0: no feed-forward
    token_shift: bool = True
    weights_of: int = -1
    act: int = ACT_XIELU
    pre_norm: bool = False
    add_embed: bool = False  # the embedding output is added to the residual stream ahead of the layer
    step: int = -1           # row of the table of vectors added ahead of the layer, -1: none
    file_layer: int = -1     # the layer's number in the model file, -1: its place in the list


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
            l.mixer.describe(o)
            o.token_shift, o.ff, o.ff_act, o.weights_of = int(l.token_shift), l.ff, l.act, l.weights_of
            o.pre_norm, o.add_embed, o.add_step = int(l.pre_norm), int(l.add_embed), int(l.step >= 0)
        return out

    def kv_bytes_per_token(self, tp=1):
        eb = 4 if self.act_dtype == F32 else 2
        return max(sum(l.mixer.cached_per_token() for l in self.layers) * eb, 1)

    def state_bytes_per_sequence(self):
        """Recurrent matrices of one sequence (f32)."""
        return sum(l.mixer.state_bytes() for l in self.layers)

    def weight_bytes_per_step(self, tp=1):
        return self.vocab * self.d * 2.0 + sum(2.0 * (l.mixer.weights(self.d) + 2 * l.ff * self.d) for l in self.layers)


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


def _pad_heads(t, heads, size, to):
    """[heads * size, ...] -> [heads * to, ...], every head padded with zeros."""
    return _pad(t.reshape(heads, size, *t.shape[1:]), heads, to, *t.shape[1:]).reshape(heads * to, *t.shape[1:])


def _out_columns(o, d, heads, size, to):
    """Output projection [d, heads * size] with padded heads, rows and columns."""
    wp = pad_to(d, 64)
    return _pad(_pad(o.reshape(d, heads, size), d, heads, to).reshape(d, heads * to), wp, pad_to(heads * to, 64))


def attention_rows(m, d, q, k, v):
    """Rows of the fused input projection of an AttentionMixer."""
    wp, dp, vp = pad_to(d, 64), pad_to(m.dim, 16), pad_to(m.v_dim, 16)
    return [_pad(_pad_heads(w, n, a, b), n * b, wp) for w, n, a, b in
            ((q, m.heads, m.dim, dp), (k, m.kv_heads, m.dim, dp), (v, m.kv_heads, m.v_dim, vp))]


def pack_attention(m, d, o, bias=None):
    """[(kind, tensor)] of an AttentionMixer besides its input projection; bias: (q, k, v)."""
    import torch
    dp, vp = pad_to(m.dim, 16), pad_to(m.v_dim, 16)
    out = [(W_ATT_OUT, _out_columns(o, d, m.heads, m.v_dim, vp))]
    if m.bias:
        out.append((W_MIX_BIAS, torch.cat([_pad_heads(b.float(), n, x, y) for b, n, x, y in
                                           zip(bias, (m.heads, m.kv_heads, m.kv_heads), (m.dim, m.dim, m.v_dim), (dp, dp, vp))])))
    return out


def delta_rows(m, d, q, k, v, g, b, a):
    """Rows of the fused input projection of a DeltaMixer."""
    wp, dp, vp, hp = pad_to(d, 64), pad_to(m.dim, 32), pad_to(m.v_dim, 16), pad_to(m.heads, 8)
    return [_pad(_pad_heads(w, n, x, y), n * y, wp) for w, n, x, y in
            ((q, m.kv_heads, m.dim, dp), (k, m.kv_heads, m.dim, dp), (v, m.heads, m.v_dim, vp), (g, m.heads, m.v_dim, vp))] + [
            _pad(b, hp, wp), _pad(a, hp, wp)]


def pack_delta(m, d, conv_q, conv_k, conv_v, a_log, dt_bias, norm, o):
    """[(kind, tensor)] of a DeltaMixer besides its input projection."""
    import torch
    dp, vp, hp = pad_to(m.dim, 32), pad_to(m.v_dim, 16), pad_to(m.heads, 8)
    conv = torch.cat([_pad_heads(w.float(), n, x, y) for w, n, x, y in
                      ((conv_q, m.kv_heads, m.dim, dp), (conv_k, m.kv_heads, m.dim, dp), (conv_v, m.heads, m.v_dim, vp))])
    return [(W_CONV, conv.T.contiguous()), (W_DELTA_DECAY, torch.stack([_pad(a_log.float(), hp), _pad(dt_bias.float(), hp)])),
            (W_DELTA_NORM, _pad(norm.float(), vp)), (W_DELTA_OUT, _out_columns(o, d, m.heads, m.v_dim, vp))]


def pack_common(d, embed, final_gain, head):
    """final_gain: one number, or [d] (pre-norm models)."""
    wp = pad_to(d, 64)
    gain = final_gain.float().reshape(-1)
    return [((-1, W_EMBD), _pad(embed, embed.shape[0], wp)), ((-1, W_OUT_NORM), _pad(gain, wp) if final_gain.dim() else gain),
            ((-1, W_LM_HEAD), _pad(head, pad_to(head.shape[0], 8), wp))]


def pack_pre_norm_block(d, ff, gain1, gain2=None, up=None, down=None):
    """[(kind, tensor)] of what surrounds a mixer in a pre-norm layer; gains in f32."""
    wp, fp = pad_to(d, 64), pad_to(ff, 64)
    out = [(W_NORM1, _pad(gain1.float(), wp))]
    if ff:
        out += [(W_NORM2, _pad(gain2.float(), wp)), (W_UP, _pad(up, fp, wp)), (W_FF_DOWN, _pad(down, wp, fp))]
    return out


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
    from . import galarax, zefedra
    return {"Galarax": galarax, "Zefedra": zefedra}


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
