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

from . import (ACT_GLU, ACT_POLYNORM, ACT_RELU2, ACT_XIELU, BF16, F32, MIX_ATTENTION, MIX_DELTA, MIX_GLA, MIX_LATENT, MIX_SSD, W_ACT, W_ATT_CONV,
               W_ATT_OUT, W_BRANCH_NORM, W_CONV, W_CONV_BIAS, W_CORRECTION, W_DELTA_DECAY, W_DELTA_NORM, W_DELTA_OUT, W_DOWN_BIAS, W_EMBD,
               W_FF_DOWN, W_GATE_MAP, W_HEAD_TEMP, W_KV_NORM, W_LAT_IN, W_LAT_OUT, W_LM_HEAD, W_MIX_BIAS, W_MIX_IN, W_NORM1, W_NORM2, W_OUT_NORM,
               W_PAIR_EMBD, W_POST1, W_POST2, W_Q_NORM, W_QK_GAIN, W_ROUTER, W_SCALARS, W_SHARED_DOWN, W_SHARED_UP, W_SHIFT, W_SINK, W_STEP, W_UKT,
               W_UKV, W_UP, W_UP_BIAS, W_UQ, LayerDesc, ModelDesc)


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
    adjacent: bool = False  # pairs (2i, 2i + 1) instead of (i, i + dims / 2)


@dataclass(frozen=True)
class AttentionMixer:
    """Softmax attention with grouped heads, optionally rotary positions, biases, normalised queries and keys (qk_norm: see
    lcu_layer_desc), a sliding window that may keep the first tokens, a sink in the softmax (1: of score 0, 2: of a learned score per
    head), a gate per head, another layer's keys and values, convolutions over time behind the projections (`conv` taps), a factor
    on the scores per head, values rotated by their positions."""
    heads: int
    kv_heads: int
    dim: int
    v_dim: int
    scale: float
    rot: Rotary
    bias: bool = True
    qk_norm: int = 1
    window: int = 0
    sink: int = 0
    out_gate: bool = False
    kv_from: int = -1  # the layer whose keys and values are used, -1: its own
    keep_first: int = 0
    conv: int = 0
    head_temp: bool = False
    rot_values: bool = False

    def describe(self, o):
        o.mixer |= MIX_ATTENTION
        o.heads, o.kv_heads, o.dim, o.v_dim, o.scale = self.heads, self.kv_heads, self.dim, self.v_dim, self.scale
        o.bias, o.qk_norm, r = int(self.bias), int(self.qk_norm), self.rot
        o.window, o.sink, o.out_gate, o.kv_from = self.window, int(self.sink), int(self.out_gate), self.kv_from + 1
        if r is not None:
            o.rot_dims, o.rot_base, o.rot_factor, o.rot_original, o.rot_fast, o.rot_slow = r.dims, r.base, r.factor, r.original, r.fast, r.slow
            o.rot_adjacent = int(r.adjacent)
        o.keep_first, o.conv, o.head_temp, o.rot_values = self.keep_first, self.conv, int(self.head_temp), int(self.rot_values)

    @property
    def own_kv_heads(self):
        return self.kv_heads if self.kv_from < 0 else 0

    def cached_per_token(self):
        return self.own_kv_heads * (pad_to(self.dim, 16) + pad_to(self.v_dim, 16))

    def state_bytes(self):
        return 0  # the convolutions' inputs are a few rows

    def weights(self, d):
        return d * ((self.heads + self.own_kv_heads) * (self.dim + self.v_dim) + (self.heads if self.out_gate else 0))


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


def describe_recurrent(m, o, kv_heads):
    o.delta_heads, o.delta_kv_heads, o.delta_dim, o.delta_v_dim = m.heads, kv_heads, m.dim, m.v_dim


def recurrent_state_bytes(m):
    return 4 * m.heads * pad_to(m.v_dim, 16) * pad_to(m.dim, 32)


@dataclass(frozen=True)
class SsdMixer:
    """State space duality: one decay per head, keys and queries (`dim` numbers) per group of heads, short convolutions with biases,
    the gated output normed in equal parts."""
    heads: int
    groups: int
    dim: int
    v_dim: int
    conv: int
    norm_parts: int

    def describe(self, o):
        o.mixer |= MIX_SSD
        describe_recurrent(self, o, self.groups)
        o.delta_conv, o.norm_parts = self.conv, self.norm_parts

    def cached_per_token(self):
        return 0

    def state_bytes(self):
        return recurrent_state_bytes(self)

    def weights(self, d):
        return d * (2 * self.groups * self.dim + 3 * self.heads * self.v_dim + self.heads)


@dataclass(frozen=True)
class GlaMixer:
    """Gated linear attention: one decay per head and key channel, sigmoid(z)^(1 / tau) with z of low rank, the output normed and gated
    per head."""
    heads: int
    dim: int
    v_dim: int
    tau: float
    rank: int

    def describe(self, o):
        o.mixer |= MIX_GLA
        describe_recurrent(self, o, self.heads)
        o.gate_tau, o.gate_rank = self.tau, self.rank

    def cached_per_token(self):
        return 0

    def state_bytes(self):
        return recurrent_state_bytes(self)

    def weights(self, d):
        return d * (2 * self.heads * self.dim + 3 * self.heads * self.v_dim + self.rank)


@dataclass(frozen=True)
class ParallelMixer:
    """Softmax attention and a recurrent mixer on the same input, their outputs added: normed over the width with a gain each (scales
    None), or with a factor each."""
    left: AttentionMixer
    right: object
    scales: tuple = None

    def describe(self, o):
        self.left.describe(o)
        self.right.describe(o)
        if self.scales:
            o.out_scale, o.out_scale2 = self.scales

    def cached_per_token(self):
        return self.left.cached_per_token() + self.right.cached_per_token()

    def state_bytes(self):
        return self.left.state_bytes() + self.right.state_bytes()

    def weights(self, d):
        return self.left.weights(d) + self.right.weights(d)


@dataclass(frozen=True)
class GluFf:
    """Gated feed-forward: g = min(W_gate x, limit), u = clamp(W_up x, +-limit), W_down (g sigmoid(alpha g) (u + shift)).  With
    `experts` > 0 every token uses `top` of that many, their inputs scaled by the sigmoids of their router logits, and the shared
    one (width `shared`, 0: none).  softmax: scores are a softmax over all experts and `identity` more that return their input;
    corrected scores choose, the chosen scores divided by their sum weigh the outputs."""
    ff: int
    limit: float
    alpha: float = 1.0
    shift: float = 0.0
    experts: int = 0
    top: int = 0
    shared: int = 0
    shared_limit: float = 0.0
    softmax: bool = False
    identity: int = 0

    def describe(self, o):
        o.ff, o.ff_act, o.experts, o.top, o.shared_ff = self.ff, ACT_GLU, self.experts, self.top, self.shared
        o.glu_limit, o.shared_limit, o.glu_alpha, o.glu_shift = self.limit, self.shared_limit, self.alpha, self.shift
        o.route_softmax, o.identity = int(self.softmax), self.identity

    def weights(self, d):
        """Weights one token meets."""
        used = self.top * self.experts / (self.experts + self.identity) if self.experts else 1
        return d * (3 * (self.ff * used + self.shared) + self.experts + self.identity)


@dataclass(frozen=True)
class PolyNormFf:
    """W_down (a z / rms(z) + b z^2 / rms(z^2) + c z^3 / rms(z^3) + e) with z = W_up x, both with biases."""
    ff: int

    def describe(self, o):
        o.ff, o.ff_act, o.ff_bias = self.ff, ACT_POLYNORM, 1

    def weights(self, d):
        return 2 * self.ff * d


@dataclass(frozen=True)
class PairEmbedding:
    """Row (previous token * prev + token * cur) mod buckets is added to a token's embedding, row `buckets` to the first one's."""
    buckets: int
    prev: int
    cur: int


@dataclass(frozen=True)
class LayerConfig:
    """One layer as it runs; a layer that runs several times is listed several times (`weights_of`)."""
    mixer: object
    ff: object = 0  # width, 0: no feed-forward; or a GluFf or PolyNormFf
    token_shift: bool = True
    weights_of: int = -1
    act: int = ACT_XIELU
    pre_norm: bool = False
    add_embed: bool = False  # the embedding output is added to the residual stream ahead of the layer
    step: int = -1           # row of the table of vectors added ahead of the layer, -1: none
    file_layer: int = -1     # the layer's number in the model file, -1: its place in the list
    post_norm: bool = False  # pre-norm layers: norms on the sublayers' outputs too
    parallel_ff: bool = False  # pre-norm layers: mixer and feed-forward read the same x, each through a norm of its own

    def ff_weights(self, d):
        return 2 * self.ff * d if isinstance(self.ff, int) else self.ff.weights(d)


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
    embed_scale: float = 1.0
    pairs: PairEmbedding = None
    logit_scale: float = 1.0
    logit_cap: float = 0.0  # logits = cap tanh(scale head x / cap), 0: not capped

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
            o.token_shift, o.weights_of = int(l.token_shift), l.weights_of
            if isinstance(l.ff, int):
                o.ff, o.ff_act = l.ff, l.act
            else:
                l.ff.describe(o)
            o.parallel_ff = int(l.parallel_ff)
            o.pre_norm, o.post_norm, o.add_embed, o.add_step = int(l.pre_norm), int(l.post_norm), int(l.add_embed), int(l.step >= 0)
        out[0].embed_scale, out[0].logit_scale, out[0].logit_cap = self.embed_scale, self.logit_scale, self.logit_cap
        if self.pairs:
            b = self.pairs.buckets
            out[0].pair_buckets, out[0].pair_prev, out[0].pair_cur = b, self.pairs.prev % b, self.pairs.cur % b
        return out

    def kv_bytes_per_token(self, tp=1):
        eb = 4 if self.act_dtype == F32 else 2
        return max(sum(l.mixer.cached_per_token() for l in self.layers) * eb, 1)

    def state_bytes_per_sequence(self):
        """Recurrent matrices of one sequence (f32)."""
        return sum(l.mixer.state_bytes() for l in self.layers)

    def weight_bytes_per_step(self, tp=1):
        return self.vocab * self.d * 2.0 + sum(2.0 * (l.mixer.weights(self.d) + l.ff_weights(self.d)) for l in self.layers)


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


def attention_rows(m, d, q, k=None, v=None, g=None):
    """Rows of the fused input projection of an AttentionMixer (k and v: unless they are another layer's)."""
    wp, dp, vp = pad_to(d, 64), pad_to(m.dim, 16), pad_to(m.v_dim, 16)
    rows = [_pad(_pad_heads(w, n, a, b), n * b, wp) for w, n, a, b in
            ((q, m.heads, m.dim, dp), (k, m.kv_heads, m.dim, dp), (v, m.kv_heads, m.v_dim, vp)) if w is not None]
    return rows + ([_pad(g, pad_to(m.heads, 8), wp)] if m.out_gate else [])


def pack_attention(m, d, o, bias=None, gains=None, conv=None, sink=None, temp=None):
    """[(kind, tensor)] of an AttentionMixer besides its input projection; bias, conv: of (q, k, v), or (q,) without own keys; gains:
    the weights of the norms of q and k, one head's or all heads' ((q,) without own keys); sink, temp: a number per head."""
    import torch
    dp, vp = pad_to(m.dim, 16), pad_to(m.v_dim, 16)
    out = [(W_ATT_OUT, _out_columns(o, d, m.heads, m.v_dim, vp))]
    if m.bias:
        out.append((W_MIX_BIAS, torch.cat([_pad_heads(b.float(), n, x, y) for b, n, x, y in
                                           zip(bias, (m.heads, m.kv_heads, m.kv_heads), (m.dim, m.dim, m.v_dim), (dp, dp, vp))])))
    if m.qk_norm == 2:
        out.append((W_QK_GAIN, torch.cat([_pad(g.float(), dp) for g in gains])))
    if m.qk_norm == 3:
        out.append((W_QK_GAIN, torch.cat([_pad_heads(g.float(), n, m.dim, dp) for g, n in zip(gains, (m.heads, m.kv_heads))])))
    if m.conv:
        taps = torch.cat([_pad_heads(c.float(), n, x, y) for c, n, x, y in
                          zip(conv, (m.heads, m.kv_heads, m.kv_heads), (m.dim, m.dim, m.v_dim), (dp, dp, vp))])
        out.append((W_ATT_CONV, taps.T.contiguous()))
    return out + [(k, t.float().contiguous()) for k, t in ((W_SINK, sink), (W_HEAD_TEMP, temp)) if t is not None]


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


def ssd_rows(m, d, w):
    """Rows of the fused input projection of an SsdMixer; w: rows z | x | B | C | dt."""
    import torch
    wp, dp, vp, hp, inner, gn = pad_to(d, 64), pad_to(m.dim, 32), pad_to(m.v_dim, 16), pad_to(m.heads, 8), m.heads * m.v_dim, m.groups * m.dim
    z, x, b, c, dt = torch.split(w, [inner, inner, gn, gn, m.heads])
    return [_pad(_pad_heads(t, n, p, q), n * q, wp) for t, n, p, q in
            ((c, m.groups, m.dim, dp), (b, m.groups, m.dim, dp), (x, m.heads, m.v_dim, vp), (z, m.heads, m.v_dim, vp))] + [_pad(dt, hp, wp)]


def pack_ssd(m, d, conv, conv_bias, a_log, dt_bias, skip, norm, o):
    """[(kind, tensor)] of an SsdMixer besides its input projection; conv [x | B | C, taps]."""
    import torch
    dp, vp, hp, inner, gn = pad_to(m.dim, 32), pad_to(m.v_dim, 16), pad_to(m.heads, 8), m.heads * m.v_dim, m.groups * m.dim

    def channels(t):
        x, b, c = torch.split(t.float(), [inner, gn, gn])
        return torch.cat([_pad_heads(c, m.groups, m.dim, dp), _pad_heads(b, m.groups, m.dim, dp), _pad_heads(x, m.heads, m.v_dim, vp)])
    return [(W_CONV, channels(conv).T.contiguous()), (W_CONV_BIAS, channels(conv_bias)),
            (W_DELTA_DECAY, torch.stack([_pad(t.float(), hp) for t in (a_log, dt_bias, skip)])),
            (W_DELTA_NORM, _pad_heads(norm.float(), m.heads, m.v_dim, vp)), (W_DELTA_OUT, _out_columns(o, d, m.heads, m.v_dim, vp))]


def gla_rows(m, d, q, k, v, g, a1):
    """Rows of the fused input projection of a GlaMixer."""
    wp, dp, vp = pad_to(d, 64), pad_to(m.dim, 32), pad_to(m.v_dim, 16)
    return [_pad(_pad_heads(w, m.heads, x, y), m.heads * y, wp) for w, x, y in ((q, m.dim, dp), (k, m.dim, dp), (v, m.v_dim, vp), (g, m.v_dim, vp))] + [
            _pad(a1, pad_to(m.rank, 8), wp)]


def pack_gla(m, d, a2, a2_bias, norm, o):
    """[(kind, tensor)] of a GlaMixer besides its input projection."""
    import torch
    dp, vp = pad_to(m.dim, 32), pad_to(m.v_dim, 16)
    gate = torch.cat([_pad_heads(a2.float(), m.heads, m.dim, dp).T, _pad_heads(a2_bias.float(), m.heads, m.dim, dp)[None]])
    return [(W_GATE_MAP, gate.contiguous()), (W_DELTA_NORM, _pad(norm.float(), vp)), (W_DELTA_OUT, _out_columns(o, d, m.heads, m.v_dim, vp))]


def glu_rows(gate, up, d, ff):
    """Gate and up rows in turn."""
    import torch
    fp, wp = pad_to(ff, 64), pad_to(d, 64)
    return torch.stack([_pad(gate, fp, wp), _pad(up, fp, wp)], 1).reshape(2 * fp, wp)


def pack_experts(f, d, router, experts, shared=None, correction=None):
    """[(kind, tensor)] of a GluFf of experts; experts: an iterable of (gate, up, down), shared: one of them or None."""
    import torch
    wp, fp = pad_to(d, 64), pad_to(f.ff, 64)
    ups, downs = torch.empty(f.experts, 2 * fp, wp, dtype=router.dtype, device=router.device), torch.empty(f.experts, wp, fp, dtype=router.dtype, device=router.device)
    for i, (gate, up, down) in enumerate(experts):
        ups[i], downs[i] = glu_rows(gate, up, d, f.ff), _pad(down, wp, fp)
    n = pad_to(f.experts + f.identity, 8)
    out = [(W_ROUTER, _pad(router, n, wp)), (W_UP, ups), (W_FF_DOWN, downs)]
    if f.softmax:
        out.append((W_CORRECTION, _pad(correction.float(), n)))
    if f.shared:
        out += [(W_SHARED_UP, glu_rows(*shared[:2], d, f.shared)), (W_SHARED_DOWN, _pad(shared[2], wp, pad_to(f.shared, 64)))]
    return out


def pack_glu(f, d, gate, up, down):
    """[(kind, tensor)] of a GluFf without experts."""
    return [(W_UP, glu_rows(gate, up, d, f.ff)), (W_FF_DOWN, _pad(down, pad_to(d, 64), pad_to(f.ff, 64)))]


def pack_poly(f, d, up, up_bias, down, down_bias, act):
    """[(kind, tensor)] of a PolyNormFf."""
    fp, wp = pad_to(f.ff, 64), pad_to(d, 64)
    return [(W_UP, _pad(up, fp, wp)), (W_FF_DOWN, _pad(down, wp, fp)), (W_UP_BIAS, _pad(up_bias.float(), fp)), (W_DOWN_BIAS, _pad(down_bias.float(), wp)),
            (W_ACT, act.float().contiguous())]


def pack_norms(d, norm1, post1=None, norm2=None, post2=None):
    """[(kind, tensor)] of the gains (f32) of a layer with norms ahead of its sublayers and on their outputs."""
    return [(k, _pad(g.float(), pad_to(d, 64))) for k, g in ((W_NORM1, norm1), (W_POST1, post1), (W_NORM2, norm2), (W_POST2, post2)) if g is not None]


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

    def shapes(self):
        return {k: tuple(v.shape) for k, v in self.items()}

    def take(self, name, *shape):
        if name not in self:
            raise ValueError(f"tensor {name} is missing")
        t = self[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, the configuration says {shape}")
        import torch
        return t if t.dtype == torch.bfloat16 else t.to(torch.bfloat16)


def architectures():
    """config.json's "architecture" -> module with read_config(dict, shapes) and pack(cfg, Tensors); shapes: {name: shape} of the
    model file, for sizes that the configuration does not name."""
    from . import galarax, gunulorn, mupuvik, zefedra
    return {"Galarax": galarax, "Gunulorn": gunulorn, "Mupuvik": mupuvik, "Zefedra": zefedra}


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
    tensors = Tensors(read_safetensors(os.path.join(path, "model.safetensors")))
    cfg = replace(known[arch].read_config(raw, tensors.shapes()), act_dtype=act_dtype)
    if nctx:
        cfg = replace(cfg, nctx=nctx)
    weights = known[arch].pack(cfg, tensors)
    tokens = kv_tokens or cfg.nctx
    pt = page_tokens or 64
    ctx = load_model(cfg, weights, device=device, kv_bytes=(tokens + pt - 1) // pt * pt * cfg.kv_bytes_per_token(), page_tokens=page_tokens,
                     max_tokens=max_tokens, max_seqs=max_seqs)
    return cfg, ctx
