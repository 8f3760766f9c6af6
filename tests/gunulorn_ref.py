"""Plain restatement of the Gunulorn design on the CPU, one function per mechanism (test infrastructure only).

Whole sequences, no cache, no batching.  It shares no code with the library; `dtype` is the precision of every operation (f64 for a
tight oracle).
"""
import math

import torch


_operand = None  # dtype that inputs of matrix products are rounded to (`forward` sets it); None: not at all


def rounded(x):
    return x if _operand is None else x.to(_operand).to(x.dtype)


def linear(x, w):
    return rounded(x) @ w.T


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(x):
    return x * torch.sigmoid(x)


def heads_of(x, heads):
    return x.reshape(x.shape[0], heads, -1)


# ---- pieces of attention

def causal_conv(x, w):
    """x [tokens, channels], w [channels, taps]; the last tap meets the current token, zeros stand before the first."""
    taps = w.shape[1]
    x = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(x[j:x.shape[0] - (taps - 1 - j)] * w[:, j] for j in range(taps))


def turn(x, dims, base, sign=1):
    """Neighbouring pairs among the first `dims` dimensions, pair i of token p by sign * p * base^(-2i / dims); x [tokens, heads, dim]."""
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = sign * torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f
    c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2), x[..., dims:]], -1)


def visible(n, window=0, keep=0):
    """[query, key]; window 0: no lower limit; the first `keep` tokens stay visible behind it."""
    i = torch.arange(n)
    d = i[:, None] - i[None]
    return (d >= 0) & ((d < window) | (i[None] < keep)) if window else d >= 0


def softmax_attention(q, k, v, scale, sink, window=0, keep=0):
    """[tokens, heads, vdim]; query head h reads key head h // (heads / kv_heads); scale [heads]; the denominator of head h also counts
    exp(sink[h])."""
    n, reps = q.shape[0], q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(reps, 1), v.repeat_interleave(reps, 1)
    s = torch.einsum("qhd,khd->hqk", rounded(q), rounded(k)) * scale[:, None, None]
    s = s.masked_fill(~visible(n, window, keep), -math.inf)
    s = torch.cat([s, sink[:, None, None].expand(-1, n, 1)], -1)
    return torch.einsum("hqk,khd->qhd", rounded(torch.softmax(s, -1)[..., :n]), rounded(v))


# ---- mixers

def conv_projection(h, w, name):
    return causal_conv(linear(h, w[name]), w[name + ".conv"])


def conv_keys(h, w, pre, m):
    """Keys and values of a layer, behind their convolutions."""
    return tuple(heads_of(conv_projection(h, w, pre + t), m["kv_heads"]) for t in "kv")


def conv_attention(h, w, pre, m, keys):
    """Without positions; keys: (k, v) of this layer, or of the layer it borrows them from."""
    q = heads_of(conv_projection(h, w, pre + "q"), m["heads"])
    o = softmax_attention(q, *keys, m["scale"] * w[pre + "temp"], w[pre + "sink"])
    return linear(o.reshape(h.shape[0], -1), w[pre + "o"])


def window_attention(h, w, pre, m):
    """Keys and queries with positions, values turned by their own positions and each output back by its token's."""
    q, k, v = (heads_of(linear(h, w[pre + t]), m[n]) for t, n in (("q", "heads"), ("k", "kv_heads"), ("v", "kv_heads")))
    d, base, vd = m["rot"]["dims"], m["rot"]["base"], m["vdim"]
    one = h.new_ones(m["heads"])
    o = softmax_attention(turn(q, d, base), turn(k, d, base), turn(v, vd, base), m["scale"] * one, 0 * one, m["mask"]["size"], m["mask"]["keep_first"])
    return linear(turn(o, vd, base, -1).reshape(h.shape[0], -1), w[pre + "o"])


# ---- feed-forwards

def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense(h, w, pre, eps):
    return linear(poly_norm(linear(h, w[pre + "up"]) + w[pre + "up.b"], w[pre + "act"], eps), w[pre + "down"]) + w[pre + "down.b"]


def expert(x, w, pre):
    return linear(silu(linear(x, w[pre + "gate"])) * linear(x, w[pre + "up"]), w[pre + "down"])


def route(h, w, pre, top):
    """(experts, their weights) of every token, [tokens, top]."""
    s = torch.softmax(linear(h, w[pre + "router"]), -1)
    e = torch.topk(s + w[pre + "correction"], top, -1).indices
    s = s.gather(-1, e)
    return e, s / (s.sum(-1, keepdim=True) + 1e-20)


def experts(h, w, pre, m):
    r = m["router"]
    chosen, weights = route(h, w, pre, r["top"])
    y = torch.zeros_like(h)
    for i in range(r["experts"] + r["identity"]):
        t, k = torch.nonzero(chosen == i, as_tuple=True)
        if len(t):
            y[t] += weights[t, k][:, None] * (expert(h[t], w, f"{pre}e{i}.") if i < r["experts"] else h[t])
    return y


# ---- model

def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def forward(raw, weights, tokens, dtype=torch.float64, keep_layers=False, operand=None):
    """Logits [tokens, vocab]; with keep_layers also the residual stream after every layer.  operand: the dtype that inputs of
    matrix products are rounded to -- what rounding alone changes, to set a tolerance by."""
    global _operand
    _operand = operand
    try:
        return _forward(raw, weights, list(tokens), dtype, keep_layers)
    finally:
        _operand = None


def _forward(raw, weights, tokens, dtype, keep_layers):
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps, x, kept, cache = raw["norm"]["eps"], w["embed"][tokens], [], {}
    for i, e in enumerate(raw["layers"]):
        p, m = f"l{i}.", e["mixer"]
        h = norm(x, w[p + "norm1"], eps)
        if e["type"] == "attention":
            cache[i] = cache[m["kv_from"]] if m.get("kv_from") is not None else conv_keys(h, w, p + "mix.", m)
            y = conv_attention(h, w, p + "mix.", m, cache[i])
        else:
            y = window_attention(h, w, p + "mix.", m)
        if e.get("mlp"):
            h = norm(x, w[p + "norm2"], eps)
            y = y + (experts(h, w, p + "mlp.", e["mlp"]) if e["mlp"]["kind"] == "moe" else dense(h, w, p + "mlp.", eps))
        x = x + y
        kept.append(x)
    logits = soft_cap(linear(norm(x, w["final.norm"], eps), w["head"]) * raw["logit_scale"], raw["logit_softcap"])
    return (logits, torch.stack(kept)) if keep_layers else logits
