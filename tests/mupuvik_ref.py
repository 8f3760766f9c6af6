"""Plain restatement of the Mupuvik design on the CPU, one function per mechanism (test infrastructure only).

Whole sequences, no cache, no batching; recurrences run token by token.  It shares no code with the library; `dtype` is the
precision of every operation (f64 for a tight oracle).
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


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


# ---- embedding

def bigram_rows(tokens, b):
    """Row of the pair table for every token; the first token of a sequence takes the last row."""
    return [b["buckets"]] + [(p * b["mul_prev"] + c * b["mul_cur"]) % b["buckets"] for p, c in zip(tokens, tokens[1:])]


def embedding(tokens, raw, w):
    e = raw["embedding"]
    return w["embed"][list(tokens)] * e["scale"] + w["bigram"][bigram_rows(tokens, e["bigram"])]


# ---- state space duality

def causal_conv(x, w, b):
    """x [tokens, channels], w [channels, taps]; the last tap meets the current token, zeros stand before the first."""
    taps = w.shape[1]
    x = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(x[j:x.shape[0] - (taps - 1 - j)] * w[:, j] for j in range(taps)) + b


def ssd_inputs(h, w, pre, m):
    """z [tokens, inner], x [tokens, heads, vdim], B and C [tokens, heads, state] (repeated for the heads of a group), step size
    [tokens, heads]."""
    n, inner, gn = h.shape[0], m["heads"] * m["vdim"], m["groups"] * m["state"]
    z, xbc, dt = torch.split(linear(h, w[pre + "in"]), [inner, inner + 2 * gn, m["heads"]], -1)
    x, b, c = torch.split(silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"])), [inner, gn, gn], -1)
    reps = m["heads"] // m["groups"]
    b, c = (t.reshape(n, m["groups"], m["state"]).repeat_interleave(reps, 1) for t in (b, c))
    return z, x.reshape(n, m["heads"], m["vdim"]), b, c, softplus(dt + w[pre + "dt_bias"])


def ssd(x, b, c, dt, rate):
    """Per head: the state decays by exp(-rate dt), takes dt b x^T up, and is read along c."""
    s = x.new_zeros(x.shape[1], b.shape[2], x.shape[2])
    out = []
    for t in range(x.shape[0]):
        s = s * torch.exp(-rate * dt[t])[:, None, None] + (dt[t][:, None] * b[t])[:, :, None] * x[t][:, None]
        out.append(torch.einsum("hnv,hn->hv", s, c[t]))
    return torch.stack(out)


def gated_norm(y, z, w, parts, eps):
    """The gate, then a norm in equal parts."""
    y = y * silu(z)
    return rms(y.reshape(y.shape[0], parts, -1), eps).reshape(y.shape) * w


def mamba2(h, w, pre, m, eps):
    z, x, b, c, dt = ssd_inputs(h, w, pre, m)
    y = ssd(x, b, c, dt, torch.exp(w[pre + "A_log"])) + w[pre + "D"][:, None] * x
    return linear(gated_norm(y.reshape(h.shape[0], -1), z, w[pre + "norm"], m["norm_groups"], eps), w[pre + "o"])


# ---- softmax attention

def rotate(x, rot):
    """Pairs of neighbouring dimensions; x [tokens, heads, dim]."""
    n = rot["dims"]
    f = torch.tensor([rot["base"] ** (-2.0 * i / n) for i in range(n // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * f
    c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    r = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
    return torch.cat([r, x[..., n:]], -1)


def visible(n, window):
    """[query, key]; window 0: no lower limit."""
    i = torch.arange(n)
    d = i[:, None] - i[None]
    return (d >= 0) & (d < window) if window else d >= 0


def softmax_attention(q, k, v, scale, window=0, sink=False):
    """[tokens, heads, vdim]; query head h reads key head h // (heads / kv_heads).  sink: the denominator counts one more key of
    score 0 and no value."""
    n, reps = q.shape[0], q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(reps, 1), v.repeat_interleave(reps, 1)
    s = torch.einsum("qhd,khd->hqk", rounded(q), rounded(k)) * scale
    s = s.masked_fill(~visible(n, window), -math.inf)
    if sink:
        s = torch.cat([s, s.new_zeros(s.shape[0], n, 1)], -1)
    return torch.einsum("hqk,khd->qhd", rounded(torch.softmax(s, -1)[..., :n]), rounded(v))


def heads_of(x, heads):
    return x.reshape(x.shape[0], heads, -1)


def gated_heads(o, h, w, pre):
    """One sigmoid gate per head, then the output projection."""
    o = o * torch.sigmoid(linear(h, w[pre + "g"]))[..., None]
    return linear(o.reshape(h.shape[0], -1), w[pre + "o"])


def window_keys(h, w, pre, m, eps):
    k, v = (linear(h, w[pre + t]) + w[pre + t + ".b"] for t in "kv")
    return heads_of(rms(k, eps) * w[pre + "k.norm"], m["kv_heads"]), heads_of(v, m["kv_heads"])


def window_attention(h, w, pre, m, eps, keys):
    """keys: (k, v) of this layer, or of the layer it borrows them from."""
    q = rms(linear(h, w[pre + "q"]) + w[pre + "q.b"], eps) * w[pre + "q.norm"]
    return gated_heads(softmax_attention(heads_of(q, m["heads"]), *keys, m["scale"], m["mask"]["size"]), h, w, pre)


def left(h, w, pre, m, eps):
    q, k = (rms(heads_of(linear(h, w[pre + t]), m[n]), eps) * w[pre + t + ".norm"] for t, n in (("q", "heads"), ("k", "kv_heads")))
    v = heads_of(linear(h, w[pre + "v"]), m["kv_heads"])
    return gated_heads(softmax_attention(rotate(q, m["rot"]), rotate(k, m["rot"]), v, m["scale"], sink=True), h, w, pre)


# ---- gated linear attention

def gla_inputs(h, w, pre, m):
    """q (scaled), k and decay [tokens, heads, dim], v [tokens, heads, vdim]."""
    q, k, v = (heads_of(linear(h, w[pre + t]), m["heads"]) for t in "qkv")
    z = linear(linear(h, w[pre + "a1"]), w[pre + "a2"]) + w[pre + "a2.b"]
    decay = torch.exp(-softplus(-z) / m["tau"])  # sigmoid(z)^(1 / tau)
    return q * m["dim"] ** -0.5, k, v, heads_of(decay, m["heads"])


def gla(q, k, v, decay):
    """Per head: every key channel of the state decays by its own factor, k v^T is added, then it is read along q."""
    s = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        s = s * decay[t][:, :, None] + k[t][:, :, None] * v[t][:, None]
        out.append(torch.einsum("hkv,hk->hv", s, q[t]))
    return torch.stack(out)


def right(h, w, pre, m, eps):
    o = (rms(gla(*gla_inputs(h, w, pre, m)), eps) * w[pre + "norm"]).reshape(h.shape[0], -1)
    return linear(o * silu(linear(h, w[pre + "g"])), w[pre + "o"])


def parallel(h, w, pre, m, eps):
    return m["left_scale"] * left(h, w, pre + "left.", m["left"], eps) + m["right_scale"] * right(h, w, pre + "right.", m["right"], eps)


# ---- feed-forward

def expert(x, w, pre, limit):
    g = torch.clamp(linear(x, w[pre + "gate"]), max=limit)
    u = torch.clamp(linear(x, w[pre + "up"]), -limit, limit)
    return linear(g * torch.sigmoid(1.702 * g) * (u + 1), w[pre + "down"])


def route(h, w, pre, top):
    """(experts, their weights) of every token, [tokens, top]."""
    s, e = torch.topk(torch.sigmoid(linear(h, w[pre + "router"])), top, -1)
    return e, s


def feed_forward(h, w, pre, m):
    """The weight of an expert scales its input."""
    experts, weights = route(h, w, pre, m["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(experts[t].tolist(), weights[t]):
            y[t] += expert(s * h[t], w, f"{pre}e{e}.", m["expert"]["limit"])
    if m.get("shared"):
        y = y + expert(h, w, pre + "shared.", m["shared"]["limit"])
    return y


# ---- model

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
    eps, x, kept, cache = raw["norm"]["eps"], embedding(tokens, raw, w), [], {}
    for i, e in enumerate(raw["layers"]):
        p, m = f"l{i}.", e["mixer"]
        h = centred_norm(x, w[p + "norm1"], eps)
        if e["type"] == "mamba2":
            y = mamba2(h, w, p + "mix.", m, eps)
        elif e["type"] == "parallel":
            y = parallel(h, w, p + "mix.", m, eps)
        else:
            cache[i] = cache[m["kv_from"]] if m.get("kv_from") is not None else window_keys(h, w, p + "mix.", m, eps)
            y = window_attention(h, w, p + "mix.", m, eps, cache[i])
        x = x + centred_norm(y, w[p + "norm1b"], eps)
        if e.get("mlp"):
            y = feed_forward(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.", e["mlp"])
            x = x + centred_norm(y, w[p + "norm2b"], eps)
        kept.append(x)
    logits = linear(centred_norm(x, w["final.norm"], eps), w["embed"])
    return (logits, torch.stack(kept)) if keep_layers else logits
