"""Plain restatement of the Galarax design on the CPU, one function per mechanism (test infrastructure only).

Whole sequences, no cache, no batching; the delta rule runs token by token.  It shares no code with the library; `dtype` is the
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


# ---- rotation

def yarn_frequencies(rot):
    """([dims / 2] frequencies, factor on cos and sin): frequencies of few turns inside the original context are divided by the
    factor, those of many are left, a linear ramp over the dimension index lies between."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    freq = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return freq, 1.0

    def index_of(turns):
        return n * math.log(sc["original"] / (turns * 2 * math.pi)) / (2 * math.log(base))
    lo, hi = max(math.floor(index_of(sc["fast"])), 0), min(math.ceil(index_of(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(freq):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(x, rot):
    """x [tokens, heads, dim]: halves of the first rot.dims dimensions are the two coordinates."""
    n = rot["dims"]
    freq, gain = yarn_frequencies(rot)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * torch.tensor(freq, dtype=torch.float64)[None]
    c, s = (torch.cos(a) * gain).to(x.dtype)[:, None], (torch.sin(a) * gain).to(x.dtype)[:, None]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], -1)


# ---- softmax attention

def attention_inputs(h, w, pre, m, eps):
    n = h.shape[0]
    q, k, v = (linear(h, w[pre + t]) + w[pre + t + ".b"] for t in "qkv")
    q, k, v = q.view(n, m["heads"], m["dim"]), k.view(n, m["kv_heads"], m["dim"]), v.view(n, m["kv_heads"], m["vdim"])
    return rms(rotate(q, m["rot"]), eps), rms(rotate(k, m["rot"]), eps), v


def causal_attention(q, k, v, scale):
    """[tokens, heads, vdim]; query head h reads key head h // (heads / kv_heads)."""
    n, reps = q.shape[0], q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(reps, 1), v.repeat_interleave(reps, 1)
    s = torch.einsum("qhd,khd->hqk", rounded(q), rounded(k)) * scale
    s = s.masked_fill(~torch.ones(n, n, dtype=torch.bool).tril(), -math.inf)
    return torch.einsum("hqk,khd->qhd", rounded(torch.softmax(s, -1)), rounded(v))


def left(h, w, pre, m, eps):
    q, k, v = attention_inputs(h, w, pre, m, eps)
    return linear(causal_attention(q, k, v, m["scale"]).reshape(h.shape[0], -1), w[pre + "o"])


# ---- gated delta rule

def causal_conv(x, w):
    """x [tokens, channels], w [channels, taps]; the last tap meets the current token, zeros stand before the first."""
    taps = w.shape[1]
    x = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x])
    return sum(x[j:x.shape[0] - (taps - 1 - j)] * w[:, j] for j in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_inputs(h, w, pre, m):
    """q, k [tokens, heads, dim] (repeated for the heads that share them), v [tokens, heads, vdim], decay and step size
    [tokens, heads]."""
    n, reps = h.shape[0], m["heads"] // m["kv_heads"]
    q, k, v = (silu(causal_conv(linear(h, w[pre + t]), w[pre + t + ".conv"])) for t in "qkv")
    q = unit(q.view(n, m["kv_heads"], m["dim"])) * m["dim"] ** -0.5
    k = unit(k.view(n, m["kv_heads"], m["dim"]))
    decay = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(linear(h, w[pre + "a"]) + w[pre + "dt_bias"]))
    beta = torch.sigmoid(linear(h, w[pre + "b"]))
    return q.repeat_interleave(reps, 1), k.repeat_interleave(reps, 1), v.view(n, m["heads"], m["vdim"]), decay, beta


def delta_rule(q, k, v, decay, beta):
    """Per head: the state decays, is corrected towards v along k, then read along q."""
    s = q.new_zeros(q.shape[1], q.shape[2], v.shape[2])
    out = []
    for t in range(q.shape[0]):
        s = s * decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None]
        out.append(torch.einsum("hkv,hk->hv", s, q[t]))
    return torch.stack(out)


def right(h, w, pre, m, eps):
    o = delta_rule(*delta_inputs(h, w, pre, m))
    o = rms(o, eps) * w[pre + "norm"] * silu(linear(h, w[pre + "g"])).view(o.shape)
    return linear(o.reshape(h.shape[0], -1), w[pre + "o"])


def parallel(h, w, pre, m, eps):
    return (rms(left(h, w, pre + "left.", m["left"], eps), eps) * w[pre + "left.out"]
            + rms(right(h, w, pre + "right.", m["right"], eps), eps) * w[pre + "right.out"]) / 2


# ---- model

def feed_forward(h, w, pre):
    return linear(torch.relu(linear(h, w[pre + "up"])).square(), w[pre + "down"])


def layer(x, raw, w, i):
    e, eps, p = raw["layers"][i], raw["norm"]["eps"], f"l{i}."
    x = x + parallel(centred_norm(x, w[p + "norm1"], eps), w, p + "mix.", e["mixer"], eps)
    if e["mlp"]:
        x = x + feed_forward(centred_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
    return x


def schedule(raw):
    """[(layer, pass that starts with it or None)]"""
    n, loop = len(raw["layers"]), raw.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def forward(raw, weights, tokens, dtype=torch.float64, keep_layers=False, operand=None):
    """Logits [tokens, vocab]; with keep_layers also the residual stream after every layer run.  operand: the dtype that inputs of
    matrix products are rounded to -- what rounding alone changes, to set a tolerance by."""
    global _operand
    _operand = operand
    try:
        return _forward(raw, weights, tokens, dtype, keep_layers)
    finally:
        _operand = None


def _forward(raw, weights, tokens, dtype, keep_layers):
    w = {k: v.to(dtype) for k, v in weights.items()}
    first = x = w["embed"][torch.tensor(list(tokens))]
    kept = []
    for i, t in schedule(raw):
        if t is not None:
            x = x + first if t else x
            x = x + w["loop.step"][t]
        x = layer(x, raw, w, i)
        kept.append(x)
    logits = linear(centred_norm(x, w["final.norm"], raw["norm"]["eps"]), w["head"])
    return (logits, torch.stack(kept)) if keep_layers else logits
