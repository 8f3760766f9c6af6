"""Plain restatement of the Zefedra design on the CPU, one function per mechanism (test infrastructure only).

Whole sequences, no cache, no batching: every function takes the full sequence and follows the equations term by term.
It shares no code with the library; `dtype` is the precision of every operation (f64 for a tight oracle).
"""
import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    return rms(x, eps) * gain


def token_shift(h, mu):
    """Row t becomes h[t] + (h[t-1] - h[t]) * mu; the row before the first is zero."""
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def latents(h, w_dq, g_q, w_dkv, g_kv, eps):
    """(query latent, cached latent), both RMS-normalised with a plain weight."""
    return rms(h @ w_dq.T, eps) * g_q, rms(h @ w_dkv.T, eps) * g_kv


def latent_scores(c_q, c, w_uq, w_uk, heads, scale):
    """Scores [heads, query, key] of explicit per-head queries and keys."""
    n = c.shape[0]
    q = (c_q @ w_uq.T).view(n, heads, -1)
    k = (c @ w_uk.T).view(n, heads, -1)
    return torch.einsum("qhd,khd->hqk", q, k) * scale


def causal_softmax(s):
    n = s.shape[-1]
    mask = torch.ones(n, n, dtype=torch.bool).tril()
    return torch.softmax(s.masked_fill(~mask, -math.inf), -1)


def latent_values(p, c, w_uv, heads):
    """[token, heads, v_dim]"""
    v = (c @ w_uv.T).view(c.shape[0], heads, -1)
    return torch.einsum("hqk,khd->qhd", p, v)


def head_gate(o, h, w_g):
    """One sigmoid per head from the mixer's input, over the head's whole output."""
    return o * torch.sigmoid(h @ w_g.T)[:, :, None]


def latent_attention(h, w, pre, m, eps, gated):
    c_q, c = latents(h, w[pre + "dq"], w[pre + "dq.norm"], w[pre + "dkv"], w[pre + "dkv.norm"], eps)
    p = causal_softmax(latent_scores(c_q, c, w[pre + "uq"], w[pre + "uk"], m["heads"], m["scale"]))
    o = latent_values(p, c, w[pre + "uv"], m["heads"])
    if gated:
        o = head_gate(o, h, w[pre + "g"])
    return o.reshape(o.shape[0], -1) @ w[pre + "o"].T


def xielu(z, p, q):
    sp, sq = torch.nn.functional.softplus(p), torch.nn.functional.softplus(q)
    return torch.where(z > 0, sp * z * z + z / 2, (0.5 + sq) * (torch.expm1(z.clamp(max=0)) - z.clamp(max=0)) + z / 2)


def feed_forward(x, w, pre):
    return xielu(x @ w[pre + "up"].T, w[pre + "act"][0], w[pre + "act"][1]) @ w[pre + "down"].T


def forward(config, weights, tokens, dtype=torch.float64, keep_layers=False):
    """Logits [n, vocab] of a whole sequence (and the residual stream after every layer)."""
    w = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    stream = []
    for i, layer in enumerate(config["layers"]):
        src = i
        while config["layers"][src].get("weights_of") is not None:
            src = config["layers"][src]["weights_of"]
        pre = f"l{src}."
        h = token_shift(x, w[pre + "shift"])
        y = latent_attention(h, w, pre + "mix.", layer["mixer"], eps, layer["type"] == "latent_attention_2")
        x = x + scalar_norm(y, w[pre + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + scalar_norm(feed_forward(x, w, pre + "mlp."), w[pre + "norm2"], eps)
        stream.append(x)
    logits = scalar_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, torch.stack(stream)) if keep_layers else logits
