"""Plain implementation of the Fezopel design on the CPU, for tests only.

One function per mechanism, each a direct restatement of its equation in the tensors' own
floating-point type (the tests use float64), one token after the other where the mechanism is a
recurrence.  Nothing here is shared with the product: the configuration is the parsed
``config.json`` as a dictionary, the weights a dictionary name -> tensor.
"""

from __future__ import annotations

import math

import torch

UNIT_EPS = 1e-6


# --------------------------------------------------------------------------- elementwise
def layer_norm(x, weight, bias, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight + bias


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + UNIT_EPS)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_erf(x):
    return 0.5 * x * (1 + torch.erf(x / math.sqrt(2.0)))


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def depth_average(outputs, coefficients):
    total = torch.zeros_like(outputs[0])
    for x, c in zip(outputs, coefficients):
        total = total + c * x
    return total


# ----------------------------------------------------------------------------- rotation
def rotate_interleaved(x, positions, base, dims):
    """x [tokens, heads, dim]; dimensions 2i and 2i + 1 of the first ``dims`` form a pair."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(angle)[:, None], torch.sin(angle)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


# ---------------------------------------------------------------------------- attention
def window_sink_attention(q, k, v, sinks, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] of one sequence from position 0; query i sees keys
    i - window + 1 .. i; exp(sink) joins the softmax's denominator."""
    tokens, heads, _ = q.shape
    share = heads // k.shape[1]
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for h in range(heads):
        keys, values = k[:, h // share], v[:, h // share]
        for i in range(tokens):
            lo = max(0, i - window + 1)
            scores = keys[lo:i + 1] @ q[i, h] * scale
            top = torch.maximum(scores.max(), sinks[h])
            weights = torch.exp(scores - top)
            out[i, h] = weights @ values[lo:i + 1] / (weights.sum() + torch.exp(sinks[h] - top))
    return out


def attention_mixer(h, w, prefix, m, eps):
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    tokens = h.shape[0]
    q = rms_norm(h @ w[prefix + "q"].T, w[prefix + "q.norm"], eps).view(tokens, heads, dim)
    k = rms_norm(h @ w[prefix + "k"].T, w[prefix + "k.norm"], eps).view(tokens, kv, dim)
    v = (h @ w[prefix + "v"].T).view(tokens, kv, vdim)
    positions = torch.arange(tokens)
    q = rotate_interleaved(q, positions, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_interleaved(k, positions, m["rot"]["base"], m["rot"]["dims"])
    out = window_sink_attention(q, k, v, w[prefix + "sink"], m["scale"], m["mask"]["size"])
    out = out * torch.sigmoid(h @ w[prefix + "g"].T)[:, :, None]
    return out.reshape(tokens, heads * vdim) @ w[prefix + "o"].T


# -------------------------------------------------------------------- linear recurrences
def gla_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, d], v [T, H, dv]: S <- diag(alpha) S + k v^T, o = S^T q.  Returns (o, S)."""
    tokens, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for t in range(tokens):
        s = alpha[t][:, :, None] * s + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", s, q[t])
    return out, s


def channel_delta_recurrence(q, k, v, g, beta, state=None):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H].  S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    tokens, heads, dim = q.shape
    s = torch.zeros(heads, dim, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for t in range(tokens):
        s = g[t][:, :, None] * s
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", s, k[t]))
        s = s + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", s, q[t])
    return out, s


def causal_conv(x, taps):
    """x [T, channels], taps [channels, n], the last column belongs to the current token."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    out = torch.zeros_like(x)
    for j in range(n):
        out = out + padded[j:j + x.shape[0]] * taps[:, j]
    return out


def gla_decay(z, tau):
    return torch.sigmoid(z) ** (1.0 / tau)


def channel_delta_decay(z, a_log):
    """z [T, H, d] (bias added), a_log [H]."""
    return torch.exp(-torch.exp(a_log)[None, :, None] * softplus(z))


def gla_mixer(h, w, prefix, m, eps):
    heads, dim, vdim = m["heads"], m["dim"], m["vdim"]
    tokens = h.shape[0]
    q = (h @ w[prefix + "q"].T * dim ** -0.5).view(tokens, heads, dim)
    k = (h @ w[prefix + "k"].T).view(tokens, heads, dim)
    v = (h @ w[prefix + "v"].T).view(tokens, heads, vdim)
    z = h @ w[prefix + "a1"].T @ w[prefix + "a2"].T + w[prefix + "a2.b"]
    out, _ = gla_recurrence(q, k, v, gla_decay(z, m["tau"]).view(tokens, heads, dim))
    out = rms_norm(out, w[prefix + "norm"], eps).reshape(tokens, heads * vdim)
    return (out * silu(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def channel_delta_mixer(h, w, prefix, m, eps):
    heads, kv, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    tokens = h.shape[0]
    q, k, v = (silu(causal_conv(h @ w[prefix + n].T, w[prefix + n + ".conv"])) for n in "qkv")
    q = unit(q.view(tokens, kv, dim)) * dim ** -0.5
    k = unit(k.view(tokens, kv, dim))
    q, k = (x.repeat_interleave(heads // kv, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ w[prefix + "b"].T)
    z = (h @ w[prefix + "a1"].T @ w[prefix + "a2"].T + w[prefix + "dt_bias"]).view(tokens, heads, dim)
    out, _ = channel_delta_recurrence(q, k, v.view(tokens, heads, vdim), channel_delta_decay(z, w[prefix + "A_log"]), beta)
    out = rms_norm(out, w[prefix + "norm"], eps).reshape(tokens, heads * vdim)
    return (out * torch.sigmoid(h @ w[prefix + "g1"].T @ w[prefix + "g2"].T)) @ w[prefix + "o"].T


MIXERS = {"attention": attention_mixer, "gla": gla_mixer, "channel_delta": channel_delta_mixer}


# ---------------------------------------------------------------------------- the model
def sublayer(x, run, w, at, which, eps):
    """x + norm_b(run(norm(x)) * sigmoid(W norm(x) + b))."""
    h = layer_norm(x, w[f"{at}norm{which}"], w[f"{at}norm{which}.b"], eps)
    y = run(h) * torch.sigmoid(h @ w[f"{at}rg{which}"].T + w[f"{at}rg{which}.b"])
    return x + layer_norm(y, w[f"{at}norm{which}b"], w[f"{at}norm{which}b.b"], eps)


def forward(config, weights, tokens, dtype=torch.float64):
    """Logits [T, vocab] of one sequence and the stream after every layer (depth average included) [L, T, width]."""
    w = {name: t.to(dtype) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    outputs, stream = [x], []
    for i, layer in enumerate(config["layers"]):
        at = f"l{i}."
        x = sublayer(x, lambda h: MIXERS[layer["type"]](h, w, at + "mix.", layer["mixer"], eps), w, at, 1, eps)
        if layer["mlp"] is not None:
            x = sublayer(x, lambda h: gelu_erf(h @ w[at + "mlp.up"].T) @ w[at + "mlp.down"].T, w, at, 2, eps)
        outputs.append(x)
        x = depth_average(outputs, w[at + "dwa"])
        stream.append(x)
    final = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    return final @ w["head"].T, torch.stack(stream)


def greedy(config, weights, prompt, count, dtype=torch.float64):
    """``count`` greedy tokens after ``prompt`` (the whole sequence again for every token) and the smallest
    gap between the two best logits met on the way."""
    tokens, gap = list(prompt), math.inf
    for _ in range(count):
        best = forward(config, weights, tokens, dtype)[0][-1].topk(2).values
        gap = min(gap, float(best[0] - best[1]))
        tokens.append(int(forward(config, weights, tokens, dtype)[0][-1].argmax()))
    return tokens[len(prompt):], gap
