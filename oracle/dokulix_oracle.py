"""Plain implementation of the Dokulix design on the CPU, for tests only.

One function per mechanism, each a direct restatement of its equation in the tensors' own
floating-point type (the tests use float64).  Nothing here is shared with the product: the
configuration is the parsed ``config.json`` as a dictionary, the weights a dictionary name -> tensor.
"""

from __future__ import annotations

import math

import torch


# --------------------------------------------------------------------------- elementwise
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def rms_norm_around_one(x, weight, eps):
    """The weight is stored as its distance from one."""
    return rms(x, eps) * (1 + weight)


def relu_glu(h, gate, up, down):
    return (torch.clamp(h @ gate.T, min=0) * (h @ up.T)) @ down.T


# ----------------------------------------------------------------------------- rotation
def rotate_half(x, positions, base, dims):
    """x [tokens, ..., dim]; dimensions i and i + dims / 2 of the first ``dims`` form a pair."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        angle = positions.to(x.dtype) * base ** (-2.0 * i / dims)
        shape = (-1,) + (1,) * (x.dim() - 2)
        c, s = torch.cos(angle).view(shape), torch.sin(angle).view(shape)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ---------------------------------------------------------------------------- attention
def sees_window(i, j, size):
    return 0 <= i - j < size


def sees_chunk(i, j, size):
    return j <= i and i // size == j // size


def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def masked_attention(q, k, v, scale, sees, slopes=None, extra_one=False):
    """q [T, H, d], k [T, G, d], v [T, G, dv] of one sequence from position 0.  ``sees(i, j)`` says which keys a
    query sees; ``slopes`` [H] times the distance is taken off the scores; ``extra_one`` adds one to the sum of
    the exponentials."""
    tokens, heads, _ = q.shape
    share = heads // k.shape[1]
    out = torch.zeros(tokens, heads, v.shape[2], dtype=q.dtype)
    for i in range(tokens):
        seen = [j for j in range(i + 1) if sees(i, j)]
        lo = seen[0]
        assert seen == list(range(lo, i + 1))
        distance = (i - torch.arange(lo, i + 1)).to(q.dtype)
        for h in range(heads):
            scores = k[lo:i + 1, h // share] @ q[i, h] * scale
            if slopes is not None:
                scores = scores - slopes[h] * distance
            top = scores.max().clamp(min=0) if extra_one else scores.max()
            weights = torch.exp(scores - top)
            total = weights.sum() + (torch.exp(-top) if extra_one else 0)
            out[i, h] = weights @ v[lo:i + 1, h // share] / total
    return out


def latent_heads(dq, dkv, w, prefix, m, eps):
    """Heads [T, H, vdim] from the rows of the two down projections."""
    heads, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    tokens, positions = dq.shape[0], torch.arange(dq.shape[0])
    q = (rms_norm(dq, w[prefix + "dq.norm"], eps) @ w[prefix + "uq"].T).view(tokens, heads, dim + rot_dim)
    q = torch.cat([q[..., :dim], rotate_half(q[..., dim:], positions, m["rot"]["base"], m["rot"]["dims"])], -1)
    latent = rms_norm(dkv[:, :rank], w[prefix + "dkv.norm"], eps)
    shared = rotate_half(dkv[:, rank:], positions, m["rot"]["base"], m["rot"]["dims"])
    keys = (latent @ w[prefix + "uk"].T).view(tokens, heads, dim)
    k = torch.cat([keys, shared[:, None].expand(tokens, heads, rot_dim)], -1)
    v = (latent @ w[prefix + "uv"].T).view(tokens, heads, vdim)
    size = m["mask"]["size"]
    return masked_attention(q, k, v, m["scale"], lambda i, j: sees_window(i, j, size))


def latent_attention_mixer(h, w, prefix, m, eps):
    out = latent_heads(h @ w[prefix + "dq"].T, h @ w[prefix + "dkv"].T, w, prefix, m, eps).flatten(1)
    return (out * torch.sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def chunk_heads(q, k, v, w, prefix, m, eps):
    """Heads [T, H, vdim] from the projections (biases added)."""
    heads, kv, dim, vdim, tokens = m["heads"], m["kv_heads"], m["dim"], m["vdim"], q.shape[0]
    q = rms_norm(q.view(tokens, heads, dim), w[prefix + "q.norm"], eps)
    k = rms_norm(k.view(tokens, kv, dim), w[prefix + "k.norm"], eps)
    size = m["mask"]["size"]
    return masked_attention(q, k, v.view(tokens, kv, vdim), m["scale"], lambda i, j: sees_chunk(i, j, size), distance_slopes(heads), True)


def attention_mixer(h, w, prefix, m, eps):
    q, k, v = (h @ w[prefix + n].T + w[prefix + n + ".b"] for n in "qkv")
    return chunk_heads(q, k, v, w, prefix, m, eps).flatten(1) @ w[prefix + "o"].T + w[prefix + "o.b"]


MIXERS = {"latent_attention": latent_attention_mixer, "attention": attention_mixer}


# ---------------------------------------------------------------------------- the model
def layer_runs(count, loop):
    """(layer, pass before which its vector is added or None) in the order they run."""
    if not loop:
        return [(i, None) for i in range(count)]
    start, stop = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(start)]
    for t in range(loop["times"]):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, count)]


def forward(config, weights, tokens, dtype=torch.float64):
    """Logits [T, vocab] of one sequence and the stream after every layer run [runs, T, width]."""
    w = {name: t.to(dtype) for name, t in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    stream = []
    for i, entering in layer_runs(len(config["layers"]), config.get("loop")):
        layer, at = config["layers"][i], f"l{i}."
        if entering is not None:
            x = x + w["loop.step"][entering]
        h = rms_norm_around_one(x, w[at + "norm1"], eps)
        x = x + MIXERS[layer["type"]](h, w, at + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            h = rms_norm_around_one(x, w[at + "norm2"], eps)
            x = x + relu_glu(h, w[at + "mlp.gate"], w[at + "mlp.up"], w[at + "mlp.down"])
        stream.append(x)
    return rms_norm_around_one(x, w["final.norm"], eps) @ w["head"].T, torch.stack(stream)


def greedy(config, weights, prompt, count, dtype=torch.float64):
    """``count`` greedy tokens after ``prompt`` (the whole sequence again for every token) and the smallest
    gap between the two best logits met on the way."""
    tokens, gap = list(prompt), math.inf
    for _ in range(count):
        logits = forward(config, weights, tokens, dtype)[0][-1]
        best = logits.topk(2).values
        gap = min(gap, float(best[0] - best[1]))
        tokens.append(int(logits.argmax()))
    return tokens[len(prompt):], gap
