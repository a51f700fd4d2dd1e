"""Plain, slow numpy implementation of the Vuvolix decoder, the oracle of tests/test_*_vuvolix.py.

One function per mechanism, everything in float32 (sums of products in float64 where numpy
allows it cheaply), whole sequences at once, no cache.  It shares no code with nerva_b200.
`weights` maps tensor names to float32 arrays; `config` is the parsed config.json dictionary.
"""
from __future__ import annotations

import math

import numpy as np

F = np.float32


def rms_norm(x, eps, w=None):
    """x / sqrt(mean(x^2) + eps), times w when given, over the last axis."""
    x = np.asarray(x, dtype=F)
    y = x / np.sqrt(np.mean(np.square(x, dtype=np.float64), axis=-1, keepdims=True) + eps)
    return (y if w is None else y * w).astype(F)


def linear(w, x):
    """Rows of x times a [out, in] matrix."""
    return (np.asarray(x, dtype=np.float64) @ np.asarray(w, dtype=np.float64).T).astype(F)


def silu(z):
    return (z / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))).astype(F)


def embedding(table, tokens, scale):
    return (np.asarray(table, dtype=F)[np.asarray(tokens)] * F(scale)).astype(F)


def rotary_frequencies(dims, base, scaling=None):
    """Angle per position of each of the dims/2 pairs, and the factor on cos and sin."""
    half = dims // 2
    plain = [float(base) ** (-2.0 * i / dims) for i in range(half)]
    if not scaling or dims == 0:
        return np.array(plain, dtype=F), 1.0

    def dim_of(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(dim_of(scaling["fast"])), 0)
    hi = min(math.ceil(dim_of(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / scaling["factor"] * ramp + f * (1.0 - ramp))
    return np.array(out, dtype=F), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, freq, magnitude):
    """x [tokens, heads, dim]: pairs (i, i + n) of the first 2n dimensions turned by position * freq[i]."""
    n = len(freq)
    out = np.array(x, dtype=F)
    angle = (np.asarray(positions, dtype=F)[:, None] * freq[None, :]).astype(F).astype(np.float64)
    c = (np.cos(angle) * magnitude)[:, None, :]
    s = (np.sin(angle) * magnitude)[:, None, :]
    u, v = np.array(out[..., :n]), np.array(out[..., n:2 * n])
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


def visible(query_positions, key_positions, window):
    """Causal sliding window: a query sees itself and the window - 1 positions before it."""
    back = np.asarray(query_positions)[:, None] - np.asarray(key_positions)[None, :]
    return (back >= 0) & (back < window) if window else back >= 0


def softmax_attention(q, k, v, scale, mask):
    """q [T, H, d], k [S, G, d], v [S, G, e], mask [T, S]; query head h reads KV head h // (H / G)."""
    heads, groups = q.shape[1], k.shape[1]
    out = np.empty((q.shape[0], heads, v.shape[2]), dtype=F)
    for h in range(heads):
        g = h // (heads // groups)
        score = (q[:, h].astype(np.float64) @ k[:, g].astype(np.float64).T) * scale
        score = np.where(mask, score, -np.inf)
        p = np.exp(score - score.max(axis=-1, keepdims=True))
        out[:, h] = (p / p.sum(axis=-1, keepdims=True)) @ v[:, g].astype(np.float64)
    return out


def attention_mixer(h, m, get, eps, positions):
    """h [T, width]; m the mixer's entry of the configuration; get(name) its tensors."""
    tokens, heads, groups, dim, vdim = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(get("q"), h).reshape(tokens, heads, dim)
    k = linear(get("k"), h).reshape(tokens, groups, dim)
    v = linear(get("v"), h).reshape(tokens, groups, vdim)
    freq, magnitude = rotary_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = rms_norm(rotate(q, positions, freq, magnitude), eps)
    k = rms_norm(rotate(k, positions, freq, magnitude), eps)
    a = softmax_attention(q, k, v, m["scale"], visible(positions, positions, m["mask"]["size"]))
    return linear(get("o"), a.reshape(tokens, heads * vdim))


def dense_feed_forward(h, get):
    return linear(get("down"), silu(linear(get("gate"), h)) * linear(get("up"), h))


def layer(x, entry, name, weights, eps, positions):
    """Parallel block: one norm, mixer and feed-forward both read it, each result scaled per channel."""
    h = rms_norm(x, eps, weights[name + ".norm1"])
    y = attention_mixer(h, entry["mixer"], lambda t: weights[f"{name}.mix.{t}"], eps, positions) * weights[name + ".ls1"]
    if entry.get("mlp"):
        y = y + dense_feed_forward(h, lambda t: weights[f"{name}.mlp.{t}"]) * weights[name + ".ls2"]
    return (x + y).astype(F)


def layer_runs(config):
    """(layer, pass) in execution order; pass is the loop's pass number before the loop's first layer, else None."""
    loop = config.get("loop")
    count = len(config["layers"])
    if not loop:
        return [(i, None) for i in range(count)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], count)]


def soft_cap(logits, cap):
    return (cap * np.tanh(logits / cap)).astype(F) if cap else logits


def forward(config, weights, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence; trace (a list) receives the stream after every layer run."""
    eps = config["norm"]["eps"]
    positions = np.arange(len(tokens))
    x = embedding(weights["embed"], tokens, config["embedding"]["scale"])
    for index, step in layer_runs(config):
        if step is not None:
            x = (x + weights["loop.step"][step]).astype(F)
        x = layer(x, config["layers"][index], f"l{index}", weights, eps, positions)
        if trace is not None:
            trace.append(x)
    logits = linear(weights["head"], rms_norm(x, eps, weights["final.norm"]))
    return soft_cap(logits, config.get("logit_softcap"))
