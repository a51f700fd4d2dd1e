"""Plain, slow numpy implementation of the Vamidra decoder, the oracle of tests/test_*_vamidra.py.

One function per mechanism, values in float32 between them and sums in float64, whole sequences at
once, the recurrence one token after the other, no cache.  It shares no code with nerva_b200.
`weights` maps tensor names to float32 arrays; `config` is the parsed config.json dictionary.
"""
from __future__ import annotations

import numpy as np

F = np.float32
D = np.float64


def layer_norm(x, eps, w):
    """Mean taken off, divided by the root of the mean squared deviation plus eps, times w."""
    x = np.asarray(x, dtype=D)
    centred = x - x.mean(axis=-1, keepdims=True)
    spread = np.sqrt(np.mean(centred * centred, axis=-1, keepdims=True) + eps)
    return (centred / spread * w).astype(F)


def grouped_rms_norm(x, groups, eps, w):
    """The last axis in `groups` equal parts, each divided by its own root mean square; then times w."""
    parts = np.asarray(x, dtype=D).reshape(*np.shape(x)[:-1], groups, -1)
    parts = parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return (parts.reshape(np.shape(x)) * w).astype(F)


def linear(w, x):
    """Rows of x times a [out, in] matrix."""
    return (np.asarray(x, dtype=D) @ np.asarray(w, dtype=D).T).astype(F)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=D)))


def silu(z):
    return (np.asarray(z, dtype=D) * sigmoid(z)).astype(F)


def gelu_tanh(z):
    z = np.asarray(z, dtype=D)
    return (0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))).astype(F)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, dtype=D))


def soft_cap(score, cap):
    return cap * np.tanh(score / cap) if cap else score


def visible(query_positions, key_positions, window, keep_first):
    """Causal; a query sees the last `window` positions, itself included (0: all), and always the first
    keep_first positions."""
    query = np.asarray(query_positions)[:, None]
    key = np.asarray(key_positions)[None, :]
    near = (query - key < window) if window else np.ones((query.shape[0], key.shape[1]), dtype=bool)
    return (key <= query) & (near | (key < keep_first))


def capped_attention(q, k, v, scale, cap, mask):
    """q [T, H, d], k [S, G, d], v [S, G, e], mask [T, S]; query head h reads KV head h // (H / G)."""
    heads, groups = q.shape[1], k.shape[1]
    out = np.empty((q.shape[0], heads, v.shape[2]), dtype=F)
    for h in range(heads):
        g = h // (heads // groups)
        score = soft_cap((q[:, h].astype(D) @ k[:, g].astype(D).T) * scale, cap)
        score = np.where(mask, score, -np.inf)
        p = np.exp(score - score.max(axis=-1, keepdims=True))
        out[:, h] = (p / p.sum(axis=-1, keepdims=True)) @ v[:, g].astype(D)
    return out


def head_gate(a, w, h):
    """a [T, H, e]: head i times sigmoid of the i-th row of w against the mixer's input."""
    return (a * sigmoid(linear(w, h))[:, :, None]).astype(F)


def attention_mixer(h, m, get, eps):
    """h [T, width]; m the mixer's entry of the configuration; get(name) its tensors."""
    tokens, heads, groups = len(h), m["heads"], m["kv_heads"]
    q = linear(get(".q"), h).reshape(tokens, heads, m["dim"])
    k = linear(get(".k"), h).reshape(tokens, groups, m["dim"])
    v = linear(get(".v"), h).reshape(tokens, groups, m["vdim"])
    mask = m.get("mask") or {}
    at = np.arange(tokens)
    see = visible(at, at, mask.get("size") or 0, mask.get("keep_first") or 0)
    a = head_gate(capped_attention(q, k, v, m["scale"], m.get("softcap"), see), get(".g"), h)
    return linear(get(".o"), a.reshape(tokens, heads * m["vdim"]))


def causal_convolution(u, w, bias):
    """u [T, channels], w [channels, taps]: per channel, the last column of w meets the current token."""
    taps = w.shape[1]
    out = np.tile(np.asarray(bias, dtype=D), (len(u), 1))
    for back in range(min(taps, len(u))):
        out[back:] += np.asarray(w, dtype=D)[:, taps - 1 - back] * np.asarray(u, dtype=D)[:len(u) - back]
    return out.astype(F)


def state_space_scan(x, b, c, step, decay_rate, skip):
    """x [T, H, P], b and c [T, G, N], step [T, H], decay_rate and skip [H].  Per head a state [N, P]:
    S <- exp(-decay_rate step) S + step b x^T, y = S^T c + skip x.  The state starts at zero."""
    tokens, heads, width = x.shape
    groups, states = b.shape[1:]
    out = np.empty_like(x, dtype=F)
    for h in range(heads):
        g = h // (heads // groups)
        s = np.zeros((states, width), dtype=D)
        for t in range(tokens):
            s = np.exp(-D(decay_rate[h]) * step[t, h]) * s + step[t, h] * np.outer(b[t, g], x[t, h]).astype(D)
            out[t, h] = s.T @ c[t, g].astype(D) + skip[h] * x[t, h]
    return out


def state_space_mixer(h, m, get, eps):
    tokens, heads, width, states, groups = len(h), m["heads"], m["vdim"], m["state"], m["groups"]
    inner, shared = heads * width, groups * states
    z, u, step = np.split(linear(get(".in"), h), [inner, 2 * inner + 2 * shared], axis=1)
    u = silu(causal_convolution(u, get(".conv"), get(".conv.b")))
    x, b, c = np.split(u, [inner, inner + shared], axis=1)
    y = state_space_scan(x.reshape(tokens, heads, width), b.reshape(tokens, groups, states),
                         c.reshape(tokens, groups, states), softplus(step + get(".dt_bias")),
                         np.exp(np.asarray(get(".A_log"), dtype=D)), get(".D")).reshape(tokens, inner)
    return linear(get(".o"), grouped_rms_norm(y * silu(z), m["norm_groups"], eps, get(".norm")))


MIXERS = {"attention": attention_mixer, "mamba2": state_space_mixer}


def feed_forward(h, get):
    return linear(get(".down"), gelu_tanh(linear(get(".gate"), h)) * linear(get(".up"), h))


def layer(x, entry, name, weights, eps):
    """A norm in front of and a norm behind each sublayer; the residual around both."""
    y = MIXERS[entry["type"]](layer_norm(x, eps, weights[name + ".norm1"]), entry["mixer"],
                              lambda t: weights[f"{name}.mix{t}"], eps)
    x = (x + layer_norm(y, eps, weights[name + ".norm1b"])).astype(F)
    if entry.get("mlp"):
        y = feed_forward(layer_norm(x, eps, weights[name + ".norm2"]), lambda t: weights[f"{name}.mlp{t}"])
        x = (x + layer_norm(y, eps, weights[name + ".norm2b"])).astype(F)
    return x


def begin_pass(x, first, weights, number):
    """Stream and embedding side by side through one matrix, then the pass's own vector."""
    return (linear(weights["loop.in"], np.concatenate([x, first], axis=-1)) + weights["loop.step"][number]).astype(F)


def layer_runs(config):
    """(layer, pass) in execution order; pass is the number of the pass that begins there, else None."""
    loop, count = config.get("loop"), len(config["layers"])
    if not loop:
        return [(i, None) for i in range(count)]
    inside = range(loop["start"], loop["stop"])
    runs = [(i, None) for i in range(loop["start"])]
    runs += [(i, t if i == loop["start"] else None) for t in range(loop["times"]) for i in inside]
    return runs + [(i, None) for i in range(loop["stop"], count)]


def forward(config, weights, tokens, trace=None):
    """Logits [T, vocab] of a whole sequence; trace (a list) receives the stream after every layer run."""
    eps = config["norm"]["eps"]
    first = np.asarray(weights["embed"], dtype=F)[np.asarray(tokens)]
    x = first
    for index, number in layer_runs(config):
        if number is not None:
            x = begin_pass(x, first, weights, number)
        x = layer(x, config["layers"][index], f"l{index}", weights, eps)
        if trace is not None:
            trace.append(x)
    return linear(weights["head"], layer_norm(x, eps, weights["final.norm"])) * F(config["logit_scale"])
