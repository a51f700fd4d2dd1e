"""Small Vamidra configurations with random weights for the tests, as config.json dictionaries."""
from __future__ import annotations

import copy

import numpy as np

from nerva_b200 import parallel_model, sandwich_model, synth
from tests.vuvolix_models import TOLERANCE, distance, round_bf16, tokens, worst_position, write_folder  # noqa: F401

__all__ = ["TOLERANCE", "distance", "round_bf16", "tokens", "worst_position", "write_folder", "attention", "space", "config",
           "full_config", "weights", "checkpoint", "marked_model", "marked_tokens", "remembering_model"]


def attention(ff=80, heads=4, kv_heads=2, dim=24, vdim=40, window=20, keep=3, scale=None, cap=6.0):
    return {"type": "attention", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "softcap": cap,
                      "mask": {"size": window, "keep_first": keep},
                      "scale": scale if scale is not None else 1.5 / dim ** 0.5}}


def space(ff=80, heads=6, vdim=24, state=40, groups=3, conv=4, norm_groups=4):
    return {"type": "mamba2", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                      "norm_groups": norm_groups}}


def config(layers, width=112, vocab=283, eps=1e-5, logit_scale=0.7, loop=None):
    out = {"architecture": "Vamidra", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "layers": copy.deepcopy(layers), "logit_scale": logit_scale}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def full_config():
    """Every mechanism at once, no two layers alike."""
    return config([space(), attention(), space(ff=0, heads=4, vdim=64, state=16, groups=1, conv=3, norm_groups=2),
                   attention(ff=136, heads=3, kv_heads=3, dim=40, vdim=16, window=37, keep=18, cap=2.0),
                   attention(ff=0, heads=8, kv_heads=1, dim=16, vdim=32, window=9, keep=0)], loop=(1, 4, 3))


def weights(cfg, seed=0):
    """name -> float32 array of bf16-representable values: matrices scaled by their fan-in, norms spread
    around values that are neither 0 nor 1, decays from slow to fast."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in sandwich_model.SandwichConfig.from_json(cfg).tensor_shapes().items():
        if "norm" in name.rsplit(".", 1)[-1]:
            w = 1.0 + 0.3 * rng.standard_normal(shape)
        elif name.endswith((".conv.b", ".D")):
            w = 0.4 * rng.standard_normal(shape)
        elif name.endswith(".dt_bias"):
            w = rng.uniform(-4.0, 0.5, shape)
        elif name.endswith(".A_log"):
            w = rng.uniform(-3.0, 1.5, shape)
        elif name.endswith(".conv"):
            w = rng.standard_normal(shape) * 0.7
        elif name in ("embed", "loop.step"):
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) * (1.5 / shape[1] ** 0.5)
        out[name] = round_bf16(w)
    return out


def checkpoint(cfg, w):
    return parallel_model.ParallelCheckpoint(sandwich_model.SandwichConfig.from_json(cfg, name="test"),
                                             {k: synth.f32_to_bf16(v).reshape(v.shape) for k, v in w.items()})


# ---- one key that stands out ----
KEY, QUERY = 0, 1  # marker tokens


def marked_model(window, keep, seed=0, **mixer):
    """A one-layer model in which token QUERY attends almost only to token KEY wherever it sees one, and the value
    of KEY changes the logits strongly: whether one key is visible decides the result.  The markers are large values
    in two channels of the embedding, read by one dimension of the queries and keys that nothing else feeds."""
    cfg = config([attention(ff=0, window=window, keep=keep, scale=0.006, cap=30.0, **mixer)], width=128, logit_scale=1.0)
    w = weights(cfg, seed)
    m = cfg["layers"][0]["mixer"]
    w["embed"][:, :2] = 0.0
    w["embed"][KEY, 0] = w["embed"][QUERY, 1] = 40.0
    w["l0.norm1"][:] = 1.0
    for name, channel, heads in (("l0.mix.k", 0, m["kv_heads"]), ("l0.mix.q", 1, m["heads"])):
        rows = w[name].reshape(heads, m["dim"], -1)
        rows[:, :, :2] = 0.0
        rows[:, 0, :] = 0.0
        rows[:, 0, channel] = 8.0
    v = w["l0.mix.v"].reshape(m["kv_heads"], m["vdim"], -1)
    v[:, :, :2] = 0.0
    v[:, 0, 0] = 2.0
    return cfg, {k: round_bf16(t) for k, t in w.items()}


def marked_tokens(cfg, length, key_at, query_at, seed=3):
    t = np.random.default_rng(seed).integers(2, cfg["vocab"], length)
    if key_at is not None:
        t[key_at] = KEY
    t[query_at] = QUERY
    return t.tolist()


def remembering_model(seed=0, **mixer):
    """A state-space layer that hardly forgets, and in which token KEY takes a far larger step than any other:
    it still shows after hundreds of tokens."""
    cfg = config([space(ff=0, **mixer)], logit_scale=1.0)
    w = weights(cfg, seed)
    w["l0.mix.A_log"][:] = -8.0
    w["l0.mix.dt_bias"][:] = -6.0
    w["embed"][:, 0] = 0.0
    w["embed"][KEY, 0] = 40.0
    w["l0.norm1"][:] = 1.0
    steps = w["l0.mix.in"][-cfg["layers"][0]["mixer"]["heads"]:]
    steps[:] *= 0.2
    steps[:, 0] = 1.5
    return cfg, {k: round_bf16(t) for k, t in w.items()}
