"""Small Vuvolix configurations with random weights for the tests, as config.json dictionaries."""
from __future__ import annotations

import copy
import json
import os

import numpy as np

from nerva_b200 import parallel_model, safetensors_file, synth

# Differences of logits (root mean square over positions and vocabulary, relative to the logits' own
# spread) a format may show against the fp32 oracle.
TOLERANCE = {"float32": 2e-5, "bfloat16": 3e-2}


def attention(heads=4, kv_heads=2, dim=32, vdim=32, window=24, rot=16, base=10000.0, scaling=None, scale=None):
    rot = {"dims": rot, "base": base}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "rot": rot,
            "scale": scale if scale is not None else 2.0 / dim ** 0.5}


YARN = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}


def layer(ff=96, **mixer):
    return {"type": "attention", "mixer": attention(**mixer), "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=128, vocab=301, eps=1e-5, scale=3.0, cap=3.0, loop=None):
    out = {"architecture": "Vuvolix", "width": width, "vocab": vocab, "norm": {"eps": eps},
           "embedding": {"scale": scale}, "layers": copy.deepcopy(layers), "logit_softcap": cap}
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def full_config():
    """Every mechanism at once, no two layers alike."""
    return config([layer(window=24, scaling=YARN), layer(heads=6, kv_heads=2, dim=48, vdim=32, ff=200, window=40, rot=24),
                   layer(ff=0, heads=3, kv_heads=3, dim=40, vdim=24, window=7, rot=40, base=500.0),
                   layer(heads=8, kv_heads=1, dim=16, vdim=64, window=33, rot=8, ff=72)], loop=(1, 3, 3))


def round_bf16(x):
    return synth.bf16_to_f32(synth.f32_to_bf16(np.asarray(x, dtype=np.float32))).reshape(np.shape(x))


def weights(cfg, seed=0):
    """name -> float32 array of bf16-representable values: matrices scaled by their fan-in, norms and
    layer scales spread around values that are neither 0 nor 1."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in parallel_model.ParallelConfig.from_json(cfg).tensor_shapes().items():
        if name.endswith(("norm1", "final.norm")):
            w = 1.0 + 0.3 * rng.standard_normal(shape)
        elif name.endswith((".ls1", ".ls2")):
            w = 0.7 + 0.4 * rng.standard_normal(shape)
        elif name in ("embed", "loop.step"):
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) * (1.5 / shape[1] ** 0.5)
        out[name] = round_bf16(w)
    return out


def checkpoint(cfg, w):
    return parallel_model.ParallelCheckpoint(parallel_model.ParallelConfig.from_json(cfg, name="test"),
                                             {k: synth.f32_to_bf16(v).reshape(v.shape) for k, v in w.items()})


def write_folder(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    safetensors_file.write_tensors(os.path.join(path, "model.safetensors"),
                                   {k: synth.f32_to_bf16(v).reshape(v.shape) for k, v in w.items()})
    return str(path)


def tokens(cfg, count, seed=1):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], count).tolist()


def distance(got, want):
    """Root mean square difference relative to the spread of the expected logits."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return float(np.sqrt(np.mean((got - want) ** 2)) / want.std())


def worst_position(got, want):
    """The largest of the positions' own distances."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return float(np.sqrt(np.mean((got - want) ** 2, axis=-1)).max() / want.std())


# ---- one key that stands out ----
KEY, QUERY = 0, 1  # marker tokens


def marked_model(window, seed=0, **mixer):
    """A one-layer model in which token QUERY attends almost only to token KEY wherever it sees one, and
    the value of KEY changes the logits strongly: whether one key is inside the window decides the result.
    The markers live in two channels of the stream that nothing else writes."""
    cfg = config([layer(ff=0, window=window, scale=1.5, **mixer)], scale=1.0, cap=0)
    w = weights(cfg, seed)
    m = cfg["layers"][0]["mixer"]
    w["embed"][:, :2] = 0.0
    w["embed"][KEY, 0] = 40.0
    w["embed"][QUERY, 1] = 40.0
    plain = 2 * (m["rot"]["dims"] // 2)  # the first dimension that no rotation touches
    for name, channel, heads in (("l0.mix.k", 0, m["kv_heads"]), ("l0.mix.q", 1, m["heads"])):
        rows = w[name].reshape(heads, m["dim"], -1)
        rows[:, :, :2] = 0.0
        rows[:, plain, channel] = 8.0
    v = w["l0.mix.v"].reshape(m["kv_heads"], m["vdim"], -1)
    v[:, :, :2] = 0.0
    v[:, 0, 0] = 2.0
    return cfg, {k: round_bf16(t) for k, t in w.items()}


def marked_tokens(cfg, length, key_at, query_at, seed=3):
    t = np.random.default_rng(seed).integers(2, cfg["vocab"], length)
    t[key_at], t[query_at] = KEY, QUERY
    return t.tolist()
