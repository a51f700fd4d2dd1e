"""Configuration and checkpoints of parallel-block decoders (the Vuvolix design).

x += ls1 * attention(norm(x)) + ls2 * mlp(norm(x)) per layer; sliding-window grouped-query attention
with a rotation of part of each head, a weightless RMS norm of q and k behind it; a range of layers
that runs several times; a scaled embedding and soft-capped logits.  The C side is
nerva_b200_session_create_parallel (include/nerva_b200_api.h); nothing here computes anything.
"""
from __future__ import annotations

import ctypes as C
import json
from dataclasses import dataclass, field

import numpy as np

from . import ffi, synth
from .safetensors_file import FileTensor

ARCHITECTURE = "Vuvolix"
COMPUTE = {"bfloat16": 1, "float32": 2}  # NERVA_DTYPE_BF16 / NERVA_DTYPE_F32


@dataclass(frozen=True)
class ParallelLayer:
    heads: int
    kv_heads: int
    qk_dim: int
    v_dim: int
    intermediate: int       # 0: no feed-forward
    window: int             # 0: every earlier key
    score_scale: float
    rotary_dims: int = 0
    rotary_base: float = 10000.0
    scaling: dict | None = None  # factor, original, fast, slow
    qk_norm: bool = True
    layer_scale: bool = True
    keep_first: int = 0     # positions below this stay visible behind the window
    score_softcap: float = 0.0
    head_gate: bool = False

    def fill(self, out) -> None:
        """This layer as a NervaB200ParallelLayer."""
        out.heads, out.kv_heads, out.qk_dim, out.v_dim = self.heads, self.kv_heads, self.qk_dim, self.v_dim
        out.intermediate, out.window, out.rotary_dims = self.intermediate, self.window, self.rotary_dims
        out.qk_norm, out.layer_scale, out.score_scale = int(self.qk_norm), int(self.layer_scale), self.score_scale
        out.keep_first, out.score_softcap, out.head_gate = self.keep_first, self.score_softcap, int(self.head_gate)
        out.rotary_base = self.rotary_base
        if self.scaling:
            out.yarn_factor, out.yarn_original = self.scaling["factor"], self.scaling["original"]
            out.yarn_fast, out.yarn_slow = self.scaling["fast"], self.scaling["slow"]


def native_model(cfg, compute: str, **fields):
    """The NervaB200ParallelModel of a configuration's layer_specs and loop; fields: the model's own."""
    layers = (ffi.structs["NervaB200ParallelLayer"] * cfg.layers)()
    for out, spec in zip(layers, cfg.layer_specs):
        spec.fill(out)
    model = ffi.structs["NervaB200ParallelModel"](
        layer_count=cfg.layers, compute=COMPUTE[compute], loop_start=cfg.loop_start, loop_stop=cfg.loop_stop,
        loop_times=cfg.loop_times, layers=C.cast(layers, C.c_void_p), **fields)
    model._keep = layers
    return model


@dataclass(frozen=True)
class ParallelConfig:
    name: str
    hidden: int
    vocab: int
    rms_eps: float
    layer_specs: tuple = field(default=())
    embedding_scale: float = 1.0
    logit_softcap: float = 0.0
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0     # 0: no loop

    # what the session's create request and the workloads ask every configuration for
    rope_theta = 0.0
    num_experts = 0

    @property
    def layers(self) -> int:
        return len(self.layer_specs)

    @property
    def layer_runs(self) -> int:
        extra = (self.loop_times - 1) * (self.loop_stop - self.loop_start) if self.loop_times else 0
        return self.layers + extra

    @property
    def heads(self) -> int:
        return max(s.heads for s in self.layer_specs)

    @property
    def kv_heads(self) -> int:
        return 1  # the request's common value; the real ones are per layer

    @property
    def head_dim(self) -> int:
        return max(max(s.qk_dim, s.v_dim) for s in self.layer_specs)

    @property
    def intermediate(self) -> int:
        return max(1, max(s.intermediate for s in self.layer_specs))

    def tensor_shapes(self) -> dict:
        """name -> shape, in upload order."""
        shapes = {"embed": (self.vocab, self.hidden)}
        if self.loop_times:
            shapes["loop.step"] = (self.loop_times, self.hidden)
        for i, s in enumerate(self.layer_specs):
            p = f"l{i}."
            shapes[p + "norm1"] = (self.hidden,)
            shapes[p + "mix.q"] = (s.heads * s.qk_dim, self.hidden)
            shapes[p + "mix.k"] = (s.kv_heads * s.qk_dim, self.hidden)
            shapes[p + "mix.v"] = (s.kv_heads * s.v_dim, self.hidden)
            if s.head_gate:
                shapes[p + "mix.g"] = (s.heads, self.hidden)
            shapes[p + "mix.o"] = (self.hidden, s.heads * s.v_dim)
            if s.intermediate:
                shapes[p + "mlp.gate"] = (s.intermediate, self.hidden)
                shapes[p + "mlp.up"] = (s.intermediate, self.hidden)
                shapes[p + "mlp.down"] = (self.hidden, s.intermediate)
            if s.layer_scale:
                shapes[p + "ls1"] = (self.hidden,)
                if s.intermediate:
                    shapes[p + "ls2"] = (self.hidden,)
        shapes["final.norm"] = (self.hidden,)
        shapes["head"] = (self.vocab, self.hidden)
        return shapes

    def streamed_bytes_per_token(self) -> int:
        """Weight bytes one decoded token streams (a looped layer counts each time)."""
        per_layer = [2 * self.hidden * (s.heads * (s.qk_dim + s.v_dim) + s.kv_heads * (s.qk_dim + s.v_dim)
                                        + 3 * s.intermediate) for s in self.layer_specs]
        looped = sum(per_layer[self.loop_start:self.loop_stop]) if self.loop_times else 0
        return sum(per_layer) + (self.loop_times - 1 if self.loop_times else 0) * looped + 2 * self.vocab * self.hidden

    def native_model(self, compute: str):
        return native_model(self, compute, embedding_scale=self.embedding_scale, logit_softcap=self.logit_softcap)

    @classmethod
    def from_json(cls, config: dict, name: str = ARCHITECTURE) -> "ParallelConfig":
        """From a parsed config.json (sizes that only tensor shapes carry come from there: see load)."""
        specs = []
        for i, entry in enumerate(config["layers"]):
            if entry["type"] != "attention":
                raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
            m, mlp = entry["mixer"], entry.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            rot = m.get("rot") or {"dims": 0, "base": 10000.0}
            specs.append(ParallelLayer(
                heads=m["heads"], kv_heads=m["kv_heads"], qk_dim=m["dim"], v_dim=m["vdim"],
                intermediate=mlp["ff"] if mlp else 0, window=(m.get("mask") or {}).get("size") or 0,
                score_scale=m["scale"], rotary_dims=rot["dims"], rotary_base=float(rot["base"]),
                scaling=rot.get("scaling")))
        loop = config.get("loop")
        return cls(name=name, hidden=config["width"], vocab=config["vocab"], rms_eps=config["norm"]["eps"],
                   layer_specs=tuple(specs), embedding_scale=(config.get("embedding") or {}).get("scale", 1.0),
                   logit_softcap=config.get("logit_softcap") or 0.0,
                   loop_start=loop["start"] if loop else 0, loop_stop=loop["stop"] if loop else 0,
                   loop_times=loop["times"] if loop else 0)


@dataclass
class ParallelCheckpoint:
    """A configuration (this module's, or one of the same interface) and its tensors: uint16 arrays of bf16
    bits, or FileTensor ranges of a file."""
    config: ParallelConfig
    tensors: dict

    def __post_init__(self):
        for name, shape in self.config.tensor_shapes().items():
            if name not in self.tensors:
                raise ValueError(f"tensor {name} is missing")
            t = self.tensors[name]
            if tuple(t.shape) != shape:
                raise ValueError(f"tensor {name} has shape {tuple(t.shape)}, the configuration says {shape}")
            if isinstance(t, FileTensor) and t.dtype != "BF16":
                raise ValueError(f"tensor {name} is {t.dtype}, not BF16")

    def upload_order(self) -> list:
        return [self.tensors[name] for name in self.config.tensor_shapes()]

    def native_model(self, compute: str):
        """The NervaB200ParallelModel of the create call."""
        return self.config.native_model(compute)


def random_checkpoint(cfg: ParallelConfig, seed: int = 0, std: float = 0.02, fill=None) -> ParallelCheckpoint:
    """Random-init weights ~ N(0, std), unit norms and scales (the workloads' counterpart of synth.dense_checkpoint)."""
    gen = fill or synth.normal_bf16
    tensors = {}
    for i, (name, shape) in enumerate(cfg.tensor_shapes().items()):
        count = int(np.prod(shape, dtype=np.int64))
        if len(shape) == 1:
            tensors[name] = np.full(shape, synth.BF16_ONE, dtype=np.uint16)
        else:
            tensors[name] = gen(seed, synth.T_LAYER_BASE + i, count, std).reshape(shape)
    return ParallelCheckpoint(cfg, tensors)


def load(folder: str, config: dict) -> ParallelCheckpoint:
    """config: the folder's parsed config.json; weights: its model.safetensors."""
    import os

    from .safetensors_file import open_tensors
    return ParallelCheckpoint(ParallelConfig.from_json(config, name=os.path.basename(os.path.abspath(folder))),
                              open_tensors(os.path.join(folder, "model.safetensors")))


def dump_config(cfg: ParallelConfig) -> str:
    """The config.json text of a configuration (what from_json reads)."""
    layers = []
    for s in cfg.layer_specs:
        rot = {"base": s.rotary_base, "dims": s.rotary_dims}
        if s.scaling:
            rot["scaling"] = s.scaling
        layers.append({"type": "attention",
                       "mixer": {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.qk_dim, "vdim": s.v_dim,
                                 "mask": {"size": s.window}, "rot": rot, "scale": s.score_scale},
                       "mlp": {"kind": "dense", "ff": s.intermediate} if s.intermediate else None})
    out = {"architecture": ARCHITECTURE, "vocab": cfg.vocab, "width": cfg.hidden, "norm": {"eps": cfg.rms_eps},
           "embedding": {"scale": cfg.embedding_scale}, "logit_softcap": cfg.logit_softcap, "layers": layers}
    if cfg.loop_times:
        out["loop"] = {"start": cfg.loop_start, "stop": cfg.loop_stop, "times": cfg.loop_times}
    return json.dumps(out)
