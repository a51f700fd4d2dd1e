"""Configuration and checkpoints of sandwich-block decoders (the Vamidra design).

A layer norm in front of and behind each sublayer, x += norm1b(mixer(norm1(x))), then
x += norm2b(mlp(norm2(x))); a mixer per layer, attention (sliding window with kept first positions,
soft-capped scores, one output gate per head, no rotation) or a selective state space; a feed-forward
gated by a tanh-form gelu; a range of layers that runs several times, every pass beginning with a
projection of the stream joined with the embedding output; scaled logits.  The C side is
nerva_b200_session_create_parallel (include/nerva_b200_api.h); nothing here computes anything.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field

import numpy as np

from . import synth
from .parallel_model import ParallelCheckpoint, ParallelLayer, native_model
from .safetensors_file import open_tensors

ARCHITECTURE = "Vamidra"
BLOCK_SANDWICH, MIXER_STATE_SPACE, NORM_LAYER, ACTIVATION_GELU_TANH = 1, 1, 1, 1  # NERVA_B200_*


@dataclass(frozen=True)
class StateSpaceLayer:
    heads: int
    v_dim: int
    state: int
    groups: int
    conv: int               # taps, the current token included
    norm_groups: int
    intermediate: int       # 0: no feed-forward

    @property
    def inner(self) -> int:
        return self.heads * self.v_dim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    def fill(self, out) -> None:
        """This layer as a NervaB200ParallelLayer."""
        out.mixer, out.heads, out.v_dim, out.intermediate = MIXER_STATE_SPACE, self.heads, self.v_dim, self.intermediate
        out.state_size, out.state_groups, out.conv_taps, out.norm_groups = self.state, self.groups, self.conv, self.norm_groups


def attention_layer(heads: int, kv_heads: int, qk_dim: int, v_dim: int, intermediate: int, window: int, keep_first: int,
                    score_scale: float, score_softcap: float) -> ParallelLayer:
    """The design's attention: no rotation, no norm of q and k, a gate per head."""
    return ParallelLayer(heads=heads, kv_heads=kv_heads, qk_dim=qk_dim, v_dim=v_dim, intermediate=intermediate, window=window,
                         score_scale=score_scale, qk_norm=False, layer_scale=False, keep_first=keep_first,
                         score_softcap=score_softcap, head_gate=True)


@dataclass(frozen=True)
class SandwichConfig:
    name: str
    hidden: int
    vocab: int
    rms_eps: float          # of every norm (the create request's name for it)
    layer_specs: tuple = field(default=())
    logit_scale: float = 1.0
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 0     # 0: no loop

    # what the session's create request and the workloads ask every configuration for
    rope_theta = 0.0
    num_experts = 0
    kv_heads = 1  # the request's common value; the real ones are per layer

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
    def head_dim(self) -> int:
        return max([1] + [max(s.qk_dim, s.v_dim) for s in self.layer_specs if isinstance(s, ParallelLayer)])

    @property
    def intermediate(self) -> int:
        return max(1, max(s.intermediate for s in self.layer_specs))

    def tensor_shapes(self) -> dict:
        """name -> shape, in upload order."""
        shapes = {"embed": (self.vocab, self.hidden)}
        if self.loop_times:
            shapes["loop.in"] = (self.hidden, 2 * self.hidden)
            shapes["loop.step"] = (self.loop_times, self.hidden)
        for i, s in enumerate(self.layer_specs):
            p = f"l{i}."
            shapes[p + "norm1"] = (self.hidden,)
            if isinstance(s, StateSpaceLayer):
                shapes[p + "mix.in"] = (s.inner + s.channels + s.heads, self.hidden)
                shapes[p + "mix.conv"] = (s.channels, s.conv)
                shapes[p + "mix.conv.b"] = (s.channels,)
                for name in ("dt_bias", "A_log", "D"):
                    shapes[p + "mix." + name] = (s.heads,)
                shapes[p + "mix.norm"] = (s.inner,)
                shapes[p + "mix.o"] = (self.hidden, s.inner)
            else:
                shapes[p + "mix.q"] = (s.heads * s.qk_dim, self.hidden)
                shapes[p + "mix.k"] = (s.kv_heads * s.qk_dim, self.hidden)
                shapes[p + "mix.v"] = (s.kv_heads * s.v_dim, self.hidden)
                shapes[p + "mix.g"] = (s.heads, self.hidden)
                shapes[p + "mix.o"] = (self.hidden, s.heads * s.v_dim)
            shapes[p + "norm1b"] = (self.hidden,)
            if s.intermediate:
                shapes[p + "norm2"] = (self.hidden,)
                shapes[p + "mlp.gate"] = (s.intermediate, self.hidden)
                shapes[p + "mlp.up"] = (s.intermediate, self.hidden)
                shapes[p + "mlp.down"] = (self.hidden, s.intermediate)
                shapes[p + "norm2b"] = (self.hidden,)
        shapes["final.norm"] = (self.hidden,)
        shapes["head"] = (self.vocab, self.hidden)
        return shapes

    def streamed_bytes_per_token(self) -> int:
        """Matrix bytes one decoded token streams (a looped layer and the join count each pass)."""
        per_layer = [0] * self.layers
        other = 2 * self.vocab * self.hidden
        for name, shape in self.tensor_shapes().items():
            if len(shape) != 2 or name in ("embed", "head", "loop.step"):
                continue
            if name == "loop.in":
                other += 2 * shape[0] * shape[1] * self.loop_times
            else:
                per_layer[int(name[1:name.index(".")])] += 2 * shape[0] * shape[1]
        looped = sum(per_layer[self.loop_start:self.loop_stop]) * max(self.loop_times - 1, 0)
        return sum(per_layer) + looped + other

    def native_model(self, compute: str):
        """The NervaB200ParallelModel of the create call."""
        return native_model(self, compute, embedding_scale=1.0, logit_scale=self.logit_scale, block=BLOCK_SANDWICH,
                            norm=NORM_LAYER, activation=ACTIVATION_GELU_TANH, loop_input=1)

    @classmethod
    def from_json(cls, config: dict, name: str = ARCHITECTURE) -> "SandwichConfig":
        specs = []
        for i, entry in enumerate(config["layers"]):
            m, mlp = entry["mixer"], entry.get("mlp")
            if mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            ff = mlp["ff"] if mlp else 0
            if entry["type"] == "attention":
                mask = m.get("mask") or {}
                specs.append(attention_layer(heads=m["heads"], kv_heads=m["kv_heads"], qk_dim=m["dim"], v_dim=m["vdim"],
                                             intermediate=ff, window=mask.get("size") or 0,
                                             keep_first=mask.get("keep_first") or 0, score_scale=m["scale"],
                                             score_softcap=m.get("softcap") or 0.0))
            elif entry["type"] == "mamba2":
                specs.append(StateSpaceLayer(heads=m["heads"], v_dim=m["vdim"], state=m["state"], groups=m["groups"],
                                             conv=m["conv"], norm_groups=m["norm_groups"], intermediate=ff))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {entry['type']!r}")
        loop = config.get("loop") or {"start": 0, "stop": 0, "times": 0}
        return cls(name=name, hidden=config["width"], vocab=config["vocab"], rms_eps=config["norm"]["eps"],
                   layer_specs=tuple(specs), logit_scale=config.get("logit_scale") or 1.0, loop_start=loop["start"],
                   loop_stop=loop["stop"], loop_times=loop["times"])


def random_checkpoint(cfg: SandwichConfig, seed: int = 0, std: float = 0.02, fill=None) -> ParallelCheckpoint:
    """Random-init matrices ~ N(0, std), unit norms, zero biases, decays between 1 and 16."""
    gen = fill or synth.normal_bf16
    tensors = {}
    for i, (name, shape) in enumerate(cfg.tensor_shapes().items()):
        count = int(np.prod(shape, dtype=np.int64))
        if name.endswith((".conv.b", ".dt_bias")):
            tensors[name] = np.zeros(shape, dtype=np.uint16)
        elif name.endswith(".A_log"):
            tensors[name] = synth.f32_to_bf16(np.log(np.linspace(1.0, 16.0, count, dtype=np.float32))).reshape(shape)
        elif len(shape) == 1:
            tensors[name] = np.full(shape, synth.BF16_ONE, dtype=np.uint16)
        else:
            scale = 0.3 if name.endswith(".conv") else std
            tensors[name] = gen(seed, synth.T_LAYER_BASE + i, count, scale).reshape(shape)
    return ParallelCheckpoint(cfg, tensors)


def load(folder: str, config: dict) -> ParallelCheckpoint:
    """config: the folder's parsed config.json; weights: its model.safetensors."""
    return ParallelCheckpoint(SandwichConfig.from_json(config, name=os.path.basename(os.path.abspath(folder))),
                              open_tensors(os.path.join(folder, "model.safetensors")))


def dump_config(cfg: SandwichConfig) -> str:
    """The config.json text of a configuration (what from_json reads)."""
    layers = []
    for s in cfg.layer_specs:
        entry = {"mlp": {"kind": "dense", "ff": s.intermediate} if s.intermediate else None}
        if isinstance(s, StateSpaceLayer):
            entry["type"] = "mamba2"
            entry["mixer"] = {"heads": s.heads, "vdim": s.v_dim, "state": s.state, "groups": s.groups, "conv": s.conv,
                              "norm_groups": s.norm_groups}
        else:
            entry["type"] = "attention"
            entry["mixer"] = {"heads": s.heads, "kv_heads": s.kv_heads, "dim": s.qk_dim, "vdim": s.v_dim,
                              "mask": {"size": s.window, "keep_first": s.keep_first}, "scale": s.score_scale,
                              "softcap": s.score_softcap}
        layers.append(entry)
    out = {"architecture": ARCHITECTURE, "vocab": cfg.vocab, "width": cfg.hidden, "norm": {"eps": cfg.rms_eps},
           "logit_scale": cfg.logit_scale, "layers": layers}
    if cfg.loop_times:
        out["loop"] = {"start": cfg.loop_start, "stop": cfg.loop_stop, "times": cfg.loop_times}
    return json.dumps(out)
