"""Model folders: config.json names the architecture, the registry names the loader.

A loader gets (folder, parsed config.json) and returns a checkpoint object that
nerva_b200.session.CudaHfDecodeSequenceSession takes: `.config` with the create request's scalars,
and either the dense tensors of nerva_b200.synth.DenseCheckpoint or `upload_order()` and
`native_model(compute)` (nerva_b200.parallel_model, nerva_b200.sandwich_model).
"""
from __future__ import annotations

import json
import os

from . import parallel_model, sandwich_model

LOADERS = {
    parallel_model.ARCHITECTURE: parallel_model.load,
    sandwich_model.ARCHITECTURE: sandwich_model.load,
}


def architecture_of(config: dict) -> str:
    name = config.get("architecture")
    if name is None:
        name = (config.get("architectures") or [None])[0]
    if name is None:
        raise ValueError("config.json names no architecture")
    return name


def load_model(folder: str):
    """The checkpoint of a model folder (config.json + weights)."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    name = architecture_of(config)
    if name not in LOADERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(LOADERS))}")
    return LOADERS[name](folder, config)
