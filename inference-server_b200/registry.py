"""Which engine serves a model: by the `architecture` of its config.json, or by the name of a built-in shape.

A family is (its built-in shapes, an engine from one of them, an engine from a model folder, the part of the kernel
library it needs).  Folders without an `architecture` key are transformers checkpoints (Qwen3-MoE), read by
`B200Backend._read_checkpoint`.
"""
from __future__ import annotations

import os
from dataclasses import dataclass
from typing import Callable

from . import checkpoint


@dataclass(frozen=True)
class Family:
    kernels: str | None                  # build.SUBSETS entry that is enough for it; None = the full library
    shapes: Callable[[], dict]           # built-in shapes by name
    from_shape: Callable                 # (shape, **engine arguments) -> engine
    from_folder: Callable | None = None  # (folder, config, **engine arguments) -> engine


def _layered_from_folder(folder: str, config: dict, **kw):
    from . import layered
    return layered.LayeredEngine(layered.LayeredConfig.from_json(config),
                                 tensors=checkpoint.read_safetensors(os.path.join(folder, "model.safetensors")), **kw)


def _layered_shapes():
    from . import layered
    return {k: c for k, c in layered.CONFIGS.items() if not c.gated}


def _gated_shapes():
    from . import layered
    return {k: c for k, c in layered.CONFIGS.items() if c.gated}


def _layered_from_shape(cfg, **kw):
    from . import layered
    return layered.LayeredEngine(cfg, **kw)


def _qwen_shapes():
    from . import engine
    return engine.CONFIGS


def _qwen_from_shape(cfg, **kw):
    from . import engine
    return engine.DecodeEngine(cfg, **kw)


QWEN3_MOE = Family(None, _qwen_shapes, _qwen_from_shape)
LAYERED = Family("layered", _layered_shapes, _layered_from_shape, _layered_from_folder)
GATED = Family("gated", _gated_shapes, _layered_from_shape, _layered_from_folder)

# config.json `architecture` -> family
ARCHITECTURES: dict[str, Family] = {"Sulepel": LAYERED, "Sefalorn": GATED}


def shape_family(name: str) -> tuple[Family, object] | None:
    """(family, shape) of a built-in shape name."""
    for family in (QWEN3_MOE, LAYERED, GATED):
        shapes = family.shapes()
        if name in shapes:
            return family, shapes[name]
    return None


def folder_family(folder: str) -> tuple[Family, dict] | None:
    """(family, config) of a model folder that names an architecture of ours; None for any other folder or name."""
    if not os.path.isfile(os.path.join(folder, "config.json")):
        return None
    config = checkpoint.read_config(folder)
    arch = config.get("architecture")
    if arch is None:
        return None
    if arch not in ARCHITECTURES:
        raise ValueError(f"{folder}: architecture {arch!r} is not one of {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[arch], config
