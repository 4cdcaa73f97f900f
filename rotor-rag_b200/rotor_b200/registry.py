"""Model registry: a model folder (config.json + model.safetensors) to a loaded model.

config.json names its design under ``architecture``; a configuration without that key is the HF-style one
of the ternary BitNet model.  A loader takes (folder, configuration dictionary, dtype, keyword arguments
of the model: max_seq, max_batch).
"""
from __future__ import annotations

import json
from pathlib import Path

from .semantics import BASELINE

_LOADERS = {}
DEFAULT = "BitNet"


class UnsupportedDtype(ValueError):
    """The design has no path in the number format asked for."""


def register(name):
    def add(loader):
        _LOADERS[name] = loader
        return loader
    return add


def architectures():
    return sorted(_LOADERS)


@register("BitNet")
def _bitnet(model_dir, config, dtype, semantics=None, **kw):
    from .bitnet_model import load_bitnet_model
    if dtype == "float32":
        raise UnsupportedDtype("the ternary model multiplies int8 activation terms; it has no float32 path")
    return load_bitnet_model(str(model_dir), semantics=semantics or BASELINE, **kw)


@register("Likerax")
def _likerax(model_dir, config, dtype, **kw):
    from .likerax import load_likerax_model
    return load_likerax_model(model_dir, config, dtype=dtype, **kw)


@register("Miborax")
def _miborax(model_dir, config, dtype, **kw):
    from .miborax import load_miborax_model
    return load_miborax_model(model_dir, config, dtype=dtype, **kw)


def load_model(model_dir, dtype: str = "bfloat16", **kw):
    model_dir = Path(model_dir)
    with open(model_dir / "config.json") as f:
        config = json.load(f)
    name = config.get("architecture", DEFAULT)
    if name not in _LOADERS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _LOADERS[name](model_dir, config, dtype, **kw)
