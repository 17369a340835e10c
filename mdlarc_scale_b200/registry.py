"""Model families by the ``architecture`` name of their ``config.json``, and loading of model folders.

A family is a function ``build(config, tensors, device, act_format, **options) -> EngineBase``.
``act_format`` is the operand format of the matrix products: ``"f16"`` (the default: bf16-rounded weights
in an IEEE-half container), ``"bf16"`` or, where the family has it, ``"f32"``.
"""
from __future__ import annotations

from typing import Callable

from .engine import Engine, EngineBase
from .weights import read_model_folder

_FAMILIES: dict[str, Callable[..., EngineBase]] = {}

# numeric formats a caller asks for by name -> act_format
DTYPES = {"bfloat16": "f16", "bfloat16-operands": "bf16", "float32": "f32"}


def register(architecture: str):
    def add(build):
        if architecture in _FAMILIES:
            raise ValueError(f"architecture {architecture!r} is registered twice")
        _FAMILIES[architecture] = build
        return build
    return add


def architectures() -> list[str]:
    _import_families()
    return sorted(_FAMILIES)


def _import_families() -> None:
    from . import logesun, vodavik  # noqa: F401  (they register themselves)


def collect_tensors(names: dict, tensors: dict) -> dict:
    """Checkpoint tensors by (kind, layer); a list of names gives the list of their tensors."""
    flat = [n for v in names.values() for n in (v if isinstance(v, list) else [v])]
    missing = sorted(n for n in flat if n not in tensors)
    if missing:
        raise ValueError(f"the checkpoint lacks {', '.join(missing[:5])}{' ...' if len(missing) > 5 else ''}")
    return {key: [tensors[n] for n in v] if isinstance(v, list) else tensors[v] for key, v in names.items()}


def build_engine(config: dict, tensors: dict, device="cuda:0", act_format: str = "f16", **options) -> EngineBase:
    _import_families()
    name = config.get("architecture")
    if name not in _FAMILIES:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _FAMILIES[name](config, tensors, device, act_format, **options)


def load_model(folder, device="cuda:0", dtype: str = "bfloat16", **options) -> EngineBase:
    """Engine for a folder with ``config.json`` and ``model.safetensors``."""
    if dtype not in DTYPES:
        raise ValueError(f"unknown dtype {dtype!r}; known: {', '.join(DTYPES)}")
    config, tensors = read_model_folder(folder)
    return build_engine(config, tensors, device, DTYPES[dtype], **options)


@register("TinyTransformer")
def _tiny(config, tensors, device, act_format, **options):
    """``config`` holds the fields of TransformerConfig (src/transformer.py:15-34), ``tensors`` its state dict."""
    if act_format == "f32":
        raise NotImplementedError("TinyTransformer has no 32-bit path")
    return Engine(tensors, config, device, act_format=act_format, **options)
