"""Which model class, engine and kernels a ``config.json`` asks for.

    entry = find_model(config)             # by "architecture", or the first of "architectures"
    model = load_model(folder, dtype)      # weights and configuration from the folder, kernels built if need be
    engine = new_engine(model, num_blocks=..., max_num_seqs=..., ...)
"""
from __future__ import annotations

from dataclasses import dataclass
from importlib import import_module

import torch

from . import _lib
from .build import build_components
from .checkpoint import load_config, load_weights


@dataclass(frozen=True)
class ModelEntry:
    module: str
    config: str
    model: str
    engine: str
    components: tuple[str, ...]
    dtypes: tuple[torch.dtype, ...]

    def resolve(self, name: str):
        return getattr(import_module(f".{self.module}", __package__), name)


MODELS: dict[str, ModelEntry] = {
    "Gotunex": ModelEntry("modeling_gotunex", "GotunexConfig", "GotunexModel", "PagedDecodeEngine", ("latent",),
                          (torch.float32, torch.bfloat16)),
    "Manirax": ModelEntry("modeling_manirax", "ManiraxConfig", "ManiraxModel", "PagedDecodeEngine", ("dense",),
                          (torch.float32, torch.bfloat16)),
    "SpikingQwen": ModelEntry("modeling", "SpikingQwenConfig", "SpikingQwenModel", "SpikeDecodeEngine", ("spike",),
                              (torch.float32, torch.bfloat16, torch.float16)),
}
# the class name the reference writes into its model folders (spikeinfer/modeling_fast.py)
ALIASES = {"FastSpikingQwenForCausalLM": "SpikingQwen"}


def find_model(config: dict) -> ModelEntry:
    name = config.get("architecture") or next(iter(config.get("architectures") or []), None)
    entry = MODELS.get(ALIASES.get(name, name))
    if entry is None:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(MODELS))})")
    return entry


def load_model(folder, dtype: torch.dtype | None = None, device: str | torch.device = "cuda"):
    """The model of a folder on ``device``; ``dtype`` None keeps the dtype of the stored weights."""
    raw = load_config(folder)
    entry = find_model(raw)
    if dtype is not None and dtype not in entry.dtypes:
        raise ValueError(f"{entry.model} does not run in {dtype}")
    _lib.use_library(build_components(entry.components))
    config = entry.resolve(entry.config).from_dict(raw)
    return entry.resolve(entry.model)(config, load_weights(folder), device=device, dtype=dtype)


def new_engine(model, **kwargs):
    """The engine that serves ``model``."""
    from .engine import decode_engine

    for entry in MODELS.values():
        if type(model).__name__ == entry.model:
            return getattr(decode_engine, entry.engine)(model, **kwargs)
    raise ValueError(f"no engine for {type(model).__name__}")
