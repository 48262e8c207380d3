"""Models the framework serves, by the architecture name of their config.json: how a configuration is
read, how its tensors are named and which engine runs it."""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable, Dict, Tuple

import torch

from .safetensors_io import load_safetensors

Weights = Dict[str, torch.Tensor]


@dataclass(frozen=True)
class ModelEntry:
    architecture: str
    read_config: Callable[[dict], Any]
    read_weights: Callable[[Any, Weights], Weights]  # stored names -> the engine's names
    engine: Callable[..., Any]  # (config, weights, *, batch, capacity) -> engine
    dtypes: Tuple[torch.dtype, ...] = (torch.float32, torch.bfloat16)
    portions: bool = False  # whether the engine has the open / forward / close step interface


_ENTRIES: Dict[str, ModelEntry] = {}


def register(entry: ModelEntry) -> None:
    _ENTRIES[entry.architecture] = entry


def architectures() -> Tuple[str, ...]:
    return tuple(sorted(_ENTRIES))


def entry_of(config: dict) -> ModelEntry:
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    try:
        return _ENTRIES[name]
    except KeyError:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(architectures())}") from None


def load_model(folder: str | Path, *, dtype: torch.dtype = torch.bfloat16, batch: int = 1, capacity: int = 4096,
               device: str | torch.device = "cuda"):
    """The engine of the model in `folder` (config.json and model.safetensors)."""

    folder = Path(folder)
    raw = json.loads((folder / "config.json").read_text())
    entry = entry_of(raw)
    if dtype not in entry.dtypes:
        raise ValueError(f"{entry.architecture} does not run in {dtype}")
    config = entry.read_config(raw)
    stored = entry.read_weights(config, load_safetensors(folder / "model.safetensors"))
    weights = {name: (tensor.to(device=device, dtype=dtype) if tensor.is_floating_point() else tensor.to(device))
               for name, tensor in stored.items()}
    return entry.engine(config, weights, batch=batch, capacity=capacity)


def _register_builtin() -> None:
    from . import bazirax, lozanex, qwen2
    from .engine import Qwen2Engine
    from .hybrid_engine import HybridEngine

    register(ModelEntry(bazirax.ARCHITECTURE, bazirax.BaziraxConfig.from_dict, lambda config, stored: stored,
                        HybridEngine, portions=True))
    register(ModelEntry(lozanex.ARCHITECTURE, lozanex.LozanexConfig.from_dict, lambda config, stored: stored,
                        HybridEngine, portions=True))
    register(ModelEntry("Qwen2ForCausalLM", qwen2.config_from_dict, qwen2.weights_from_checkpoint, Qwen2Engine,
                        dtypes=(torch.float32, torch.bfloat16, torch.float16)))


_register_builtin()
