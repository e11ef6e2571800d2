"""Model registry: the architecture a checkpoint's config.json names -> a model class and its configuration.
Model modules register themselves; importing ``pace_b200.llm.models`` registers all of them."""
import os
from dataclasses import dataclass
from typing import Callable, Dict, List, Tuple

import torch

from pace_b200.llm.weights import read_config, read_safetensors


class UnsupportedDtype(ValueError):
    """The architecture has no kernels for the requested number format."""


@dataclass
class ModelEntry:
    make: Callable[[dict, torch.dtype], torch.nn.Module]   # (config.json, dtype) -> model with empty weights
    dtypes: Tuple[torch.dtype, ...]


class ModelRegistry:
    def __init__(self):
        self._entries: Dict[str, ModelEntry] = {}

    def register(self, architecture: str, make: Callable[[dict, torch.dtype], torch.nn.Module],
                 dtypes: Tuple[torch.dtype, ...] = (torch.bfloat16,)) -> None:
        if architecture in self._entries:
            raise AssertionError(f"duplicate registration of {architecture}")
        self._entries[architecture] = ModelEntry(make, dtypes)

    def architectures(self) -> List[str]:
        return sorted(self._entries)

    def find(self, config: dict) -> ModelEntry:
        """``architecture``, or the first known one of the ``architectures`` list other toolkits write."""
        names = [config["architecture"]] if "architecture" in config else list(config.get("architectures", []))
        for n in names:
            if n in self._entries:
                return self._entries[n]
        raise ValueError(f"no model for architecture {names}; known: {self.architectures()}")


model_registry = ModelRegistry()


def build_model(config: dict, dtype: torch.dtype = torch.bfloat16, device="cuda:0"):
    """An uninitialised model of the architecture ``config`` names."""
    import pace_b200.llm.models  # noqa: F401  (registration)
    entry = model_registry.find(config)
    if dtype not in entry.dtypes:
        raise UnsupportedDtype(f"this architecture runs in {[str(d) for d in entry.dtypes]}, not {dtype}")
    with torch.device(device):
        return entry.make(config, dtype).eval()


def load_model(folder: str, dtype: torch.dtype = torch.bfloat16, device="cuda:0"):
    """The model of a checkpoint folder (config.json + model.safetensors) with its weights on ``device``."""
    model = build_model(read_config(folder), dtype, device)
    model.load_weights(read_safetensors(os.path.join(folder, "model.safetensors")))
    return model
