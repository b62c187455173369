"""Which model class runs a checkpoint directory: decided by its ``config.json``
(``Architecture::detect``, crates/orion-models/src/config.rs:106-131, for the Hugging Face layouts)."""
from __future__ import annotations

import json
import os

from .backend import CudaBackend
from .errors import ModelError
from .layered import READERS, CudaLayeredModel
from .model import CudaModel, CudaTransformerModel

#: config.json "architecture" -> model class; configs without that key are Hugging Face ones
ARCHITECTURES = {name: CudaLayeredModel for name in READERS}


def model_class(directory: str):
    path = os.path.join(directory, "config.json")
    try:
        with open(path) as f:
            config = json.load(f)
    except OSError as e:
        raise ModelError(f"{path}: {e}") from e
    except ValueError as e:
        raise ModelError(f"config.json is malformed: {e}") from e
    name = config.get("architecture")
    if name is None:
        return CudaTransformerModel
    if name not in ARCHITECTURES:
        raise ModelError(f"unsupported architecture {name}")
    return ARCHITECTURES[name]


def load_model(directory: str, num_blocks: int, block_size: int, backend: CudaBackend, **kw) -> CudaModel:
    """``from_directory`` of the class that ``config.json`` asks for. ``num_state_slots`` is passed on to models
    that carry state and dropped for the others."""
    cls = model_class(directory)
    if cls is CudaTransformerModel:
        kw.pop("num_state_slots", None)
    return cls.from_directory(directory, num_blocks, block_size, backend, **kw)
