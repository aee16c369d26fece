"""Which class serves a model folder: `config.json` names the architecture, the registry maps it to a model class.

A registered class offers `from_dir(directory, device, dtype, max_tokens, max_sequences)` and the serving interface the
engine drives: `table` (a `SequenceTable`), `max_portion` (most tokens of one sequence in a step), `vocab` and
`forward(entries, want) -> f32 logits`."""
from __future__ import annotations

import importlib
import json
import os

# architecture name in config.json -> module, class (imported on use)
ARCHITECTURES = {
    "Vumipel": ("scratchy_b200.vumipel", "Vumipel"),
    "Vekurax": ("scratchy_b200.vekurax", "Vekurax"),
    "LlamaForCausalLM": ("scratchy_b200.llama_serving", "LlamaServing"),
}


def read_config(directory: str) -> dict:
    path = os.path.join(directory, "config.json")
    with open(path) as f:
        return json.load(f)


def architecture_of(config: dict) -> str:
    """The name under `architecture`, or the first of `architectures`."""
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ValueError(f"architecture {name!r} is not one of {sorted(ARCHITECTURES)}")
    return name


def model_class(config: dict):
    module, cls = ARCHITECTURES[architecture_of(config)]
    return getattr(importlib.import_module(module), cls)


def prepare_library(directory: str) -> None:
    """Compiles, where needed, the kernels that the model in `directory` runs on (for programs of a source checkout)."""
    from . import _lib
    from .build import DESIGNS
    name = architecture_of(read_config(directory))
    if name in DESIGNS:
        _lib.models_lib(build_for=name)
    else:
        from .build import LIB, build_library
        build_library(LIB)


def load_model(directory: str, device="cuda", dtype: str = "bfloat16", max_tokens: int = 8192, max_sequences: int = 8):
    """The model in `directory`, ready to serve.  `max_tokens`: the most tokens that live sequences hold together."""
    return model_class(read_config(directory)).from_dir(directory, device, dtype, max_tokens=max_tokens, max_sequences=max_sequences)
