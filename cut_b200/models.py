"""The model registry: which class serves a model, chosen by the model's own files.

A folder with config.json and model.safetensors is looked up by the configuration's "architecture"; a .gguf file by its
general.architecture key (the C++ runner reads it).  A new design adds an entry."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from . import bigerax, lenesun
from .layer_list import LayerListDecoder
from .safetensors_io import SafetensorsFile


@dataclass(frozen=True)
class ModelEntry:
    parse_config: Callable      # dict of config.json -> configuration
    gather_weights: Callable    # (configuration, get, has) -> weights of `decoder`
    decoder: type               # constructed as decoder(configuration, weights, device=, dtype=, max_seq=, ...)
    dtypes: tuple


REGISTRY = {
    bigerax.ARCHITECTURE: ModelEntry(bigerax.parse_config, bigerax.gather_weights, LayerListDecoder, ("bfloat16", "float32")),
    lenesun.ARCHITECTURE: ModelEntry(lenesun.parse_config, lenesun.gather_weights, LayerListDecoder, ("bfloat16", "float32")),
}


def read_config(folder: str):
    """(registry entry, parsed configuration) of a model folder."""
    with open(os.path.join(folder, "config.json")) as f:
        raw = json.load(f)
    arch = raw.get("architecture")
    if arch not in REGISTRY:
        raise ValueError(f"{folder}: unknown architecture {arch!r} (known: {', '.join(sorted(REGISTRY))})")
    entry = REGISTRY[arch]
    return entry, entry.parse_config(raw)


def load_model(folder: str, dtype: str = "bfloat16", **options):
    """Reads a model folder and puts the model on the device; options go to the decoder (max_seq, max_portion, slots, device)."""
    entry, cfg = read_config(folder)
    if dtype not in entry.dtypes:
        raise ValueError(f"{dtype} is not among this model's element types {entry.dtypes}")
    f = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    return entry.decoder(cfg, entry.gather_weights(cfg, f.get, f.__contains__), dtype=dtype, **options)
