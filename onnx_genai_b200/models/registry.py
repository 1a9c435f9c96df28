"""Model families: which executor, weights and caches a configuration gets, and which checkpoint directories are read natively.

A decoder lowered from an ONNX package has a :class:`~.config.DecoderConfig`.  A checkpoint directory whose ``config.json``
names an architecture registered here is read without a graph: its configuration selects the family.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from . import decoder, dezudra, fizesun, hybrid, midisun, rilelorn
from .config import DecoderConfig


@dataclass(frozen=True)
class Family:
    config: type                 # configurations of this class belong to the family
    model: type                  # executor: (cfg, weights, device, max_tokens, max_rows, tp, rank, comm)
    random_weights: Callable     # (cfg, device, tp, rank, seed, dtype)
    compute_dtypes: tuple        # what EngineConfig.compute_dtype may be on a GPU


@dataclass(frozen=True)
class Architecture:
    name: str                    # config.json "architecture"
    read_config: Callable        # (document, name) -> configuration
    load_weights: Callable       # (configuration, tensors, dtype, device) -> weights
    kernels: str | None = None   # kernel subset the architecture needs (build.SUBSETS)


FAMILIES = (
    Family(DecoderConfig, decoder.DecoderModel, lambda cfg, device, tp, rank, seed, dtype: decoder.random_weights(cfg, device, tp, rank, seed=seed, dtype=dtype),
           ("bf16",)),
    Family(hybrid.HybridConfig, hybrid.HybridModel, lambda cfg, device, tp, rank, seed, dtype: hybrid.random_weights(cfg, device, seed=seed, dtype=dtype),
           ("bf16", "f32")),
)
ARCHITECTURES = {a.name: a for a in (Architecture("Rilelorn", rilelorn.read_config, rilelorn.load_weights, "hybrid"),
                                     Architecture("Dezudra", dezudra.read_config, dezudra.load_weights, "delta"),
                                     Architecture("Fizesun", fizesun.read_config, fizesun.load_weights, "latent_moe"),
                                     Architecture("Midisun", midisun.read_config, midisun.load_weights, "memory"))}


def family_of(cfg) -> Family:
    for f in FAMILIES:
        if isinstance(cfg, f.config):
            return f
    raise TypeError(f"no model family takes a {type(cfg).__name__}")


def native_config(path: str) -> dict | None:
    """The ``config.json`` of a checkpoint directory with a registered architecture, else None."""
    p = os.path.join(path, "config.json")
    if not os.path.exists(p) or not os.path.exists(os.path.join(path, "model.safetensors")):
        return None
    try:
        with open(p, encoding="utf-8") as f:
            doc = json.load(f)
    except ValueError:
        return None
    return doc if isinstance(doc, dict) and doc.get("architecture") in ARCHITECTURES else None


def load_checkpoint(path: str, doc: dict, dtype, device):
    """(configuration, weights) of a native checkpoint directory."""
    from ..package.safetensors import SafetensorsFile

    arch = ARCHITECTURES[doc["architecture"]]
    cfg = arch.read_config(doc, os.path.basename(os.path.abspath(path)) or arch.name)
    return cfg, arch.load_weights(cfg, SafetensorsFile(os.path.join(path, "model.safetensors")), dtype, device)
