"""Which configuration reader and which model class a checkpoint or preset takes.

A ``config.json`` with an "architecture" key names its design directly; everything else is read as a Hugging Face
config of the Llama / Qwen families (``ModelConfig``)."""
from __future__ import annotations

import dataclasses
import json
import os
from dataclasses import dataclass
from typing import Callable


@dataclass(frozen=True)
class Architecture:
    read_config: Callable                 # parsed config.json -> configuration object
    model: Callable                       # () -> model class
    trainable: bool = True                # False: forward / serving only (no backward kernels)
    fp32_on_gpu: bool = False             # the kernels also run with float32 weights and activations
    component: str | None = None          # part of the kernel library that serving it takes (None: all of it)


def _transformer():
    from .transformer import TransformerLM

    return TransformerLM


def _hybrid():
    from .hybrid import HybridLM

    return HybridLM


def _read_hf(d: dict):
    from .config import ModelConfig

    return ModelConfig.from_hf_dict(d)


def _read_hybrid(d: dict):
    from .hybrid_config import HybridConfig

    return HybridConfig.from_dict(d)


HF = Architecture(_read_hf, _transformer)
ARCHITECTURES: dict[str, Architecture] = {
    "Sigisun": Architecture(_read_hybrid, _hybrid, trainable=False, fp32_on_gpu=True, component="serve_hybrid"),
}
_MODEL_TYPES = {"sigisun": "Sigisun"}


def architecture_of(cfg_or_dict) -> Architecture:
    """Entry of a configuration object or of a parsed config.json."""
    if isinstance(cfg_or_dict, dict):
        name = cfg_or_dict.get("architecture")
        if name is not None and name not in ARCHITECTURES:
            raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)} and HF configs")
        return ARCHITECTURES.get(name, HF)
    return ARCHITECTURES.get(_MODEL_TYPES.get(cfg_or_dict.model_type), HF)


def read_config(path_or_preset: str):
    from .config import PRESETS

    if path_or_preset in PRESETS:
        return dataclasses.replace(PRESETS[path_or_preset])
    with open(os.path.join(path_or_preset, "config.json")) as f:
        d = json.load(f)
    return architecture_of(d).read_config(d)


def build_model(cfg, **kw):
    """Instantiate the model class of a configuration (``TransformerLM`` arguments)."""
    return architecture_of(cfg).model()(cfg, **kw)


def require_trainable(cfg) -> None:
    if not architecture_of(cfg).trainable:
        raise NotImplementedError(f"{cfg.model_type} models are served only: this framework has no backward kernels "
                                  "for their mixers")
