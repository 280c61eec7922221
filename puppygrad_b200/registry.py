"""Model registry: which class serves a model directory, by the "architecture" entry of its config.json (GPT-2
configurations have none)."""
from __future__ import annotations

import json
import os
from typing import Dict, Optional, Type

from .decoder import CudaConfig, DecoderModel
from .dirurax import DiruraxModel
from .errors import DesignError
from .gpt2 import Gpt2Model
from .sanesun import SanesunModel

MODELS: Dict[str, Type[DecoderModel]] = {"gpt2": Gpt2Model, **{m.architecture: m for m in (DiruraxModel, SanesunModel)}}


def architecture_of(model_dir: str) -> str:
    path = os.path.join(str(model_dir), "config.json")
    try:
        with open(path) as f:
            name = json.load(f).get("architecture")
    except (OSError, ValueError, AttributeError) as err:
        raise DesignError("Asset", f"failed to read config file {path}: {err}") from err
    return name if isinstance(name, str) else "gpt2"


def model_class(architecture: str) -> Type[DecoderModel]:
    if architecture not in MODELS:
        raise DesignError("InvalidConfig", f"unknown architecture {architecture!r} (known: {', '.join(MODELS)})")
    return MODELS[architecture]


def load_model(model_dir: str, cuda_config: Optional[CudaConfig] = None, use_tuning: bool = True,
               tuning_file: Optional[str] = None) -> DecoderModel:
    """Loads a model directory with the class its configuration names."""
    return model_class(architecture_of(model_dir)).from_dir(model_dir, cuda_config, use_tuning=use_tuning,
                                                             tuning_file=tuning_file)
