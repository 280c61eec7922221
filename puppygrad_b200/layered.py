"""Models described layer by layer: what their classes share. The layers, their sizes and their constants come from
config.json; the weights from model.safetensors (BF16 or F32). The compute runs in the native library: `csrc/design.cpp`
reads the configuration, `csrc/layered.cu` runs the layers."""
from __future__ import annotations

import ctypes as C
import json
import os
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from . import _native as N
from .decoder import CudaConfig, DecoderModel
from .errors import DesignError


@dataclass
class LayeredConfig:
    """config.json, with the names the decoding calls use."""
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    layers: List[Dict[str, Any]] = field(default_factory=list)
    n_positions: int = 0  # the cache's limit: positions themselves have none
    embed_scale: Optional[float] = None  # designs that scale the token embedding

    @classmethod
    def from_dict(cls, d: Dict[str, Any], n_positions: int = 0) -> "LayeredConfig":
        scale = d["embedding"]["scale"] if "embedding" in d else None
        return cls(d["architecture"], d["vocab"], d["width"], d["norm"]["eps"], list(d["layers"]), n_positions, scale)

    def to_dict(self) -> Dict[str, Any]:
        out = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": self.layers}
        if self.embed_scale is not None:
            out["embedding"] = {"scale": self.embed_scale}
        return out

    @property
    def n_layer(self) -> int:
        return len(self.layers)


class LayeredModel(DecoderModel):
    architecture = ""
    error_class = DesignError

    @classmethod
    def default_cuda_config(cls) -> CudaConfig:
        return CudaConfig(math_mode="bf16")  # the weights are BF16 in the file

    @classmethod
    def from_dir(cls, model_dir: str, cuda_config: Optional[CudaConfig] = None, use_tuning: bool = True,
                 tuning_file: Optional[str] = None) -> "LayeredModel":
        """Loads a model directory (config.json, model.safetensors). Without an explicit configuration the tuning file of
        the directory is used when it exists, as for GPT-2."""
        self = cls.__new__(cls)
        if cuda_config is None and use_tuning:
            from .autotune import load_tuning
            cuda_config = load_tuning(str(model_dir), tuning_file)
        self.cuda_config = cuda_config or cls.default_cuda_config()
        b = self.cuda_config.to_native()
        self._h = C.c_void_p()
        self._check(N.lib.pg_model_load_dir(str(model_dir).encode(), C.byref(b), C.byref(self._h)))
        with open(os.path.join(str(model_dir), "config.json")) as f:
            self.config = LayeredConfig.from_dict(json.load(f), self.max_context_len())
        return self

    def state_bytes_per_sequence(self) -> int:
        return int(N.lib.pg_model_state_bytes_per_sequence(self._h))
