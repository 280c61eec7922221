"""Host-side mirror of the reference's GPT-2 model API over the CUDA library.

Names, argument meaning and error behaviour follow puppygrad src/models/gpt2/rust.rs:
`Gpt2Config` (31-100), `Gpt2Model` (798-1027), `Gpt2KvCache` (178-249), `Gpt2Output` (150-175). The calls
that are the same for every model family are in decoder.py.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import numpy as np

from . import _native as N
from .decoder import _MATH, CudaConfig, DecoderCache, DecoderModel, ModelOutput, _fp  # noqa: F401  (_MATH: operator calls)
from .errors import Gpt2Error, check

Gpt2CudaConfig = CudaConfig
Gpt2Output = ModelOutput


@dataclass
class Gpt2Config:
    vocab_size: int
    n_positions: int
    n_embd: int
    n_layer: int
    n_head: int
    n_inner: int = 0
    layer_norm_epsilon: float = 1e-5

    def __post_init__(self):
        if not self.n_inner:
            self.n_inner = 4 * self.n_embd

    @classmethod
    def from_dict(cls, d: dict) -> "Gpt2Config":
        return cls(d["vocab_size"], d["n_positions"], d["n_embd"], d["n_layer"], d["n_head"],
                   d.get("n_inner") or 0, d.get("layer_norm_epsilon", 1e-5))

    @classmethod
    def from_json(cls, path: str) -> "Gpt2Config":
        """load_config, rust.rs:696-711"""
        c = N.PgConfig()
        check(N.lib.pg_config_load_json(str(path).encode(), C.byref(c)))
        return cls._from_native(c)

    @classmethod
    def _from_native(cls, c: N.PgConfig) -> "Gpt2Config":
        return cls(c.vocab_size, c.n_positions, c.n_embd, c.n_layer, c.n_head, c.n_inner, c.layer_norm_epsilon)

    def to_native(self) -> N.PgConfig:
        return N.PgConfig(self.vocab_size, self.n_positions, self.n_embd, self.n_layer, self.n_head,
                          self.n_inner, self.layer_norm_epsilon)

    def validate(self) -> None:
        c = self.to_native()
        check(N.lib.pg_config_validate(C.byref(c)))

    def head_dim(self) -> int:
        return self.n_embd // self.n_head


class Gpt2KvCache(DecoderCache):
    """Paged device-resident KV cache for `max_batch` independent sequences."""

    def read_layer(self, layer: int, slot: int = 0):
        """Keys and values in the reference layout [head][max_seq_len][head_dim]."""
        cfg = self.model.config
        n = cfg.n_positions * cfg.n_embd
        k = np.empty(n, np.float32)
        v = np.empty(n, np.float32)
        self._check(N.lib.pg_cache_read_layer(self._h, slot, layer, _fp(k), _fp(v)))
        shape = (cfg.n_head, cfg.n_positions, cfg.head_dim())
        return k.reshape(shape), v.reshape(shape)


class Gpt2Model(DecoderModel):
    cache_class = Gpt2KvCache

    def __init__(self, config, weights, cuda_config: Optional[Gpt2CudaConfig] = None):
        """Gpt2Model::new_with_rust_config (rust.rs:803-825). `weights` maps Hugging Face tensor
        names to float32 arrays (dense matrices `[in, out]`), or is the flat list in ABI order."""
        from .synthetic import tensor_names
        self.config = config if isinstance(config, Gpt2Config) else Gpt2Config.from_dict(config)
        self.cuda_config = cuda_config or Gpt2CudaConfig()
        if isinstance(weights, dict):
            names = tensor_names({"n_layer": self.config.n_layer})
            missing = [n for n in names if n not in weights]
            if missing:
                raise Gpt2Error("Asset", f"tensor {missing[0]} not found")
            weights = [weights[n] for n in names]
        tensors = [np.ascontiguousarray(t, np.float32).reshape(-1) for t in weights]
        n = len(tensors)
        ptrs = (C.POINTER(C.c_float) * n)(*[_fp(t) for t in tensors])
        lens = np.array([t.size for t in tensors], np.uint64)
        c, b = self.config.to_native(), self.cuda_config.to_native()
        self._h = C.c_void_p()
        check(N.lib.pg_model_from_host_weights(C.byref(c), ptrs, lens.ctypes.data_as(C.POINTER(C.c_uint64)), n,
                                               C.byref(b), C.byref(self._h)))

    @classmethod
    def from_dir(cls, model_dir: str, cuda_config: Optional[Gpt2CudaConfig] = None, use_tuning: bool = True,
                 tuning_file: Optional[str] = None) -> "Gpt2Model":
        """The model half of Gpt2Runtime::from_dir_with_backend (rust.rs:382-396). Without an explicit
        configuration the tuning file of the model directory is used when it exists (the reference's
        `puppygrad-tune.json` behaviour, main.rs:1333-1342, 2564-2585; `use_tuning=False` is its --no-tuning)."""
        self = cls.__new__(cls)
        if cuda_config is None and use_tuning:
            from .autotune import load_tuning
            cuda_config = load_tuning(str(model_dir), tuning_file)
        self.cuda_config = cuda_config or Gpt2CudaConfig()
        b = self.cuda_config.to_native()
        self._h = C.c_void_p()
        check(N.lib.pg_model_load_dir(str(model_dir).encode(), C.byref(b), C.byref(self._h)))
        c = N.PgConfig()
        check(N.lib.pg_model_config(self._h, C.byref(c)))
        self.config = Gpt2Config._from_native(c)
        return self
