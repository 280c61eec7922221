"""The reference's error type for this path (puppygrad src/models/gpt2/error.rs:4-25)."""
from __future__ import annotations

from . import _native as N


class Gpt2Error(Exception):
    """One of Asset / InvalidConfig / InvalidInput / InvalidWeights, plus Cuda and Timeout, which
    only this backend can raise. `str()` gives the same text as the reference's Display impl."""

    KINDS = {N.PG_ASSET: "Asset", N.PG_INVALID_CONFIG: "InvalidConfig", N.PG_INVALID_INPUT: "InvalidInput",
             N.PG_INVALID_WEIGHTS: "InvalidWeights", N.PG_CUDA: "Cuda", N.PG_TIMEOUT: "Timeout"}
    _PREFIX = {"Asset": "GPT-2 asset error: ", "InvalidConfig": "invalid GPT-2 config: ",
               "InvalidInput": "invalid GPT-2 input: ", "InvalidWeights": "invalid GPT-2 weights: ",
               "Cuda": "GPT-2 CUDA error: ", "Timeout": "GPT-2 device timeout: "}

    def __init__(self, kind: str, message: str):
        super().__init__(self.prefix(kind) + message)
        self.kind = kind
        self.message = message


    @classmethod
    def prefix(cls, kind: str) -> str:
        return cls._PREFIX.get(kind, "")


class DesignError(Gpt2Error):
    """The same for models of other designs than GPT-2."""

    @classmethod
    def prefix(cls, kind: str) -> str:
        return Gpt2Error._PREFIX.get(kind, "").replace("GPT-2", "model").replace("model asset", "asset")


def check(status: int, error=Gpt2Error) -> None:
    if status != N.PG_OK:
        raise error(Gpt2Error.KINDS.get(status, "Cuda"), N.lib.pg_last_error_message().decode())
