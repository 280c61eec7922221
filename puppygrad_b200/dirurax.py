"""Dirurax: a decoder whose layers mix tokens by gated linear attention ("gla") or by chunked attention beside a
generalized delta rule ("parallel"), each layer with an optional dense feed-forward."""
from __future__ import annotations

from .layered import LayeredConfig, LayeredModel

DiruraxConfig = LayeredConfig


class DiruraxModel(LayeredModel):
    architecture = "Dirurax"
