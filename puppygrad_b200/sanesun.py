"""Sanesun: a decoder whose layers mix tokens by rotated attention in a window that keeps the first tokens, with mixed heads and
a sink ("attention"), by a delta rule with a decay per key channel ("channel_delta"), or by attention over one latent row
per token ("latent_attention"); each layer has an optional feed-forward beside the mixer, reading the same normed input."""
from __future__ import annotations

from .layered import LayeredConfig, LayeredModel

SanesunConfig = LayeredConfig


class SanesunModel(LayeredModel):
    architecture = "Sanesun"
