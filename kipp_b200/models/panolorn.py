"""The Panolorn decoder: attention in blocks of positions with unit-norm queries
and keys, a distance term per head in place of a rotation, capped scores, a sink
of score 0 and a gate per element, beside feed-forwards that are dense (gelu) or
experts chosen by sigmoid scores which weigh the experts' inputs, with a norm on
either side of every sublayer.  Its configuration checks and its plan are the
host core's (csrc/host/panolorn.hpp); this module registers the configuration
class on the Python side.
"""
from __future__ import annotations

from ..config.panolorn import PanolornConfig
from ..config.registry import register_architecture
from .spec import ModelSpec


def build_panolorn(config: PanolornConfig) -> ModelSpec:
    return ModelSpec.from_library(config)


register_architecture("Panolorn", PanolornConfig, build_panolorn)
