"""The Nogavik decoder: layers of three kinds (the selective state space layer in its
matrix-state form; attention over a cached latent with a gate per element, some
layers reading another one's latent; grouped-query attention without positions
beside the gated delta rule, each normed over the width), a feed-forward that
reads a norm of its own of the same stream, and an embedding of the token per
layer that joins the stream behind them.  Its configuration checks and its plan
are the host core's (csrc/host/nogavik.hpp); this module registers the
configuration class on the Python side.
"""
from __future__ import annotations

from ..config.nogavik import NogavikConfig
from ..config.registry import register_architecture
from .spec import ModelSpec


def build_nogavik(config: NogavikConfig) -> ModelSpec:
    return ModelSpec.from_library(config)


register_architecture("Nogavik", NogavikConfig, build_nogavik)
