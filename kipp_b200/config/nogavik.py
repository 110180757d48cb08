"""Configuration of the Nogavik decoder, from its ``config.json`` keys.

The file is nested: ``layers`` lists the layers one by one (``type`` ``mamba2``,
``latent_attention`` or ``parallel``, the mixer's sizes and constants under
``mixer`` -- a parallel mixer's under ``left`` and ``right`` -- and the feed-forward
under ``mlp``: ``kind`` ``dense`` and ``ff``, or null), ``token_side.dim`` is the size
of every layer's own embedding of a token, ``norm.eps`` the eps of every norm, and
``vocab`` / ``width`` are the two global sizes.  A latent attention layer with
``kv_from`` reads the latent that an earlier one cached.  ``decay_rank`` and
``gate_rank`` of a parallel mixer's ``right`` (the widths of its two bottlenecks) are
needed only where weights are made from a seed.  The model class is named by the
key ``architecture``.  The checks are the host core's (csrc/host/nogavik.hpp);
this class keeps the keys as they are.
"""
from __future__ import annotations

import copy
import dataclasses
import json
from typing import Any

from .base import ConfigError, ModelConfig, architecture_name


@dataclasses.dataclass(frozen=True)
class NogavikConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm: dict = dataclasses.field(default_factory=dict)
    layers: tuple = ()
    token_side: dict | None = None

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "NogavikConfig":
        if not isinstance(data, dict):
            raise ConfigError("config.json must hold a JSON object")
        for key in ("vocab", "width", "norm", "layers"):
            if key not in data:
                raise ConfigError(f"config.json lacks required key {key!r}")
        if not isinstance(data["layers"], (list, tuple)):
            raise ConfigError("config key 'layers' must be a list of layers")
        config = cls(architecture=architecture_name(data), vocab=data["vocab"], width=data["width"],
                     norm=copy.deepcopy(data["norm"]), layers=tuple(copy.deepcopy(list(data["layers"]))),
                     token_side=copy.deepcopy(data.get("token_side")))
        config.validate()
        return config

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": copy.deepcopy(self.norm), "layers": copy.deepcopy(list(self.layers))}
        if self.token_side is not None:
            out["token_side"] = copy.deepcopy(self.token_side)
        return out

    # what code that sizes a run asks of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def initializer_range(self) -> float:
        return 0.02

    def normalized(self) -> dict:
        """The keys after the host core's checks and defaults."""
        from .. import native as N
        return json.loads(N.text_result(N.lib().kipp_config_normalize, json.dumps(self.to_dict()).encode()))

    def validate(self) -> None:
        self.normalized()
