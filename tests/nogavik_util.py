"""Small Nogavik configurations for the tests (sizes of their own, each unlike the
others in head counts, head sizes, ranks, taps, layer order and what is left out)
and helpers to write them as model folders with random weights."""
from __future__ import annotations

import functools
import os
import tempfile

import torch

from zunilorn_util import random_tokens, set_tensors  # noqa: F401  (the same helpers)


def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def mamba_layer(heads, groups, vdim, state, conv, norm_groups, mlp) -> dict:
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "groups": groups, "vdim": vdim, "state": state, "conv": conv, "norm_groups": norm_groups}}


def latent_layer(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, mlp, base=10000.0, kv_from=None) -> dict:
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale}
    if rot_dim:
        m["rot"] = {"base": base, "dims": rot_dim}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel_layer(left, right, mlp) -> dict:
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def left(heads, kv_heads, dim, vdim, scale) -> dict:
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}


def right(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank) -> dict:
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": decay_rank, "gate_rank": gate_rank}


CONFIGS = {
    # every kind of layer; one without a feed-forward; a latent read by two later layers with other
    # heads and ranks of their own; groups of heads in both halves of the parallel mixer; values wider than
    # keys on one side and narrower on the other
    "A": {"architecture": "Nogavik", "vocab": 300, "width": 64, "norm": {"eps": 1e-5}, "token_side": {"dim": 12},
          "layers": [latent_layer(4, 16, 8, 24, 32, 40, 0.25, dense(96)),
                     parallel_layer(left(4, 2, 16, 24, 0.3), right(4, 2, 16, 8, 3, 12, 20), dense(80)),
                     latent_layer(2, 24, 8, 16, 32, 16, 0.2, None, kv_from=0),
                     mamba_layer(4, 2, 16, 24, 3, 2, dense(64)),
                     latent_layer(3, 8, 8, 8, 32, 24, 0.35, dense(48), kv_from=0)]},
    # as many key heads as heads, one tap (no convolution to carry), a rotation with another base, two lenders
    # in turn, a token side as wide as the model's narrowest part, no feed-forward in the first layer
    "B": {"architecture": "Nogavik", "vocab": 257, "width": 96, "norm": {"eps": 3e-6}, "token_side": {"dim": 8},
          "layers": [mamba_layer(3, 3, 32, 8, 2, 1, None),
                     latent_layer(2, 16, 16, 32, 48, 24, 0.3, dense(40), base=77.0),
                     latent_layer(6, 32, 16, 16, 48, 32, 0.2, dense(64), base=500.0),
                     latent_layer(2, 16, 16, 32, 48, 24, 0.3, dense(40), base=77.0, kv_from=1),
                     parallel_layer(left(3, 3, 32, 16, 0.25), right(2, 2, 8, 24, 1, 8, 8), dense(72)),
                     latent_layer(4, 8, 16, 8, 48, 16, 0.4, None, base=500.0, kv_from=2)]},
    # head sizes the tensor-core kernels take: values of 192 and of 256, a state of 128 rows, states of 64 x 64
    # and 96 x 32, a latent of 128
    "C": {"architecture": "Nogavik", "vocab": 512, "width": 128, "norm": {"eps": 1e-6}, "token_side": {"dim": 32},
          "layers": [parallel_layer(left(4, 2, 96, 192, 0.1), right(4, 1, 64, 64, 4, 16, 32), dense(256)),
                     latent_layer(8, 64, 32, 48, 128, 96, 0.1, dense(384)),
                     mamba_layer(4, 1, 32, 128, 4, 4, dense(192)),
                     parallel_layer(left(2, 1, 64, 256, 0.12), right(2, 2, 96, 32, 2, 24, 8), None)]},
    # sizes that fit no vector width: an odd vocabulary, a width that is no multiple of 8, heads of 6 and 5, a
    # latent of 11 and a rotated part of 2, five taps, bottlenecks of 3 and 5, a token side of 7
    "D": {"architecture": "Nogavik", "vocab": 101, "width": 100, "norm": {"eps": 2e-5}, "token_side": {"dim": 7},
          "layers": [parallel_layer(left(3, 1, 6, 5, 0.7), right(3, 3, 5, 7, 5, 3, 5), dense(11)),
                     mamba_layer(2, 2, 9, 3, 1, 2, dense(13)),
                     latent_layer(3, 5, 2, 7, 11, 9, 0.6, dense(9), base=100.0),
                     latent_layer(1, 3, 2, 5, 11, 6, 0.9, None, base=100.0, kv_from=2)]},
    # no token side and no rotation: what a design beside this one may leave out
    "E": {"architecture": "Nogavik", "vocab": 120, "width": 48, "norm": {"eps": 1e-5},
          "layers": [latent_layer(2, 16, 0, 16, 24, 16, 0.4, dense(40)),
                     parallel_layer(left(2, 1, 8, 8, 0.5), right(2, 1, 8, 8, 4, 4, 4), None)]},
}
INIT = {"A": dict(seed=3, sigma=0.15, norm_jitter=0.2), "B": dict(seed=5, sigma=0.12, norm_jitter=0.1),
        "C": dict(seed=9, sigma=0.08, norm_jitter=0.15), "D": dict(seed=12, sigma=0.2, norm_jitter=0.1),
        "E": dict(seed=15, sigma=0.2, norm_jitter=0.1)}

_tmp = tempfile.TemporaryDirectory(prefix="kipp_b200_nogavik_")


def write_folder(folder: str, cfg: dict, init: dict, dtype=torch.bfloat16) -> str:
    """Weights are stored in bfloat16, as this design's checkpoints are: both engines and the plain model start
    from the same numbers."""
    from kipp_b200.config import config_from_dict
    from kipp_b200.weights import write_random_model
    return write_random_model(folder, config_from_dict(cfg), init["seed"], sigma=init["sigma"],
                              norm_jitter=init["norm_jitter"], dtype=dtype)


@functools.lru_cache(maxsize=None)
def model_folder(name: str) -> str:
    return write_folder(os.path.join(_tmp.name, name), CONFIGS[name], INIT[name])
