"""Small Panolorn configurations for the tests (sizes of their own, each unlike the
others in head counts, head sizes, block sizes, caps, experts and layer order) and
helpers to write them as model folders with random weights."""
from __future__ import annotations

import functools
import os
import tempfile

import torch


def moe(experts, top, ff, shared=None) -> dict:
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def dense(ff) -> dict:
    return {"kind": "dense", "ff": ff}


def attention_layer(heads, kv_heads, dim, vdim, mlp, scale, softcap=None, block=None) -> dict:
    m = {"heads": heads, "dim": dim, "scale": scale}
    if kv_heads is not None:
        m["kv_heads"] = kv_heads
    if vdim is not None:
        m["vdim"] = vdim
    if softcap is not None:
        m["softcap"] = softcap
    if block is not None:
        m["mask"] = {"size": block}
    return {"type": "attention", "mixer": m, "mlp": mlp}


CONFIGS = {
    # blocks of two sizes that are no multiple of a page, value heads wider and narrower than key heads, two
    # and three experts per token, a layer without a feed-forward
    "A": {"architecture": "Panolorn", "vocab": 300, "width": 64, "norm": {"eps": 1e-5}, "embedding": {"scale": 3.0},
          "layers": [attention_layer(4, 2, 16, 24, dense(96), 0.5, 6.0, 37),
                     attention_layer(6, 2, 16, 16, moe(5, 2, 40, 48), 0.4, 10.0, 21),
                     attention_layer(2, 1, 32, 16, None, 0.3, 20.0, 37),
                     attention_layer(4, 4, 16, 32, moe(7, 3, 24), 0.25, 4.0, 50)]},
    # what may be left out: no mask, no cap, no scale of the embedding, as many key heads as heads, values of
    # the keys' size, no shared expert; a router that takes every expert
    "B": {"architecture": "Panolorn", "vocab": 257, "width": 96, "norm": {"eps": 3e-6},
          "layers": [attention_layer(3, None, 16, None, moe(2, 2, 32), 0.3),
                     attention_layer(6, 2, 32, 16, dense(64), 0.2, None, 64),
                     attention_layer(5, 1, 16, 48, moe(1, 1, 24, 16), 0.6, 3.0)]},
    # head sizes of 64 and 128, blocks of one page and of several key tiles, sixteen experts
    "C": {"architecture": "Panolorn", "vocab": 512, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 11.3},
          "layers": [attention_layer(4, 2, 64, 128, moe(16, 4, 64, 128), 0.125, 50.0, 128),
                     attention_layer(8, 2, 128, 64, dense(256), 0.05, 15.0, 16),
                     attention_layer(4, 1, 64, 64, moe(16, 1, 64, 64), 0.2, 8.0, 90)]},
    # sizes that fit no vector width: an odd vocabulary, a width that is no multiple of 8, heads of 6 and 5,
    # a block of 7 positions
    "D": {"architecture": "Panolorn", "vocab": 101, "width": 100, "norm": {"eps": 2e-5}, "embedding": {"scale": 0.7},
          "layers": [attention_layer(3, 1, 6, 5, moe(3, 2, 7, 9), 0.7, 5.0, 7),
                     attention_layer(2, 2, 10, 3, dense(11), 0.5, 2.0, 33),
                     attention_layer(7, 7, 4, 9, moe(4, 1, 7), 0.9, None, 1)]},
}
INIT = {"A": dict(seed=3, sigma=0.15, norm_jitter=0.2), "B": dict(seed=5, sigma=0.12, norm_jitter=0.1),
        "C": dict(seed=9, sigma=0.08, norm_jitter=0.15), "D": dict(seed=12, sigma=0.2, norm_jitter=0.1)}

_tmp = tempfile.TemporaryDirectory(prefix="kipp_b200_panolorn_")


def write_folder(folder: str, cfg: dict, init: dict, dtype=torch.bfloat16) -> str:
    """Weights are stored in bfloat16, as this design's checkpoints are: the 32-bit engine, the
    16-bit engine (which keeps its routers in float32) and the plain model then all start from
    the same numbers."""
    from kipp_b200.config import config_from_dict
    from kipp_b200.weights import write_random_model
    return write_random_model(folder, config_from_dict(cfg), init["seed"], sigma=init["sigma"],
                              norm_jitter=init["norm_jitter"], dtype=dtype)


@functools.lru_cache(maxsize=None)
def model_folder(name: str) -> str:
    return write_folder(os.path.join(_tmp.name, name), CONFIGS[name], INIT[name])


def random_tokens(vocab: int, n: int, seed: int) -> list:
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def set_tensors(folder: str, changed: dict) -> None:
    """Rewrite ``folder/model.safetensors`` with some tensors replaced."""
    from kipp_b200.weights.safetensors_io import write_safetensors
    from tiny import read_weights
    w = read_weights(folder)
    for name, t in changed.items():
        assert tuple(w[name].shape) == tuple(t.shape), name
        w[name] = t.to(w[name].dtype)
    write_safetensors(os.path.join(folder, "model.safetensors"), list(w.items()), metadata={"format": "pt"})
