"""Arrangement of norm, mixer and feed-forward in one layer."""
from __future__ import annotations

from .base import Block, FeedForward, Mixer, Norm
from .embedding import TokenSide


class PreNormBlock(Block):
    """x += mixer(norm1(x)); x += ffn(norm2(x)): the un-normed x is the
    residual stream (src/kipp.c:2948, 2994).  ``post_norm`` and ``ffn`` None: a
    block with the first sublayer only.  The part itself: csrc/host/parts.hpp."""
    kind = "pre_norm_block"

    def __init__(self, input_norm: Norm, mixer: Mixer, post_norm: Norm, ffn: FeedForward,
                 names: tuple[str, str, str, str] = ("input_layernorm.", "self_attn.",
                                                     "post_attention_layernorm.", "mlp.")):
        self.input_norm, self.mixer, self.post_norm, self.ffn = input_norm, mixer, post_norm, ffn
        self.names = tuple(names)

    def params(self, prefix, ctx) -> dict:
        parts = (self.input_norm, self.mixer, self.post_norm, self.ffn)
        described = [None if p is None else p.describe(prefix + n, ctx) for p, n in zip(parts, self.names)]
        return {"names": list(self.names), "input_norm": described[0], "mixer": described[1],
                "post_norm": described[2], "ffn": described[3]}


class ParallelBlock(Block):
    """x += mixer(n) + ffn(n) with n = norm(x): ONE norm whose output both
    sublayers read, or (``ffn_norm``) one each, of the same x.  ``ffn`` None: the
    mixer only.  ``side``: a ``TokenSide`` behind them.  ``names``: prefixes of norm,
    mixer and feed-forward and, where given, of ``ffn_norm`` and ``side``.  The part
    itself: csrc/host/parts.hpp."""
    kind = "parallel_block"

    def __init__(self, norm: Norm, mixer: Mixer, ffn: FeedForward | None, names: tuple = ("norm.", "mix.", "mlp."), *,
                 ffn_norm: Norm | None = None, side: TokenSide | None = None):
        self.parts = (norm, mixer, ffn, ffn_norm, side)
        self.norm, self.mixer, self.ffn = norm, mixer, ffn
        self.names = tuple(names) if len(names) == 5 or (ffn_norm is None and side is None) else tuple(names) + ("", "side.")

    def params(self, prefix, ctx) -> dict:
        roles = ("norm", "mixer", "ffn", "ffn_norm", "side")
        names = self.names + ("",) * (5 - len(self.names))
        described = {r: None if p is None else p.describe(prefix + n, ctx) for r, p, n in zip(roles, self.parts, names)}
        return {"names": list(self.names), **described}


class SandwichNormBlock(Block):
    """x += residual_mult * mixer_out_norm(mixer(input_norm(x))); x += residual_mult *
    ffn_out_norm(ffn(post_norm(x))): an RMS norm on either side of every sublayer.  ``ffn``
    None (with its two norms): the mixer only.  ``names``: prefixes of the six parts in this
    order.  The part itself: csrc/host/parts.hpp."""
    kind = "sandwich_norm_block"

    def __init__(self, input_norm: Norm, mixer: Mixer, mixer_out_norm: Norm, post_norm: Norm | None = None,
                 ffn: FeedForward | None = None, ffn_out_norm: Norm | None = None, *, residual_mult: float = 1.0,
                 names: tuple = ("", "mix.", "", "", "mlp.", "")):
        self.parts = (input_norm, mixer, mixer_out_norm, post_norm, ffn, ffn_out_norm)
        self.residual_mult, self.names = float(residual_mult), tuple(names)

    def params(self, prefix, ctx) -> dict:
        roles = ("input_norm", "mixer", "mixer_out_norm", "post_norm", "ffn", "ffn_out_norm")
        described = {r: None if p is None else p.describe(prefix + n, ctx) for r, p, n in zip(roles, self.parts, self.names)}
        return {"names": list(self.names), "residual_mult": self.residual_mult, **described}


class HyperConnectionBlock(Block):
    """The residual stream as ``streams`` copies: sublayer q reads
    u = sum_s in_q[s] x_s through its RMS norm and its output y joins every copy,
    x_t <- sum_s mix_q[s, t] x_s + residual_mult * out_q[t] * y.  ``connections``
    False: one stream and the plain x <- x + residual_mult * sublayer(norm(x)).
    ``names``: prefixes of the two norms, the mixer, the feed-forward and the two
    sets of connection tensors.  The part itself: csrc/host/parts.hpp."""
    kind = "hyper_connection_block"

    def __init__(self, input_norm: Norm, mixer: Mixer, post_norm: Norm, ffn: FeedForward, *, streams: int = 1,
                 connections: bool = True, residual_mult: float = 1.0,
                 names: tuple = ("", "mix.", "", "mlp.", "hc1.", "hc2.")):
        self.input_norm, self.mixer, self.post_norm, self.ffn = input_norm, mixer, post_norm, ffn
        self.streams, self.connections, self.residual_mult = int(streams), bool(connections), float(residual_mult)
        self.names = tuple(names)

    def params(self, prefix, ctx) -> dict:
        parts = (self.input_norm, self.mixer, self.post_norm, self.ffn)
        described = [None if p is None else p.describe(prefix + n, ctx) for p, n in zip(parts, self.names)]
        return {"names": list(self.names), "streams": self.streams, "connections": self.connections,
                "residual_mult": self.residual_mult, "input_norm": described[0], "mixer": described[1],
                "post_norm": described[2], "ffn": described[3]}
