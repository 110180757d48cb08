"""Mixers with a matrix state per request, a mixer made of several side by side,
and the feed-forward with a PolyNorm activation.  The parts themselves:
csrc/host/recurrent_parts.hpp; their kernels: csrc/recurrent.cu.

``RetentionMixer``      S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t per head (q, k rotated,
                        k scaled), each head's o divided by its root mean square, gated, projected.
``DeltaRuleMixer``      S_t = diag(w_t) S_{t-1} - (a_t u_t)(u_t^T S_{t-1}) + k_t v_t^T, o_t = S_t^T r_t.
``GatedMemoryMixer``    m_t = max(f_t + m_{t-1}, i_t), S_t = e^(f_t + m_{t-1} - m_t) S_{t-1} + e^(i_t - m_t) k_t v_t^T,
                        n_t alike, o_t = S_t^T q_t / (max(|n_t . q_t|, e^(-m_t)) + 1e-6): the matrix memory of the xLSTM.
``GatedDeltaMixer``     S <- diag(g_t) S, u_t = beta_t (v_t - S^T k_t), S <- S + k_t u_t^T, o_t = S^T q_t, with short
                        convolutions on q, k and v.
``ParallelMixer``       the sum of its branches, each with its own cache or state and output_scale, or of
                        their normed outputs.
``PolyNormFeedForward`` W_down (c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3), z = W_up h.
"""
from __future__ import annotations

from typing import Optional, Sequence

from .base import FeedForward, Mixer, PositionEncoding


class RetentionMixer(Mixer):
    kind = "retention"

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, decay: Sequence[float],
                 position: PositionEncoding, eps: float, *, value_dim: Optional[int] = None,
                 gate: str = "silu", output_scale: float = 1.0, key_scale: Optional[float] = None,
                 names: Optional[dict] = None):
        self.hidden_size, self.num_heads, self.head_dim = hidden_size, num_heads, head_dim
        self.decay, self.position, self.eps = [float(d) for d in decay], position, eps
        self.value_dim, self.gate, self.output_scale = value_dim or head_dim, gate, output_scale
        self.key_scale, self.names = key_scale, dict(names or {})

    def params(self, prefix, ctx) -> dict:
        out = {"hidden_size": self.hidden_size, "num_heads": self.num_heads, "head_dim": self.head_dim,
               "value_dim": self.value_dim, "decay": self.decay, "position": self.position.describe(prefix, ctx),
               "eps": self.eps, "gate": self.gate, "output_scale": float(self.output_scale), "names": self.names}
        if self.key_scale is not None:
            out["key_scale"] = float(self.key_scale)
        return out


class DeltaRuleMixer(Mixer):
    kind = "delta_rule"

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, decay_rank: int, eps: float, *,
                 gate: str = "sigmoid", output_scale: float = 1.0, names: Optional[dict] = None):
        self.hidden_size, self.num_heads, self.head_dim = hidden_size, num_heads, head_dim
        self.decay_rank, self.eps, self.gate, self.output_scale = decay_rank, eps, gate, output_scale
        self.names = dict(names or {})

    def params(self, prefix, ctx) -> dict:
        return {"hidden_size": self.hidden_size, "num_heads": self.num_heads, "head_dim": self.head_dim,
                "decay_rank": self.decay_rank, "eps": self.eps, "gate": self.gate,
                "output_scale": float(self.output_scale), "names": self.names}


class ParallelMixer(Mixer):
    kind = "parallel"

    def __init__(self, branches: Sequence[tuple], *, out_norms: Optional[Sequence[str]] = None, size: int = 0, eps: float = 1e-6,
                 offset: float = 0.0, out_scale: float = 1.0):
        """``branches``: (prefix, mixer) pairs; each mixer brings its own output_scale.  ``out_norms``: the
        weight names of an RMS norm (of ``size``, with ``eps``; weights stored less ``offset``) over every
        branch's output; ``out_scale`` times the sum of the normed outputs then joins the stream."""
        self.branches, self.out_norms = list(branches), list(out_norms) if out_norms else None
        self.size, self.eps, self.offset, self.out_scale = size, float(eps), float(offset), float(out_scale)

    def params(self, prefix, ctx) -> dict:
        out = {"branches": [{"prefix": p, "part": m.describe(prefix + p, ctx)} for p, m in self.branches]}
        if self.out_norms is not None:
            for branch, name in zip(out["branches"], self.out_norms):
                branch["norm"] = name
            out["out_norm"] = {"size": self.size, "eps": self.eps, "offset": self.offset}
            out["out_scale"] = self.out_scale
        return out


class PolyNormFeedForward(FeedForward):
    kind = "polynorm_mlp"

    def __init__(self, hidden_size: int, intermediate_size: int, eps: float, names: Optional[dict] = None):
        self.hidden_size, self.intermediate_size, self.eps = hidden_size, intermediate_size, eps
        self.names = dict(names or {})

    def params(self, prefix, ctx) -> dict:
        return {"hidden_size": self.hidden_size, "intermediate_size": self.intermediate_size, "eps": self.eps,
                "names": self.names}


class GatedMemoryMixer(Mixer):
    kind = "gated_memory"

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, gate_cap: float, eps: float, *,
                 value_dim: Optional[int] = None, gate: str = "sigmoid", output_scale: float = 1.0,
                 query_scale: Optional[float] = None, names: Optional[dict] = None):
        self.hidden_size, self.num_heads, self.head_dim = hidden_size, num_heads, head_dim
        self.gate_cap, self.eps, self.value_dim = float(gate_cap), eps, value_dim or head_dim
        self.gate, self.output_scale, self.query_scale, self.names = gate, output_scale, query_scale, dict(names or {})

    def params(self, prefix, ctx) -> dict:
        out = {"hidden_size": self.hidden_size, "num_heads": self.num_heads, "head_dim": self.head_dim,
               "value_dim": self.value_dim, "gate_cap": self.gate_cap, "eps": self.eps, "gate": self.gate,
               "output_scale": float(self.output_scale), "names": self.names}
        if self.query_scale is not None:
            out["query_scale"] = float(self.query_scale)
        return out


class StateSpaceMixer(Mixer):
    """The selective state space layer in its matrix-state form: one projection
    [z | x | B | C | dt], a causal convolution of ``conv`` taps over x, B and C,
    S_t = exp(-exp(A) dt) S_(t-1) + dt B_t x_t^T per head (the heads of a group share
    B and C), y = S^T C + D x, the gate silu(z), a root-mean-square division in
    ``norm_groups`` parts.  Per request: S and the convolution's last inputs."""
    kind = "state_space"

    def __init__(self, hidden_size: int, num_heads: int, value_dim: int, state_dim: int, conv: int, eps: float, *,
                 groups: int = 1, norm_groups: int = 1, names: Optional[dict] = None):
        self.hidden_size, self.num_heads, self.value_dim, self.state_dim = hidden_size, num_heads, value_dim, state_dim
        self.conv, self.eps, self.groups, self.norm_groups, self.names = conv, eps, groups, norm_groups, dict(names or {})

    def params(self, prefix, ctx) -> dict:
        return {"hidden_size": self.hidden_size, "num_heads": self.num_heads, "value_dim": self.value_dim,
                "state_dim": self.state_dim, "conv": self.conv, "eps": self.eps, "groups": self.groups,
                "norm_groups": self.norm_groups, "names": self.names}


class GatedDeltaMixer(Mixer):
    """The gated delta rule: q, k (``num_kv_heads`` heads, unit vectors, q times ``query_scale``, default
    head_dim^-1/2) and v (``num_heads``) behind causal convolutions of ``conv`` taps and silu, a write rate per
    head, a decay per head and key channel from a bottleneck of ``decay_rank``, the output divided by its root
    mean square per head, times a weight all heads share, times a gate from a bottleneck of ``gate_rank`` (a rank
    of 0 is read from the checkpoint).  Per request: S and the convolutions' last inputs."""
    kind = "gated_delta"

    def __init__(self, hidden_size: int, num_heads: int, head_dim: int, conv: int, eps: float, *,
                 num_kv_heads: Optional[int] = None, value_dim: Optional[int] = None, decay_rank: int = 0, gate_rank: int = 0,
                 gate: str = "sigmoid", output_scale: float = 1.0, query_scale: Optional[float] = None,
                 names: Optional[dict] = None):
        self.hidden_size, self.num_heads, self.head_dim, self.conv, self.eps = hidden_size, num_heads, head_dim, conv, eps
        self.num_kv_heads, self.value_dim = num_kv_heads or num_heads, value_dim or head_dim
        self.decay_rank, self.gate_rank, self.gate, self.output_scale = decay_rank, gate_rank, gate, output_scale
        self.query_scale, self.names = query_scale, dict(names or {})

    def params(self, prefix, ctx) -> dict:
        out = {"hidden_size": self.hidden_size, "num_heads": self.num_heads, "num_kv_heads": self.num_kv_heads,
               "head_dim": self.head_dim, "value_dim": self.value_dim, "conv": self.conv, "eps": self.eps,
               "decay_rank": self.decay_rank, "gate_rank": self.gate_rank, "gate": self.gate,
               "output_scale": float(self.output_scale), "names": self.names}
        if self.query_scale is not None:
            out["query_scale"] = float(self.query_scale)
        return out
