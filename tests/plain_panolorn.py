"""A plain, slow Panolorn in float64 on the CPU: the oracle of the GPU tests.

One function per mechanism, each written from its equation; whole sequences
only (no cache: a position's logits are those of the whole prefix run at once).
Nothing here is shared with the engine.

Notation: x residual stream [T, W]; n(.) = division by the root mean square with
eps inside the root; a layer is x <- x + wb n(sublayer(w n(x))), twice.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_divide(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return rms_divide(x, eps) * weight


def embed(cfg: dict, w: dict, tokens: list) -> torch.Tensor:
    return w["embed"][torch.tensor(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)


# ------------------------------------------------------------------------------------------------
# attention, piece by piece
def capped(s: torch.Tensor, cap) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap else s


def slope(head: int, heads: int) -> float:
    """What a head takes off a score per position of distance: 2^(-8 (head + 1) / heads)."""
    return 2.0 ** (-8.0 * (head + 1) / heads)


def distances(T: int) -> torch.Tensor:
    t = torch.arange(T, dtype=F64)
    return t[:, None] - t[None, :]


def same_block(T: int, size: int) -> torch.Tensor:
    """[T, T] bool: key j of query i lies at or before it and in the same block of ``size`` positions
    counted from the start of the sequence (size 0: every earlier key)."""
    out = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        first = i // size * size if size else 0
        out[i, first:i + 1] = True
    return out


def softmax_plus_one(s: torch.Tensor, seen: torch.Tensor) -> torch.Tensor:
    """e^s_j / (1 + sum over the seen keys of e^s)."""
    s = s.masked_fill(~seen, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, V = m.get("kv_heads") or H, m.get("vdim") or D
    q = rms_divide((h @ w[p + "q"].T).view(T, H, D), eps)
    k = rms_divide((h @ w[p + "k"].T).view(T, G, D), eps)
    v = (h @ w[p + "v"].T).view(T, G, V)
    seen = same_block(T, (m.get("mask") or {}).get("size", 0))
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = capped((q[:, a] @ k[:, g].T) * m["scale"], m.get("softcap")) - slope(a, H) * distances(T)
        heads.append(softmax_plus_one(s, seen) @ v[:, g])
    y = torch.cat(heads, -1) * torch.sigmoid(h @ w[p + "g"].T)
    return y @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------
# feed-forwards
def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gated(act, w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return (act(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(f: dict, w: dict, p: str, h: torch.Tensor) -> tuple:
    """(chosen [T, top], weights [T, top]): the largest sigmoid scores, as they are."""
    s = torch.sigmoid(h @ w[p + "router"].T)
    best = torch.topk(s, f["router"]["top"], dim=-1)
    return best.indices, best.values


def mixture(f: dict, w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    """An expert reads its weight times the token's input; the outputs are added as they are."""
    chosen, weights = route(f, w, p, h)
    rows = []
    for t in range(h.shape[0]):
        rows.append(sum(gated(silu, w, f"{p}e{e}.", a * h[t:t + 1]) for e, a in zip(chosen[t].tolist(), weights[t]))[0])
    out = torch.stack(rows)
    if f.get("shared"):
        out = out + gated(silu, w, p + "shared.", h)
    return out


def feed_forward(f: dict, w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return gated(gelu_tanh, w, p, h) if f["kind"] == "dense" else mixture(f, w, p, h)


# ------------------------------------------------------------------------------------------------
# the layer and the model
def layer_forward(cfg: dict, w: dict, i: int, x: torch.Tensor) -> torch.Tensor:
    layer, p, eps = cfg["layers"][i], f"l{i}.", cfg["norm"]["eps"]
    y = attention(layer["mixer"], w, p + "mix.", norm(x, w[p + "norm1"], eps), eps)
    x = x + norm(y, w[p + "norm1b"], eps)
    if layer.get("mlp"):
        y = feed_forward(layer["mlp"], w, p + "mlp.", norm(x, w[p + "norm2"], eps))
        x = x + norm(y, w[p + "norm2b"], eps)
    return x


def forward(cfg: dict, w: dict, tokens: list, layers_out: list = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence; layers_out collects the stream after every layer."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in w.items()}
    x = embed(cfg, w, tokens)
    for i in range(len(cfg["layers"])):
        x = layer_forward(cfg, w, i, x)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T
