"""A plain, slow Nogavik in float64 on the CPU: the oracle of the GPU tests.

One function per mechanism, each written from its equation; whole sequences
only (no cache, no state carried between calls: a position's logits are those of
the whole prefix run at once).  Nothing here is shared with the engine.

Notation: T tokens, W the width, n(x; w) = x / sqrt(mean(x^2) + eps) * w.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_divide(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """The model's norm: the weight is stored as its distance from one."""
    return rms_divide(x, eps) * (1.0 + w)


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(x: torch.Tensor) -> torch.Tensor:
    return torch.logaddexp(x, torch.zeros_like(x))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def rotate_neighbours(x: torch.Tensor, positions: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, H, D]: coordinate 2i pairs with 2i + 1 for 2i < dims and turns by p * base^(-2i/dims); the rest stays."""
    dims = rot["dims"] if rot else 0
    if dims == 0:
        return x
    freq = torch.tensor([rot["base"] ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = positions.to(F64)[:, None, None] * freq
    c, s = torch.cos(ang), torch.sin(ang)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def causal_softmax(scores: torch.Tensor) -> torch.Tensor:
    """scores [T, T] (query, key) -> weights over the keys j <= i"""
    T = scores.shape[0]
    return torch.softmax(scores.masked_fill(~torch.tril(torch.ones(T, T, dtype=torch.bool)), -math.inf), -1)


def causal_conv(x: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor = None) -> torch.Tensor:
    """x [T, C], weight [C, taps]: the last column meets the token itself, the one before it the token before, ..."""
    T, taps = x.shape[0], weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x], 0)
    out = torch.zeros_like(x) if bias is None else bias.expand(T, -1).clone()
    for j in range(taps):
        out = out + padded[j:j + T] * weight[:, j]
    return out


# ------------------------------------------------------------------------------------------------
# mixers
def attention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Grouped-query attention without positions: biases on q, k and v, then q and k normed per head."""
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, V = m.get("kv_heads") or H, m.get("vdim") or D
    q = (h @ w[p + "q"].T + w[p + "q.b"]).view(T, H, D)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).view(T, G, D)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, V)
    q, k = rms_divide(q, eps) * w[p + "q.norm"], rms_divide(k, eps) * w[p + "k.norm"]
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        out[:, hd] = causal_softmax(q[:, hd] @ k[:, g].T * m["scale"]) @ v[:, g]
    return out.reshape(T, H * V) @ w[p + "o"].T


def delta_vectors(m: dict, w: dict, p: str, h: torch.Tensor) -> tuple:
    """(q, k [T, H, D] unit vectors, q times D^-1/2; v [T, H, V]; the write rate beta [T, H]; the decay g [T, H, D])"""
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    G, V = m.get("kv_heads") or H, m.get("vdim") or D
    q, k, v = (silu(causal_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in ("q", "k", "v"))
    head_of = torch.arange(H) // (H // G)
    q = unit(q.view(T, G, D))[:, head_of] * D ** -0.5
    k = unit(k.view(T, G, D))[:, head_of]
    beta = torch.sigmoid(h @ w[p + "b"].T)
    rate = softplus((h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(w[p + "A_log"])[:, None] * rate)
    return q, k, v.view(T, H, V), beta, g


def gated_delta_rule(q, k, v, beta, g) -> torch.Tensor:
    """Per head: every row of S decays, u = beta (v - S^T k), S += k u^T, o = S^T q."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def gated_delta(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    T, H = h.shape[0], m["heads"]
    V = m.get("vdim") or m["dim"]
    o = gated_delta_rule(*delta_vectors(m, w, p, h))
    o = rms_divide(o, eps) * w[p + "norm"]
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).view(T, H, V)
    return (o * gate).reshape(T, H * V) @ w[p + "o"].T


def parallel(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """Half the sum of the two mixers' outputs, each normed over the width."""
    left = attention(m["left"], w, p + "left.", h, eps)
    right = gated_delta(m["right"], w, p + "right.", h, eps)
    return 0.5 * (rms_divide(left, eps) * w[p + "left.out"] + rms_divide(right, eps) * w[p + "right.out"])


def mamba2(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> torch.Tensor:
    """S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T per head, y_t = S_t^T C_t + D x_t; the
    gate silu(z) first, then a root-mean-square division in norm_groups parts."""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m.get("groups") or 1
    inner = H * P
    proj = h @ w[p + "in"].T
    z, xbc, dt = proj[:, :inner], proj[:, inner:2 * inner + 2 * G * N], proj[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x = xbc[:, :inner].view(T, H, P)
    B = xbc[:, inner:inner + G * N].view(T, G, N)
    C = xbc[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + w[p + "dt_bias"])
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    head_of = torch.arange(H) // (H // G)
    S = torch.zeros(H, N, P, dtype=h.dtype)
    y = torch.zeros(T, H, P, dtype=h.dtype)
    for t in range(T):
        S = decay[t][:, None, None] * S + dt[t][:, None, None] * B[t, head_of][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", S, C[t, head_of]) + w[p + "D"][:, None] * x[t]
    y = y.reshape(T, inner) * silu(z)
    parts = m.get("norm_groups") or 1
    y = rms_divide(y.view(T, parts, inner // parts), eps).reshape(T, inner) * w[p + "norm"]
    return y @ w[p + "o"].T


def latent_keys(m: dict, w: dict, p: str, h: torch.Tensor, eps: float) -> tuple:
    """(the normed latent [T, kv_rank], the rotated key part [T, rot_dim] all heads share)"""
    R = m["kv_rank"]
    both = h @ w[p + "dkv"].T
    c = rms_divide(both[:, :R], eps) * w[p + "dkv.norm"]
    k_rot = rotate_neighbours(both[:, None, R:], torch.arange(h.shape[0]), m.get("rot"))[:, 0]
    return c, k_rot


def latent_attention(m: dict, w: dict, p: str, h: torch.Tensor, eps: float, keys: tuple) -> torch.Tensor:
    """Keys and values out of the latent; every element of the concatenated heads has a gate."""
    T = h.shape[0]
    H, D, R = m["heads"], m["dim"], m["rot_dim"]
    V = m.get("vdim") or D
    c, k_rot = keys
    c_q = rms_divide(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = (c_q @ w[p + "uq"].T).view(T, H, D + R)
    q_rot = rotate_neighbours(q[..., D:], torch.arange(T), m.get("rot"))
    k = (c @ w[p + "uk"].T).view(T, H, D)
    v = (c @ w[p + "uv"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for hd in range(H):
        out[:, hd] = causal_softmax((q[:, hd, :D] @ k[:, hd].T + q_rot[:, hd] @ k_rot.T) * m["scale"]) @ v[:, hd]
    return (out.reshape(T, H * V) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# ------------------------------------------------------------------------------------------------
def feed_forward(w: dict, p: str, h: torch.Tensor) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def token_side(w: dict, p: str, x: torch.Tensor, e: torch.Tensor, eps: float) -> torch.Tensor:
    """What a layer's own embedding e of the token adds: gated by the stream, brought to its width, normed."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms_divide(y, eps) * w[p + "norm"]


def mixer(cfg: dict, w: dict, i: int, h: torch.Tensor, lent: dict) -> torch.Tensor:
    """`lent` holds every latent attention layer's own keys for the layers that read them."""
    layer, p, eps = cfg["layers"][i], f"l{i}.mix.", cfg["norm"]["eps"]
    m = layer["mixer"]
    if layer["type"] == "parallel":
        return parallel(m, w, p, h, eps)
    if layer["type"] == "mamba2":
        return mamba2(m, w, p, h, eps)
    if m.get("kv_from") is None:
        lent[i] = latent_keys(m, w, p, h, eps)
    return latent_attention(m, w, p, h, eps, lent[i if m.get("kv_from") is None else m["kv_from"]])


def layer_forward(cfg: dict, w: dict, i: int, x: torch.Tensor, tokens: torch.Tensor, lent: dict) -> torch.Tensor:
    eps = cfg["norm"]["eps"]
    y = mixer(cfg, w, i, norm_one_plus(x, w[f"l{i}.norm1"], eps), lent)
    if cfg["layers"][i].get("mlp"):
        y = y + feed_forward(w, f"l{i}.mlp.", norm_one_plus(x, w[f"l{i}.norm2"], eps))
    x = x + y
    side = cfg.get("token_side")
    if side:
        d = side["dim"]
        x = x + token_side(w, f"l{i}.side.", x, w["side.embed"][tokens, i * d:(i + 1) * d], eps)
    return x


def forward(cfg: dict, w: dict, tokens: list, layers_out: list = None) -> torch.Tensor:
    """Logits [T, vocab] of a whole sequence; layers_out collects the stream after every layer."""
    w = {k: (v.to(F64) if v.is_floating_point() else v) for k, v in w.items()}
    ids = torch.tensor(tokens)
    x = w["embed"][ids]
    lent = {}
    for i in range(len(cfg["layers"])):
        x = layer_forward(cfg, w, i, x, ids, lent)
        if layers_out is not None:
            layers_out.append(x)
    return norm_one_plus(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T
