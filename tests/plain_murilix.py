"""A plain, slow implementation of the Murilix design: one function per mechanism, float64 on the CPU, whole sequences
only (positions count from 0, every state starts at zero).  It shares no code with the package: the tests compare the
package's kernels, cache and scheduler with it.

A model is (config, tensors): ``config`` is the design's config.json as a dict, ``tensors`` maps checkpoint names to
torch tensors.  ``forward(config, tensors, tokens)`` returns (logits [T, vocab], stream after every layer
[layers, T, width], every token's closest routing call).
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional, Tuple

import torch

F64 = torch.float64


def _w(tensors: Mapping[str, torch.Tensor], name: str) -> torch.Tensor:
    return tensors[name].to(F64)


# ---------------------------------------------------------------------------------------------- small pieces
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """x over the root of (its mean square + eps), along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """(x - mean) over the root of (mean squared deviation + eps), times the weight."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """y_t[c] = sum_j w[c, j] h_(t - taps + 1 + j)[c]; h [T, C], w [C, taps]; zeros before the start."""
    T, C = h.shape
    taps = w.shape[1]
    pad = torch.cat([torch.zeros(taps - 1, C, dtype=h.dtype), h], 0)
    y = torch.zeros_like(h)
    for j in range(taps):
        y = y + pad[j:j + T] * w[:, j]
    return y


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, ..., d]: coordinates 2i and 2i + 1, i < dims / 2, turned by position * base^(-2 i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        a = positions.to(F64) * base ** (-2.0 * i / dims)
        a = a.view(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        y[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return y


# ---------------------------------------------------------------------------------------------- mixers
def windowed_softmax(scores: torch.Tensor, window: int) -> torch.Tensor:
    """scores [H, T, T] (query, key) -> weights; query i sees j with 0 <= i - j (< window, if any)."""
    T = scores.shape[1]
    i = torch.arange(T)
    gap = i[:, None] - i[None, :]
    seen = gap >= 0
    if window:
        seen &= gap < window
    return torch.softmax(scores.masked_fill(~seen, -math.inf), dim=-1)


def latent_attention(m: torch.Tensor, positions: torch.Tensor, p: str, c: Mapping, tensors, eps: float,
                     records: Dict[int, Tuple[torch.Tensor, torch.Tensor]], index: int) -> torch.Tensor:
    """Per-head keys [W_uk c | kr] and values W_uv c from one latent c and one rotated key part kr per token; queries
    through a normed latent of their own.  ``records`` holds (c, kr) by layer: this layer's are made and put there, or
    with ``kv_from`` those of the named layer are read."""
    T = m.shape[0]
    H, dn, dr, dv, r = (int(c[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rot = c.get("rot")
    base, dims = (float(rot["base"]), int(rot["dims"])) if rot else (1.0, 0)
    c_q = rms_unit(m @ _w(tensors, p + "dq").T, eps) * _w(tensors, p + "dq.norm")
    q = (c_q @ _w(tensors, p + "uq").T).view(T, H, dn + dr)
    q_plain, q_rot = q[..., :dn], rotate_pairs(q[..., dn:], positions, base, dims)
    if c.get("kv_from") is None:
        down = m @ _w(tensors, p + "dkv").T
        records[index] = (rms_unit(down[:, :r], eps) * _w(tensors, p + "dkv.norm"),
                          rotate_pairs(down[:, r:], positions, base, dims))
        lat, kr = records[index]
    else:
        lat, kr = records[int(c["kv_from"])]
    k = (lat @ _w(tensors, p + "uk").T).view(T, H, dn)
    v = (lat @ _w(tensors, p + "uv").T).view(T, H, dv)
    scores = (torch.einsum("ihd,jhd->hij", q_plain, k) + torch.einsum("ihd,jd->hij", q_rot, kr)) * float(c["scale"])
    mask = c.get("mask")
    w = windowed_softmax(scores, int(mask["size"]) if mask else 0)
    return torch.einsum("hij,jhd->ihd", w, v).reshape(T, H * dv) @ _w(tensors, p + "o").T


def gated_recurrence(z: torch.Tensor, cand: torch.Tensor) -> torch.Tensor:
    """S_t = (1 - z_t) S_(t-1) + z_t cand_t, S before the first token 0; z, cand [T, W] -> all S."""
    S = torch.zeros_like(z[0])
    out = []
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        out.append(S)
    return torch.stack(out)


def candidate(u: torch.Tensor) -> torch.Tensor:
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def mingru(m: torch.Tensor, p: str, tensors) -> torch.Tensor:
    z = torch.sigmoid(m @ _w(tensors, p + "z").T + _w(tensors, p + "z.b"))
    u = m @ _w(tensors, p + "x").T + _w(tensors, p + "x.b")
    S = gated_recurrence(z, candidate(u))
    return (S * silu(m @ _w(tensors, p + "g").T)) @ _w(tensors, p + "o").T


# ---------------------------------------------------------------------------------------------- feed-forwards
def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    a, b, c, e = (coef[i] for i in range(4))
    return a * rms_unit(z, eps) + b * rms_unit(z ** 2, eps) + c * rms_unit(z ** 3, eps) + e


def dense_ff(h: torch.Tensor, p: str, tensors, eps: float) -> torch.Tensor:
    return poly_norm(h @ _w(tensors, p + "up").T, _w(tensors, p + "act"), eps) @ _w(tensors, p + "down").T


def route(z: torch.Tensor, top: int, tilt: float = 0.0):
    """The ``top`` largest logits of every row and the softmax over those alone; also how far the last chosen logit is
    above the first one left out.  ``tilt`` is added to the even experts' logits for the choice only."""
    T, E = z.shape
    c = z.clone()
    c[:, 0::2] += tilt
    order = c.topk(min(top + 1, E), -1)
    margin = order.values[:, top - 1] - order.values[:, top] if top < E else torch.full((T,), math.inf, dtype=F64)
    idx = order.indices[:, :top]
    return idx, torch.softmax(z.gather(1, idx), -1), margin


def moe_ff(h: torch.Tensor, p: str, c: Mapping, tensors, tilt: float = 0.0):
    idx, wgt, margin = route(h @ _w(tensors, p + "router").T, int(c["router"]["top"]), tilt)
    out = torch.zeros_like(h)
    for e in range(int(c["router"]["experts"])):
        t, j = (idx == e).nonzero(as_tuple=True)
        if len(t):
            x = h[t]
            a = silu(x @ _w(tensors, f"{p}e{e}.gate").T) * (x @ _w(tensors, f"{p}e{e}.up").T)
            out[t] += wgt[t, j][:, None] * (a @ _w(tensors, f"{p}e{e}.down").T)
    return out, margin


# ---------------------------------------------------------------------------------------------- the per-layer token input
def token_input(x: torch.Tensor, rows: torch.Tensor, p: str, tensors, eps: float) -> torch.Tensor:
    """rows [T, dim]: the layer's part of the tokens' rows in the model's side table."""
    g = gelu_tanh(x @ _w(tensors, p + "gate").T) * rows
    return rms_unit(g @ _w(tensors, p + "proj").T, eps) * _w(tensors, p + "norm")


# ---------------------------------------------------------------------------------------------- the model
def forward(config: Mapping, tensors: Mapping[str, torch.Tensor], tokens: List[int], tilt: float = 0.0):
    """-> (logits [T, vocab], the stream after every layer [layers, T, width], every token's closest routing call)."""
    eps = float(config["norm"]["eps"])
    dim = int(config["token_side"]["dim"])
    T = len(tokens)
    ids, positions = torch.tensor(tokens), torch.arange(T)
    x = _w(tensors, "embed")[ids] * float((config.get("embedding") or {}).get("scale", 1.0))
    side = _w(tensors, "side.embed")[ids]
    streams, records = [], {}
    closest = torch.full((T,), math.inf, dtype=F64)
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = layer_norm(x, _w(tensors, p + "norm1"), eps)
        m = h + causal_conv(h, _w(tensors, p + "canon1"))
        if layer["type"] == "latent_attention":
            y = latent_attention(m, positions, p + "mix.", layer["mixer"], tensors, eps, records, i)
        else:
            y = mingru(m, p + "mix.", tensors)
        ff = layer.get("mlp")
        if ff is not None and ff["kind"] == "dense":
            y = y + dense_ff(h, p + "mlp.", tensors, eps)
        elif ff is not None:
            f, margin = moe_ff(h, p + "mlp.", ff, tensors, tilt)
            y = y + f
            closest = torch.minimum(closest, margin)
        x = x + y
        x = x + token_input(x, side[:, i * dim:(i + 1) * dim], p + "side.", tensors, eps)
        streams.append(x.clone())
    logits = layer_norm(x, _w(tensors, "final.norm"), eps) @ _w(tensors, "embed").T
    return logits, torch.stack(streams), closest
