"""A plain, slow implementation of the Lolivik design: one function per mechanism, float64 on the CPU, whole sequences
only (positions count from 0, every state starts at zero).  It shares no code with the package: the tests compare the
package's kernels, cache and scheduler with it.

A model is (config, tensors): ``config`` is the design's config.json as a dict, ``tensors`` maps checkpoint names to
torch tensors.  ``forward(config, tensors, tokens)`` returns (logits [T, vocab], stream after every layer
[layers, T, width], every token's closest routing call, how much is left of every token's memory read-outs after
cancellation).
"""
from __future__ import annotations

import math
from typing import Dict, List, Mapping, Optional, Tuple

import torch

F64 = torch.float64


def _w(tensors: Mapping[str, torch.Tensor], name: str) -> torch.Tensor:
    return tensors[name].to(F64)


# ---------------------------------------------------------------------------------------------- small pieces
def rms_norm(x: torch.Tensor, weight: Optional[torch.Tensor], eps: float) -> torch.Tensor:
    """x / sqrt(mean(x^2) + eps) over the last axis, times the weight."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if weight is None else y * weight


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softcap(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap else s


# ---------------------------------------------------------------------------------------------- positions
def rotary_frequencies(rot: Mapping) -> torch.Tensor:
    """base^(-2i/dims), i < dims / 2; with ``scaling`` short wavelengths keep their frequency, long ones are divided by
    the factor, those between get a mixture."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    sc = rot.get("scaling")
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc is not None:
            wavelength = 2.0 * math.pi / f
            if wavelength > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif not wavelength < sc["original"] / sc["high"]:
                s = (sc["original"] / wavelength - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_neighbours(x: torch.Tensor, rot: Optional[Mapping]) -> torch.Tensor:
    """x [T, heads, dim], token t at position t: coordinates 2i and 2i + 1 of the first rot.dims are a pair."""
    if rot is None or int(rot["dims"]) == 0:
        return x
    dims = int(rot["dims"])
    a = torch.arange(x.shape[0], dtype=F64)[:, None] * rotary_frequencies(rot)[None, :]
    cos, sin = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    return out


def query_temperature(T: int, t: Optional[Mapping]) -> torch.Tensor:
    """The factor on a query, by its position."""
    if t is None:
        return torch.ones(T, dtype=F64)
    return torch.tensor([1.0 + t["coef"] * math.log(math.floor((p + 1) / t["every"]) + 1.0) for p in range(T)], dtype=F64)


def distance_bucket(n: int, rows: int, far: int) -> int:
    """Which row of the bias table a distance reads: one each up to half of the rows, then logarithmically wider."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(T: int, table: torch.Tensor, far: int) -> torch.Tensor:
    """[T, T, heads]: the bias of query i on key j (j <= i)."""
    rows = torch.tensor([distance_bucket(n, table.shape[0], far) for n in range(T)])
    n = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp_min(0)
    return table[rows[n]]


def window_with_first_tokens(T: int, mask: Optional[Mapping]) -> torch.Tensor:
    """seen[i, j]: j not after i, and close enough or among the first tokens that are kept."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    if mask is None:
        return j <= i
    return (j <= i) & ((i - j < int(mask["size"])) | (j < int(mask.get("keep_first", 0))))


# ---------------------------------------------------------------------------------------------- attention
def attend(q, k, v, scale: float, seen, cap: float = 0.0, bias=None, sink=None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H * V]; bias [T, T, H]; sink [H]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = softcap((q[:, h] @ k[:, g].T) * scale, cap)
        if bias is not None:
            s = s + bias[..., h]
        s = s.masked_fill(~seen, -math.inf)
        m = s.max(-1, keepdim=True).values
        if sink is not None:
            m = m.clamp_min(float(sink[h]))
        e = torch.exp(s - m)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - m)
        out[:, h] = (e / den) @ v[:, g]
    return out.reshape(T, -1)


def mixed_values(v: torch.Tensor, p: str, c: Mapping, tensors, first: Dict[str, torch.Tensor]) -> torch.Tensor:
    """The first layer that mixes keeps its values for the others, which blend them into their own."""
    if not c.get("v_mix"):
        return v
    if "v" not in first:
        first["v"] = v
        return v
    lam = _w(tensors, p + "vmix")
    return (1.0 - lam) * v + lam * first["v"]


def attention(h, p: str, c: Mapping, tensors, eps: float, first) -> torch.Tensor:
    """Every earlier key, no rotation: norms over the whole projections, a temperature on the query, capped scores, a
    learned bias by distance, a learned sink."""
    T = h.shape[0]
    H, G, D, V = int(c["heads"]), int(c.get("kv_heads", c["heads"])), int(c["dim"]), int(c["vdim"])
    q = rms_norm(h @ _w(tensors, p + "q").T, _w(tensors, p + "q.norm"), eps).view(T, H, D)
    k = rms_norm(h @ _w(tensors, p + "k").T, _w(tensors, p + "k.norm"), eps).view(T, G, D)
    v = mixed_values(h @ _w(tensors, p + "v").T, p, c, tensors, first).view(T, G, V)
    q = q * query_temperature(T, c.get("q_temp"))[:, None, None]
    bias = distance_bias(T, _w(tensors, p + "rel"), int(c["bias_max"]))
    o = attend(q, k, v, float(c["scale"]), window_with_first_tokens(T, None), float(c.get("softcap") or 0.0), bias,
               _w(tensors, p + "sink"))
    return o @ _w(tensors, p + "o").T


def attention_2(h, p: str, c: Mapping, tensors, eps: float, first) -> torch.Tensor:
    """A sliding window beside the first tokens: norms per head, rotation of neighbouring pairs, ordinary softmax."""
    T = h.shape[0]
    H, G, D, V = int(c["heads"]), int(c.get("kv_heads", c["heads"])), int(c["dim"]), int(c["vdim"])
    q = rms_norm((h @ _w(tensors, p + "q").T).view(T, H, D), _w(tensors, p + "q.norm"), eps)
    k = rms_norm((h @ _w(tensors, p + "k").T).view(T, G, D), _w(tensors, p + "k.norm"), eps)
    v = mixed_values(h @ _w(tensors, p + "v").T, p, c, tensors, first).view(T, G, V)
    q, k = rotate_neighbours(q, c.get("rot")), rotate_neighbours(k, c.get("rot"))
    o = attend(q, k, v, float(c["scale"]), window_with_first_tokens(T, c.get("mask")))
    return o @ _w(tensors, p + "o").T


# ---------------------------------------------------------------------------------------------- matrix memory
def empty_memory(H: int, D: int, V: int):
    return torch.zeros(H, D, V, dtype=F64), torch.zeros(H, D, dtype=F64), torch.zeros(H, dtype=F64)


def matrix_memory(q, k, v, i, f, state=None, left=None):
    """q, k [T, H, D], v [T, H, V], log gates i, f [T, H] -> ([T, H, V], the state after them), token by token with the
    running maximum; ``state`` (S, n, m): where to start, nothing and a maximum of 0 if not given.  ``left`` [T] is lowered
    to |S^T q| / sum_d |S_d| |q_d|, the smallest of the heads': where that is tiny, the read-out is what rounding leaves."""
    T, H, D = q.shape
    S, n, m = state if state is not None else empty_memory(H, D, v.shape[2])
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        read = torch.einsum("hdv,hd->hv", S, q[t])
        out[t] = read / den[:, None]
        if left is not None:
            left[t] = torch.minimum(left[t], (read.norm(dim=-1) / (S.norm(dim=-1) * q[t].abs()).sum(-1).clamp_min(1e-30)).min())
    return out, (S, n, m)


def memory_gates(h, p: str, c: Mapping, tensors) -> Tuple[torch.Tensor, torch.Tensor]:
    cap = float(c["gate_cap"])
    i = softcap(h @ _w(tensors, p + "i").T + _w(tensors, p + "i.b"), cap)
    f = torch.nn.functional.logsigmoid(softcap(h @ _w(tensors, p + "f").T + _w(tensors, p + "f.b"), cap))
    return i, f


def mlstm(h, p: str, c: Mapping, tensors, eps: float, left=None) -> torch.Tensor:
    T = h.shape[0]
    H, D, V = int(c["heads"]), int(c["dim"]), int(c["vdim"])
    q = (h @ _w(tensors, p + "q").T).view(T, H, D) * D ** -0.5
    k = (h @ _w(tensors, p + "k").T).view(T, H, D)
    v = (h @ _w(tensors, p + "v").T).view(T, H, V)
    i, f = memory_gates(h, p, c, tensors)
    o = rms_norm(matrix_memory(q, k, v, i, f, left=left)[0], None, eps).reshape(T, H * V)
    return (o * _w(tensors, p + "norm") * torch.sigmoid(h @ _w(tensors, p + "g").T)) @ _w(tensors, p + "o").T


# ---------------------------------------------------------------------------------------------- feed-forward
def dense(h, p: str, tensors) -> torch.Tensor:
    return (gelu_tanh(h @ _w(tensors, p + "gate").T) * (h @ _w(tensors, p + "up").T)) @ _w(tensors, p + "down").T


def expert(h, p: str, limit: float, tensors) -> torch.Tensor:
    g = (h @ _w(tensors, p + "gate").T).clamp_max(limit)
    u = (h @ _w(tensors, p + "up").T).clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ _w(tensors, p + "down").T


def choose(z: torch.Tensor, top: int, tilt: float = 0.0) -> Tuple[List[Tuple[int, float]], float]:
    """One token's router logits -> its experts with their weights, and how far the choice is from another one (the
    last chosen logit over the best refused one).  ``tilt`` moves that call by as much, for tests that ask whether
    anything hangs on it."""
    s = torch.softmax(z, -1)
    order = torch.argsort(z, descending=True, stable=True).tolist()
    margin = float(z[order[top - 1]] - z[order[top]]) if top < len(order) else math.inf
    if margin < abs(tilt):
        order[top - 1], order[top] = order[top], order[top - 1]
    picked = order[:top]
    total = float(s[picked].sum()) + 1e-20
    return [(e, float(s[e]) / total) for e in picked], margin


def mixture(h, p: str, c: Mapping, tensors, tilt: float = 0.0) -> Tuple[torch.Tensor, torch.Tensor]:
    T, E = h.shape[0], int(c["router"]["experts"])
    z = h @ _w(tensors, p + "router").T
    y = torch.zeros_like(h)
    margin = torch.zeros(T, dtype=F64)
    weight = torch.zeros(T, E, dtype=F64)
    for t in range(T):
        picked, margin[t] = choose(z[t], int(c["router"]["top"]), tilt)
        for e, w in picked:
            weight[t, e] = w
    for e in range(E):
        rows = (weight[:, e] != 0).nonzero().flatten()
        if len(rows):
            y[rows] += weight[rows, e, None] * expert(h[rows], p + f"e{e}.", float(c["expert"]["limit"]), tensors)
    if c.get("shared"):
        y = y + expert(h, p + "shared.", float(c["shared"]["limit"]), tensors)
    return y, margin


# ---------------------------------------------------------------------------------------------- the model
def forward(config: Mapping, tensors: Mapping[str, torch.Tensor], tokens, tilt: float = 0.0):
    eps, m = float(config["norm"]["eps"]), float(config.get("residual_mult", 1.0))
    x = _w(tensors, "embed")[torch.as_tensor(list(tokens), dtype=torch.long)]
    margin = torch.full((x.shape[0],), math.inf, dtype=F64)
    left = torch.ones(x.shape[0], dtype=F64)
    first: Dict[str, torch.Tensor] = {}
    layers = []
    for i, l in enumerate(config["layers"]):
        p, c, ff = f"l{i}.", l["mixer"], l.get("mlp")
        if l["type"] == "attention":
            y = attention(x, p + "mix.", c, tensors, eps, first)
        elif l["type"] == "attention_2":
            y = attention_2(x, p + "mix.", c, tensors, eps, first)
        elif l["type"] == "mlstm":
            y = mlstm(x, p + "mix.", c, tensors, eps, left)
        else:
            raise ValueError(l["type"])
        x = x + m * rms_norm(y, _w(tensors, p + "norm1"), eps)
        if ff is not None:
            if ff["kind"] == "dense":
                y = dense(x, p + "mlp.", tensors)
            else:
                y, close = mixture(x, p + "mlp.", ff, tensors, tilt)
                margin = torch.minimum(margin, close)
            x = x + m * rms_norm(y, _w(tensors, p + "norm2"), eps)
        layers.append(x)
    logits = rms_norm(x, _w(tensors, "final.norm"), eps) @ _w(tensors, "head").T
    return logits, torch.stack(layers), margin, left
