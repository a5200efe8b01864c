"""Grouped-query attention whose q, k and v pass through a short causal convolution over time, with a sink in the
softmax and a gate on the output.

    q, k, v = conv(W_q x), conv(W_k x), conv(W_v x)     per channel: y_t = sum_j w[:, j] u_(t - taps + 1 + j), zeros
                                                        before the sequence's start
    q, k <- unit_norm per head over head_dim (``qk_norm``; no weight, no rotation: positions do not enter the scores)
    s_ij = q_i . k_j * scale   for 0 <= i - j < window (window 0: all earlier tokens)
    p_ij = exp(s_ij) / (1 + sum_j exp(s_ij))            (``sink``: one more term of score 0 that has no value)
    y = W_o (concat_h(p v) * sigmoid(W_g x))

Options that other designs use: ``conv=False`` (no convolution and no ``*_conv`` tensors); ``qk_norm`` "head" (RMS norm
per head with one weight of head_dim shared by the heads, tensors ``q_norm.weight`` / ``k_norm.weight``) or "row" (RMS
norm over the whole projection, all heads of q, or of k, at once, with a weight per channel); ``position`` (a registered
rotation whose frequencies the kernel reads, after the norm); ``gate="none"`` (no gate and no ``g_proj``).  In the general
form that any of these asks for, also:

``keep``           with a window: 0 <= i - j < window, or j < keep (the sequence's first tokens stay visible)
``softcap``        s <- softcap * tanh(s / softcap), ahead of a bias and of the softmax
``distance_bias``  {"far": D}: s <- s + table[bucket(i - j), h] with a learned table of B rows (tensor ``bias``): bucket(n) = n
                   up to B/2, then B/2 + floor(ln(n / (B/2)) / ln(D / (B/2)) * (B - B/2)), at most B - 1
``learned_sink``   the sink's score is a learned number per head (tensor ``sinks``) instead of 0
``q_temp``         {"coef": c, "every": n}: q is multiplied by 1 + c ln(floor((pos + 1) / n) + 1)
``v_mix``          "source": the layer's values are kept for later layers of the step; "reader": v <- (1 - lambda) v + lambda
                   v_source, lambda the learned number ``v_mix``; what the cache holds is the mixed v

Query head h reads kv head h // (heads / kv_heads).  Keys are ``head_dim`` wide and values ``v_dim``; in the cache
both are padded with zeros to one width, so that the pages have the layout the library's attention kernels read.  The
last taps - 1 projected values of a sequence are its state (``StateRequest``).
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Mapping, Optional, Union

import torch

from ..kernels import PAGE_TOKENS, pad_bias
from ..registry import POSITION_ENCODINGS, lookup, register_mixer
from .base import CacheRequest, LayerIO, Mixer, ParamSpec, StateRequest, StepContext


def distance_rows(rows: int, far: int) -> List[int]:
    """Which row of a bias table of ``rows`` rows each distance 0 .. far reads (from ``far`` on all read the last)."""
    half = rows // 2
    out = []
    for n in range(far + 1):
        if n < half or half == 0:
            out.append(min(n, rows - 1))
        else:
            out.append(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))
    return out


@register_mixer("conv_attention")
class ConvAttention(Mixer):
    reads_input_by_products = True       # x goes into the fused projection and nowhere else

    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_dim: int, conv_taps: int,
                 scale: float, norm_eps: float, window: int = 0, qk_norm: Union[bool, str] = True, sink: bool = True,
                 gate: str = "sigmoid", conv: bool = True, position: Optional[Mapping[str, Any]] = None, keep: int = 0,
                 softcap: float = 0.0, distance_bias: Optional[Mapping[str, int]] = None, learned_sink: bool = False,
                 q_temp: Optional[Mapping[str, Any]] = None, v_mix: Optional[str] = None):
        if num_heads % num_kv_heads:
            raise ValueError(f"attention: {num_heads} heads over {num_kv_heads} kv heads")
        if gate not in ("silu", "sigmoid", "none"):
            raise ValueError(f"attention: gate={gate!r}")
        qk_norm = {True: "unit", False: "none"}.get(qk_norm, qk_norm)
        if qk_norm not in ("none", "unit", "head", "row"):
            raise ValueError(f"attention: qk_norm={qk_norm!r}")
        self.hidden = int(hidden_size)
        self.H, self.G, self.D, self.V = int(num_heads), int(num_kv_heads), int(head_dim), int(v_dim)
        self.taps, self.scale, self.eps = int(conv_taps), float(scale), float(norm_eps)
        self.window, self.qk_norm, self.sink, self.gate = int(window), qk_norm, bool(sink), gate
        self.conv = bool(conv)
        if not self.conv:
            self.taps = 1
        if self.taps < 1:
            raise ValueError(f"attention: a convolution of {self.taps} taps")
        position = dict(position or {"kind": "none"})
        self.position = lookup(POSITION_ENCODINGS, "position encoding", position.pop("kind"))(**position)
        if not getattr(self.position, "fused", False):
            raise ValueError("attention: the rotation must be one whose frequencies the kernel reads (rope_half_split, "
                             "rope_interleaved or none)")
        if int(getattr(self.position, "n_rot", 0) or 0) > self.D:
            raise ValueError(f"attention: {self.position.n_rot} rotated dimensions in a head of {self.D}")
        # what the first kernel of this kind took (convolution, per-head unit norm, a gate) stays on it
        self.general = (not self.conv) or self.qk_norm in ("head", "row") or bool(getattr(self.position, "n_rot", 0))
        self.keep, self.softcap, self.learned_sink, self.v_mix = int(keep), float(softcap), bool(learned_sink), v_mix
        if self.learned_sink:
            self.sink = True
        if self.keep < 0 or (self.keep and not self.window) or self.softcap < 0:
            raise ValueError(f"attention: {keep} first tokens beside a window of {window}, softcap {softcap}")
        self.far = None if distance_bias is None else int(distance_bias["far"])
        if self.far is not None and self.far < 1:
            raise ValueError(f"attention: a distance bias up to {self.far}")
        self.q_temp = None if q_temp is None else (float(q_temp["coef"]), int(q_temp["every"]))
        if self.q_temp is not None and self.q_temp[1] < 1:
            raise ValueError(f"attention: a temperature that changes every {self.q_temp[1]} positions")
        if v_mix not in (None, "source", "reader"):
            raise ValueError(f"attention: v_mix={v_mix!r}")
        if not self.general and (self.q_temp is not None or v_mix is not None):
            raise ValueError("attention: q_temp and v_mix belong to the general form (a norm with weights, a rotation or no convolution)")
        # keys and values share one padded width in the cache (a multiple of 16: what the tensor-core kernels take)
        self.hdp = (max(self.D, self.V) + 15) // 16 * 16
        self.C = (self.H + self.G) * self.D + self.G * self.V          # convolved channels: q, k, v
        self.HV = self.H * self.V
        self.GW = self.HV if self.gate != "none" else 0        # the gate's columns in the fused projection

    def attach(self, rt) -> None:
        super().attach(rt)
        self.position.attach(rt)

    def param_specs(self) -> Dict[str, ParamSpec]:
        H, G, D, V, K, t = self.H, self.G, self.D, self.V, self.hidden, self.taps
        s = {"q_proj.weight": ParamSpec((H * D, K)), "k_proj.weight": ParamSpec((G * D, K)),
             "v_proj.weight": ParamSpec((G * V, K)), "o_proj.weight": ParamSpec((K, self.HV))}
        if self.gate != "none":
            s["g_proj.weight"] = ParamSpec((self.HV, K))
        if self.conv:
            s.update({"q_conv.weight": ParamSpec((H * D, t)), "k_conv.weight": ParamSpec((G * D, t)),
                      "v_conv.weight": ParamSpec((G * V, t))})
        if self.qk_norm in ("head", "row"):
            nq, nk = ((D,), (D,)) if self.qk_norm == "head" else ((H * D,), (G * D,))
            s["q_norm.weight"] = ParamSpec(nq, kind="vector", init="one_plus_normal")
            s["k_norm.weight"] = ParamSpec(nk, kind="vector", init="one_plus_normal")
        if self.far is not None:
            s["bias"] = ParamSpec((-1, self.H), kind="vector")          # (the checkpoint says how many rows)
        if self.learned_sink:
            s["sinks"] = ParamSpec((self.H,), kind="vector")
        if self.v_mix is not None:
            s["v_mix"] = ParamSpec((), kind="vector", ignorable=self.v_mix == "source")
        return s

    def cache_request(self) -> Optional[CacheRequest]:
        return CacheRequest(self.G, self.hdp, self.window, keep=self.keep)

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((self.taps - 1, self.C), self.rt.dtype) if (self.conv and self.taps > 1) else None

    def step_key(self, ctx: StepContext):
        # the decode kernel cuts the longest sequence's pages into parts (as for the rotary attention mixer)
        if not ctx.is_decode:
            return None
        from ..kernels import attention_len_bucket
        # (behind a window a query's keys span the window's pages and the kept ones at most, however long the sequence)
        reach = ctx.max_len
        if self.window and self.general:
            reach = min(reach, (self.keep + PAGE_TOKENS - 1) // PAGE_TOKENS * PAGE_TOKENS + self.window + PAGE_TOKENS)
        return ("gqa_attention", attention_len_bucket(reach))

    def bind(self, params: Dict[str, torch.Tensor]) -> None:
        # one fused projection: rows [q | k | v | g]; the convolutions' taps in the same channel order
        rows = [params.pop("q_proj.weight"), params.pop("k_proj.weight"), params.pop("v_proj.weight")]
        if self.gate != "none":
            rows.append(params.pop("g_proj.weight"))
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.w_conv = (torch.cat([params.pop("q_conv.weight"), params.pop("k_conv.weight"), params.pop("v_conv.weight")],
                                 dim=0).contiguous() if self.conv else None)
        self.q_norm, self.k_norm = params.pop("q_norm.weight", None), params.pop("k_norm.weight", None)
        if self.q_norm is not None and self.q_norm.dtype != self.k_norm.dtype:
            self.q_norm, self.k_norm = self.q_norm.float(), self.k_norm.float()
        # the bias of every distance up to ``far``, head by head; sinks; the share of the first layer's values: 32-bit
        self.stored = {n: params.pop(n) for n in ("bias", "sinks", "v_mix") if n in params}
        self.bias = self.sinks = None
        if self.far is not None:
            table = self.stored["bias"]
            if table.shape[0] // 2 >= self.far and table.shape[0] > 1:
                raise ValueError(f"attention: a distance bias of {table.shape[0]} rows up to a distance of {self.far}")
            rows = torch.tensor(distance_rows(table.shape[0], self.far), device=table.device)
            self.bias = pad_bias(table.float()[rows].t())
        if self.learned_sink:
            self.sinks = self.stored["sinks"].float().contiguous()
        self.lam = float(self.stored["v_mix"].float()) if self.v_mix == "reader" else 0.0
        self.w_o = params.pop("o_proj.weight")
        self.w_o_stored = self.w_o
        if self.gate == "none" and self.V < self.hdp:
            # no gate kernel drops the heads' padding: the projection gets zero columns there instead
            wide = torch.zeros((self.hidden, self.H, self.hdp), dtype=self.w_o.dtype, device=self.w_o.device)
            wide[:, :, :self.V] = self.w_o.view(self.hidden, self.H, self.V)
            self.w_o = wide.view(self.hidden, self.H * self.hdp).contiguous()
        self.check_products(in_proj=self.w_in, o_proj=self.w_o)

    def tensors(self) -> Dict[str, torch.Tensor]:
        a, b, c = self.H * self.D, (self.H + self.G) * self.D, self.C
        out = {"q_proj.weight": self.w_in[:a], "k_proj.weight": self.w_in[a:b], "v_proj.weight": self.w_in[b:c],
               "o_proj.weight": self.w_o_stored}
        if self.gate != "none":
            out["g_proj.weight"] = self.w_in[c:]
        if self.conv:
            out.update({"q_conv.weight": self.w_conv[:a], "k_conv.weight": self.w_conv[a:b], "v_conv.weight": self.w_conv[b:]})
        if self.q_norm is not None:
            out.update({"q_norm.weight": self.q_norm, "k_norm.weight": self.k_norm})
        out.update(self.stored)
        return out

    def _values(self, ctx: StepContext, T: int):
        """(the values to mix in, where to keep this layer's): what the layers of one step hand on to each other."""
        if self.v_mix is None:
            return None, None
        if self.v_mix == "source":
            ctx.extras["v_mix.first"] = keep = self.rt.ws.get("v_mix.first", (T, self.G * self.V), self.rt.dtype)
            return None, keep
        first = ctx.extras["v_mix.first"]
        if first.shape[1] != self.G * self.V:
            raise ValueError(f"attention: values of {self.G} x {self.V} columns mixed with values of {first.shape[1]}")
        return first, None

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: StepContext, io: LayerIO) -> None:
        rt, k = self.rt, self.rt.k
        T = x.shape[0]
        cache = io.cache
        proj = rt.ws.get("conv_attn.proj", (T, self.C + self.GW), rt.dtype)
        k.linear(proj, x, self.w_in)
        q = rt.ws.get("conv_attn.q", (T, self.H * self.hdp), rt.dtype)
        if self.general:
            v_first, v_keep = self._values(ctx, T)
            k.attn_prep(q, proj, self.w_conv, io.state, ctx, cache.block_table, cache.pool, self.H, self.G, self.D, self.V,
                        self.taps, self.qk_norm, self.q_norm, self.k_norm, self.eps, self.position.inv_freq,
                        int(getattr(self.position, "n_rot", 0) or 0), float(getattr(self.position, "mscale", 1.0)),
                        interleaved=bool(getattr(self.position, "interleaved", False)), q_temp=self.q_temp, v_first=v_first,
                        v_lambda=self.lam, v_keep=v_keep)
        else:
            k.conv_norm_write(q, proj, self.w_conv, io.state, ctx, cache.block_table, cache.pool, self.H, self.G, self.D,
                              self.V, self.taps, self.qk_norm == "unit", self.eps)
        out = rt.ws.get("conv_attn.out", (T, self.H * self.hdp), rt.dtype)
        key = self.step_key(ctx)
        k.attention(out, q, cache.pool, cache.block_table, ctx.token_pos, ctx.token_slot, self.H, self.G, self.hdp,
                    self.scale, self.window, ctx, len_bucket=key[1] if key else None,
                    v_dim=self.V if self.V < self.hdp else None, sink=self.sink, softcap=self.softcap, sinks=self.sinks,
                    keep=self.keep, bias=self.bias)
        if self.gate == "none":
            y = out             # (the output projection has zero columns where the heads are padded)
        else:
            y = rt.ws.get("conv_attn.gated", (T, self.HV), rt.dtype)
            k.head_gate(y, out.view(T, self.H, self.hdp), proj[:, self.C:], self.H, self.V, False, self.eps, self.gate)
        k.linear(residual, y, self.w_o, accumulate=True, defer=True)       # a norm reads the stream next
