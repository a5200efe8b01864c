"""What a layer reads beside the normed stream.

``causal_conv`` (a mixer input): the mixer reads h + conv(h) instead of h, conv a causal convolution over time on each
channel, conv(h)_t = sum_j w[:, j] * h_(t - taps + 1 + j), zeros before the sequence's start.  The last taps - 1 rows h of
a sequence are its state, in the compute dtype (what the mixer's products read).

``gated_token_input`` (a layer input): every token has, beside its row in the embedding, a row in one table of the model
of which each layer owns ``dim`` columns (from ``offset`` on).  After the sublayers

    e = table[token, offset : offset + dim],  g = gelu_tanh(W_gate x) * e,  y = W_proj g
    x <- x + y / sqrt(mean(y^2) + eps) * w                                       (an RMS norm whatever the model's norm is)

The layers' parts name the same table tensor; it is loaded once and shared.
"""
from __future__ import annotations

from typing import Any, Dict, Mapping, Optional

import torch

from ..kernels import pad_inner
from ..registry import NORMS, lookup, register_layer_input, register_mixer_input
from .base import Norm, ParamSpec, Part, StateRequest, StepContext


@register_mixer_input("causal_conv")
class CausalConvInput(Part):
    def __init__(self, hidden_size: int, taps: int):
        self.hidden, self.taps = int(hidden_size), int(taps)
        if self.taps < 1:
            raise ValueError(f"causal_conv: a convolution of {self.taps} taps")

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.hidden, self.taps))}

    def state_request(self) -> Optional[StateRequest]:
        return StateRequest((self.taps - 1, self.hidden), self.rt.dtype) if self.taps > 1 else None

    def bind(self, params: Dict[str, torch.Tensor]) -> None:
        # tap by tap, so that neighbouring channels' weights are neighbours
        self.w_taps = params.pop("weight").t().contiguous()

    def tensors(self) -> Dict[str, torch.Tensor]:
        return {"weight": self.w_taps.t()}

    def forward(self, out: torch.Tensor, h: torch.Tensor, ctx: StepContext, state: Optional[torch.Tensor]) -> None:
        self.rt.k.input_conv(out, h, self.w_taps, state, ctx)

    def fusable(self, out: torch.Tensor, ctx: StepContext, state: Optional[torch.Tensor]):
        """What ``RMSNorm.add_into_then_norm`` takes to convolve the rows it norms, or None where the step has more
        than one token a sequence (a row's neighbours are then other blocks' work)."""
        return (out, self.w_taps, state, ctx) if ctx.is_decode and ctx.T == ctx.R else None


@register_layer_input("gated_token_input")
class GatedTokenInput(Part):
    def __init__(self, hidden_size: int, vocab_size: int, dim: int, offset: int, table_width: int, norm: Mapping[str, Any]):
        self.hidden, self.vocab, self.dim = int(hidden_size), int(vocab_size), int(dim)
        self.offset, self.width = int(offset), int(table_width)
        if self.dim <= 0 or self.offset < 0 or self.offset + self.dim > self.width:
            raise ValueError(f"gated_token_input: {self.dim} columns from {self.offset} on of a table of {self.width}")
        norm = dict(norm)
        self.norm: Norm = lookup(NORMS, "norm", norm.pop("kind"))(size=self.hidden, **norm)

    def param_specs(self) -> Dict[str, ParamSpec]:
        s = {"table": ParamSpec((self.vocab, self.width)), "gate": ParamSpec((self.dim, self.hidden)),
             "proj": ParamSpec((self.hidden, self.dim))}
        s.update({"norm." + n: p for n, p in self.norm.param_specs().items()})
        return s

    def attach(self, rt) -> None:
        super().attach(rt)
        self.norm.attach(rt)

    def bind(self, params: Dict[str, torch.Tensor]) -> None:
        self.table = params.pop("table")
        self.w_gate = params.pop("gate")
        self.w_proj = pad_inner(params.pop("proj"))
        self.norm.bind({n[5:]: t for n, t in params.items() if n.startswith("norm.")})
        self.check_products(gate=self.w_gate, proj=self.w_proj)

    def tensors(self) -> Dict[str, torch.Tensor]:
        out = {"table": self.table, "gate": self.w_gate, "proj": self.w_proj[:, :self.dim]}
        out.update({"norm." + n: t for n, t in self.norm.tensors().items()})
        return out

    def project(self, hidden: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        """y = W_proj g for the step's rows of the stream, fp32 [T, hidden] (scratch)."""
        rt, k = self.rt, self.rt.k
        T, cols = hidden.shape[0], self.w_proj.shape[1]
        g = rt.ws.get("token_input.g", (T, cols), rt.dtype)
        few = getattr(k, "token_gate_few_supported", None)
        if few is not None and few(T, self.w_gate):
            k.token_gate_few(g, hidden, self.w_gate, self.table, self.offset, ctx.token_ids)
        else:
            x = hidden
            if rt.dtype != torch.float32:
                x = rt.ws.get("token_input.x", hidden.shape, rt.dtype)
                k.cast_rows(x, hidden)
            z = rt.ws.get("token_input.z", (T, cols), rt.dtype)[:, :self.dim]
            k.linear(z, x, self.w_gate)
            k.token_gate(g, z, self.table, self.offset, ctx.token_ids)
        y = rt.ws.get("token_input.y", hidden.shape, torch.float32)
        k.linear(y, g, self.w_proj)
        return y

    def forward(self, hidden: torch.Tensor, ctx: StepContext) -> None:
        self.norm.add_into(hidden, self.project(hidden, ctx))
