"""Dense SwiGLU feed-forward: down(silu(gate x) * up x), silu(g) = g / (1 + e^-g)
(src/architectures/impl/qwen3/block.zig:36-39,
src/kernels/transformer/activation.zig:8-13).  Gate and up are one fused
projection [gate | up], as the reference fuses them for decode
(src/kernels/linear/matvec/form/fused.zig:27-86).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..kernels import pad_inner
from ..registry import register_feed_forward
from .base import FeedForward, ParamSpec, StepContext


@register_feed_forward("swiglu")
class SwiGLU(FeedForward):
    reads_input_by_products = True       # x goes into the gate/up product and nowhere else

    def __init__(self, hidden_size: int, intermediate_size: int, activation: str = "silu", limit: float = 0.0,
                 alpha: float = 1.702):
        """``activation``: what the gate passes through, "silu" or "gelu_tanh"
        (0.5 z (1 + tanh(sqrt(2/pi) (z + 0.044715 z^3)))), or "swish_limit": with g = min(gate, limit) and
        u = clamp(up, -limit, limit) the product of the two halves is g sigmoid(alpha g) (u + 1)."""
        self.hidden = int(hidden_size)
        self.inter = int(intermediate_size)
        if activation not in ("silu", "gelu_tanh", "swish_limit"):
            raise ValueError(f"gated feed-forward: activation={activation!r}")
        self.act = activation
        self.limit, self.alpha = float(limit), float(alpha)
        if activation == "swish_limit" and not self.limit > 0:
            raise ValueError(f"gated feed-forward: limit={limit!r}")

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {"gate_proj.weight": ParamSpec((self.inter, self.hidden)),
                "up_proj.weight": ParamSpec((self.inter, self.hidden)),
                "down_proj.weight": ParamSpec((self.hidden, self.inter))}

    def bind(self, params: Dict[str, torch.Tensor]) -> None:
        gate, up, down = params.pop("gate_proj.weight"), params.pop("up_proj.weight"), params.pop("down_proj.weight")
        # bf16: channels of zeros up to a multiple of 8 (act(0) * 0 = 0 in every form): what the products read at a time
        self.cols = self.inter + (-self.inter % 8 if gate.dtype == torch.bfloat16 else 0)
        if self.cols > self.inter:
            more = (0, 0, 0, self.cols - self.inter)
            gate, up, down = torch.nn.functional.pad(gate, more), torch.nn.functional.pad(up, more), pad_inner(down)
        # bf16: gate and up rows interleaved in eights, so that the product's epilogue holds
        # a channel's gate and up together and writes act(gate) * up directly
        self.fused = (gate.dtype == torch.bfloat16 and hasattr(self.rt.k, "linear_swiglu")
                      and (self.act == "silu" or getattr(self.rt.k, "gated_activations", ()).count(self.act)))
        if self.fused:
            from ..kernels import interleave_gate_up
            self.w_gu = interleave_gate_up(gate, up)
        else:
            self.w_gu = torch.cat([gate, up], dim=0).contiguous()
        self.w_down = down
        self.check_products(gate_up_proj=self.w_gu, down_proj=self.w_down)

    def tensors(self) -> Dict[str, torch.Tensor]:
        I, K, n = self.cols, self.hidden, self.inter
        if self.fused:
            gu = self.w_gu.view(I // 8, 2, 8, K)
            gate, up = gu[:, 0].reshape(I, K), gu[:, 1].reshape(I, K)
        else:
            gate, up = self.w_gu[:I], self.w_gu[I:]
        return {"gate_proj.weight": gate[:n], "up_proj.weight": up[:n], "down_proj.weight": self.w_down[:, :n]}

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: StepContext) -> None:
        rt, k = self.rt, self.rt.k
        T = x.shape[0]
        act = rt.ws.get("ffn.act", (T, self.cols), rt.dtype)
        if self.fused:
            if self.act == "silu":
                k.linear_swiglu(act, x, self.w_gu)
            elif self.act == "swish_limit":
                k.linear_swiglu(act, x, self.w_gu, act=self.act, limit=self.limit, alpha=self.alpha)
            else:
                k.linear_swiglu(act, x, self.w_gu, act=self.act)
        else:
            gu = rt.ws.get("ffn.gu", (T, 2 * self.cols), rt.dtype)
            k.linear(gu, x, self.w_gu)
            if self.act == "silu":
                k.swiglu(act, gu)
            elif self.act == "swish_limit":
                k.gated_limit(act, gu, self.limit, self.alpha)
            else:
                k.gated_act(act, gu, self.act)
        k.linear(residual, act, self.w_down, accumulate=True, defer=True)      # a norm reads the stream next


@register_feed_forward("poly_norm")
class PolyNormMLP(FeedForward):
    """W_down act(W_up x) without a gate: act(z) = a N(z) + b N(z^2) + c N(z^3) + e with powers taken element by element
    and N dividing a token's vector of ff values by its root mean square (eps inside the root); (a, b, c, e) is the
    checkpoint's vector ``act``."""

    def __init__(self, hidden_size: int, intermediate_size: int, norm_eps: float):
        self.hidden, self.inter, self.eps = int(hidden_size), int(intermediate_size), float(norm_eps)
        if self.inter <= 0:
            raise ValueError(f"poly_norm feed-forward: intermediate_size={self.inter}")

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {"up_proj.weight": ParamSpec((self.inter, self.hidden)),
                "down_proj.weight": ParamSpec((self.hidden, self.inter)),
                "act": ParamSpec((4,), kind="vector", init="one_plus_normal")}

    def bind(self, params: Dict[str, torch.Tensor]) -> None:
        self.w_up = params.pop("up_proj.weight")
        self.w_down = pad_inner(params.pop("down_proj.weight"))
        self.coef = params.pop("act").contiguous()
        self.check_products(up_proj=self.w_up, down_proj=self.w_down)

    def tensors(self) -> Dict[str, torch.Tensor]:
        return {"up_proj.weight": self.w_up, "down_proj.weight": self.w_down[:, :self.inter], "act": self.coef}

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx: StepContext) -> None:
        rt, k = self.rt, self.rt.k
        T, cols = x.shape[0], self.w_down.shape[1]
        z = rt.ws.get("ffn.z", (T, cols), rt.dtype)[:, :self.inter]
        k.linear(z, x, self.w_up)
        act = rt.ws.get("ffn.act", (T, cols), rt.dtype)
        k.poly_norm(act, z, self.coef, self.eps)
        k.linear(residual, act, self.w_down, accumulate=True, defer=True)      # a norm reads the stream next
