"""The dense SwiGLU feed-forward: ``h = silu(xn Wg^T) * (xn Wu^T)``, ``x += h Wd^T``
(src/model.cpp:301-305; src/kernels.cpp:291-298).  gate_proj and up_proj are stacked by
rows into one matrix so that one product yields rows laid out [gate | up]
(src/model.cpp:162-164).  SiLU is the only activation the reference has; no biases.
``activation="gelu_tanh"`` makes it ``h = gelu_tanh(xn Wg^T) * (xn Wu^T)`` with ``gelu_tanh(z) = 0.5 z (1
+ tanh(sqrt(2 / pi) (z + 0.044715 z^3)))``."""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..weights.loader import MATRIX, ParamSpec
from .base import FeedForward, StepContext, register_feed_forward


ACTIVATIONS = ("silu", "gelu_tanh")


class SwiGLU(FeedForward):
    graph_safe = True  # kernels only: a step through this part can be captured

    def __init__(self, width: int, intermediate: int, names=("gate_proj", "up_proj", "down_proj"),
                 suffix: str = ".weight", activation: str = "silu"):
        if activation not in ACTIVATIONS:
            raise ValueError(f"gated feed-forward: activation {activation!r} (known: {', '.join(ACTIVATIONS)})")
        self.activation = activation
        self.width, self.intermediate = width, intermediate
        self.names = names
        self.suffix = suffix  # what follows a matrix's name in the checkpoint
        self.w_gate_up: Optional[torch.Tensor] = None  # rows [gate | up], or interleaved when fused
        self.w_down: Optional[torch.Tensor] = None
        self.fused = False  # gate/up product and SwiGLU in one kernel

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        g, u, d = self.names
        sfx = self.suffix
        return [ParamSpec(f"{prefix}.{g}{sfx}", (self.intermediate, self.width), MATRIX),
                ParamSpec(f"{prefix}.{u}{sfx}", (self.intermediate, self.width), MATRIX),
                ParamSpec(f"{prefix}.{d}{sfx}", (self.width, self.intermediate), MATRIX)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        g, u, d = self.names
        sfx = self.suffix
        self.w_gate_up = torch.cat([state[f"{prefix}.{g}{sfx}"], state[f"{prefix}.{u}{sfx}"]], 0).contiguous()
        self.w_down = state[f"{prefix}.{d}{sfx}"]

    def param_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_gate_up, self.w_down))

    def prepare(self, ops) -> None:
        """Kernels that apply SwiGLU in the epilogue of the gate/up product want the two
        matrices interleaved in blocks of 64 rows."""
        if not self.fused and getattr(ops, "fuses_swiglu", None) and ops.fuses_swiglu(self.width, self.intermediate,
                                                                                      **self._act):
            gate, up = self.w_gate_up[:self.intermediate], self.w_gate_up[self.intermediate:]
            self.w_gate_up = ops.interleave_gate_up(gate, up)
            self.fused = True

    @property
    def _act(self):
        # (only an activation other than SiLU is named to the kernels' bindings)
        return {} if self.activation == "silu" else {"activation": self.activation}

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, accumulate: bool = True,
                then: Optional[tuple] = None) -> None:
        """``accumulate`` False: the output is written to ``x`` (float32) instead of added to it.  ``then``: the norm that
        follows on the finished rows (``TanhNorm.after``)."""
        ops, n = ctx.ops, ctx.n
        h = ctx.workspace.rows("ffn_h", n, self.intermediate, ctx.act_dtype)
        if self.fused:
            ops.linear_swiglu(xn, self.w_gate_up, h, **self._act)
        else:
            gate_up = ctx.workspace.rows("gate_up", n, 2 * self.intermediate, ctx.act_dtype)
            ops.linear(xn, self.w_gate_up, gate_up)
            if self.activation == "gelu_tanh":
                ops.glu_gelu(gate_up, h)
            else:
                ops.swiglu(gate_up, h)
        ops.linear(h, self.w_down, x, residual=x if accumulate else None, **({"then": then} if then else {}))


class DenseFFN(FeedForward):
    """``x += W_down act(W_up xn)``: no gate, no biases.  ``activation``: "relu2", the square of relu.  On the serving
    precision the activation is applied in the up product's epilogue."""
    graph_safe = True  # kernels only

    def __init__(self, width: int, intermediate: int, names=("up", "down"), suffix: str = "", activation: str = "relu2"):
        if activation != "relu2":
            raise ValueError(f"feed-forward: activation {activation!r} (known: relu2)")
        self.width, self.intermediate, self.names, self.suffix, self.activation = width, intermediate, names, suffix, activation
        self.w_up: Optional[torch.Tensor] = None
        self.w_down: Optional[torch.Tensor] = None

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        u, d = self.names
        return [ParamSpec(f"{prefix}.{u}{self.suffix}", (self.intermediate, self.width), MATRIX),
                ParamSpec(f"{prefix}.{d}{self.suffix}", (self.width, self.intermediate), MATRIX)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        u, d = self.names
        self.w_up, self.w_down = state[f"{prefix}.{u}{self.suffix}"], state[f"{prefix}.{d}{self.suffix}"]

    def param_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_up, self.w_down))

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, accumulate: bool = True) -> None:
        """``accumulate`` False: the output is written to ``x`` (float32) instead of added to it."""
        h = ctx.workspace.rows("ffn_h", ctx.n, self.intermediate, ctx.act_dtype)
        ctx.ops.linear(xn, self.w_up, h, activation=self.activation)
        ctx.ops.linear(h, self.w_down, x, residual=x if accumulate else None)


register_feed_forward("swiglu", SwiGLU)
register_feed_forward("dense", DenseFFN)
