"""Two mixers side by side on the same input: half the sum of their outputs, each first divided by its root mean
square over the width, times a weight.

The left one may keep pages; the right one keeps slot state.  Where both project their input with one stacked
matrix (``stacks_input``), the two matrices are stacked once more and one product feeds both.  The mean, and the layer
norm that a block puts behind its mixer, are one kernel (``forward_into_norm``).  Norms and sums are float32.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..weights.loader import KEEP32, ParamSpec
from .base import Mixer, PagedKVView, StepContext, register_mixer
from .norm import LayerNorm


class PairedMixer(Mixer):
    NAMES = {"left": "left", "right": "right", "left_norm": "left.out", "right_norm": "right.out"}

    def __init__(self, width: int, left: Mixer, right: Mixer, eps: float, names: Optional[Dict[str, str]] = None):
        if left.state_need() is not None or right.state_need() is not None:
            raise NotImplementedError("a pair keeps one cache on the left and one slot state on the right")
        self.width, self.left, self.right, self.eps = width, left, right, float(eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.graph_safe = getattr(left, "graph_safe", False) and getattr(right, "graph_safe", False)
        self.left_norm = self.right_norm = self.w_in = None
        self.left_cols = 0

    def cache_need(self):
        return self.left.cache_need()

    def state_need(self):
        return self.right.cache_need()

    def query_tile_rows(self, ops=None):
        sizes = set()
        for part in (self.left, self.right):
            fn = getattr(part, "query_tile_rows", None)
            if fn is not None:
                got = fn(ops)
                sizes.update(got if isinstance(got, (list, tuple, set)) else [got])
        return sorted(sizes)

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        n = self.names
        return (self.left.param_specs(f"{prefix}.{n['left']}") + self.right.param_specs(f"{prefix}.{n['right']}")
                + [ParamSpec(f"{prefix}.{n[k]}", (self.width,), KEEP32, init="ones") for k in ("left_norm", "right_norm")])

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        n = self.names
        self.left.load_params(state, f"{prefix}.{n['left']}")
        self.right.load_params(state, f"{prefix}.{n['right']}")
        self.left_norm, self.right_norm = state[f"{prefix}.{n['left_norm']}"], state[f"{prefix}.{n['right_norm']}"]
        if getattr(self.left, "stacks_input", False) and getattr(self.right, "stacks_input", False):
            from .state_recurrence import stacked_rows
            rows = self.left.w_in.shape[0]
            left = stacked_rows([self.left.w_in])
            self.left_cols = left.shape[0]
            self.w_in = torch.cat([left, self.right.w_in], 0).contiguous()
            self.left.w_in, self.right.w_in = self.w_in[:rows], self.w_in[self.left_cols:]

    def param_bytes(self) -> int:
        own = sum(t.numel() * t.element_size() for t in (self.left_norm, self.right_norm))
        return self.left.param_bytes() + self.right.param_bytes() + own

    def prepare(self, ops) -> None:
        self.left.prepare(ops)
        self.right.prepare(ops)

    def _both(self, ctx: StepContext, xn: torch.Tensor, cache: PagedKVView):
        ws, n = ctx.workspace, ctx.n
        a = ws.rows("pair_left32", n, self.width, torch.float32)
        b = ws.rows("pair_right32", n, self.width, torch.float32)
        left, right = {}, {}
        if self.w_in is not None:
            u = ws.rows("pair_in32", n, self.w_in.shape[0], torch.float32)
            ctx.ops.linear(xn, self.w_in, u)
            left["projected"], right["projected"] = u[:, :self.left.w_in.shape[0]], u[:, self.left_cols:]
        self.left.forward(ctx, xn, a, cache, accumulate=False, **left)
        self.right.forward(ctx, xn, b, cache.state, accumulate=False, **right)
        return a, b

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, cache: PagedKVView,
                accumulate: bool = True) -> None:
        a, b = self._both(ctx, xn, cache)
        y = ctx.workspace.rows("pair_mean32", ctx.n, self.width, torch.float32) if accumulate else x
        ctx.ops.pair_mean(a, self.left_norm, b, self.right_norm, self.eps, y=y)
        if accumulate:
            ctx.ops.add_rows(x, y)

    def forward_into_norm(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, cache: PagedKVView, norm, rounded) -> None:
        """``x += norm(mixer(xn))``, the summed rows also into ``rounded`` (activation type) where that is given."""
        if type(norm) is not LayerNorm:
            y = ctx.workspace.rows("pair_mean32", ctx.n, self.width, torch.float32)
            self.forward(ctx, xn, y, cache, accumulate=False)
            if rounded is None:
                norm.forward_residual(ctx, y, x)
            else:
                norm.forward_residual_round(ctx, y, x, rounded)
            return
        a, b = self._both(ctx, xn, cache)
        ctx.ops.pair_mean(a, self.left_norm, b, self.right_norm, self.eps, norm_weight=norm.weight, norm_eps=norm.eps, x=x,
                          rounded=rounded)


register_mixer("paired", PairedMixer)
