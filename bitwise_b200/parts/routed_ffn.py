"""A routed feed-forward: many small experts, a few per row, and a shared expert for all rows.

Router: ``z = W_r h`` in 32-bit, scores ``s = sigmoid(z)``.  The choice uses ``s + correction``
(a stored vector), the weights use ``s`` alone, times ``weight_scale``, not renormalised.  The
experts form ``groups`` equal groups of neighbours; a group counts as the sum of its two largest
corrected scores and only the experts of the ``keep_groups`` best groups can be chosen; of those
the ``top`` with the largest corrected scores are.  An expert is ``W_down (act(W_gate h, W_up
h))`` with ``act(g, u) = g' sigmoid(alpha g') (u' + 1)``, ``g' = min(g, limit)``, ``u' = clamp(u,
-limit, limit)``.  The output is the weighted sum of the chosen experts' outputs, in the order
of choice, plus the shared expert's.

By constructor arguments: other scores (``scoring``), groups that count as their largest score (``group_score``), weights
divided by their sum (``sum_eps``), experts ``W_down relu(W_up h)^2`` without a gate (``activation="relu2"``), and a shared
expert that is multiplied by the sigmoid of one number per row (``shared_gate``).

On the device: the router's product, ``route`` (one warp per row), ``group_rows`` (the (row,
choice) pairs listed expert by expert), one grouped product for gate and up of all experts, the
activation, one grouped product for down, and ``combine``, which adds the weighted outputs into
the stream.  Nothing is read back to the host: a step's launches depend on its sizes only.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..weights.loader import KEEP32, MATRIX, ParamSpec
from .base import FeedForward, StepContext, register_feed_forward
from .state_recurrence import stacked_rows


class ClampedGLU(FeedForward):
    """gate / up / down with the clamped activation: the shared expert, the form of every
    routed one, and a dense feed-forward of its own."""
    graph_safe = True  # kernels only

    def __init__(self, width: int, inner: int, limit: float, alpha: float):
        self.width, self.inner, self.limit, self.alpha = width, inner, float(limit), float(alpha)
        self.w_gate_up: Optional[torch.Tensor] = None
        self.w_down: Optional[torch.Tensor] = None

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        return [ParamSpec(f"{prefix}.gate", (self.inner, self.width), MATRIX),
                ParamSpec(f"{prefix}.up", (self.inner, self.width), MATRIX),
                ParamSpec(f"{prefix}.down", (self.width, self.inner), MATRIX)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        self.w_gate_up = torch.cat([state[f"{prefix}.gate"], state[f"{prefix}.up"]], 0).contiguous()
        self.w_down = state[f"{prefix}.down"]

    def param_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.w_gate_up, self.w_down))

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, accumulate: bool = True) -> None:
        """``accumulate`` False: the output is written to ``x`` (float32) instead of added to it."""
        ops, n = ctx.ops, ctx.n
        gate_up = ctx.workspace.rows("glu_gate_up", n, 2 * self.inner, ctx.act_dtype)
        ops.linear(xn, self.w_gate_up, gate_up)
        h = ctx.workspace.rows("glu_h", n, self.inner, ctx.act_dtype)
        ops.glu_clamped(gate_up, h, self.limit, self.alpha)
        ops.linear(h, self.w_down, x, residual=x if accumulate else None)


class RoutedFFN(FeedForward):
    graph_safe = True  # kernels only; nothing of the routing is read on the host

    def __init__(self, width: int, experts: int, top: int, inner: int, limit: float, alpha: float,
                 weight_scale: float = 1.0, groups: int = 1, keep_groups: int = 1, correction: bool = True,
                 shared: Optional[FeedForward] = None, scoring: str = "sigmoid", activation: str = "clamped",
                 group_score: str = "top2", sum_eps: Optional[float] = None, shared_gate: Optional[str] = None):
        """``scoring``: "sigmoid" (the weights are the chosen experts' sigmoid scores), "softmax_top" (the
        largest logits are chosen and the weights are the softmax over the chosen logits only) or "softmax" (the
        scores are the softmax over all experts).  ``activation``: "clamped" (``limit``, ``alpha``), "silu" (``silu(gate) *
        up``) or "relu2" (no gate: the square of relu of up).  ``group_score``: a group counts as the sum of its two
        largest choice scores ("top2") or as its largest ("max").  ``sum_eps``: the weights are divided by (their sum +
        sum_eps) before ``weight_scale``.  ``shared_gate``: the name, after the feed-forward's, of a ``[1, width]``
        projection whose sigmoid multiplies the shared expert's output."""
        if scoring not in ("sigmoid", "softmax_top", "softmax") or activation not in ("clamped", "silu", "relu2"):
            raise ValueError(f"unknown scoring {scoring!r} or activation {activation!r}")
        if group_score not in ("top2", "max") or (sum_eps is not None and (scoring == "softmax_top" or sum_eps < 0)):
            raise ValueError(f"unknown group score {group_score!r}, or weights over their sum + {sum_eps!r} with {scoring!r} scores")
        if shared_gate is not None and shared is None:
            raise ValueError("a shared expert's gate without a shared expert")
        self.scoring, self.activation, self.group_score = scoring, activation, group_score
        self.sum_eps, self.shared_gate = sum_eps, shared_gate
        self.gated = activation != "relu2"
        # what the routing asks of the kernels beyond the first design's
        self._route_options = {}
        if scoring != "sigmoid":
            self._route_options.update({"softmax_top": True} if scoring == "softmax_top" else {"scoring": scoring})
        if group_score == "max":
            self._route_options["group_max"] = True
        if sum_eps is not None:
            self._route_options["sum_eps"] = float(sum_eps)
        if experts <= 0 or groups <= 0 or experts % groups:
            raise ValueError(f"{experts} experts do not form {groups} equal groups")
        if not (0 < keep_groups <= groups) or not (0 < top <= keep_groups * (experts // groups)):
            raise ValueError(f"{top} choices among {keep_groups} groups of {experts // groups} experts")
        self.width, self.experts, self.top, self.inner = width, experts, top, inner
        self.limit, self.alpha, self.weight_scale = float(limit), float(alpha), float(weight_scale)
        self.groups, self.keep_groups, self.has_correction, self.shared = groups, keep_groups, correction, shared
        # (w_gate_up: [experts, 2 * inner, width], or [experts, inner, width] where the experts have no gate)
        self.w_router = self.correction = self.w_gate_up = self.w_down = None

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        specs = []
        for e in range(self.experts):
            specs += [ParamSpec(f"{prefix}.e{e}.{n}", (self.inner, self.width), MATRIX) for n in self._inputs]
            specs.append(ParamSpec(f"{prefix}.e{e}.down", (self.width, self.inner), MATRIX))
        specs.append(ParamSpec(f"{prefix}.router", (self.experts, self.width), MATRIX))
        if self.has_correction:
            specs.append(ParamSpec(f"{prefix}.correction", (self.experts,), KEEP32))
        if self.shared is not None:
            specs += self.shared.param_specs(f"{prefix}.shared")
        if self.shared_gate is not None:
            specs.append(ParamSpec(f"{prefix}.{self.shared_gate}", (1, self.width), MATRIX))
        return specs

    @property
    def _inputs(self):
        return ("gate", "up") if self.gated else ("up",)

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        # all experts in two tensors: [experts, 2 * inner, width] (gate rows, then up rows) and
        # [experts, width, inner]
        self.w_gate_up = torch.stack([torch.cat([state[f"{prefix}.e{e}.{n}"] for n in self._inputs], 0)
                                      for e in range(self.experts)]).contiguous()
        self.w_down = torch.stack([state[f"{prefix}.e{e}.down"] for e in range(self.experts)]).contiguous()
        self.w_router = state[f"{prefix}.router"]
        if self.shared_gate is not None:  # the gate's row rides behind the router's in one product
            self.w_router = stacked_rows([self.w_router, state[f"{prefix}.{self.shared_gate}"]])
        self.correction = state[f"{prefix}.correction"] if self.has_correction else None
        if self.shared is not None:
            self.shared.load_params(state, f"{prefix}.shared")

    def param_bytes(self) -> int:
        own = sum(t.numel() * t.element_size() for t in (self.w_gate_up, self.w_down, self.w_router, self.correction)
                  if t is not None)
        return own + (self.shared.param_bytes() if self.shared is not None else 0)

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, then: Optional[tuple] = None) -> None:
        """``then``: the norm that follows on the finished rows (``TanhNorm.after``)."""
        self.forward_sum(ctx, xn, None, x, then=then)

    def forward_scaled(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, scale: torch.Tensor) -> None:
        """``x += scale * feed_forward(xn)`` column by column (``scale`` float32 [width])."""
        if self.shared is not None:
            raise NotImplementedError("a scaled sum with a shared expert")
        self.forward_sum(ctx, xn, None, x, scale=scale)

    def forward_sum(self, ctx: StepContext, xn: torch.Tensor, d: Optional[torch.Tensor], x: torch.Tensor,
                    scale: Optional[torch.Tensor] = None, then: Optional[tuple] = None) -> None:
        """``x += d + feed_forward(xn)``; ``d`` (float32 rows, or None) is used as scratch."""
        ops, ws, n, top = ctx.ops, ctx.workspace, ctx.n, self.top
        act = ctx.act_dtype
        pairs = n * top
        # routing
        z = ws.rows("route_logits", n, self.w_router.shape[0], torch.float32)
        ops.linear(xn, self.w_router, z)
        logits, d_gate = z, None
        if self.shared_gate is not None:
            logits, d_gate = z[:, :self.experts], z[:, self.experts:self.experts + 1]
        chosen = ws.rows("route_chosen", n, top, torch.int32)
        weights = ws.rows("route_weights", n, top, torch.float32)
        lists = ws.rows("route_lists", 3, self.experts + 1, torch.int32)
        order = ws.rows("route_order", n, top, torch.int32)
        place = ws.rows("route_place", n, top, torch.int32)
        ops.route(logits, self.correction, self.groups, self.keep_groups, top, self.weight_scale, chosen, weights,
                  lists=(lists[0], lists[1:3], order, place), **self._route_options)
        grouped = (lists[0], lists[1:3], order)
        # the chosen experts, all in one product each for gate/up and down
        cols = self.w_gate_up.shape[1]
        sorted_x = None
        if getattr(ops, "grouped_takes_tiles", None) and ops.grouped_takes_tiles(pairs, self.experts, cols, self.width):
            sorted_x = ws.rows("routed_x", n, top * self.width, act).view(pairs, self.width)
        h = ws.rows("routed_h", n, top * self.inner, act).view(pairs, self.inner)
        if self.gated:
            gate_up = ws.rows("routed_gate_up", n, top * cols, act).view(pairs, cols)
            ops.grouped_linear(xn, self.w_gate_up, gate_up, pairs, lists=grouped, order_div=top, sorted_x=sorted_x, max_rows=n)
            if self.activation == "silu":
                ops.swiglu(gate_up, h)
            else:
                ops.glu_clamped(gate_up, h, self.limit, self.alpha)
        else:
            ops.grouped_linear(xn, self.w_gate_up, h, pairs, lists=grouped, order_div=top, sorted_x=sorted_x, max_rows=n, activation=self.activation)
        y = ws.rows("routed_y", n, top * self.width, torch.float32).view(pairs, self.width)
        ops.grouped_linear(h, self.w_down, y, pairs, lists=grouped, gather=False, max_rows=n)
        # the shared expert adds into d (or, without d, into the stream), then everything into the stream
        if d_gate is not None:
            # a gated one waits in a buffer of its own for its factor
            if d is not None:
                ops.add_rows(x, d)
            d = ws.rows("shared_out", n, self.width, torch.float32)
            self.shared.forward(ctx, xn, d, accumulate=False)
            ops.combine(x, d, y, place, weights, top, scale=scale, d_gate=d_gate, **({"then": then} if then else {}))
            return
        if self.shared is not None:
            self.shared.forward(ctx, xn, d if d is not None else x)
        ops.combine(x, d, y, place, weights, top, scale=scale, **({"then": then} if then else {}))


register_feed_forward("routed", RoutedFFN)
