"""Mixers whose memory is a matrix of state per head, beside gated linear attention.

* :class:`ChannelDelta`: the gated delta rule.  q, k and v pass a short causal convolution over time and SiLU, q and k are
  unit vectors per head; per head ``S <- g S`` with a decay g per key channel, ``S <- S + k (beta (v - S^T
  k))^T``, ``o = S^T q``.
* :class:`ShiftedRecurrence`: every projection reads its own mix of the current and the previous row; ``o = (S +
  diag(u) k v^T)^T r``, then ``S <- diag(w) S + k v^T`` with a decay w from the input and a bonus u.
* :class:`StateSpace`: x, B and C pass a short causal convolution over time and SiLU; per head ``S <- e^(-rate t) S + t B
  x^T``, ``y = S^T C + D x`` with a step t from the input.
* :class:`MatrixMemory`: exponential input and forget gates under a running maximum, a normaliser beside S.

In all of them but the state space a head's output is divided by its root mean square, times a weight and a gate, and
projected by W_o; the state space's is gated first and normed in equal parts of the row.

The state is float32 and lives in a state slot of the request, as do a convolution's last inputs and the
previous row.  The projections may run in the activation type; the convolution, decays, gates of the recurrence,
unit norms, state, outputs and their norm are float32 in both precisions.  The recurrence is walked token by token in
one order whatever the step's cut, so a position's result does not depend on how the prompt was portioned.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..weights.loader import KEEP32, MATRIX, ParamSpec
from .base import Mixer, SlotStateNeed, SlotStateView, StepContext, register_mixer
from .scored_attention import SEQUENCE_TILE


def stacked_rows(tensors, multiple: int = 8) -> torch.Tensor:
    """The matrices one under the other, with rows of zeros up to a multiple of ``multiple`` rows (so that the columns of
    their product start and lie on 16 bytes)."""
    w = torch.cat(list(tensors), 0)
    pad = -w.shape[0] % multiple
    if pad:
        w = torch.cat([w, torch.zeros(pad, w.shape[1], dtype=w.dtype, device=w.device)], 0)
    return w.contiguous()


def _padded(count: int, multiple: int = 8) -> int:
    return count + -count % multiple


def one_row_each(ctx: StepContext) -> bool:
    """Whether every sequence of the step has one row (a function of the step's sizes)."""
    return ctx.query_tiles(SEQUENCE_TILE)[3] == ctx.n


def _check(what: str, **sizes) -> None:
    for name, v in sizes.items():
        if v <= 0:
            raise ValueError(f"{what}: {name} must be positive, got {v}")


class _StateMixer(Mixer):
    graph_safe = True  # kernels only; launches depend on the step's sizes

    def query_tile_rows(self, ops=None):
        return [SEQUENCE_TILE]

    def _tensors(self):
        raise NotImplementedError

    def param_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self._tensors())


class ChannelDelta(_StateMixer):
    NAMES = {"q": "q", "k": "k", "v": "v", "out": "o", "conv": ".conv", "beta": "b", "decay_down": "a1", "decay_up": "a2",
             "decay_bias": "dt_bias", "decay_log": "A_log", "gate_down": "g1", "gate_up": "g2", "norm": "norm"}

    def __init__(self, width: int, heads: int, kv_heads: int, dim: int, vdim: int, conv_taps: int, decay_rank: int,
                 gate_rank: int, eps: float = 1e-6, names: Optional[Dict[str, str]] = None):
        _check("delta rule", heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv_taps=conv_taps, decay_rank=decay_rank,
               gate_rank=gate_rank)
        if heads % kv_heads:
            raise ValueError(f"{heads} heads are not a multiple of {kv_heads} query/key heads")
        self.width, self.heads, self.kv_heads, self.dim, self.vdim, self.taps = width, heads, kv_heads, dim, vdim, conv_taps
        self.decay_rank, self.gate_rank, self.eps = decay_rank, gate_rank, float(eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.qk_cols, self.v_cols = kv_heads * dim, heads * vdim
        self.channels = 2 * self.qk_cols + self.v_cols
        # columns of the stacked product: q | k | v | decay, down | gate, down | beta
        self.low0 = _padded(self.channels)
        self.low_cols = _padded(decay_rank) + _padded(gate_rank)
        self.beta0 = self.low0 + self.low_cols
        self.in_cols = _padded(self.beta0 + heads)
        self.w_in = self.w_low = self.conv_t = self.decay_bias = self.decay_log = self.norm = self.w_o = None

    def cache_need(self):
        """A head's value columns one after the other."""
        return SlotStateNeed((self.heads, self.vdim, self.dim), torch.float32)

    def state_need(self):
        """The convolution's inputs of the last ``taps - 1`` positions."""
        return SlotStateNeed((self.taps - 1, self.channels), torch.float32) if self.taps > 1 else None

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        n = self.names
        specs = []
        for key, cols in (("q", self.qk_cols), ("k", self.qk_cols), ("v", self.v_cols)):
            specs += [ParamSpec(f"{prefix}.{n[key]}", (cols, self.width), MATRIX),
                      ParamSpec(f"{prefix}.{n[key]}{n['conv']}", (cols, self.taps), KEEP32)]
        return specs + [ParamSpec(f"{prefix}.{n['beta']}", (self.heads, self.width), MATRIX),
                        ParamSpec(f"{prefix}.{n['decay_log']}", (self.heads,), KEEP32),
                        ParamSpec(f"{prefix}.{n['norm']}", (self.vdim,), KEEP32, init="ones"),
                        ParamSpec(f"{prefix}.{n['decay_down']}", (self.decay_rank, self.width), MATRIX),
                        ParamSpec(f"{prefix}.{n['decay_up']}", (self.heads * self.dim, self.decay_rank), MATRIX),
                        ParamSpec(f"{prefix}.{n['decay_bias']}", (self.heads * self.dim,), KEEP32),
                        ParamSpec(f"{prefix}.{n['gate_down']}", (self.gate_rank, self.width), MATRIX),
                        ParamSpec(f"{prefix}.{n['gate_up']}", (self.v_cols, self.gate_rank), MATRIX),
                        ParamSpec(f"{prefix}.{n['out']}", (self.width, self.v_cols), MATRIX)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        t = {k: state[f"{prefix}.{v}"] for k, v in self.names.items() if k != "conv"}
        qkv = stacked_rows([t["q"], t["k"], t["v"]])
        low = torch.cat([stacked_rows([t["decay_down"]]), stacked_rows([t["gate_down"]])], 0)
        self.w_in = torch.cat([qkv, low, stacked_rows([t["beta"]])], 0).contiguous()
        # both second projections in one product over [decay, down | gate, down]; the blocks off the diagonal are zero
        a, g = t["decay_up"], t["gate_up"]
        self.w_low = torch.zeros(a.shape[0] + g.shape[0], self.low_cols, dtype=a.dtype, device=a.device)
        self.w_low[:a.shape[0], :self.decay_rank] = a
        self.w_low[a.shape[0]:, _padded(self.decay_rank):_padded(self.decay_rank) + self.gate_rank] = g
        self.conv_t = torch.cat([state[f"{prefix}.{self.names[k]}{self.names['conv']}"] for k in ("q", "k", "v")],
                                0).t().contiguous()
        self.decay_bias, self.decay_log, self.norm, self.w_o = t["decay_bias"], t["decay_log"], t["norm"], t["out"]

    def _tensors(self):
        return (self.w_in, self.w_low, self.conv_t, self.decay_bias, self.decay_log, self.norm, self.w_o)

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, cache: SlotStateView,
                accumulate: bool = True) -> None:
        """``accumulate`` False: the output is written to ``x`` instead of added to it."""
        ops, ws, n, H = ctx.ops, ctx.workspace, ctx.n, self.heads
        tiles = ctx.query_tiles(SEQUENCE_TILE)
        conv_state = cache.beside.state if self.taps > 1 else None
        u = ws.rows("delta_in32", n, self.in_cols, torch.float32)
        ops.linear(xn, self.w_in, u)
        low = ws.rows("delta_low", n, self.low_cols, ctx.act_dtype)
        ops.activate_rows(u[:, self.low0:self.beta0], low)
        z = ws.rows("delta_low32", n, H * self.dim + self.v_cols, torch.float32)
        ops.linear(low, self.w_low, z)
        decay, gate = z[:, :H * self.dim], z[:, H * self.dim:]
        ready = ws.rows("delta_ready32", n, _padded(self.channels + H + self.kv_heads), torch.float32)
        keep = one_row_each(ctx)
        ops.delta_prepare(u, self.beta0, self.conv_t, conv_state, decay, self.decay_bias, self.decay_log, ready, ctx, H,
                          self.kv_heads, self.dim, self.vdim, self.dim ** -0.5, keep=keep)
        if conv_state is not None and not keep:
            ops.conv_state_update(u[:, :self.channels], conv_state, ctx, self.taps, tiles)
        o = ws.rows("scan_out32", n, self.v_cols, torch.float32)
        a, b, c = self.qk_cols, 2 * self.qk_cols, self.channels
        ops.state_scan("delta", ready[:, :a], ready[:, a:b], ready[:, b:c], cache.state, o, ctx, tiles, H, self.dim, self.vdim,
                       decay=decay, beta=ready[:, c:c + H], qk=ready[:, c + H:c + H + self.kv_heads])
        gated = ws.rows("scan_gated", n, self.v_cols, ctx.act_dtype)
        ops.scan_finish(o, self.norm, gate, self.eps, gated, H, self.vdim)
        ops.linear(gated, self.w_o, x, residual=x if accumulate else None)


class ShiftedRecurrence(_StateMixer):
    reads_stream = True  # the mixes are formed from the float32 rows

    NAMES = {"mix": "mu.{}", "r": "r", "k": "k", "v": "v", "gate": "g", "decay_down": "w1", "decay_up": "w2", "decay_bias": "w0",
             "bonus": "u", "norm": "norm", "out": "o"}
    MIXES = ("r", "k", "v", "g", "w")

    def __init__(self, width: int, heads: int, dim: int, decay_rank: int, eps: float = 1e-6,
                 names: Optional[Dict[str, str]] = None):
        _check("shifted recurrence", heads=heads, dim=dim, decay_rank=decay_rank)
        self.width, self.heads, self.dim, self.decay_rank, self.eps = width, heads, dim, decay_rank, float(eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.cols = heads * dim
        self.mu = self.w = self.w_down = self.w_up = self.decay_bias = self.bonus = self.norm = self.w_o = None

    def cache_need(self):
        return SlotStateNeed((self.heads, self.dim, self.dim), torch.float32)

    def state_need(self):
        """The previous row of the stream."""
        return SlotStateNeed((1, self.width), torch.float32)

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        n = self.names
        specs = [ParamSpec(f"{prefix}.{n['mix'].format(s)}", (self.width,), KEEP32) for s in self.MIXES]
        specs += [ParamSpec(f"{prefix}.{n[k]}", (self.cols, self.width), MATRIX) for k in ("r", "k", "v", "gate")]
        return specs + [ParamSpec(f"{prefix}.{n['decay_down']}", (self.decay_rank, self.width), MATRIX),
                        ParamSpec(f"{prefix}.{n['decay_up']}", (self.cols, self.decay_rank), MATRIX),
                        ParamSpec(f"{prefix}.{n['decay_bias']}", (self.cols,), KEEP32),
                        ParamSpec(f"{prefix}.{n['bonus']}", (self.heads, self.dim), KEEP32),
                        ParamSpec(f"{prefix}.{n['norm']}", (self.cols,), KEEP32, init="ones"),
                        ParamSpec(f"{prefix}.{n['out']}", (self.width, self.cols), MATRIX)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        n = self.names
        self.mu = torch.stack([state[f"{prefix}.{n['mix'].format(s)}"] for s in self.MIXES]).contiguous()
        self.w = [state[f"{prefix}.{n[k]}"] for k in ("r", "k", "v", "gate")]
        self.w_down = stacked_rows([state[f"{prefix}.{n['decay_down']}"]])
        up = state[f"{prefix}.{n['decay_up']}"]
        self.w_up = torch.zeros(up.shape[0], self.w_down.shape[0], dtype=up.dtype, device=up.device)
        self.w_up[:, :self.decay_rank] = up
        self.decay_bias, self.bonus = state[f"{prefix}.{n['decay_bias']}"], state[f"{prefix}.{n['bonus']}"]
        self.norm, self.w_o = state[f"{prefix}.{n['norm']}"], state[f"{prefix}.{n['out']}"]

    def _tensors(self):
        return (self.mu, *self.w, self.w_down, self.w_up, self.decay_bias, self.bonus, self.norm, self.w_o)

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, cache: SlotStateView,
                accumulate: bool = True) -> None:
        """``xn``: the float32 rows (``reads_stream``).  ``accumulate`` False: the output is written to ``x``."""
        ops, ws, n = ctx.ops, ctx.workspace, ctx.n
        tiles = ctx.query_tiles(SEQUENCE_TILE)
        mixes = ws.rows("shift_mixes", n, 5 * self.width, ctx.act_dtype).view(5, n, self.width)
        last = cache.beside.state
        keep = one_row_each(ctx)
        ops.shift_mix(xn, self.mu, last, mixes, ctx, keep=keep)
        if not keep:
            ops.conv_state_update(xn, last, ctx, 2, tiles)
        r, k, v, gate = (ws.rows(f"shift_{s}32", n, self.cols, torch.float32) for s in "rkvg")
        for s, (w, dst) in enumerate(zip(self.w, (r, k, v, gate))):
            ops.linear(mixes[s], w, dst)
        low = ws.rows("shift_low", n, self.w_down.shape[0], ctx.act_dtype)
        ops.linear(mixes[4], self.w_down, low, activation="tanh")
        z = ws.rows("shift_z32", n, self.cols, torch.float32)
        ops.linear(low, self.w_up, z)
        o = ws.rows("scan_out32", n, self.cols, torch.float32)
        ops.state_scan("bonus", r, k, v, cache.state, o, ctx, tiles, self.heads, self.dim, self.dim, decay=z,
                       decay_bias=self.decay_bias, bonus=self.bonus)
        gated = ws.rows("scan_gated", n, self.cols, ctx.act_dtype)
        ops.scan_finish(o, self.norm, gate, self.eps, gated, self.heads, self.dim, gate_kind="silu")
        ops.linear(gated, self.w_o, x, residual=x if accumulate else None)


class MatrixMemory(_StateMixer):
    stacks_input = True  # ``w_in`` is one product of the mixer's input, and ``forward`` takes its result ready-made

    NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "input": "i", "forget": "f", "bias": ".b", "norm": "norm", "out": "o"}

    def __init__(self, width: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float = 1e-6,
                 names: Optional[Dict[str, str]] = None):
        _check("matrix memory", heads=heads, dim=dim, vdim=vdim, gate_cap=gate_cap)
        self.width, self.heads, self.dim, self.vdim = width, heads, dim, vdim
        self.gate_cap, self.eps = float(gate_cap), float(eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.qk_cols, self.v_cols = heads * dim, heads * vdim
        self.in_cols = _padded(2 * self.qk_cols + 2 * self.v_cols + 2 * heads)
        self.w_in = self.input_bias = self.forget_bias = self.norm = self.w_o = None

    def cache_need(self):
        """Per head the value columns and the normaliser as one more, each followed by the running maximum (every column
        keeps its own copy, so that the thread blocks of a head share nothing) and three spare numbers."""
        return SlotStateNeed((self.heads, self.vdim + 1, self.dim + 4), torch.float32)

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        n = self.names
        return [ParamSpec(f"{prefix}.{n['q']}", (self.qk_cols, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['k']}", (self.qk_cols, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['v']}", (self.v_cols, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['gate']}", (self.v_cols, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['out']}", (self.width, self.v_cols), MATRIX),
                ParamSpec(f"{prefix}.{n['norm']}", (self.v_cols,), KEEP32, init="ones"),
                ParamSpec(f"{prefix}.{n['input']}", (self.heads, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['input']}{n['bias']}", (self.heads,), KEEP32),
                ParamSpec(f"{prefix}.{n['forget']}", (self.heads, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['forget']}{n['bias']}", (self.heads,), KEEP32)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        n = self.names
        # one product yields rows laid out [q | k | v | gate | input gate | forget gate]
        self.w_in = stacked_rows([state[f"{prefix}.{n[k]}"] for k in ("q", "k", "v", "gate", "input", "forget")])
        self.input_bias = state[f"{prefix}.{n['input']}{n['bias']}"]
        self.forget_bias = state[f"{prefix}.{n['forget']}{n['bias']}"]
        self.norm, self.w_o = state[f"{prefix}.{n['norm']}"], state[f"{prefix}.{n['out']}"]

    def _tensors(self):
        return (self.w_in, self.input_bias, self.forget_bias, self.norm, self.w_o)

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, cache: SlotStateView,
                accumulate: bool = True, projected: Optional[torch.Tensor] = None) -> None:
        """``accumulate`` False: the output is written to ``x`` instead of added to it.  ``projected``: the product
        of ``xn`` with ``w_in`` (float32 rows) where the caller has formed it."""
        ops, ws, n, H = ctx.ops, ctx.workspace, ctx.n, self.heads
        u = projected
        if u is None:
            u = ws.rows("memory_in32", n, self.in_cols, torch.float32)
            ops.linear(xn, self.w_in, u)
        a, b, c = self.qk_cols, 2 * self.qk_cols, 2 * self.qk_cols + self.v_cols
        d = c + self.v_cols
        o = ws.rows("scan_out32", n, self.v_cols, torch.float32)
        aux = ws.rows("scan_aux32", n, 2 * H, torch.float32)
        ops.state_scan("memory", u[:, :a], u[:, a:b], u[:, b:c], cache.state, o, ctx, ctx.query_tiles(SEQUENCE_TILE), H, self.dim,
                       self.vdim, inp=u[:, d:d + H], forget=u[:, d + H:d + 2 * H], inp_bias=self.input_bias,
                       forget_bias=self.forget_bias, cap=self.gate_cap, aux=aux)
        gated = ws.rows("scan_gated", n, self.v_cols, ctx.act_dtype)
        ops.scan_finish(o, self.norm, u[:, c:d], self.eps, gated, H, self.vdim, aux=aux, q_scale=self.dim ** -0.5)
        ops.linear(gated, self.w_o, x, residual=x if accumulate else None)


class StateSpace(_StateMixer):
    """Per head h with vdim values and a state of ``state`` numbers each: ``t = ln(1 + e^(dt + dt_bias_h))``, ``S <- e^(-e^(A_log_h)
    t) S + t B x^T``, ``y = S^T C + D_h x``.  B and C belong to ``groups`` groups of heads.  One projection gives [z | x | B | C |
    dt]; x, B and C pass a causal convolution over time with a bias, and SiLU.  The row y is multiplied by ``silu(z)``, each of
    its ``norm_groups`` equal parts divided by its own root mean square, times a weight, and projected by W_o."""

    NAMES = {"in": "in", "out": "o", "conv": "conv", "conv_bias": "conv.b", "step_bias": "dt_bias", "decay_log": "A_log", "skip": "D",
             "norm": "norm"}

    def __init__(self, width: int, heads: int, vdim: int, state: int, groups: int, conv_taps: int, norm_groups: int = 1,
                 eps: float = 1e-6, names: Optional[Dict[str, str]] = None):
        _check("state space", heads=heads, vdim=vdim, state=state, groups=groups, conv_taps=conv_taps, norm_groups=norm_groups)
        if heads % groups:
            raise ValueError(f"{heads} heads are not a multiple of {groups} groups")
        if heads * vdim % norm_groups:
            raise ValueError(f"{heads * vdim} entries do not form {norm_groups} equal parts")
        self.width, self.heads, self.vdim, self.state, self.groups = width, heads, vdim, state, groups
        self.taps, self.norm_groups, self.eps = conv_taps, norm_groups, float(eps)
        self.names = dict(self.NAMES, **(names or {}))
        self.inner = heads * vdim
        self.channels = self.inner + 2 * groups * state
        self.step0 = self.inner + self.channels             # where the steps' columns of the projection begin
        self.w_in = self.conv_t = self.conv_b = self.step_bias = self.rate = self.skip = self.norm = self.w_o = None

    def cache_need(self):
        """A head's value columns one after the other."""
        return SlotStateNeed((self.heads, self.vdim, self.state), torch.float32)

    def state_need(self):
        """The convolution's inputs of the last ``taps - 1`` positions."""
        return SlotStateNeed((self.taps - 1, self.channels), torch.float32) if self.taps > 1 else None

    def param_specs(self, prefix: str) -> List[ParamSpec]:
        n = self.names
        return [ParamSpec(f"{prefix}.{n['in']}", (self.step0 + self.heads, self.width), MATRIX),
                ParamSpec(f"{prefix}.{n['conv']}", (self.channels, self.taps), KEEP32),
                ParamSpec(f"{prefix}.{n['conv_bias']}", (self.channels,), KEEP32),
                ParamSpec(f"{prefix}.{n['step_bias']}", (self.heads,), KEEP32),
                ParamSpec(f"{prefix}.{n['decay_log']}", (self.heads,), KEEP32),
                ParamSpec(f"{prefix}.{n['skip']}", (self.heads,), KEEP32, init="ones"),
                ParamSpec(f"{prefix}.{n['norm']}", (self.inner,), KEEP32, init="ones"),
                ParamSpec(f"{prefix}.{n['out']}", (self.width, self.inner), MATRIX)]

    def load_params(self, state: Dict[str, torch.Tensor], prefix: str) -> None:
        t = {k: state[f"{prefix}.{v}"] for k, v in self.names.items()}
        self.w_in = stacked_rows([t["in"]], 64)  # (whole pieces of 64 columns: what the product's wide tiles take)
        self.conv_t, self.conv_b = t["conv"].t().contiguous(), t["conv_bias"]
        self.step_bias, self.skip, self.norm, self.w_o = t["step_bias"], t["skip"], t["norm"], t["out"]
        self.rate = torch.exp(t["decay_log"].double()).float()

    def _tensors(self):
        return (self.w_in, self.conv_t, self.conv_b, self.step_bias, self.rate, self.skip, self.norm, self.w_o)

    def forward(self, ctx: StepContext, xn: torch.Tensor, x: torch.Tensor, cache: SlotStateView,
                accumulate: bool = True, then: Optional[tuple] = None) -> None:
        """``accumulate`` False: the output is written to ``x`` instead of added to it.  ``then``: the norm that follows on
        the finished rows (``TanhNorm.after``)."""
        ops, ws, n, H, ch = ctx.ops, ctx.workspace, ctx.n, self.heads, self.channels
        tiles = ctx.query_tiles(SEQUENCE_TILE)
        conv_state = cache.beside.state if self.taps > 1 else None
        u = ws.rows("space_in32", n, self.w_in.shape[0], torch.float32)
        ops.linear(xn, self.w_in, u)
        step = _padded(ch)
        ready = ws.rows("space_ready32", n, _padded(step + 2 * H), torch.float32)
        keep = one_row_each(ctx)
        ops.space_prepare(u, self.inner, self.step0, self.conv_t, self.conv_b, conv_state, self.step_bias, self.rate, ready, step, ctx,
                          keep=keep)
        if conv_state is not None and not keep:
            ops.conv_state_update(u[:, self.inner:self.step0], conv_state, ctx, self.taps, tiles)
        o = ws.rows("scan_out32", n, self.inner, torch.float32)
        b, c = self.inner, self.inner + self.groups * self.state
        ops.state_scan("space", ready[:, c:ch], ready[:, b:c], ready[:, :b], cache.state, o, ctx, tiles, H, self.state, self.vdim,
                       step=ready[:, step:step + H], decay=ready[:, step + H:step + 2 * H], skip=self.skip)
        gated = ws.rows("scan_gated", n, self.inner, ctx.act_dtype)
        ops.gated_group_norm(o, u[:, :self.inner], self.norm, self.eps, gated, self.norm_groups)
        ops.linear(gated, self.w_o, x, residual=x if accumulate else None, **({"then": then} if then else {}))


register_mixer("channel_delta", ChannelDelta)
register_mixer("state_space", StateSpace)
register_mixer("shifted_recurrence", ShiftedRecurrence)
register_mixer("matrix_memory", MatrixMemory)
