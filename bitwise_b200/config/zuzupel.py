"""Typed configuration of the Zuzupel design, read from config.json.

Keys: ``architecture`` ("Zuzupel"), ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list with one entry per layer:
``type`` (``wkv``, ``channel_delta`` or ``parallel``), ``mixer``, ``mlp`` (null for none, else ``kind`` "dense" with ``ff``)
and optionally ``weights_of``, the earlier layer whose tensors the layer uses (the rest of its entry equals that
layer's).  A mixer's keys by type:

* ``wkv``: ``heads``, ``dim``;
* ``channel_delta``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps of the short convolution);
* ``parallel``: ``left`` with ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale`` and optionally ``rot.base`` / ``rot.dims`` /
  ``rot.scaling.factor`` and ``mask.size`` (the chunk); ``right`` with ``heads``, ``dim``, ``vdim``, ``gate_cap``.

The inner sizes of the low-rank projections are tensors' shapes (``with_tensor_shapes``).
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Optional, Tuple

from .base import ConfigError

MIXER_TYPES = ("wkv", "channel_delta", "parallel")


def _get(d, key: str, where: str):
    if not isinstance(d, dict) or key not in d:
        raise ConfigError(f"config.json: {where} lacks the key {key!r}")
    return d[key]


def _positive_int(v, what: str) -> int:
    if not isinstance(v, int) or isinstance(v, bool) or v <= 0:
        raise ConfigError(f"config.json: {what} must be a positive integer, got {v!r}")
    return v


def _int_of(d, key: str, where: str) -> int:
    return _positive_int(_get(d, key, where), f"{where}.{key}")


def _positive(v, what: str) -> float:
    v = float(v)
    if not v > 0:
        raise ConfigError(f"config.json: {what} must be positive, got {v!r}")
    return v


def _whole_groups(heads: int, kv_heads: int, where: str) -> None:
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: {heads} heads are no multiple of {kv_heads} key/value heads")


@dataclass(frozen=True)
class WkvConfig:
    heads: int
    dim: int
    decay_rank: Optional[int] = None  # a tensor's shape, no key of config.json

    kind = "wkv"

    @staticmethod
    def from_json(d: dict, where: str) -> "WkvConfig":
        return WkvConfig(_int_of(d, "heads", where), _int_of(d, "dim", where))

    def to_json(self) -> dict:
        return {"dim": self.dim, "heads": self.heads}


@dataclass(frozen=True)
class ChannelDeltaConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: Optional[int] = None  # tensors' shapes, no keys of config.json
    gate_rank: Optional[int] = None

    kind = "channel_delta"

    @staticmethod
    def from_json(d: dict, where: str) -> "ChannelDeltaConfig":
        c = ChannelDeltaConfig(*(_int_of(d, k, where) for k in ("heads", "kv_heads", "dim", "vdim", "conv")))
        _whole_groups(c.heads, c.kv_heads, where)
        return c

    def to_json(self) -> dict:
        return {"conv": self.conv, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "vdim": self.vdim}


@dataclass(frozen=True)
class ChunkAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: Optional[float] = None
    rot_dims: Optional[int] = None     # how many leading entries of a head turn
    rot_factor: Optional[float] = None  # every rotary frequency is divided by it
    chunk: Optional[int] = None

    @staticmethod
    def from_json(d: dict, where: str) -> "ChunkAttentionConfig":
        heads, kv_heads, dim, vdim = (_int_of(d, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
        _whole_groups(heads, kv_heads, where)
        rot, mask = d.get("rot"), d.get("mask")
        base = dims = factor = None
        if rot is not None:
            base = _positive(_get(rot, "base", where + ".rot"), where + ".rot.base")
            dims = _int_of(rot, "dims", where + ".rot")
            if dims > dim or dims % 2:
                raise ConfigError(f"config.json: {where}.rot.dims = {dims} must be even and at most dim = {dim}")
            if rot.get("scaling") is not None:
                factor = _positive(_get(rot["scaling"], "factor", where + ".rot.scaling"), where + ".rot.scaling.factor")
        return ChunkAttentionConfig(heads, kv_heads, dim, vdim, float(_get(d, "scale", where)), base, dims, factor,
                                    _int_of(mask, "size", where + ".mask") if mask is not None else None)

    def to_json(self) -> dict:
        d = {"dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.chunk is not None:
            d["mask"] = {"size": self.chunk}
        if self.rot_dims is not None:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_factor is not None:
                d["rot"]["scaling"] = {"factor": self.rot_factor}
        return d


@dataclass(frozen=True)
class MatrixMemoryConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_json(d: dict, where: str) -> "MatrixMemoryConfig":
        return MatrixMemoryConfig(*(_int_of(d, k, where) for k in ("heads", "dim", "vdim")),
                                  _positive(_get(d, "gate_cap", where), where + ".gate_cap"))

    def to_json(self) -> dict:
        return {"dim": self.dim, "gate_cap": self.gate_cap, "heads": self.heads, "vdim": self.vdim}


@dataclass(frozen=True)
class ParallelConfig:
    left: ChunkAttentionConfig
    right: MatrixMemoryConfig

    kind = "parallel"

    @staticmethod
    def from_json(d: dict, where: str) -> "ParallelConfig":
        return ParallelConfig(ChunkAttentionConfig.from_json(_get(d, "left", where), where + ".left"),
                              MatrixMemoryConfig.from_json(_get(d, "right", where), where + ".right"))

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "right": self.right.to_json()}


_MIXERS = {c.kind: c for c in (WkvConfig, ChannelDeltaConfig, ParallelConfig)}


@dataclass(frozen=True)
class ZuzupelLayerConfig:
    mixer: object                      # WkvConfig, ChannelDeltaConfig or ParallelConfig
    ff: Optional[int] = None           # inner size of the feed-forward; None: the layer has none
    weights_of: Optional[int] = None   # the layer whose tensors this one uses


@dataclass(frozen=True)
class ZuzupelConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[ZuzupelLayerConfig, ...]
    architectures: tuple = ("Zuzupel",)
    eos_token_id: int = -1

    architecture_name = "Zuzupel"

    def __post_init__(self):
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        if not self.eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {self.eps!r}")
        if not self.layers:
            raise ConfigError("config.json: no layers")
        for i, layer in enumerate(self.layers):
            if layer.weights_of is None:
                continue
            j = self.owner(i)
            other = self.layers[j]
            if layer.mixer.to_json() != other.mixer.to_json() or layer.mixer.kind != other.mixer.kind or layer.ff != other.ff:
                raise ConfigError(f"config.json: layers {i} and {j} share weights and differ in their sizes")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        seen = [i]
        while self.layers[seen[-1]].weights_of is not None:
            j = self.layers[seen[-1]].weights_of
            if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < len(self.layers) or j in seen:
                raise ConfigError(f"config.json: layer {seen[-1]} uses the weights of layer {j!r}, which is no other layer with "
                                  f"tensors of its own")
            seen.append(j)
        return seen[-1]

    def with_tensor_shapes(self, shapes) -> "ZuzupelConfig":
        """The sizes that only a checkpoint's tensors give (name -> shape): the inner sizes of the low-rank projections
        are the row counts of ``l<i>.mix.w1`` (wkv) and ``l<i>.mix.a1`` / ``.g1`` (channel_delta)."""

        def rows(i: int, name: str):
            shape = shapes.get(f"l{self.owner(i)}.mix.{name}")
            return int(shape[0]) if shape is not None and len(shape) == 2 else None

        layers = []
        for i, layer in enumerate(self.layers):
            if layer.mixer.kind == "wkv":
                layer = replace(layer, mixer=replace(layer.mixer, decay_rank=rows(i, "w1")))
            elif layer.mixer.kind == "channel_delta":
                layer = replace(layer, mixer=replace(layer.mixer, decay_rank=rows(i, "a1"), gate_rank=rows(i, "g1")))
            layers.append(layer)
        return replace(self, layers=tuple(layers))

    @staticmethod
    def from_json(d: dict) -> "ZuzupelConfig":
        layers = []
        for i, entry in enumerate(_get(d, "layers", "the model")):
            where = f"layers[{i}]"
            kind = _get(entry, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where} has the unknown type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            mixer = _MIXERS[kind].from_json(_get(entry, "mixer", where), where + ".mixer")
            mlp, ff = entry.get("mlp"), None
            if mlp:
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind = {mlp.get('kind')!r} is not supported (supported: 'dense')")
                ff = _int_of(mlp, "ff", where + ".mlp")
            layers.append(ZuzupelLayerConfig(mixer, ff, entry.get("weights_of")))
        eos = d.get("eos_token_id", -1)
        return ZuzupelConfig(vocab=_get(d, "vocab", "the model"), width=_get(d, "width", "the model"),
                             eps=float(_get(_get(d, "norm", "the model"), "eps", "norm")), layers=tuple(layers),
                             eos_token_id=-1 if eos is None else int(eos))

    def to_json(self) -> dict:
        layers = []
        for l in self.layers:
            e = {"mixer": l.mixer.to_json(), "mlp": {"ff": l.ff, "kind": "dense"} if l.ff else None, "type": l.mixer.kind}
            if l.weights_of is not None:
                e["weights_of"] = l.weights_of
            layers.append(e)
        return {"architecture": "Zuzupel", "layers": layers, "norm": {"eps": self.eps}, "vocab": self.vocab, "width": self.width}
