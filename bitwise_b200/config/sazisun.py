"""Typed configuration of the Sazisun design, read from config.json.

Keys: ``architecture`` ("Sazisun"), ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list with one entry per layer:
``type`` (``attention`` or ``mamba2``), ``mixer`` and ``mlp`` (null for none).  A mixer's keys by type:

* ``attention``: ``heads``, ``kv_heads``, ``dim`` (per map), ``vdim``, ``scale``, ``diff`` and optionally ``softcap``, ``rot.base`` /
  ``rot.dims`` / ``rot.scaling.{factor, low, high, original}`` and ``kv_from``, the earlier attention layer whose keys and values
  the layer reads;
* ``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` (taps of the short convolution), ``norm_groups``.

A feed-forward is ``kind`` "dense" with ``ff``, or "moe" with ``expert.ff``, ``router.{experts, top, scale}``, optionally
``router.groups.{count, keep}`` and ``shared.ff``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError

MIXER_TYPES = ("attention", "mamba2")


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


def _multiple(a: int, b: int, where: str, what: str) -> None:
    if a % b:
        raise ConfigError(f"config.json: {where}: {a} is no multiple of {b} ({what})")


@dataclass(frozen=True)
class WavelengthScalingConfig:
    factor: float
    low: float
    high: float
    original: float

    @staticmethod
    def from_json(d: dict, where: str) -> "WavelengthScalingConfig":
        c = WavelengthScalingConfig(*(_positive(_get(d, k, where), f"{where}.{k}") for k in ("factor", "low", "high", "original")))
        if c.low > c.high:
            raise ConfigError(f"config.json: {where}: low = {c.low} is above high = {c.high}")
        return c

    def to_json(self) -> dict:
        return {"factor": self.factor, "high": self.high, "low": self.low, "original": self.original}


@dataclass(frozen=True)
class TwoMapAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    softcap: Optional[float] = None
    rot_base: Optional[float] = None
    rot_dims: Optional[int] = None      # how many leading entries of a map's head turn
    rot_scaling: Optional[WavelengthScalingConfig] = None
    kv_from: Optional[int] = None

    kind = "attention"

    @staticmethod
    def from_json(d: dict, where: str) -> "TwoMapAttentionConfig":
        heads, kv_heads, dim, vdim = (_int_of(d, k, where) for k in ("heads", "kv_heads", "dim", "vdim"))
        _multiple(heads, kv_heads, where, "heads on key/value heads")
        rot = d.get("rot")
        base = dims = scaling = None
        if rot is not None:
            base = _positive(_get(rot, "base", where + ".rot"), where + ".rot.base")
            dims = _int_of(rot, "dims", where + ".rot")
            if dims > dim or dims % 2:
                raise ConfigError(f"config.json: {where}.rot.dims = {dims} must be even and at most dim = {dim}")
            if rot.get("scaling") is not None:
                scaling = WavelengthScalingConfig.from_json(rot["scaling"], where + ".rot.scaling")
        cap = d.get("softcap")
        return TwoMapAttentionConfig(heads, kv_heads, dim, vdim, float(_get(d, "scale", where)), float(_get(d, "diff", where)),
                                     None if cap is None else _positive(cap, where + ".softcap"), base, dims, scaling, d.get("kv_from"))

    def to_json(self) -> dict:
        d = {"diff": self.diff, "dim": self.dim, "heads": self.heads, "kv_heads": self.kv_heads, "scale": self.scale, "vdim": self.vdim}
        if self.softcap is not None:
            d["softcap"] = self.softcap
        if self.rot_dims is not None:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.rot_scaling is not None:
                d["rot"]["scaling"] = self.rot_scaling.to_json()
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d

    def shared_sizes(self):
        """What a layer and the one whose keys and values it reads have in common."""
        return (self.heads, self.kv_heads, self.dim, self.vdim, self.rot_base, self.rot_dims, self.rot_scaling)


@dataclass(frozen=True)
class StateSpaceConfig:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    kind = "mamba2"

    @staticmethod
    def from_json(d: dict, where: str) -> "StateSpaceConfig":
        c = StateSpaceConfig(*(_int_of(d, k, where) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        _multiple(c.heads, c.groups, where, "heads in groups")
        _multiple(c.heads * c.vdim, c.norm_groups, where, "entries in norm_groups")
        return c

    def to_json(self) -> dict:
        return {"conv": self.conv, "groups": self.groups, "heads": self.heads, "norm_groups": self.norm_groups, "state": self.state,
                "vdim": self.vdim}


@dataclass(frozen=True)
class FeedForwardConfig:
    ff: int

    kind = "dense"

    @staticmethod
    def from_json(d: dict, where: str) -> "FeedForwardConfig":
        return FeedForwardConfig(_int_of(d, "ff", where))

    def to_json(self) -> dict:
        return {"ff": self.ff, "kind": "dense"}


@dataclass(frozen=True)
class ExpertsConfig:
    ff: int
    experts: int
    top: int
    scale: float = 1.0
    groups: int = 1
    keep_groups: int = 1
    shared_ff: Optional[int] = None

    kind = "moe"

    @staticmethod
    def from_json(d: dict, where: str) -> "ExpertsConfig":
        router, at = _get(d, "router", where), where + ".router"
        groups, shared = router.get("groups"), d.get("shared")
        c = ExpertsConfig(_int_of(_get(d, "expert", where), "ff", where + ".expert"), _int_of(router, "experts", at),
                          _int_of(router, "top", at), float(router.get("scale", 1.0)),
                          _int_of(groups, "count", at + ".groups") if groups else 1,
                          _int_of(groups, "keep", at + ".groups") if groups else 1,
                          _int_of(shared, "ff", where + ".shared") if shared else None)
        _multiple(c.experts, c.groups, at, "experts in groups")
        if c.keep_groups > c.groups or c.top > c.keep_groups * (c.experts // c.groups):
            raise ConfigError(f"config.json: {at}: {c.top} choices among {c.keep_groups} of {c.groups} groups of {c.experts} experts")
        return c

    def to_json(self) -> dict:
        return {"expert": {"ff": self.ff}, "kind": "moe",
                "router": {"experts": self.experts, "groups": {"count": self.groups, "keep": self.keep_groups}, "scale": self.scale,
                           "top": self.top},
                "shared": {"ff": self.shared_ff} if self.shared_ff else None}


_MIXERS = {c.kind: c for c in (TwoMapAttentionConfig, StateSpaceConfig)}
_FEED_FORWARDS = {c.kind: c for c in (FeedForwardConfig, ExpertsConfig)}


@dataclass(frozen=True)
class SazisunLayerConfig:
    mixer: object                      # TwoMapAttentionConfig or StateSpaceConfig
    mlp: Optional[object] = None       # FeedForwardConfig or ExpertsConfig; None: the layer has no feed-forward


@dataclass(frozen=True)
class SazisunConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[SazisunLayerConfig, ...]
    architectures: tuple = ("Sazisun",)
    eos_token_id: int = -1

    architecture_name = "Sazisun"

    def __post_init__(self):
        _positive_int(self.vocab, "vocab")
        _positive_int(self.width, "width")
        if not self.eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {self.eps!r}")
        if not self.layers:
            raise ConfigError("config.json: no layers")
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            j = getattr(m, "kv_from", None)
            if j is None:
                continue
            if not isinstance(j, int) or isinstance(j, bool) or not 0 <= j < i or self.layers[j].mixer.kind != "attention" or \
                    self.layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from = {j!r} is no earlier attention layer with keys of its own")
            if self.layers[j].mixer.shared_sizes() != m.shared_sizes():
                raise ConfigError(f"config.json: layers {i} and {j} share keys and values and differ in their heads or rotation")

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @staticmethod
    def from_json(d: dict) -> "SazisunConfig":
        layers = []
        for i, entry in enumerate(_get(d, "layers", "the model")):
            where = f"layers[{i}]"
            kind = _get(entry, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"config.json: {where} has the unknown type {kind!r} (known: {', '.join(MIXER_TYPES)})")
            mixer = _MIXERS[kind].from_json(_get(entry, "mixer", where), where + ".mixer")
            mlp = entry.get("mlp")
            if mlp:
                ff = mlp.get("kind", "dense")
                if ff not in _FEED_FORWARDS:
                    raise ConfigError(f"config.json: {where}.mlp.kind = {ff!r} is not supported (supported: 'dense', 'moe')")
                mlp = _FEED_FORWARDS[ff].from_json(mlp, where + ".mlp")
            layers.append(SazisunLayerConfig(mixer, mlp or None))
        eos = d.get("eos_token_id", -1)
        return SazisunConfig(vocab=_get(d, "vocab", "the model"), width=_get(d, "width", "the model"),
                             eps=float(_get(_get(d, "norm", "the model"), "eps", "norm")), layers=tuple(layers),
                             eos_token_id=-1 if eos is None else int(eos))

    def to_json(self) -> dict:
        return {"architecture": "Sazisun",
                "layers": [{"mixer": l.mixer.to_json(), "mlp": l.mlp.to_json() if l.mlp else None, "type": l.mixer.kind}
                           for l in self.layers],
                "norm": {"eps": self.eps}, "vocab": self.vocab, "width": self.width}
