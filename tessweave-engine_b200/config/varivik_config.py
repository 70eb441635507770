"""Typed view of a Varivik ``config.json``.

The file names the design under ``architecture`` and gives the residual width, the vocabulary, the norms' eps and a list
of layers.  Every layer's mixer (``type: attention``) is softmax attention with grouped heads, keys and values of their
own sizes, a rotation of neighbouring pairs over the first part of a head (optionally with scaled frequencies), chunks
of positions that see only themselves, a gate per head, and, where ``v_mix`` is set, values blended with those of the
first such layer.  A layer's feed-forward under ``mlp`` is ``dense`` (gated, with biases), ``moe`` (routed experts
without gates, optionally with a shared one) or null.  Every size and constant comes from here; anything this engine
does not implement is refused before a weight is read.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path

from .linurax_config import _finite, _need, _positive_int
from .model_config import ConfigError

MAX_HEAD = 1024         # the attention kernels' largest head (above 256: the exact kernel alone)


@dataclass(frozen=True)
class BandsConfig:
    """Frequency scaling: pairs by how often they turn over ``original`` positions (``low`` and ``high`` turns)."""
    factor: float
    low: float
    high: float
    original: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "BandsConfig":
        cfg = cls(*(_finite(_need(d, k, where), f"{where}.{k}") for k in ("factor", "low", "high", "original")))
        if min(cfg.factor, cfg.original) <= 0 or cfg.low < 0 or cfg.high <= cfg.low:
            raise ConfigError(f"config.json: {where}: factor and original must be positive, low not negative, high above low")
        return cfg

    def as_dict(self) -> dict:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class RotationConfig:
    dims: int
    base: float
    scaling: BandsConfig | None

    @classmethod
    def from_dict(cls, d: dict, where: str, head_dim: int) -> "RotationConfig":
        dims = _need(d, "dims", where)
        if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > head_dim:
            raise ConfigError(f"config.json: {where}.dims must be even and at most the head size {head_dim}, got {dims!r}")
        base = _finite(_need(d, "base", where), f"{where}.base")
        if not base > 0:
            raise ConfigError(f"config.json: {where}.base must be positive")
        scaling = d.get("scaling")
        return cls(dims, base, None if scaling is None else BandsConfig.from_dict(scaling, f"{where}.scaling"))


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    """``chunk`` None: causal over everything.  ``rot`` None: no rotation."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int | None
    rot: RotationConfig | None
    v_mix: bool

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ChunkedAttentionConfig":
        dim = _positive_int(_need(d, "dim", where), f"{where}.dim")
        mask, rot, v_mix = d.get("mask"), d.get("rot"), d.get("v_mix", False)
        if not isinstance(v_mix, bool):
            raise ConfigError(f"config.json: {where}.v_mix must be true or false")
        cfg = cls(heads=_positive_int(_need(d, "heads", where), f"{where}.heads"),
                  kv_heads=_positive_int(_need(d, "kv_heads", where), f"{where}.kv_heads"), dim=dim,
                  vdim=_positive_int(_need(d, "vdim", where), f"{where}.vdim"),
                  scale=_finite(_need(d, "scale", where), f"{where}.scale"),
                  chunk=None if mask is None else _positive_int(_need(mask, "size", f"{where}.mask"), f"{where}.mask.size"),
                  rot=None if rot is None else RotationConfig.from_dict(rot, f"{where}.rot", dim), v_mix=v_mix)
        if cfg.heads % cfg.kv_heads:
            raise ConfigError(f"config.json: {where}: heads must be a multiple of kv_heads")
        if max(cfg.dim, cfg.vdim) > MAX_HEAD:
            raise ConfigError(f"config.json: {where}: head sizes above {MAX_HEAD} are not supported")
        return cfg

    @property
    def value_width(self) -> int:
        return self.kv_heads * self.vdim


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "DenseConfig":
        return cls(_positive_int(_need(d, "ff", where), f"{where}.ff"))


@dataclass(frozen=True)
class MixtureConfig:
    experts: int
    top: int
    ff: int
    shared_ff: int | None

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "MixtureConfig":
        router, expert, shared = _need(d, "router", where), _need(d, "expert", where), d.get("shared")
        cfg = cls(experts=_positive_int(_need(router, "experts", f"{where}.router"), f"{where}.router.experts"),
                  top=_positive_int(_need(router, "top", f"{where}.router"), f"{where}.router.top"),
                  ff=_positive_int(_need(expert, "ff", f"{where}.expert"), f"{where}.expert.ff"),
                  shared_ff=None if shared is None else _positive_int(_need(shared, "ff", f"{where}.shared"), f"{where}.shared.ff"))
        if cfg.top > cfg.experts:
            raise ConfigError(f"config.json: {where}.router: top exceeds the number of experts")
        return cfg


MLPS = {"dense": DenseConfig, "moe": MixtureConfig}


@dataclass(frozen=True)
class VarivikLayer:
    mixer: ChunkedAttentionConfig
    mlp: DenseConfig | MixtureConfig | None


@dataclass(frozen=True)
class VarivikConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[VarivikLayer, ...]
    eos_token_ids: tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, d: dict) -> "VarivikConfig":
        raw_layers = _need(d, "layers", "the top level")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, layer in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind != "attention":
                raise ConfigError(f"config.json: {where}: mixer type {kind!r} is not implemented (known: attention)")
            mixer = ChunkedAttentionConfig.from_dict(_need(layer, "mixer", where), f"{where}.mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                form = _need(mlp, "kind", f"{where}.mlp")
                if form not in MLPS:
                    raise ConfigError(f"config.json: {where}.mlp: feed-forward kind {form!r} is not implemented (known: {', '.join(sorted(MLPS))})")
                mlp = MLPS[form].from_dict(mlp, f"{where}.mlp")
            layers.append(VarivikLayer(mixer, mlp))
        mixing = [layer.mixer.value_width for layer in layers if layer.mixer.v_mix]
        if len(set(mixing)) > 1:
            raise ConfigError("config.json: layers with v_mix blend values of one another, so kv_heads * vdim must be equal in all of them")
        cfg = cls(architecture=str(d.get("architecture", "Varivik")),
                  vocab=_positive_int(_need(d, "vocab", "the top level"), "vocab"),
                  width=_positive_int(_need(d, "width", "the top level"), "width"),
                  norm_eps=_finite(_need(_need(d, "norm", "the top level"), "eps", "norm"), "norm.eps"), layers=tuple(layers))
        if not cfg.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        return cfg

    @classmethod
    def read(cls, folder) -> "VarivikConfig":
        return cls.from_dict(json.loads((Path(folder) / "config.json").read_text()))
