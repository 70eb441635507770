"""Typed view of a Bavetar ``config.json``.

The file names the design under ``architecture`` and gives the residual width, the vocabulary, the norms' eps, the
factor and the cap of the logits, and a list of layers.  A layer names its mixer by ``type`` -- ``latent_attention``
(queries and keys/values through low-rank latents, a rotated key part shared by the heads, a learned sink and an output
gate per head) or ``mamba2`` (a state-space recurrence) -- with the mixer's sizes and constants under ``mixer``, and its
feed-forward under ``mlp``: ``dense`` (two matrices around the square of relu), ``moe`` (routed experts, chosen within
the best groups) or null.  Every size and constant comes from here.  Anything this engine does not implement is refused
before a weight is read.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path

from .linurax_config import _finite, _need, _positive_int
from .model_config import ConfigError

MAX_CACHED_ROW = 1024       # the attention kernels' largest head (a cached row is one key); above 256: the exact kernel alone
MAX_STATE, MAX_VALUE, MAX_TAPS = 256, 255, 17      # the recurrence's and the convolution's limits


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "LatentAttentionConfig":
        rot = _need(d, "rot", where)
        rot_dim = _need(d, "rot_dim", where)
        if isinstance(rot_dim, bool) or not isinstance(rot_dim, int) or rot_dim <= 0 or rot_dim % 2:
            raise ConfigError(f"config.json: {where}.rot_dim must be a positive even integer, got {rot_dim!r}")
        if _need(rot, "dims", f"{where}.rot") != rot_dim:
            raise ConfigError(f"config.json: {where}.rot.dims must equal rot_dim: the rotated part is rotated as a whole")
        if rot.get("scaling") is not None:
            raise ConfigError(f"config.json: {where}.rot.scaling is not part of this design's rotation")
        if d.get("mask") is not None:
            raise ConfigError(f"config.json: {where}.mask: this design's attention sees every earlier token")
        ints = {k: _positive_int(_need(d, k, where), f"{where}.{k}") for k in ("heads", "dim", "vdim", "q_rank", "kv_rank")}
        cfg = cls(rot_dim=rot_dim, scale=_finite(_need(d, "scale", where), f"{where}.scale"),
                  rot_base=_finite(_need(rot, "base", f"{where}.rot"), f"{where}.rot.base"), **ints)
        if not cfg.rot_base > 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive")
        if cfg.kv_rank + cfg.rot_dim > MAX_CACHED_ROW:
            raise ConfigError(f"config.json: {where}: kv_rank + rot_dim above {MAX_CACHED_ROW} is not supported (a cached row is one key)")
        return cfg


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "Mamba2Config":
        cfg = cls(**{k: _positive_int(_need(d, k, where), f"{where}.{k}")
                     for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")})
        if cfg.heads % cfg.groups:
            raise ConfigError(f"config.json: {where}: heads must be a multiple of groups")
        if (cfg.heads * cfg.vdim) % cfg.norm_groups:
            raise ConfigError(f"config.json: {where}: norm_groups must divide heads * vdim")
        if cfg.state > MAX_STATE or cfg.vdim > MAX_VALUE:
            raise ConfigError(f"config.json: {where}: a head of {cfg.state} x {cfg.vdim} does not fit the recurrence kernel "
                              f"({MAX_STATE} x {MAX_VALUE})")
        if cfg.conv > MAX_TAPS:
            raise ConfigError(f"config.json: {where}.conv: more than {MAX_TAPS} taps are not supported")
        return cfg


@dataclass(frozen=True)
class DenseConfig:
    ff: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "DenseConfig":
        return cls(_positive_int(_need(d, "ff", where), f"{where}.ff"))


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    scale: float
    groups: tuple[int, int] | None       # (count, keep)
    ff: int

    @classmethod
    def from_dict(cls, d: dict, where: str) -> "ExpertsConfig":
        router, expert = _need(d, "router", where), _need(d, "expert", where)
        at = f"{where}.router"
        groups = router.get("groups")
        if groups is not None:
            groups = tuple(_positive_int(_need(groups, k, f"{at}.groups"), f"{at}.groups.{k}") for k in ("count", "keep"))
        cfg = cls(experts=_positive_int(_need(router, "experts", at), f"{at}.experts"),
                  top=_positive_int(_need(router, "top", at), f"{at}.top"),
                  scale=_finite(router.get("scale", 1.0), f"{at}.scale"), groups=groups,
                  ff=_positive_int(_need(expert, "ff", f"{where}.expert"), f"{where}.expert.ff"))
        if cfg.top > cfg.experts:
            raise ConfigError(f"config.json: {at}: top exceeds the number of experts")
        if groups is not None:
            count, keep = groups
            if cfg.experts % count or keep > count or keep * (cfg.experts // count) < cfg.top:
                raise ConfigError(f"config.json: {at}.groups: {count} equal groups of {cfg.experts} experts, of which {keep} hold at "
                                  f"least {cfg.top}, are not possible")
        return cfg


MIXERS = {"latent_attention": LatentAttentionConfig, "mamba2": Mamba2Config}
FEED_FORWARDS = {"dense": DenseConfig, "moe": ExpertsConfig}


@dataclass(frozen=True)
class BavetarLayer:
    type: str
    mixer: LatentAttentionConfig | Mamba2Config
    mlp: DenseConfig | ExpertsConfig | None


@dataclass(frozen=True)
class BavetarConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    logit_scale: float
    logit_softcap: float | None
    layers: tuple[BavetarLayer, ...]
    eos_token_ids: tuple[int, ...] = ()

    @classmethod
    def from_dict(cls, d: dict) -> "BavetarConfig":
        raw_layers = _need(d, "layers", "the top level")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, layer in enumerate(raw_layers):
            where = f"layers[{i}]"
            kind = _need(layer, "type", where)
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}: mixer type {kind!r} is not implemented (known: {', '.join(sorted(MIXERS))})")
            mixer = MIXERS[kind].from_dict(_need(layer, "mixer", where), f"{where}.mixer")
            mlp = layer.get("mlp")
            if mlp is not None:
                ff = _need(mlp, "kind", f"{where}.mlp")
                if ff not in FEED_FORWARDS:
                    raise ConfigError(f"config.json: {where}.mlp: feed-forward kind {ff!r} is not implemented (known: {', '.join(sorted(FEED_FORWARDS))})")
                mlp = FEED_FORWARDS[ff].from_dict(mlp, f"{where}.mlp")
            layers.append(BavetarLayer(kind, mixer, mlp))
        cap, scale = d.get("logit_softcap"), d.get("logit_scale")
        cfg = cls(architecture=str(d.get("architecture", "Bavetar")),
                  vocab=_positive_int(_need(d, "vocab", "the top level"), "vocab"),
                  width=_positive_int(_need(d, "width", "the top level"), "width"),
                  norm_eps=_finite(_need(_need(d, "norm", "the top level"), "eps", "norm"), "norm.eps"),
                  logit_scale=1.0 if scale is None else _finite(scale, "logit_scale"),
                  logit_softcap=None if cap is None else _finite(cap, "logit_softcap"), layers=tuple(layers))
        if not cfg.norm_eps > 0:
            raise ConfigError("config.json: norm.eps must be positive")
        if cfg.logit_softcap is not None and not cfg.logit_softcap > 0:
            raise ConfigError("config.json: logit_softcap must be positive or null")
        return cfg

    @classmethod
    def read(cls, folder) -> "BavetarConfig":
        return cls.from_dict(json.loads((Path(folder) / "config.json").read_text()))
