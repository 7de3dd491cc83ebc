"""Typed configuration of the ``Zinesun`` architecture.

``config.json`` gives ``vocab``, ``width``, ``norm.eps``, ``canon.taps``, ``embedding.scale`` and a list
``layers``; every entry names its mixer (``type``: ``"latent_attention"``), the mixer's sizes (``mixer``)
and its feed-forward (``mlp``: dense, a mixture of experts, or null for none).  Layers may differ from one
another in everything.  Nothing here has a default that stands for a size: a missing key is an error.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .registry import ConfigError


def _need(m: Mapping[str, Any], key: str, where: str):
    if not isinstance(m, Mapping) or key not in m or m[key] is None:
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    return m[key]


def _positive(m: Mapping[str, Any], key: str, where: str) -> int:
    v = _need(m, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v <= 0:
        raise ConfigError(f"config.json: {where}.{key} must be a positive integer, got {v!r}")
    return v


@dataclass(frozen=True)
class LatentMixerConfig:
    heads: int
    dim: int                  # unrotated query/key dimensions of a head
    rot_dim: int              # rotated ones
    vdim: int
    kv_rank: int
    q_rank: int
    window: int
    scale: float
    rot_base: float
    rot_dims: int


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class ExpertsConfig:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class ZinesunLayer:
    mixer: LatentMixerConfig
    mlp: DenseConfig | ExpertsConfig | None


@dataclass(frozen=True)
class ZinesunConfig:
    vocab: int
    width: int
    eps: float
    taps: int                 # of the convolution in front of every mixer
    embedding_scale: float
    layers: tuple[ZinesunLayer, ...]

    @classmethod
    def from_json(cls, raw: Mapping[str, Any]) -> "ZinesunConfig":
        layers = _need(raw, "layers", "the top level")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        return cls(
            vocab=_positive(raw, "vocab", "the top level"),
            width=_positive(raw, "width", "the top level"),
            eps=float(_need(_need(raw, "norm", "the top level"), "eps", "norm")),
            taps=_positive(_need(raw, "canon", "the top level"), "taps", "canon"),
            embedding_scale=float(_need(_need(raw, "embedding", "the top level"), "scale", "embedding")),
            layers=tuple(_layer(l, f"layers[{i}]") for i, l in enumerate(layers)),
        )


def _mixer(m: Mapping[str, Any], where: str) -> LatentMixerConfig:
    rot = _need(m, "rot", where)
    c = LatentMixerConfig(
        heads=_positive(m, "heads", where), dim=_positive(m, "dim", where), rot_dim=_positive(m, "rot_dim", where),
        vdim=_positive(m, "vdim", where), kv_rank=_positive(m, "kv_rank", where), q_rank=_positive(m, "q_rank", where),
        window=_positive(_need(m, "mask", where), "size", where + ".mask"), scale=float(_need(m, "scale", where)),
        rot_base=float(_need(rot, "base", where + ".rot")), rot_dims=_positive(rot, "dims", where + ".rot"),
    )
    if c.rot_dims % 2 or c.rot_dims > c.rot_dim:
        raise ConfigError(f"config.json: {where}.rot.dims={c.rot_dims} must be even and at most rot_dim={c.rot_dim}")
    return c


def _layer(raw: Mapping[str, Any], where: str) -> ZinesunLayer:
    kind = _need(raw, "type", where)
    if kind != "latent_attention":
        raise ConfigError(f"config.json: {where}.type {kind!r} is not 'latent_attention'")
    mixer = _mixer(_need(raw, "mixer", where), where + ".mixer")
    mlp = raw.get("mlp")
    ff: DenseConfig | ExpertsConfig | None = None
    if mlp is not None:
        fw = where + ".mlp"
        mlp_kind = _need(mlp, "kind", fw)
        if mlp_kind == "dense":
            ff = DenseConfig(_positive(mlp, "ff", fw))
        elif mlp_kind == "moe":
            router, expert = _need(mlp, "router", fw), _need(mlp, "expert", fw)
            ff = ExpertsConfig(experts=_positive(router, "experts", fw + ".router"),
                               top=_positive(router, "top", fw + ".router"), ff=_positive(expert, "ff", fw + ".expert"))
            if ff.top > ff.experts:
                raise ConfigError(f"config.json: {fw}.router: top={ff.top} of {ff.experts} experts")
        else:
            raise ConfigError(f"config.json: {fw}.kind {mlp_kind!r} is neither 'dense' nor 'moe'")
    return ZinesunLayer(mixer, ff)
