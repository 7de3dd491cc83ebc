"""Typed configuration of the ``Gotivik`` architecture.

``config.json`` gives ``vocab``, ``width``, ``norm.eps``, ``residual_mult`` and a list ``layers``; every entry
names its mixer (``type``: ``"attention"``, windowed attention behind short convolutions, or ``"attention_2"``,
differential attention), the mixer's sizes (``mixer``) and its feed-forward (``mlp``: dense, or null for none).
An entry with ``weights_of: j`` runs layer ``j``'s weights with a cache and a state of its own; the rest of the
entry repeats layer ``j``'s.  Layers may differ from one another in everything.  Nothing here has a default
that stands for a size: a missing key is an error.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping

from .registry import ConfigError


def _need(m: Mapping[str, Any], key: str, where: str):
    if not isinstance(m, Mapping) or key not in m or m[key] is None:
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    return m[key]


def _integer(m: Mapping[str, Any], key: str, where: str, least: int = 1) -> int:
    v = _need(m, key, where)
    if isinstance(v, bool) or not isinstance(v, int) or v < least:
        kind = "a positive integer" if least == 1 else f"an integer from {least} on"
        raise ConfigError(f"config.json: {where}.{key} must be {kind}, got {v!r}")
    return v


@dataclass(frozen=True)
class YarnScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class WindowAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int                           # taps of the short convolutions on q, k and v
    window: int
    keep_first: int                     # first positions of the sequence that stay visible
    rot_base: float
    rot_dims: int                       # 0: no rotation
    rot_scaling: YarnScaling | None


@dataclass(frozen=True)
class DifferentialAttentionConfig:
    heads: int
    kv_heads: int
    dim: int                            # of one map's queries and keys
    vdim: int
    scale: float
    softcap: float
    temp_coef: float
    temp_every: int
    diff: float


@dataclass(frozen=True)
class GotivikLayer:
    type: str
    mixer: WindowAttentionConfig | DifferentialAttentionConfig
    ff: int                             # 0: no feed-forward
    weights: int                        # the layer whose tensors this one runs (its own index: its own)


@dataclass(frozen=True)
class GotivikConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    layers: tuple[GotivikLayer, ...]

    @classmethod
    def from_json(cls, raw: Mapping[str, Any]) -> "GotivikConfig":
        layers = _need(raw, "layers", "the top level")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        parsed = [_layer(entry, i, layers) for i, entry in enumerate(layers)]
        for i, layer in enumerate(parsed):
            o = parsed[layer.weights]
            if (o.type, o.mixer, o.ff) != (layer.type, layer.mixer, layer.ff):
                raise ConfigError(f"config.json: layers[{i}] runs layer {layer.weights}'s weights but differs from it")
        return cls(
            vocab=_integer(raw, "vocab", "the top level"),
            width=_integer(raw, "width", "the top level"),
            eps=float(_need(_need(raw, "norm", "the top level"), "eps", "norm")),
            residual_mult=float(_need(raw, "residual_mult", "the top level")),
            layers=tuple(parsed),
        )


def _owner(layers, i: int) -> int:
    """The layer whose tensors layer ``i`` runs: ``weights_of`` followed to a layer that has its own."""
    seen = {i}
    while isinstance(layers[i], Mapping) and layers[i].get("weights_of") is not None:
        j = layers[i]["weights_of"]
        if isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < len(layers) or j in seen:
            raise ConfigError(f"config.json: layers[{i}].weights_of={j!r} names no layer with weights of its own")
        seen.add(j)
        i = j
    return i


def _heads(m: Mapping[str, Any], where: str) -> tuple[int, int]:
    heads, kv_heads = _integer(m, "heads", where), _integer(m, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}: {heads} heads cannot share {kv_heads} key/value heads")
    return heads, kv_heads


def _window_attention(m: Mapping[str, Any], where: str) -> WindowAttentionConfig:
    heads, kv_heads = _heads(m, where)
    dim, rot, mask = _integer(m, "dim", where), m.get("rot"), _need(m, "mask", where)
    scaling = None
    if rot and rot.get("scaling"):
        sw = where + ".rot.scaling"
        scaling = YarnScaling(*(float(_need(rot["scaling"], k, sw)) for k in ("factor", "original", "fast", "slow")))
        if not (scaling.factor > 0 and scaling.original > 0 and scaling.fast > 0 and scaling.slow > 0):
            raise ConfigError(f"config.json: {sw}: every number must be positive")
    rot_dims = _integer(rot, "dims", where + ".rot") if rot else 0
    if rot_dims % 2 or rot_dims > dim:
        raise ConfigError(f"config.json: {where}.rot.dims={rot_dims} must be even and at most dim={dim}")
    return WindowAttentionConfig(
        heads=heads, kv_heads=kv_heads, dim=dim, vdim=_integer(m, "vdim", where),
        scale=float(_need(m, "scale", where)), conv=_integer(m, "conv", where),
        window=_integer(mask, "size", where + ".mask"), keep_first=_integer(mask, "keep_first", where + ".mask", 0),
        rot_base=float(_need(rot, "base", where + ".rot")) if rot else 0.0, rot_dims=rot_dims, rot_scaling=scaling)


def _differential_attention(m: Mapping[str, Any], where: str) -> DifferentialAttentionConfig:
    heads, kv_heads = _heads(m, where)
    temp = m.get("q_temp")
    cap = m.get("softcap")
    if cap is not None and not float(cap) > 0:
        raise ConfigError(f"config.json: {where}.softcap must be positive, got {cap!r}")
    return DifferentialAttentionConfig(
        heads=heads, kv_heads=kv_heads, dim=_integer(m, "dim", where), vdim=_integer(m, "vdim", where),
        scale=float(_need(m, "scale", where)), softcap=float(cap) if cap is not None else 0.0,
        temp_coef=float(_need(temp, "coef", where + ".q_temp")) if temp else 0.0,
        temp_every=_integer(temp, "every", where + ".q_temp") if temp else 1,
        diff=float(_need(m, "diff", where)))


def _layer(raw: Mapping[str, Any], index: int, layers) -> GotivikLayer:
    where = f"layers[{index}]"
    kind = _need(raw, "type", where)
    m = _need(raw, "mixer", where)
    if kind == "attention":
        mixer = _window_attention(m, where + ".mixer")
    elif kind == "attention_2":
        mixer = _differential_attention(m, where + ".mixer")
    else:
        raise ConfigError(f"config.json: {where}.type {kind!r} is neither 'attention' nor 'attention_2'")
    mlp, ff = raw.get("mlp"), 0
    if mlp is not None:
        mlp_kind = _need(mlp, "kind", where + ".mlp")
        if mlp_kind != "dense":
            raise ConfigError(f"config.json: {where}.mlp.kind {mlp_kind!r} is not 'dense'")
        ff = _integer(mlp, "ff", where + ".mlp")
    return GotivikLayer(kind, mixer, ff, _owner(layers, index))
