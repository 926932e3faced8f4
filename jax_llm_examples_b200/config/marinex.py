"""Typed configuration of the Marinex decoder, read from config.json's own keys.

A Marinex model is a list of layers whose sublayers read the residual rows as they are and whose OUTPUTS are normed before
they are added (plain RMS norms).  A layer has one of two mixers,

* ``attention``: grouped-query softmax attention over all earlier positions; q and k RMS-normed per head and then rotated
  in neighbouring pairs on their first entries, values divided by their root mean square, a number per head on the
  scores, soft-capped scores, one added to the softmax's denominator;
* ``latent_attention``: low-rank queries and one cached latent per token over a sliding window, a rotated key part shared
  by the heads (rotate-half), a learned sink per head, a sigmoid gate per head;

and a feed-forward that is a mixture of experts (exact gelu; sigmoid router with a correction on the choice and a limit to
the best groups) or missing.  Embedding and head are tensors of their own.  Every size and constant that can differ between
two models is a key of the file.
"""

from __future__ import annotations

import dataclasses
from typing import Any, Mapping

from .base import ConfigError, read_key, require


@dataclasses.dataclass(frozen=True)
class RotSpec:
    base: float
    dims: int


@dataclasses.dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float | None
    rot: RotSpec | None
    window: int | None


@dataclasses.dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotSpec
    window: int | None


@dataclasses.dataclass(frozen=True)
class MoeSpec:
    experts: int
    top: int
    groups: int
    keep: int
    ff: int


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    type: str
    mixer: "AttentionSpec | LatentAttentionSpec"
    mlp: MoeSpec | None


def _rot(m: Mapping[str, Any], size: int, where: str) -> RotSpec | None:
    rot = read_key(m, "rot", dict, None)
    if rot is None:
        return None
    base, dims = read_key(rot, "base", float), read_key(rot, "dims", int)
    require(base > 0, f"{where}.rot.base must be positive")
    require(dims % 2 == 0 and 0 <= dims <= size, f"{where}: rot.dims = {dims} must be even and at most {size}")
    return RotSpec(base, dims)


def _window(m: Mapping[str, Any], where: str) -> int | None:
    mask = read_key(m, "mask", dict, None)
    if mask is None:
        return None
    size = read_key(mask, "size", int)
    require(size > 0, f"{where}: mask.size must be positive")
    return size


def _moe(ml: Mapping[str, Any], at: str) -> MoeSpec:
    kind = read_key(ml, "kind", str)
    if kind != "moe":
        raise ConfigError(f"config.json: {at}.kind = {kind!r}; this architecture has 'moe'")
    r = read_key(ml, "router", dict)
    g = read_key(r, "groups", dict, None)
    groups, keep = (1, 1) if g is None else (read_key(g, "count", int), read_key(g, "keep", int))
    spec = MoeSpec(read_key(r, "experts", int), read_key(r, "top", int), groups, keep, read_key(read_key(ml, "expert", dict), "ff", int))
    require(spec.experts > 0 and spec.ff > 0, f"{at}: sizes must be positive")
    require(groups >= 1 and spec.experts % groups == 0 and 1 <= keep <= groups,
            f"{at}.router.groups: {groups} groups (keep {keep}) of {spec.experts} experts")
    require(1 <= spec.top <= spec.experts // groups * keep,
            f"{at}.router: top-{spec.top} of the {spec.experts // groups * keep} experts of the kept groups")
    return spec


@dataclasses.dataclass(frozen=True)
class MarinexConfig:
    vocab: int
    width: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float

    # the names the rest of the framework asks a configuration for
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "MarinexConfig":
        raw_layers = read_key(d, "layers", list)
        require(len(raw_layers) > 0, "'layers' is empty")
        layers: list[LayerSpec] = []
        for i, L in enumerate(raw_layers):
            require(isinstance(L, dict), f"layers[{i}] must be an object")
            kind = read_key(L, "type", str)
            m = read_key(L, "mixer", dict)
            where = f"layers[{i}].mixer"
            heads, dim, vdim = read_key(m, "heads", int), read_key(m, "dim", int), read_key(m, "vdim", int)
            require(heads > 0 and dim > 0 and vdim > 0, f"{where}: sizes must be positive")
            scale = read_key(m, "scale", float)
            if kind == "attention":
                kv_heads = read_key(m, "kv_heads", int)
                require(kv_heads > 0 and heads % kv_heads == 0, f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
                cap = read_key(m, "softcap", float, None)
                require(cap is None or cap > 0, f"{where}: softcap must be positive")
                mixer: Any = AttentionSpec(heads, kv_heads, dim, vdim, scale, cap, _rot(m, dim, where), _window(m, where))
            elif kind == "latent_attention":
                rot_dim, q_rank, kv_rank = read_key(m, "rot_dim", int), read_key(m, "q_rank", int), read_key(m, "kv_rank", int)
                require(rot_dim >= 0 and q_rank > 0 and kv_rank > 0, f"{where}: sizes must be positive")
                rot = _rot(m, rot_dim, where)
                require(rot is not None and rot.dims == rot_dim, f"{where}: rot.dims must be rot_dim = {rot_dim}")
                mixer = LatentAttentionSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, _window(m, where))
            else:
                raise ConfigError(f"config.json: layers[{i}].type = {kind!r} is no mixer of this architecture "
                                  "(attention, latent_attention)")
            mlp = None if L.get("mlp") is None else _moe(read_key(L, "mlp", dict), f"layers[{i}].mlp")
            layers.append(LayerSpec(kind, mixer, mlp))
        cfg = MarinexConfig(vocab=read_key(d, "vocab", int), width=read_key(d, "width", int), layers=tuple(layers),
                            norm_eps=read_key(read_key(d, "norm", dict), "eps", float))
        require(cfg.vocab > 0 and cfg.width > 0, "vocab and width must be positive")
        require(cfg.norm_eps > 0, "norm.eps must be positive")
        return cfg
