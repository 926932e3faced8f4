"""Typed configuration of the Samerax decoder, read from config.json's own keys.

A Samerax model is a list of pre-norm layers (plain RMS norms) over a scaled embedding.  A layer's mixer is ``attention``:
grouped-query attention whose heads are each the difference of two softmax maps over the same values, with biased
projections, a rotate-half rotation of part of every map (optionally with YaRN-scaled frequencies) and a sliding window
that keeps the sequence's first keys.  Its feed-forward is dense (a gated silu unit), a mixture of such experts that a table
of token ids chooses from, or missing.  A layer with ``weights_of`` j has no tensors of its own: it runs layer j's once more,
with a cache of its own.  The logits come from a head of their own and are soft-capped.  Every size and constant that can
differ between two models is a key of the file.
"""

from __future__ import annotations

import dataclasses
from typing import Any, Mapping

from .base import ConfigError, read_key, require
from .koduzen import YarnSpec


@dataclasses.dataclass(frozen=True)
class RotSpec:
    base: float
    dims: int
    scaling: YarnSpec | None


@dataclasses.dataclass(frozen=True)
class DifferentialSpec:
    heads: int
    kv_heads: int
    dim: int  # entries of one map's query or key
    vdim: int
    scale: float
    diff: float
    window: int | None
    keep_first: int
    rot: RotSpec | None


@dataclasses.dataclass(frozen=True)
class DenseSpec:
    ff: int


@dataclasses.dataclass(frozen=True)
class TableMoeSpec:
    experts: int
    top: int
    ff: int


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    mixer: DifferentialSpec
    mlp: "DenseSpec | TableMoeSpec | None"
    weights_of: int | None


def _rot(m: Mapping[str, Any], dim: int, where: str) -> RotSpec | None:
    rot = read_key(m, "rot", dict, None)
    if rot is None:
        return None
    base, dims = read_key(rot, "base", float), read_key(rot, "dims", int)
    require(base > 0, f"{where}.rot.base must be positive")
    require(dims % 2 == 0 and 0 <= dims <= dim, f"{where}: rot.dims = {dims} must be even and at most dim = {dim}")
    if dims == 0:
        return None
    sc = read_key(rot, "scaling", dict, None)
    scaling = None
    if sc is not None:
        scaling = YarnSpec(*(read_key(sc, k, float) for k in ("factor", "original", "fast", "slow")))
        require(min(scaling.factor, scaling.original, scaling.fast, scaling.slow) > 0 and base != 1.0,
                f"{where}.rot.scaling: factor, original, fast and slow must be positive (and the base not 1)")
    return RotSpec(base, dims, scaling)


@dataclasses.dataclass(frozen=True)
class SameraxConfig:
    vocab: int
    width: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float
    embedding_scale: float
    logit_softcap: float | None

    # the names the rest of the framework asks a configuration for
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i uses."""
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
        return i

    @staticmethod
    def from_dict(d: Mapping[str, Any]) -> "SameraxConfig":
        raw_layers = read_key(d, "layers", list)
        require(len(raw_layers) > 0, "'layers' is empty")
        layers: list[LayerSpec] = []
        for i, L in enumerate(raw_layers):
            require(isinstance(L, dict), f"layers[{i}] must be an object")
            kind = read_key(L, "type", str)
            require(kind == "attention", f"layers[{i}].type = {kind!r} is no mixer of this architecture (attention)")
            m, where = read_key(L, "mixer", dict), f"layers[{i}].mixer"
            heads, kv_heads, dim, vdim = (read_key(m, k, int) for k in ("heads", "kv_heads", "dim", "vdim"))
            require(min(heads, kv_heads, dim, vdim) > 0, f"{where}: sizes must be positive")
            require(heads % kv_heads == 0, f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
            mask = read_key(m, "mask", dict, None)
            window, keep = (None, 0) if mask is None else (read_key(mask, "size", int), read_key(mask, "keep_first", int, 0))
            require(window is None or (window > 0 and keep >= 0), f"{where}.mask: size must be positive and keep_first not negative")
            mixer = DifferentialSpec(heads, kv_heads, dim, vdim, read_key(m, "scale", float), read_key(m, "diff", float), window, keep,
                                     _rot(m, dim, where))
            mlp: Any = None
            if L.get("mlp") is not None:
                ml, at = read_key(L, "mlp", dict), f"layers[{i}].mlp"
                mk = read_key(ml, "kind", str)
                if mk == "dense":
                    mlp = DenseSpec(read_key(ml, "ff", int))
                elif mk == "moe":
                    r = read_key(ml, "router", dict)
                    mlp = TableMoeSpec(read_key(r, "experts", int), read_key(r, "top", int), read_key(read_key(ml, "expert", dict), "ff", int))
                    require(mlp.experts > 0 and 1 <= mlp.top <= mlp.experts, f"{at}.router: top-{mlp.top} of {mlp.experts} experts")
                else:
                    raise ConfigError(f"config.json: {at}.kind = {mk!r}; this architecture has 'dense' and 'moe'")
                require(mlp.ff > 0, f"{at}: ff must be positive")
            layers.append(LayerSpec(mixer, mlp, read_key(L, "weights_of", int, None)))
        for i, L in enumerate(layers):
            seen, j = {i}, L.weights_of
            while j is not None:
                require(0 <= j < len(layers) and j not in seen, f"layers[{i}].weights_of leads to no layer with tensors of its own")
                require((layers[j].mixer, layers[j].mlp) == (L.mixer, L.mlp), f"layers[{i}].weights_of = {j}, but the two layers differ")
                seen.add(j)
                j = layers[j].weights_of
        cfg = SameraxConfig(vocab=read_key(d, "vocab", int), width=read_key(d, "width", int), layers=tuple(layers),
                            norm_eps=read_key(read_key(d, "norm", dict), "eps", float),
                            embedding_scale=read_key(read_key(d, "embedding", dict, {}), "scale", float, 1.0),
                            logit_softcap=read_key(d, "logit_softcap", float, None))
        require(cfg.vocab > 0 and cfg.width > 0, "vocab and width must be positive")
        require(cfg.norm_eps > 0, "norm.eps must be positive")
        require(cfg.logit_softcap is None or cfg.logit_softcap > 0, "logit_softcap must be positive")
        return cfg
