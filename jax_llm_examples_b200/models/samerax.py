"""Samerax: its tensors by name and how its layers are put together from parts.

Tensor names: ``embed``, ``head``, ``final.norm`` and per layer with tensors of its own ``l<i>.``: ``norm1``, ``norm2`` (if the
layer has a feed-forward), ``mix.{q,k,v}`` with ``mix.{q,k,v}.b``, ``mix.{lq1,lk1,lq2,lk2}`` [dim], ``mix.o``, and
``mlp.{gate,up,down}`` (dense) or ``mlp.e<j>.{gate,up,down}`` with ``mlp.table`` [vocab, top] (mixture).  Linear weights are
[out, in]; the rows of q and k lie head by head as [map 1, map 2].

Layer rules (config: :class:`..config.samerax.SameraxConfig`): x += mixer(norm1(x)); x += ff(norm2(x)), plain RMS norms.
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..config.registry import Architecture, register_architecture
from ..config.samerax import DenseSpec, SameraxConfig
from ..parts import DecoderModel, DifferentialAttention, Runtime, make_part, rotary_frequencies, yarn_frequencies
from ..weights.loader import TensorSpec


def tensor_specs(cfg: SameraxConfig) -> dict[str, TensorSpec]:
    D, V = cfg.width, cfg.vocab
    specs: list[TensorSpec] = [TensorSpec("embed", (V, D))]

    def glu(prefix: str, ff: int):
        return [TensorSpec(prefix + "gate", (ff, D)), TensorSpec(prefix + "up", (ff, D)), TensorSpec(prefix + "down", (D, ff))]

    for i, L in enumerate(cfg.layers):
        if L.weights_of is not None:
            continue
        p, m, q = f"l{i}.", L.mixer, f"l{i}.mix."
        specs.append(TensorSpec(p + "norm1", (D,), "norm"))
        for name, rows in (("q", 2 * m.heads * m.dim), ("k", 2 * m.kv_heads * m.dim), ("v", m.kv_heads * m.vdim)):
            specs += [TensorSpec(q + name, (rows, D)), TensorSpec(q + name + ".b", (rows,), "bias")]
        specs += [TensorSpec(q + name, (m.dim,)) for name in ("lq1", "lk1", "lq2", "lk2")]
        specs.append(TensorSpec(q + "o", (D, m.heads * m.vdim)))
        if L.mlp is not None:
            specs.append(TensorSpec(p + "norm2", (D,), "norm"))
            if isinstance(L.mlp, DenseSpec):
                specs += glu(p + "mlp.", L.mlp.ff)
            else:
                for e in range(L.mlp.experts):
                    specs += glu(f"{p}mlp.e{e}.", L.mlp.ff)
                specs.append(TensorSpec(p + "mlp.table", (V, L.mlp.top), "choices", high=L.mlp.experts))
    specs += [TensorSpec("final.norm", (D,), "norm"), TensorSpec("head", (V, D))]
    return {s.name: s for s in specs}


def build(cfg: SameraxConfig, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> DecoderModel:
    """Puts the decoder together.  ``tensors`` (by spec name) is consumed as the weights are stacked into the layouts
    the kernels read."""
    t = dict(tensors) if not isinstance(tensors, dict) else tensors
    dev, eps = runtime.device, cfg.norm_eps

    def take(name: str) -> torch.Tensor:
        return t.pop(name).to(dev)

    def stack(prefix: str, names) -> torch.Tensor:
        return torch.cat([take(prefix + n) for n in names], dim=0).contiguous()

    def norm(name: str):
        return make_part("norm", "rms", weight=take(name), eps=eps)

    def rotation(rot):
        """(frequencies, rotated entries, amplitude) of a mixer's rotation."""
        if rot is None:
            return None, 0, 1.0
        if rot.scaling is None:
            return rotary_frequencies(rot.base, rot.dims).to(dev), rot.dims, 1.0
        sc = rot.scaling
        f, amplitude = yarn_frequencies(rot.base, rot.dims, sc.factor, sc.original, sc.fast, sc.slow)
        return f.to(dev), rot.dims, amplitude

    blocks, block_of = [], {}
    for i, L in enumerate(cfg.layers):
        if L.weights_of is not None:
            continue
        p, m, q = f"l{i}.", L.mixer, f"l{i}.mix."
        inv_freq, rot_dims, amplitude = rotation(m.rot)
        mixer = make_part(
            "mixer", "differential_attention", w_in=stack(q, ("q", "k", "v")), in_bias=stack(q, ("q.b", "k.b", "v.b")),
            w_o=take(q + "o").contiguous(), heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps,
            map_weight=DifferentialAttention.map_weight_of(*(take(q + s) for s in ("lq1", "lk1", "lq2", "lk2")), m.diff), diff=m.diff,
            inv_freq=inv_freq, rot_dims=rot_dims, rot_amplitude=amplitude, window=m.window, keep_first=m.keep_first,
            padded_dim=DifferentialAttention.padded_size(m.dim, m.vdim, runtime.dtype))
        ff = None
        if isinstance(L.mlp, DenseSpec):
            ff = make_part("feed_forward", "dense_swiglu", w_gate_up=stack(p + "mlp.", ("gate", "up")), w_down=take(p + "mlp.down").contiguous())
        elif L.mlp is not None:
            e = f"{p}mlp."
            ff = make_part("feed_forward", "table_routed_glu_experts", table=take(e + "table"),
                           we_gate_up=torch.stack([stack(f"{e}e{j}.", ("gate", "up")) for j in range(L.mlp.experts)]),
                           we_down=torch.stack([take(f"{e}e{j}.down") for j in range(L.mlp.experts)]))
        block_of[i] = len(blocks)
        blocks.append(make_part("block", "pre_norm", norm1=norm(p + "norm1"), mixer=mixer, norm2=None if ff is None else norm(p + "norm2"),
                                feed_forward=ff))
    # a layer with another's weights is that layer's block once more, with a cache of its own
    schedule = DecoderModel.schedule_of([(block_of[cfg.owner(i)],) for i in range(len(cfg.layers))], blocks)
    return DecoderModel(runtime, take("embed").contiguous(), blocks, norm("final.norm"), take("head").contiguous(), schedule=schedule,
                        config=cfg, embedding_scale=cfg.embedding_scale, logit_softcap=cfg.logit_softcap)


SAMERAX = Architecture(name="Samerax", parse_config=SameraxConfig.from_dict, tensor_specs=tensor_specs, build=build)
register_architecture(SAMERAX)
