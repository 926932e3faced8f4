"""Marinex: its tensors by name and how its layers are put together from parts.

Tensor names: ``embed``, ``head``, ``final.norm`` and per layer ``l<i>.``: ``norm1`` (on the mixer's output), ``norm2`` (on
the feed-forward's, if the layer has one), ``mix.*`` and ``mlp.*``.  Linear weights are [out, in].

* ``attention`` mixer: ``mix.{q,k,v,o}``, ``mix.q.norm``, ``mix.k.norm`` [dim], ``mix.temp`` [heads].
* ``latent_attention`` mixer: ``mix.{dq,uq,dkv,uk,uv,g,o}``, ``mix.dq.norm`` [q_rank], ``mix.dkv.norm`` [kv_rank],
  ``mix.sink`` [heads].
* mixture: ``mlp.router`` [experts, width], ``mlp.correction`` [experts], ``mlp.e<j>.{up,down}``.

Layer rules (config: :class:`..config.marinex.MarinexConfig`): x += norm1(mixer(x)); x += norm2(ff(x)).
"""

from __future__ import annotations

from typing import Mapping

import torch

from ..config.marinex import AttentionSpec, LatentAttentionSpec, MarinexConfig
from ..config.registry import Architecture, register_architecture
from ..parts import DecoderModel, GatedPagedAttention, Runtime, make_part, rotary_frequencies
from ..weights.loader import TensorSpec

GROUP_TOP = 2  # a group of experts is as good as the sum of its two largest choice scores


def tensor_specs(cfg: MarinexConfig) -> dict[str, TensorSpec]:
    D, V = cfg.width, cfg.vocab
    specs: list[TensorSpec] = [TensorSpec("embed", (V, D))]
    for i, L in enumerate(cfg.layers):
        p, m, q = f"l{i}.", L.mixer, f"l{i}.mix."
        H = m.heads
        specs.append(TensorSpec(p + "norm1", (D,), "norm"))
        if isinstance(m, AttentionSpec):
            specs += [TensorSpec(q + "q", (H * m.dim, D)), TensorSpec(q + "k", (m.kv_heads * m.dim, D)),
                      TensorSpec(q + "v", (m.kv_heads * m.vdim, D)), TensorSpec(q + "q.norm", (m.dim,), "norm"),
                      TensorSpec(q + "k.norm", (m.dim,), "norm"), TensorSpec(q + "temp", (H,), "norm"),
                      TensorSpec(q + "o", (D, H * m.vdim))]
        else:
            assert isinstance(m, LatentAttentionSpec)
            specs += [TensorSpec(q + "dq", (m.q_rank, D)), TensorSpec(q + "dq.norm", (m.q_rank,), "norm"),
                      TensorSpec(q + "uq", (H * (m.dim + m.rot_dim), m.q_rank)), TensorSpec(q + "dkv", (m.kv_rank + m.rot_dim, D)),
                      TensorSpec(q + "dkv.norm", (m.kv_rank,), "norm"), TensorSpec(q + "uk", (H * m.dim, m.kv_rank)),
                      TensorSpec(q + "uv", (H * m.vdim, m.kv_rank)), TensorSpec(q + "sink", (H,), "bias"),
                      TensorSpec(q + "g", (H, D)), TensorSpec(q + "o", (D, H * m.vdim))]
        if L.mlp is not None:
            specs.append(TensorSpec(p + "norm2", (D,), "norm"))
            for e in range(L.mlp.experts):
                specs += [TensorSpec(f"{p}mlp.e{e}.up", (L.mlp.ff, D)), TensorSpec(f"{p}mlp.e{e}.down", (D, L.mlp.ff))]
            specs += [TensorSpec(p + "mlp.router", (L.mlp.experts, D)), TensorSpec(p + "mlp.correction", (L.mlp.experts,), "bias")]
    specs += [TensorSpec("final.norm", (D,), "norm"), TensorSpec("head", (V, D))]
    return {s.name: s for s in specs}


def build(cfg: MarinexConfig, tensors: Mapping[str, torch.Tensor], runtime: Runtime) -> DecoderModel:
    """Puts the decoder together.  ``tensors`` (by spec name) is consumed as the weights are stacked into the layouts
    the kernels read."""
    t = dict(tensors) if not isinstance(tensors, dict) else tensors
    dev, eps = runtime.device, cfg.norm_eps

    def take(name: str) -> torch.Tensor:
        return t.pop(name).to(dev)

    def stack(prefix: str, names) -> torch.Tensor:
        return torch.cat([take(prefix + n) for n in names], dim=0).contiguous()

    def norm(name: str):
        return make_part("norm", "group_rms", weight=take(name), eps=eps)

    blocks = []
    for i, L in enumerate(cfg.layers):
        p, m, q = f"l{i}.", L.mixer, f"l{i}.mix."
        if isinstance(m, AttentionSpec):
            dims = 0 if m.rot is None else m.rot.dims
            mixer = make_part(
                "mixer", "gated_paged_attention", w_in=stack(q, ("q", "k", "v")), w_o=take(q + "o").contiguous(), n_heads=m.heads,
                n_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim, scale=m.scale, eps=eps, q_norm_weight=take(q + "q.norm"),
                k_norm_weight=take(q + "k.norm"), norm="before", inv_freq=rotary_frequencies(m.rot.base, dims).to(dev) if dims else None,
                rot_dims=dims, pairing="pairs", window=m.window, gate="none", sink=torch.zeros(m.heads, device=dev),
                head_temperature=take(q + "temp"), softcap=m.softcap, value_norm=True,
                padded_dim=GatedPagedAttention.padded_size(m.dim, m.vdim, runtime.dtype))
        else:
            mixer = make_part(
                "mixer", "latent_attention", w_down=stack(q, ("dq", "dkv", "g")), q_norm_weight=take(q + "dq.norm"),
                w_uq=take(q + "uq").contiguous(), kv_norm_weight=take(q + "dkv.norm"), w_uk=take(q + "uk"), w_uv=take(q + "uv"),
                w_o=take(q + "o").contiguous(), sink=take(q + "sink"), heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim,
                q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale, rot_base=m.rot.base, rot_dims=m.rot.dims, eps=eps,
                window=m.window, pairing="halves", gated=True)
        ff = None
        if L.mlp is not None:
            r, e = L.mlp, f"{p}mlp."
            ff = make_part("feed_forward", "routed_mlp", w_router=take(e + "router"), router_bias=None, correction=take(e + "correction"),
                           we_up=torch.stack([take(f"{e}e{j}.up") for j in range(r.experts)]),
                           we_down=torch.stack([take(f"{e}e{j}.down") for j in range(r.experts)]), top_k=r.top, activation="gelu",
                           weight_form="sigmoid_corrected", groups=r.groups, keep=r.keep, group_top=GROUP_TOP)
        blocks.append(make_part("block", "post_norm", norm1=norm(p + "norm1"), mixer=mixer,
                                norm2=None if ff is None else norm(p + "norm2"), feed_forward=ff))
    return DecoderModel(runtime, take("embed").contiguous(), blocks, norm("final.norm"), take("head").contiguous(), config=cfg)


MARINEX = Architecture(name="Marinex", parse_config=MarinexConfig.from_dict, tensor_specs=tensor_specs, build=build)
register_architecture(MARINEX)
