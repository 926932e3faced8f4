"""Shared by the Marinex tests: small configurations of their own, model folders from a seed, the plain implementation's
logits and the comparison of a trace's rows with them."""

from __future__ import annotations

import copy
import functools
import json
from pathlib import Path

import numpy as np
import torch

from tests.plain import marinex_plain as plain


def attention(heads, kv, dim, vdim, scale, softcap, rot=None, mlp=None, window=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if softcap is not None:
        m["softcap"] = softcap
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, window, scale, base=10000.0, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if window is not None:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def moe(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


CONFIGS = {
    # every size small and odd (no size is a multiple of 8: every product runs on the 32-bit FMA kernel in both precisions);
    # three query heads per key head, values of another size than keys, part of the head rotated, a cap that bends most
    # scores; a window shorter than a page; groups of which two are kept; the last layer has no feed-forward
    "small": {
        "architecture": "Marinex", "vocab": 61, "width": 36, "norm": {"eps": 1e-5},
        "layers": [attention(6, 2, 10, 7, 0.5, 1.5, (60.0, 6), moe(6, 2, 14, (3, 2))),
                   latent(3, 5, 6, 9, 11, 13, 7, 0.3, 50.0, moe(5, 3, 9)),
                   attention(2, 2, 6, 11, 0.7, 4.0, (900.0, 6), moe(4, 1, 10, (2, 1))),
                   latent(2, 7, 2, 5, 6, 10, 19, 0.4, 1000.0)],
    },
    # sizes in multiples of 8 (bfloat16 products on the tcgen05 streaming kernel, attention on the tensor-core kernels at
    # head sizes 64 and 128); one key head for four query heads; the whole head rotated; a window that straddles page
    # borders; eight experts in four groups of which two are kept; the first layer has no feed-forward
    "wide": {
        "architecture": "Marinex", "vocab": 96, "width": 128, "norm": {"eps": 1e-6},
        "layers": [attention(4, 1, 64, 64, 0.3, 6.0, (10000.0, 64)),
                   latent(4, 40, 16, 24, 48, 64, 36, 0.15, 10000.0, moe(8, 2, 64, (4, 2))),
                   attention(2, 2, 128, 128, 0.2, 12.0, (500000.0, 32), moe(6, 4, 32, (2, 2))),
                   latent(6, 16, 32, 40, 40, 96, 24, 0.2, 300.0, moe(8, 3, 48, (2, 1)))],
    },
    # keys shorter than values and values shorter than keys, both padded in the cache (to 64 in bfloat16); no rotation of
    # the attention at all; a window of one token (a query sees itself and the sink); one without a window; a cap that
    # hardly bends, and none; top-1 of one group
    "padded": {
        "architecture": "Marinex", "vocab": 50, "width": 48, "norm": {"eps": 1e-6},
        "layers": [attention(3, 3, 24, 40, 0.25, 60.0, None, moe(3, 1, 16)),
                   latent(2, 8, 8, 16, 16, 24, 1, 0.4, 100.0, moe(4, 2, 24, (1, 1))),
                   attention(2, 1, 40, 24, 0.2, None, (10000.0, 8), moe(6, 3, 8, (2, 1))),
                   latent(5, 12, 4, 8, 24, 40, None, 0.3, 10000.0, moe(2, 2, 16))],
    },
}


def random_config(rng) -> dict:
    """A configuration drawn at random: two to six layers of the two mixers in any order, odd and even sizes, one to four
    query heads per key head, windows from one token to more than a prompt, caps from hard to none, every kind of router."""
    width = rng.choice([24, 40, 64, 96, 128])

    def mlp():
        if rng.random() < 0.15:
            return None
        experts = rng.choice([2, 3, 4, 6, 8, 12])
        divisors = [g for g in (1, 2, 3, 4) if experts % g == 0]
        groups = None
        if rng.random() < 0.75:
            g = rng.choice(divisors)
            groups = (g, rng.randint(1, g))
        usable = experts if groups is None else experts // groups[0] * groups[1]
        return moe(experts, rng.randint(1, min(5, usable)), rng.choice([8, 12, 16, 32, 40]), groups)

    layers = []
    for _ in range(rng.randint(2, 6)):
        if rng.random() < 0.5:
            kv = rng.choice([1, 2, 3])
            dim = rng.choice([8, 12, 16, 32, 64, 96, 128])
            rot = None if rng.random() < 0.15 else (rng.choice([100.0, 10000.0, 500000.0]), rng.choice([d for d in (2, 4, 8, dim // 2, dim) if d % 2 == 0]))
            cap = None if rng.random() < 0.1 else rng.choice([0.8, 2.0, 7.0, 25.0])
            layers.append(attention(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([8, 20, 16, 64, 128]), rng.uniform(0.05, 0.4), cap, rot, mlp(),
                                    None if rng.random() < 0.85 else rng.choice([5, 33])))
        else:
            layers.append(latent(rng.choice([1, 2, 3, 5, 8]), rng.choice([4, 8, 16, 32]), rng.choice([2, 6, 8, 16, 32]), rng.choice([5, 8, 16, 24, 48]),
                                 rng.choice([7, 16, 24, 64]), rng.choice([9, 24, 32, 64, 128]), rng.choice([1, 2, 5, 16, 17, 31, 64, 100, None]),
                                 rng.uniform(0.1, 0.4), rng.choice([50.0, 10000.0, 1e6]), mlp()))
    return {"architecture": "Marinex", "vocab": rng.choice([37, 64, 100]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}


def mid_size_config(rng) -> dict:
    """A configuration drawn at random at sizes between the tiny ones above and a real model's: widths of 192 to 512, head
    sizes 32 to 128, up to 16 query heads, latents of 64 to 320, windows of 40 to 300 tokens, 6 to 40 experts."""
    width = rng.choice([192, 256, 384, 512])

    def mlp():
        experts = rng.choice([6, 12, 24, 40])
        divisors = [g for g in (2, 3, 4, 8) if experts % g == 0]
        g = rng.choice(divisors)
        keep = rng.randint(max(1, g // 2), g)
        return moe(experts, rng.randint(1, min(6, experts // g * keep)), rng.choice([48, 64, 80, 128]), (g, keep))

    layers = []
    for i in range(rng.randint(3, 6)):
        if rng.random() < 0.5:
            kv = rng.choice([1, 2, 4])
            dim = rng.choice([32, 64, 96, 128])
            layers.append(attention(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([32, 64, 128]), dim ** -0.5, rng.choice([5.0, 15.0, 50.0]),
                                    (rng.choice([1e4, 5e5]), rng.choice([d for d in (16, 32, 64, dim) if d <= dim])), mlp()))
        else:
            layers.append(latent(rng.choice([2, 4, 6, 12, 16]), rng.choice([32, 64, 128]), rng.choice([16, 32, 64]), rng.choice([32, 64, 96]),
                                 rng.choice([48, 96, 160]), rng.choice([64, 160, 256, 320]), rng.choice([48, 64, 100, 130, 300]), rng.uniform(0.08, 0.2),
                                 rng.choice([1e4, 1e6]), mlp()))
    return {"architecture": "Marinex", "vocab": rng.choice([300, 500, 1000]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])}, "layers": layers}


def config(name: str, **overrides) -> dict:
    c = copy.deepcopy(CONFIGS[name])
    c.update(overrides)
    return c


def write_model(path, cfg: dict, seed: int, std: float = 0.15):
    from jax_llm_examples_b200 import write_random_model

    return write_random_model(path, cfg, seed, norm_noise=0.1, std=std)


def make_dir(path, name: str, seed: int, **overrides):
    return write_model(path, config(name, **overrides), seed)


@functools.lru_cache(maxsize=32)
def plain_model(folder: str):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), plain.read_safetensors(folder / "model.safetensors")


def routed_layers(folder) -> list[int]:
    cfg, _ = plain_model(str(folder))
    return [i for i, L in enumerate(cfg["layers"]) if L.get("mlp")]


def plain_logits(folder, tokens, forced=None):
    """(logits [T, V], the share of (token, routed layer) pairs whose forced experts are not the set the plain router
    chose itself)."""
    cfg, P = plain_model(str(folder))
    trace = []
    with torch.no_grad():
        logits = plain.forward(cfg, P, list(tokens), forced, trace)
    differ = total = 0
    for _, used, own in trace:
        if used is not None:
            total += used.shape[0]
            differ += int((torch.sort(used, dim=1).values != torch.sort(own, dim=1).values).any(dim=1).sum())
    return logits.numpy(), differ / max(total, 1)


# float32: a few thousand roundings of 6e-8 per logit.  bfloat16: activations are rounded (4e-3) several times per layer,
# and a tiny model's logits are sums of few terms, so single rows scatter: the mean over all rows is held tight and a
# single row is capped where a fault (a key off by one, a sink left out) would still stand out by far.
TOL = {"float32": 3e-5, "bfloat16": 1.2e-1}
TOL_MEAN = {"float32": 1e-5, "bfloat16": 3e-2}
# The share of choices that may differ from the plain router's: two scores that tie within the precision go either way; a
# fault in the routing (a group, a correction, a tie rule) changes tens of percent.
OTHER_CHOICES = {"float32": 0.004, "bfloat16": 0.04}


def row_err(got: np.ndarray, ref: np.ndarray) -> float:
    """Difference of two logit rows, each with its mean taken off, relative to the reference row's spread."""
    d = (got - got.mean()) - (ref - ref.mean())
    return float(np.sqrt((d ** 2).mean()) / max(np.sqrt(((ref - ref.mean()) ** 2).mean()), 1e-9))


def compare(folder, requests: dict, got: dict, routing: dict | None, dtype: str, stray: int = 0) -> float:
    """Every logit row a trace produced against the plain implementation's row at that place.  With ``routing`` (the
    engine's expert choices by (request, position)) the plain implementation takes those experts; they must be its own
    choice too but for a small share of near-ties.  Among hundreds of rows `stray` of them may scatter past the cap for
    a single row, up to twice as far; the mean stays as tight."""
    errs, shares = [], []
    routed = routed_layers(folder)
    for rid, toks in requests.items():
        forced = None
        if routing is not None and routed:
            forced = {layer: torch.as_tensor(np.stack([routing[(rid, p)][j] for p in range(len(toks))])) for j, layer in enumerate(routed)}
        ref, share = plain_logits(folder, toks, forced)
        shares.append((share, len(toks)))
        for pos in range(len(toks)):
            if (rid, pos) in got:
                err = row_err(got[(rid, pos)], ref[pos])
                assert err < TOL[dtype] * (2 if stray else 1), f"{dtype}: request {rid} position {pos}: relative error {err:.3e}"
                errs.append(err)
    total = max(sum(n for _, n in shares), 1)
    other = sum(s * n for s, n in shares) / total
    few = 3 / (total * max(len(routed), 1)) if dtype == "bfloat16" else 0.0  # a handful of tokens: three near-ties are no share
    assert other <= max(OTHER_CHOICES[dtype], few), f"{dtype}: {other:.2%} of the expert choices differ from the plain router's"
    assert sum(e >= TOL[dtype] for e in errs) <= stray, f"{dtype}: more than {stray} rows beyond {TOL[dtype]}"
    mean = float(np.mean(errs))
    assert mean < TOL_MEAN[dtype], f"{dtype}: mean relative error {mean:.3e} over {len(errs)} rows"
    return max(errs)


def engine_choices(model, tokens, tail: int) -> dict | None:
    """The experts the engine takes for every token of a sequence whose last ``tail`` tokens it decodes one by one, in the form
    that ``plain_logits`` takes as ``forced``."""
    import jax_llm_examples_b200 as J
    from tests import helpers as H

    routed = [i for i, L in enumerate(model.config.layers) if L.mlp is not None]
    if not routed:
        return None
    engine = J.Engine(model, max_tokens=-(-len(tokens) // 64) * 64, page_size=64, max_slots=1)
    _, routing = H.run_trace(engine, H.trace_tail_decode({"a": list(tokens)}, tail), record_routing=True)
    return {layer: torch.as_tensor(np.stack([routing[("a", p)][j] for p in range(len(tokens))])) for j, layer in enumerate(routed)}


def greedy_checked(folder, model, prompt, got, dtype: str) -> None:
    """``got`` must be the plain implementation's greedy continuation, except where its two best logits are closer than the
    precision tells apart (the plain implementation follows the engine's tokens).  In bfloat16 it also takes the engine's
    experts: where two choice scores tie, one token through another expert is another logit, not a rounding."""
    toks = list(prompt) + list(got)
    tol = 1e-4 if dtype == "float32" else 8e-2
    forced = engine_choices(model, toks, len(got)) if dtype == "bfloat16" else None
    logits, other = plain_logits(folder, toks, forced)
    assert other <= 0.1, f"{dtype}: {other:.1%} of the expert choices differ from the plain router's"
    for step, g in enumerate(got):
        row = logits[len(prompt) - 1 + step]
        best = int(np.argmax(row))
        if g != best:
            gap = float(row[best] - row[g]) / float(np.abs(row - row.mean()).max())
            assert gap < tol, f"{dtype}: step {step}: engine chose {g}, plain {best}, relative logit gap {gap:.2e}"
