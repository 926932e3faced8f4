"""Shared by the Samerax tests: small configurations of their own, model folders from a seed, the plain implementation's
logits and the comparison of a trace's rows with them."""

from __future__ import annotations

import copy
import functools
import json
from pathlib import Path

import numpy as np
import torch

from tests.plain import samerax_plain as plain


def layer(heads, kv, dim, vdim, window, keep, scale, diff, rot=None, mlp=None, weights_of=None):
    """``rot``: (base, dims) or (base, dims, (factor, original, fast, slow)); ``window`` None: no mask."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "diff": diff}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), rot[2]))
    out = {"type": "attention", "mlp": mlp, "mixer": m}
    if weights_of is not None:
        out["weights_of"] = weights_of
    return out


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def again(layers, j):
    """Layer j once more, with its weights."""
    return dict(copy.deepcopy(layers[j]), weights_of=j)


def _with_repeats(layers, repeats):
    out = list(layers)
    for j in repeats:
        out.append(again(out, j))
    return out


CONFIGS = {
    # every size small and odd (no size is a multiple of 8: every product runs on the 32-bit FMA kernel in both precisions);
    # values shorter and longer than two maps' keys; a window shorter than a page that keeps tokens of the first page only,
    # one longer that keeps more tokens than its size; lambda near one (a difference of nearly equal maps); a layer that
    # runs three times, a repeat of a repeat
    "small": {
        "architecture": "Samerax", "vocab": 61, "width": 36, "norm": {"eps": 1e-5}, "embedding": {"scale": 1.7}, "logit_softcap": 4.0,
        "layers": _with_repeats([layer(6, 2, 5, 7, 7, 3, 0.5, 0.2, (60.0, 4, (4.0, 30, 4.0, 1.0)), moe(5, 2, 14)),
                                 layer(3, 3, 6, 13, 11, 18, 0.4, 0.9, (900.0, 6), dense(22))], (0, 2)) +
                  [layer(2, 1, 10, 9, 19, 0, 0.3, 0.5, None, moe(3, 1, 10))],
    },
    # sizes in multiples of 8 (bfloat16 products on the tcgen05 streaming kernel, attention on the tensor-core kernels at
    # padded sizes 64 and 128); ten query rows for a key head (more than a prefill block takes), 24 (more than a decode
    # block takes); maps of 64, of 40 (their border inside a 16-entry step), values below the padded size; many experts;
    # windows at and across page borders; no feed-forward in one layer
    "wide": {
        "architecture": "Samerax", "vocab": 96, "width": 128, "norm": {"eps": 1e-6}, "embedding": {"scale": 0.5}, "logit_softcap": 25.0,
        "layers": _with_repeats([layer(5, 1, 32, 64, 36, 5, 0.08, 0.4, (10000.0, 32), moe(8, 3, 48)),
                                 layer(4, 2, 64, 128, 64, 20, 0.05, 0.6, (500000.0, 64, (8.0, 128, 16.0, 2.0)), moe(12, 2, 32)),
                                 layer(12, 1, 40, 72, 50, 70, 0.06, 0.1, (300.0, 16), dense(96)),
                                 layer(2, 1, 64, 96, 40, 1, 0.05, 0.8, (10000.0, 32), None)], (1,)),
    },
    # no window at all in one layer, a window of one token that keeps the first, kept tokens over several pages, no cap on the
    # logits, no kept tokens; a head wider than the tensor-core attention kernels; every expert chosen
    "padded": {
        "architecture": "Samerax", "vocab": 50, "width": 48, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
        "layers": [layer(3, 3, 8, 40, None, 0, 0.25, 0.3, (100.0, 8), moe(4, 4, 16)),
                   layer(4, 2, 24, 16, 1, 1, 0.2, 0.5, (10000.0, 12), moe(3, 2, 24)),
                   layer(2, 1, 80, 144, 30, 37, 0.1, 0.45, (10000.0, 80), dense(40))],
    },
}


def random_config(rng) -> dict:
    """A configuration drawn at random: one to six layers, odd and even sizes, one to six query heads per key head, windows
    from one token to more than a prompt, from none to many kept tokens, repeats of any earlier layer."""
    width = rng.choice([24, 40, 64, 96, 128])
    layers = []
    for i in range(rng.randint(1, 6)):
        if layers and rng.random() < 0.3:
            layers.append(again(layers, rng.randrange(len(layers))))
            continue
        kv, dim = rng.choice([1, 2, 3]), rng.choice([4, 8, 12, 16, 32, 48, 64])
        rot = None
        if rng.random() < 0.9:
            rot = (rng.choice([100.0, 10000.0, 500000.0]), rng.choice([d for d in (2, 4, 8, dim // 2, dim) if d % 2 == 0 and d <= dim]))
            if rng.random() < 0.7:
                rot += ((rng.choice([1.0, 2.0, 8.0]), rng.choice([32, 200, 4096]), rng.choice([4.0, 32.0]), rng.choice([1.0, 2.0])),)
        mlp = None if rng.random() < 0.12 else dense(rng.choice([16, 20, 64])) if rng.random() < 0.4 else None
        if mlp is None and rng.random() < 0.85:
            experts = rng.choice([1, 2, 3, 6, 8, 20])
            mlp = moe(experts, rng.randint(1, min(5, experts)), rng.choice([8, 12, 16, 32]))
        layers.append(layer(kv * rng.choice([1, 2, 3, 6]), kv, dim, rng.choice([8, 20, 16, 64, 96, 128]), rng.choice([1, 2, 5, 16, 17, 31, 64, 100, None]),
                            rng.choice([0, 1, 2, 5, 16, 17, 40, 64, 90]), rng.uniform(0.05, 0.4), rng.uniform(0.0, 0.9), rot, mlp))
    cfg = {"architecture": "Samerax", "vocab": rng.choice([37, 64, 100]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])},
           "embedding": {"scale": rng.choice([0.3, 1.0, 5.0])}, "layers": layers}
    if rng.random() < 0.8:
        cfg["logit_softcap"] = rng.choice([2.0, 10.0, 50.0])
    return cfg


def mid_size_config(rng) -> dict:
    """A configuration drawn at random at sizes between the tiny ones above and a real model's: widths of 192 to 512, maps of
    16 to 64, up to 16 query heads, windows of 40 to 300 tokens that keep up to 200, 6 to 40 experts."""
    width = rng.choice([192, 256, 384, 512])
    layers = []
    for i in range(rng.randint(3, 6)):
        if layers and rng.random() < 0.25:
            layers.append(again(layers, rng.randrange(len(layers))))
            continue
        kv, dim = rng.choice([1, 2, 4]), rng.choice([16, 32, 40, 64])
        rot = (rng.choice([1e4, 5e5]), rng.choice([d for d in (8, 16, 32, dim) if d <= dim]), (rng.choice([2.0, 4.0]), rng.choice([256, 2048]), 32.0, 1.0))
        experts = rng.choice([6, 12, 24, 40])
        mlp = dense(rng.choice([128, 320])) if rng.random() < 0.4 else moe(experts, rng.randint(1, 4), rng.choice([48, 64, 80, 128]))
        layers.append(layer(kv * rng.choice([1, 2, 4]), kv, dim, rng.choice([32, 64, 80, 128]), rng.choice([48, 64, 100, 130, 300]),
                            rng.choice([0, 1, 4, 64, 70, 130, 200]), dim ** -0.5, rng.uniform(0.1, 0.8), rot, mlp))
    return {"architecture": "Samerax", "vocab": rng.choice([300, 500, 1000]), "width": width, "norm": {"eps": rng.choice([1e-5, 1e-6])},
            "embedding": {"scale": rng.choice([1.0, 4.0])}, "logit_softcap": rng.choice([5.0, 30.0]), "layers": layers}


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


def plain_logits(folder, tokens) -> np.ndarray:
    cfg, P = plain_model(str(folder))
    with torch.no_grad():
        return plain.forward(cfg, P, list(tokens)).numpy()


# float32: a few thousand roundings of 6e-8 per logit.  bfloat16: activations are rounded (4e-3) several times per layer,
# and a tiny model's logits are sums of few terms, so single rows scatter: the mean over all rows is held tight and a
# single row is capped where a fault (a key off by one, a kept token left out) would still stand out by far.
TOL = {"float32": 3e-5, "bfloat16": 1.2e-1}
TOL_MEAN = {"float32": 1e-5, "bfloat16": 3e-2}


def row_err(got: np.ndarray, ref: np.ndarray) -> float:
    """Difference of two logit rows, each with its mean taken off, relative to the reference row's spread."""
    d = (got - got.mean()) - (ref - ref.mean())
    return float(np.sqrt((d ** 2).mean()) / max(np.sqrt(((ref - ref.mean()) ** 2).mean()), 1e-9))


def compare(folder, requests: dict, got: dict, dtype: str, stray: int = 0) -> float:
    """Every logit row a trace produced against the plain implementation's row at that place.  Among hundreds of rows
    ``stray`` of them may scatter past the cap for a single row, up to twice as far; the mean stays as tight."""
    errs = []
    for rid, toks in requests.items():
        ref = plain_logits(folder, toks)
        for pos in range(len(toks)):
            if (rid, pos) in got:
                err = row_err(got[(rid, pos)], ref[pos])
                assert err < TOL[dtype] * (2 if stray else 1), f"{dtype}: request {rid} position {pos}: relative error {err:.3e}"
                errs.append(err)
    assert sum(e >= TOL[dtype] for e in errs) <= stray, f"{dtype}: more than {stray} rows beyond {TOL[dtype]}"
    mean = float(np.mean(errs))
    assert mean < TOL_MEAN[dtype], f"{dtype}: mean relative error {mean:.3e} over {len(errs)} rows"
    return max(errs)


def greedy_checked(folder, prompt, got, dtype: str) -> None:
    """``got`` must be the plain implementation's greedy continuation, except where its two best logits are closer than the
    precision tells apart (the plain implementation follows the engine's tokens)."""
    toks = list(prompt) + list(got)
    tol = 1e-4 if dtype == "float32" else 8e-2
    logits = plain_logits(folder, toks)
    for step, g in enumerate(got):
        row = logits[len(prompt) - 1 + step]
        best = int(np.argmax(row))
        if g != best:
            gap = float(row[best] - row[g]) / float(np.abs(row - row.mean()).max())
            assert gap < tol, f"{dtype}: step {step}: engine chose {g}, plain {best}, relative logit gap {gap:.2e}"
