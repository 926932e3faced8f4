"""Samerax on the GPU against the plain implementation: each mechanism alone (kernel or part against the plain function of
the same name), inputs made so that a fault shows (a far token, a window's edge, the last kept token and the first one that
is not, the weight of the second map, a token's experts), then whole models through the engine's step function under every
kind of cut, batches against requests alone, pages and slots that are used again, long decoding, and greedy generation
through the scheduler.  All configurations are this file's own (``tests/samerax_helpers.py``)."""

import json
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import helpers as H
from tests import samerax_helpers as SX
from tests.plain import samerax_plain as plain
from tests.test_koduzen_gpu import LONG_PORTIONS, PORTIONS
from tests.test_tebivik_gpu import _close, _ctx

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [("float32", torch.float32, 2e-5), ("bfloat16", torch.bfloat16, 3e-2)]
F64 = torch.float64


# ------------------------------------------------------------------------------------- kernels alone
def _attention_kernel(kind, q, pages, table, req, pos, tiles, scale, window, keep, diff=None, out=None):
    """One of the four attention kernels over all rows of q."""
    from jax_llm_examples_b200.kernels import api as K

    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    out = torch.full_like(q, float("nan")) if out is None else out
    if kind == "generic":
        K.attention_generic(q, pages, table, req, pos, out, scale, 0, window, 0.0, 1.0, st, keep=keep)
    elif kind == "decode":
        keys, splits = K.attention_decode_plan(int(pos.max()) + 1, 0, window, 600)  # as few keys per split as there may be
        n = q.shape[0] * q.shape[1] * splits
        K.attention_decode(q, pages, table, req, pos, out, scale, 0, window, 0.0, 1.0, torch.empty(n * q.shape[2], device=DEV),
                           torch.empty(2 * n, device=DEV), splits, keys, st, keep=keep, diff=diff)
    else:
        fn, rows = (K.attention_prefill, 16) if kind == "flash" else (K.attention_prefill_tc, 128)
        t = torch.tensor([(f + o, min(rows, n - o)) for f, n in tiles for o in range(0, n, rows)], dtype=torch.int32, device=DEV)
        fn(q, pages, table, req, pos, out, t, t.shape[0], scale, 0, window, 0.0, 1.0, st, keep=keep, diff=diff)
    assert int(st) == 0
    return out


def _cache(lens, Hkv, dh, page, dtype):
    """Random pages of requests of those lengths: (pages, table, keys [r] float64, values [r])."""
    width = -(-max(lens) // page)
    pages = torch.randn(len(lens) * width + 3, 2, Hkv, page, dh, device=DEV).to(dtype)
    table = torch.randperm(pages.shape[0])[:len(lens) * width].to(torch.int32).view(len(lens), width).to(DEV)
    flat = [pages[table[r].long()].double().cpu().permute(1, 2, 0, 3, 4).reshape(2, Hkv, -1, dh)[:, :, :n] for r, n in enumerate(lens)]
    return pages, table, [f[0] for f in flat], [f[1] for f in flat]


def _reference(q, ks, vs, req, pos, scale, window, keep):
    """[N, Hq, dh] float64: every query row over its request's visible keys."""
    N, Hq, dh = q.shape
    out = torch.empty(N, Hq, dh, dtype=F64)
    for n in range(N):
        r, p = int(req[n]), int(pos[n])
        T = p + 1
        mask = plain.window_with_kept_start(T, window or T, keep)[p]
        for h in range(Hq):
            g = h // (Hq // ks[r].shape[0])
            w = plain.masked_softmax((ks[r][g, :T] @ q[n, h].double().cpu() * scale)[None], mask[None])[0]
            out[n, h] = w @ vs[r][g, :T]
    return out


@pytest.mark.parametrize("kind, dtype, dh, page, tol", [
    ("generic", torch.float32, 24, 16, 2e-5), ("generic", torch.bfloat16, 144, 16, 1e-2), ("decode", torch.bfloat16, 64, 16, 1e-2), ("decode", torch.bfloat16, 128, 64, 1e-2),
    ("decode", torch.bfloat16, 128, 24, 1e-2), ("flash", torch.bfloat16, 64, 16, 1e-2), ("flash", torch.bfloat16, 128, 64, 1e-2), ("flash", torch.bfloat16, 64, 40, 1e-2),
    ("tc", torch.bfloat16, 128, 64, 1e-2)])
@pytest.mark.parametrize("Hq, Hkv", [(2, 1), (20, 2), (36, 2)])
@pytest.mark.parametrize("window, keep", [(40, 5), (130, 64), (1, 1), (600, 70), (64, 200), (100, 0)])
def test_kept_first_keys_in_every_attention_kernel(kind, dtype, dh, page, tol, Hq, Hkv, window, keep):
    """A window that keeps the sequence's first keys, in the four kernels: more kept keys than the window has, kept keys across
    tiles and pages, several splits (which share the kept tiles), groups of more query heads than a block takes, also with
    the pages that no query sees taken out of the table."""
    torch.manual_seed(window + Hq)
    single = kind == "decode"
    lens = [1400, 9, 130, 1] if single else [700, 30]
    starts = [n - 1 for n in lens] if single else [650 if kind != "tc" else 560, 0]
    if kind == "tc":
        lens, starts = [700, 80], [560, 0]
    pages, table, ks, vs = _cache(lens, Hkv, dh, page, dtype)
    q_lens = [n - s for n, s in zip(lens, starts)]
    req = torch.tensor([r for r, n in enumerate(q_lens) for _ in range(n)], dtype=torch.int32, device=DEV)
    pos = torch.tensor([s + i for s, n in zip(starts, q_lens) for i in range(n)], dtype=torch.int32, device=DEV)
    q = (torch.randn(len(req), Hq, dh, device=DEV) * 1.5).to(dtype)
    tiles = [(sum(q_lens[:r]), n) for r, n in enumerate(q_lens)]
    some = torch.randperm(len(req))[:12].sort().values
    some = torch.unique(torch.cat([some, torch.tensor([0, len(req) - 1])]))
    want = _reference(q[some], ks, vs, req[some], pos[some], dh ** -0.5, window, keep)
    got = _attention_kernel(kind, q, pages, table, req, pos, tiles, dh ** -0.5, window, keep)
    assert not got.isnan().any()
    _close(got[some], want, tol, kind)
    gone = table.clone()
    for r, s in enumerate(starts):
        first = max(0, s - window + 1) // page
        kept = -(-keep // page)
        if first > kept:
            gone[r, kept:first] = -1
    if kind != "generic":  # (the generic kernel reports a missing page that it would read; it reads none of these either)
        pages[[i for i in range(pages.shape[0]) if i not in set(gone[gone >= 0].tolist())]] = 0.25  # finite, as released pages are
    again = _attention_kernel(kind, q, pages, gone, req, pos, tiles, dh ** -0.5, window, keep)
    assert torch.equal(again, got)


@pytest.mark.parametrize("kind, dh, page", [("decode", 64, 16), ("decode", 128, 64), ("decode", 128, 24), ("flash", 64, 16), ("flash", 128, 64), ("flash", 64, 40),
                                            ("flash", 128, 40), ("tc", 128, 64)])
@pytest.mark.parametrize("H_, G, d, dv", [(2, 1, 32, 64), (12, 2, 20, 33), (20, 1, 8, 48), (3, 3, 64, 128), (4, 2, 41, 100), (4, 2, 16, 8)])
def test_the_difference_of_two_maps_in_the_kernels_last_lines(kind, dh, page, H_, G, d, dv):
    """The three tensor-core kernels, which end in the difference, its norm and the store, against the generic kernel's 32-bit
    maps and the difference as a kernel of its own; and that one against the plain function.  Also into a column range."""
    from jax_llm_examples_b200.kernels import api as K

    if max(2 * d, dv) > dh:
        pytest.skip("does not fit this head size")
    torch.manual_seed(H_ + d)
    lens = [1300, 40, 1] if kind == "decode" else [300, 75]
    starts = [n - 1 for n in lens] if kind == "decode" else [130, 0]
    pages, table, ks, vs = _cache(lens, G, dh, page, torch.bfloat16)
    pages[:, 0, ..., 2 * d:] = 0
    pages[:, 1, ..., dv:] = 0
    q_lens = [n - s for n, s in zip(lens, starts)]
    req = torch.tensor([r for r, n in enumerate(q_lens) for _ in range(n)], dtype=torch.int32, device=DEV)
    pos = torch.tensor([s + i for s, n in zip(starts, q_lens) for i in range(n)], dtype=torch.int32, device=DEV)
    N = len(req)
    q = torch.zeros(N, 2 * H_, dh, device=DEV)
    q[:, 0::2, :d], q[:, 1::2, d:2 * d] = torch.randn(N, H_, d, device=DEV), torch.randn(N, H_, d, device=DEV)
    q = (q * 2).bfloat16()
    window, keep, lam, mult, eps, scale = 90, 20, 0.9, 0.35, 1e-5, d ** -0.5
    maps = torch.empty(N, 2 * H_, dh, device=DEV)
    _attention_kernel("generic", q, pages, table, req, pos, None, scale, window, keep, out=maps)
    want = torch.empty(N, H_ * dv, device=DEV)
    K.map_difference(maps, want, K.map_difference_spec(d, lam, mult, eps, want, H_))
    m64 = maps.double().cpu()[..., :dv]
    ref = plain.rms_divide(m64[:, 0::2] - lam * m64[:, 1::2], eps) * mult
    _close(want, ref.reshape(N, -1), 2e-5, "the difference alone")
    got = torch.full((N, H_ * dv), float("nan"), device=DEV, dtype=torch.bfloat16)
    _attention_kernel(kind, q, pages, table, req, pos, [(sum(q_lens[:r]), n) for r, n in enumerate(q_lens)], scale, window, keep,
                      K.map_difference_spec(d, lam, mult, eps, got, H_), got)
    _close(got, want, 3e-2, kind)
    wide = torch.full((N, H_ * dv + 24), 7.0, device=DEV, dtype=torch.bfloat16)
    part = wide[:, 16:16 + H_ * dv]
    _attention_kernel(kind, q, pages, table, req, pos, [(sum(q_lens[:r]), n) for r, n in enumerate(q_lens)], scale, window, keep,
                      K.map_difference_spec(d, lam, mult, eps, part, H_), part)
    if kind != "decode" or int(pos.max()) < 512:
        assert torch.equal(part, got)
    _close(part, want, 3e-2, kind)
    assert bool((wide[:, :16] == 7).all()) and bool((wide[:, 16 + H_ * dv:] == 7).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H_, G, d, dv, dpad, rot, splits", [(3, 1, 5, 7, 10, 4, 1), (4, 2, 32, 64, 64, 32, 3), (2, 2, 24, 100, 128, 10, 2), (6, 3, 64, 128, 128, 0, 1),
                                                          (3, 1, 20, 36, 64, 16, 2)])
def test_biased_projections_turned_and_laid_side_by_side(dtype, H_, G, d, dv, dpad, rot, splits):
    """Partial sums added, the bias added, every map turned with an amplitude, keys of both maps in one cached row, queries
    at their map's place with zeros elsewhere; few tokens and many."""
    from jax_llm_examples_b200.kernels import api as K

    for N in (3, 70):
        torch.manual_seed(N + d)
        cols, page = 2 * H_ * d + 2 * G * d + G * dv, 16
        off = 4 if d % 4 == 0 else 5  # the first projected column (in fours: the rows that take 16 bytes at a time)
        proj, bias = torch.randn(splits, N, cols + off, device=DEV), torch.randn(cols, device=DEV)
        pos = torch.arange(40, 40 + N, dtype=torch.int32, device=DEV)
        width = (40 + N) // page + 1
        pages = torch.full((width, 2, G, page, dpad), 9.0, device=DEV, dtype=dtype)
        table = torch.randperm(width).to(torch.int32).view(1, width).to(DEV)
        q, st = torch.full((N, 2 * H_, dpad), 9.0, device=DEV, dtype=dtype), torch.zeros(1, dtype=torch.int32, device=DEV)
        f = torch.rand(max(rot // 2, 1), device=DEV)
        K.rope_norm_kv_store(K.rows_view(proj, splits, off), 2 * H_ * d, 2 * (H_ + G) * d, q, pages, table, torch.zeros(N, dtype=torch.int32, device=DEV), pos, None,
                             None, 1e-6, f if rot else None, rot, 2 * H_, G, d, dv, st, "halves", "none", 1.3, bias=bias, maps=2)
        assert int(st) == 0
        rows = proj.sum(0)[:, off:].double().cpu() + bias.double().cpu()

        def turned(x):
            y, half = x.clone(), rot // 2
            for i in range(half):
                a = (pos.float() * f[i]).double().cpu()[:, None]
                u, v = x[..., i], x[..., i + half]
                y[..., i], y[..., i + half] = 1.3 * (u * torch.cos(a) - v * torch.sin(a)), 1.3 * (v * torch.cos(a) + u * torch.sin(a))
            return y

        qr, kr = turned(rows[:, :2 * H_ * d].view(N, 2 * H_, d)), turned(rows[:, 2 * H_ * d:2 * (H_ + G) * d].view(N, 2 * G, d))
        want_q, want = torch.zeros(N, 2 * H_, dpad, dtype=F64), torch.zeros(2, N, G, dpad, dtype=F64)
        want_q[:, 0::2, :d], want_q[:, 1::2, d:2 * d] = qr[:, 0::2], qr[:, 1::2]
        want[0, :, :, :2 * d] = kr.reshape(N, G, 2 * d)
        want[1, :, :, :dv] = rows[:, 2 * (H_ + G) * d:].view(N, G, dv)
        tol = 1e-5 if dtype == torch.float32 else 5e-3
        _close(q, want_q, tol, "queries")
        at = pos.long()
        got = pages[table[0, at // page].long(), :, :, at % page]  # [N, 2, G, dpad]
        _close(got.permute(1, 0, 2, 3), want, tol, "cache")
        assert bool((q.float().cpu()[want_q == 0] == 0).all())


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("N, D, copies, k, splits", [(3, 36, 2, 3, 1), (5, 2048, 4, 2, 3), (40, 1024, 1, 1, 2), (17, 200, 16, 4, 1), (2, 30, 3, 5, 2), (70, 4096, 2, 2, 1)])
def test_the_norm_writes_its_rows_where_they_are_wanted(out_dtype, N, D, copies, k, splits):
    """x += scale * (the sum of a token's rows in expert order + a second term); the normed row goes to all its places, in the
    one-block kernel and in the cluster kernel of a decode step."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(D + N)
    x, y, z = torch.randn(N, D, device=DEV), torch.randn(splits, N * k, D, device=DEV), torch.randn(N, D, device=DEV)
    idx, places = (torch.randperm(N * m).to(torch.int32).to(DEV) for m in (k, copies))
    w, out = torch.randn(D, device=DEV), torch.full((N * copies, D), float("nan"), device=DEV, dtype=out_dtype)
    ref = x.double() + y.double().sum(0)[idx.long()].view(N, k, D).sum(1) / k + z.double() / k
    K.add_rmsnorm(x, [(y, splits, idx, k, 0), (z, 1, None, 1, 0)], w, 1e-5, out, places=places, copies=copies, delta_scale=1.0 / k)
    _close(x, ref, 2e-6, "residual")
    normed = plain.rms_norm(ref, w.double(), 1e-5)
    _close(out[places.long()].view(N, copies, D), normed[:, None].expand(N, copies, D), 2e-6 if out_dtype == torch.float32 else 5e-3, "rows")
    first = out[places.long()].view(N, copies, D)
    assert torch.equal(first, first[:, :1].expand_as(first))


@pytest.mark.parametrize("N, k, V, E, tile_rows", [(1, 2, 50, 5, 16), (7, 3, 20, 3, 0), (300, 2, 999, 256, 32), (700, 2, 64, 8, 128), (2048, 2, 5000, 16, 96), (4000, 5, 300, 200, 64)])
def test_sort_by_a_table_of_token_ids(N, k, V, E, tile_rows):
    """The pairs of a step sorted by the experts that a table gives its tokens: what the sort of the looked-up choices gives,
    in both sort kernels, with and without the choices handed back."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(N)
    table = torch.rand(V, E).argsort(1)[:, :k].to(torch.int32).contiguous().to(DEV)
    ids = torch.randint(0, V, (N,), dtype=torch.int32, device=DEV)
    choice, P = table[ids.long()].contiguous(), N * k
    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device=DEV)  # noqa: E731

    def run(given, **kw):
        off, pair, pos = i32(E + 1), i32(P), i32(P)
        tiles = (i32(2 * (-(-P // tile_rows) + E)), i32(1)) if tile_rows else ()
        K.expert_sort(given, off, pair, pos, E, st, 0, tile_rows, *tiles, **kw)
        n = int(tiles[1]) if tiles else 0
        return [off, pair, pos] + ([tiles[0][:2 * n], tiles[1]] if tiles else [])

    want = run(choice)
    handed = i32(P)
    for given in (None, handed):
        got = run(given, token_ids=ids, table=table)
        assert all(torch.equal(a, b) for a, b in zip(want, got))
    assert torch.equal(handed.view(N, k), choice) and int(st) == 0
    bad = ids.clone()
    bad[0] = V  # a token id outside the table is reported, not followed
    run(None, token_ids=bad, table=table)
    assert int(st) == 2


def test_soft_cap_in_place():
    from jax_llm_examples_b200.kernels import api as K

    for n, cap in ((1, 3.0), (4099, 15.0), (300001, 0.5)):
        x = torch.randn(n, device=DEV) * 20
        ref = plain.soft_cap(x.double().cpu(), cap)
        K.soft_cap(x, cap)
        _close(x, ref, 1e-6)


# --------------------------------------------------------------------------------------------- parts alone
def _mixer(wd, m, eps, dtype):
    from jax_llm_examples_b200.parts import DifferentialAttention, rotary_frequencies, yarn_frequencies

    c = lambda n: wd[n].to(dtype).to(DEV)  # noqa: E731
    rot, inv, amp = m.get("rot"), None, 1.0
    if rot:
        sc = rot.get("scaling")
        inv, amp = (rotary_frequencies(rot["base"], rot["dims"]), 1.0) if sc is None else \
            yarn_frequencies(rot["base"], rot["dims"], sc["factor"], sc["original"], sc["fast"], sc["slow"])
        inv = inv.to(DEV)
    mask = m.get("mask") or {}
    return DifferentialAttention(
        torch.cat([c("q"), c("k"), c("v")]), c("o"), m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps,
        map_weight=DifferentialAttention.map_weight_of(wd["lq1"], wd["lk1"], wd["lq2"], wd["lk2"], m["diff"]), diff=m["diff"],
        in_bias=torch.cat([c("q.b"), c("k.b"), c("v.b")]), inv_freq=inv, rot_dims=rot["dims"] if rot else 0, rot_amplitude=amp, window=mask.get("size"),
        keep_first=mask.get("keep_first", 0), padded_dim=DifferentialAttention.padded_size(m["dim"], m["vdim"], dtype))


def _weights(m, D, dtype, spread=0.3):
    g = lambda *s: (torch.randn(*s) * spread).to(dtype)  # noqa: E731
    Hh, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    return {"q": g(2 * Hh * d, D), "q.b": g(2 * Hh * d), "k": g(2 * G * d, D), "k.b": g(2 * G * d), "v": g(G * dv, D), "v.b": g(G * dv), "o": g(D, Hh * dv),
            "lq1": g(d), "lk1": g(d), "lq2": g(d), "lk2": g(d)}


def _in_portions(mixer, rt, hs, dtype, portions, page):
    """The part over one request's rows, in portions; before each, the pages that the manager would have taken back by then
    are gone from the table."""
    from jax_llm_examples_b200.parts import LayerCache

    need, r = mixer.kv_need(), mixer.kv_need().retention
    width = -(-hs.shape[0] // page)
    pages = torch.zeros(width + 5, need.planes, need.num_kv_heads, page, need.head_dim, device=DEV, dtype=dtype)
    table = torch.randperm(width + 5)[:width].reshape(1, width).to(torch.int32).to(DEV)
    outs = []
    for lo, hi in portions:
        if r.kind == 2:
            dead, kept = max(0, lo - r.size + 1) // page, -(-r.keep // page)
            if dead > kept:
                table[0, kept:dead] = -1
        ctx = _ctx(rt, [hi - lo], [lo], planners=mixer.step_planners(), page_size=page)
        outs.append(H.as_rows_sum(mixer.forward(ctx, hs[lo:hi].to(DEV), LayerCache(pages, table, True, None))))
        assert int(ctx.status) == 0
    return torch.cat(outs)


ROT = {"base": 60.0, "dims": 4, "scaling": {"factor": 4.0, "original": 30, "fast": 4.0, "slow": 1.0}}


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("m, portions", [
    ({"heads": 6, "kv_heads": 2, "dim": 5, "vdim": 7, "scale": 0.5, "diff": 0.2, "mask": {"size": 7, "keep_first": 3}, "rot": ROT}, PORTIONS),
    ({"heads": 4, "kv_heads": 1, "dim": 32, "vdim": 64, "scale": 0.2, "diff": 0.5, "mask": {"size": 20, "keep_first": 17}, "rot": {"base": 1e4, "dims": 32}}, PORTIONS),
    ({"heads": 2, "kv_heads": 2, "dim": 24, "vdim": 16, "scale": 0.3, "diff": 0.8}, PORTIONS),
    ({"heads": 8, "kv_heads": 2, "dim": 64, "vdim": 128, "scale": 0.1, "diff": 0.4, "mask": {"size": 90, "keep_first": 6},
      "rot": {"base": 5e5, "dims": 48, "scaling": {"factor": 8.0, "original": 64, "fast": 8.0, "slow": 2.0}}}, LONG_PORTIONS),
    ({"heads": 18, "kv_heads": 1, "dim": 40, "vdim": 72, "scale": 0.15, "diff": 0.0, "mask": {"size": 64, "keep_first": 64}, "rot": {"base": 300.0, "dims": 2}}, LONG_PORTIONS),
    ({"heads": 3, "kv_heads": 3, "dim": 16, "vdim": 33, "scale": 0.2, "diff": 0.6, "mask": {"size": 1, "keep_first": 1}, "rot": {"base": 100.0, "dims": 16}}, PORTIONS),
    ({"heads": 2, "kv_heads": 1, "dim": 80, "vdim": 144, "scale": 0.1, "diff": 0.3, "mask": {"size": 30, "keep_first": 37}, "rot": {"base": 900.0, "dims": 80}}, PORTIONS),
])
def test_differential_attention_in_portions(name, dtype, tol, m, portions):
    """The mixer as a part: biased projections, scaled rotation of part of every map, the window with its kept tokens, the
    difference and its norm; portions that start inside a page, two tokens, single tokens; padded size 128 on the tcgen05
    kernel in bfloat16; pages that the window has passed are gone."""
    from jax_llm_examples_b200.parts import Runtime

    torch.manual_seed(m["heads"] + m["dim"])
    D, eps, T = 48, 1e-5, portions[-1][1]
    wd = _weights(m, D, dtype)
    hs = torch.randn(T, D).to(dtype)
    page = 64 if max(2 * m["dim"], m["vdim"]) in range(65, 129) else 16
    got = _in_portions(_mixer(wd, m, eps, dtype), Runtime(dtype, torch.device(DEV)), hs, dtype, portions, page)
    _close(got, plain.differential_attention(hs.double(), {"m." + k: v.double() for k, v in wd.items()}, "m.", m, eps), tol, name)


def _needle_mixer(size, window, keep, dtype):
    """One head over rows of `size`: map 1 scores entry 3 of query and key, map 2 scores nothing (all keys alike)."""
    from jax_llm_examples_b200.parts import DifferentialAttention

    eye, zero, values = torch.eye(size), torch.zeros(size, size), torch.eye(size)
    values[3, 3] = 0.0  # what the keys are found by is no part of the values
    return DifferentialAttention(torch.cat([eye, zero, eye, zero, values]).to(dtype).to(DEV), eye.to(dtype).to(DEV), 1, 1, size, size, 1.0, 1e-6, map_weight=0.5,
                                 diff=0.25, window=window, keep_first=keep, padded_dim=DifferentialAttention.padded_size(size, size, dtype))


def _marker(mixer, dtype, T, at, decoded, page, size):
    from jax_llm_examples_b200.parts import Runtime

    hs = torch.randn(T, size) * 0.3
    hs[:, 3] = hs[:, 8] = 0.0
    hs[T - 1] = 0.0
    hs[T - 1, 3] = 4.0
    hs[at] = 0.0
    hs[at, 3], hs[at, 8] = 4.0, 2.0
    cuts = {"prompt": [(0, T)], "alone": [(0, T - 1), (T - 1, T)], "two": [(0, T // 2), (T // 2, T - 2), (T - 2, T)]}[decoded]
    out = _in_portions(mixer, Runtime(dtype, torch.device(DEV)), hs.to(dtype), dtype, [c for c in cuts if c[1] > c[0]], page)
    return float(out[-1, 8])


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("size", [16, 64])
@pytest.mark.parametrize("window, keep", [(5, 3), (16, 16), (21, 1), (64, 17), (64, 64), (100, 33)])
def test_keys_at_the_windows_edge_and_at_the_last_kept_token(name, dtype, tol, size, window, keep):
    """ONE earlier token's first-map key points where the query points, and its value carries a marker: window - 1 tokens back
    it is seen, window tokens back it is not; the sequence's token keep - 1 is seen from any distance, its token keep is not.
    In a prompt, for a token decoded alone and in a portion of two; at and across page borders, at both kernel sizes."""
    torch.manual_seed(window + keep)
    mixer, page = _needle_mixer(size, window, keep, dtype), 64 if size == 64 else 16
    for T in (window + keep + 4, 199, 260):
        for at, seen in ((T - window, True), (T - 1 - window, False), (keep - 1, True), (keep, False), (0, True)):
            if at >= T - 1 or at < 0 or (not seen and (at < keep or at > T - 1 - window)):
                continue
            for how in ("prompt", "alone", "two"):
                marker = _marker(mixer, dtype, T, at, how, page, size)
                assert (marker > 1.0) == seen and (seen or abs(marker) < 0.03), \
                    f"{name} window {window} keep {keep}: query {T - 1} ({how}), key {at}: marker {marker:.3f}"


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("size, page", [(16, 16), (64, 64)])
def test_edges_far_out_with_split_keys(name, dtype, tol, size, page):
    """The same 1500 tokens out with a window of 700 that keeps 150: several splits of a decode step share the kept tokens."""
    torch.manual_seed(size)
    mixer, T = _needle_mixer(size, 700, 150, dtype), 1500
    for at, seen in ((149, True), (150, False), (0, True), (64, True), (T - 700, True), (T - 701, False), (1023, True)):
        for how in ("prompt", "alone"):
            marker = _marker(mixer, dtype, T, at, how, page, size)
            assert (marker > 1.0) == seen and (seen or abs(marker) < 0.03), f"{name}: key {at} ({how}): marker {marker:.3f}"


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("lam", [0.0, 0.5, 0.999, 1.7])
def test_the_second_maps_weight_made_to_show(name, dtype, tol, lam):
    """Map 1 of every query looks at tokens of kind A only, map 2 at tokens of kind B only, and the values name the kinds: the
    head is (1, -lambda) before its norm, in closed form; with both maps on one token it is (1 - lambda) of that token's value."""
    from jax_llm_examples_b200.parts import DifferentialAttention, Runtime

    size, T, diff, eps = 32, 90, 0.3, 1e-7
    wq, wk = torch.zeros(2 * size, size), torch.zeros(2 * size, size)
    wq[0, 0] = wq[size, 0] = 6.0  # every query asks entry 0 of map 1 and of map 2
    wk[0, 1] = wk[size, 2] = 6.0  # kind A answers in map 1, kind B in map 2
    hs = torch.zeros(T, size)
    hs[:, 0] = 1.0
    hs[0::2, 1] = 1.0
    hs[1::2, 2] = 1.0
    hs[0] = torch.tensor([1.0, 1.0, 1.0] + [0.0] * (size - 3))  # the first token is both
    mixer = DifferentialAttention(torch.cat([wq, wk, torch.eye(size)]).to(dtype).to(DEV), torch.eye(size).to(dtype).to(DEV), 1, 1, size, size, 1.0, eps, map_weight=lam,
                                  diff=diff, window=8, padded_dim=DifferentialAttention.padded_size(size, size, dtype))
    for portions in (((0, T),), ((0, 64), (64, 70)) + tuple((p, p + 1) for p in range(70, T))):
        got = _in_portions(mixer, Runtime(dtype, torch.device(DEV)), hs.to(dtype), dtype, portions, 16).double().cpu()
        first = torch.zeros(size, dtype=F64)
        first[:3] = 1.0 - lam
        _close(got[0], plain.rms_divide(first, eps) * (1 - diff), 0.05 if lam == 0.999 and dtype == torch.bfloat16 else 1e-2, f"{name}: one token")
        for p in (20, 63, 64, 71, 89):
            o = torch.zeros(size, dtype=F64)
            o[0], o[1], o[2] = 1.0 - lam, 1.0, -lam
            _close(got[p], plain.rms_divide(o, eps) * (1 - diff), 1e-2, f"{name}: position {p}")


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("mask", [None, {"size": 33, "keep_first": 2}, {"size": 300, "keep_first": 100}, {"size": 1000, "keep_first": 5}])
@pytest.mark.parametrize("d, dv", [(12, 20), (64, 128)])
def test_decoding_of_unequal_requests_beside_portions(name, dtype, tol, mask, d, dv):
    """Requests decode one token each over contexts from one token to 1300, then some of them bring portions: the maps are put
    together from split ranges, single tokens go beside the portions by their row list."""
    from jax_llm_examples_b200.parts import LayerCache, Runtime

    torch.manual_seed(7)
    D, eps, page = 48, 1e-5, 64
    m = {"heads": 4, "kv_heads": 2, "dim": d, "vdim": dv, "scale": d ** -0.5, "diff": 0.4, "rot": {"base": 1e4, "dims": 8}}
    if mask:
        m["mask"] = mask
    wd = _weights(m, D, dtype)
    mixer, rt = _mixer(wd, m, eps, dtype), Runtime(dtype, torch.device(DEV))
    lens = [1300, 1, 33, 64, 257, 600]
    P = {"m." + k: v.double() for k, v in wd.items()}
    seqs = [torch.randn(n + 80, D).to(dtype) for n in lens]
    refs = [plain.differential_attention(s.double(), P, "m.", m, eps) for s in seqs]
    need, width = mixer.kv_need(), 1400 // page + 1
    table = torch.randperm(len(lens) * width).to(torch.int32).view(len(lens), width).to(DEV)
    pages = torch.zeros(len(lens) * width, 2, need.num_kv_heads, page, need.head_dim, device=DEV, dtype=dtype)

    def step(live, q_lens, starts):
        ctx = _ctx(rt, q_lens, starts, planners=mixer.step_planners(), page_size=page)
        rows = torch.cat([seqs[r][s:s + n] for r, n, s in zip(live, q_lens, starts)]).to(DEV)
        out = H.as_rows_sum(mixer.forward(ctx, rows, LayerCache(pages, table[live].contiguous(), True, None)))
        assert int(ctx.status) == 0
        return out

    for r, n in enumerate(lens):
        _close(step([r], [n], [0]), refs[r][:n], tol, f"{name}: prompt of {n}")
    every = list(range(len(lens)))
    got = step(every, [1] * len(lens), lens)
    for r, n in enumerate(lens):
        _close(got[r:r + 1], refs[r][n:n + 1], 2 * tol, f"{name}: token after {n}")
    q, at = [1, 11, 1, 66, 2, 1], 0
    got = step(every, q, [n + 1 for n in lens])
    for r, n in enumerate(lens):
        _close(got[at:at + q[r]], refs[r][n + 1:n + 1 + q[r]], 2 * tol, f"{name}: mixed step, request {r}")
        at += q[r]


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
def test_a_window_that_keeps_the_first_tokens_and_biases_in_plain_grouped_attention(name, dtype, tol):
    """The same two mechanisms in the general attention part, where another design can use them."""
    from jax_llm_examples_b200.parts import GatedPagedAttention, Runtime

    torch.manual_seed(3)
    D, T, Hh, G, d, dv, window, keep = 40, 154, 4, 2, 64, 64, 30, 9
    g = lambda *s: (torch.randn(*s) * 0.3).to(dtype)  # noqa: E731
    w, b, o = g(Hh * d + G * d + G * dv, D), g(Hh * d + G * d + G * dv), g(D, Hh * dv)
    mixer = GatedPagedAttention(w.to(DEV), o.to(DEV), Hh, G, d, dv, 0.15, 1e-5, gate="none", window=window, keep_first=keep, in_bias=b.to(DEV),
                                padded_dim=GatedPagedAttention.padded_size(d, dv, dtype))
    hs = torch.randn(T, D).to(dtype)
    got = _in_portions(mixer, Runtime(dtype, torch.device(DEV)), hs, dtype, LONG_PORTIONS, 16)
    rows = hs.double() @ w.double().T + b.double()
    q, k, v = rows[:, :Hh * d].view(T, Hh, d), rows[:, Hh * d:(Hh + G) * d].view(T, G, d), rows[:, (Hh + G) * d:].view(T, G, dv)
    mask = plain.window_with_kept_start(T, window, keep)
    heads = [plain.masked_softmax(q[:, a] @ k[:, a // 2].T * 0.15, mask) @ v[:, a // 2] for a in range(Hh)]
    _close(got, torch.cat(heads, -1) @ o.double().T, tol, name)


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("E, k, ff, D, n", [(5, 2, 14, 36, 9), (8, 3, 48, 128, 1), (8, 2, 64, 128, 16), (12, 5, 80, 1024, 20), (16, 1, 32, 64, 300), (3, 3, 16, 64, 5),
                                            (40, 20, 16, 64, 6), (16, 2, 64, 256, 1100)])
def test_experts_by_table(name, dtype, tol, E, k, ff, D, n):
    """The feed-forward as a part, from one row to a portion: behind a norm that writes the rows where the experts read them
    (sorted ahead on the second stream), and behind one that does not; more choices than the norm has places for."""
    from jax_llm_examples_b200.parts import RMSNorm, RowPlaces, RowSum, Runtime, TableRoutedGLUExperts, as_rows

    torch.manual_seed(E + n)
    V, eps = 30, 1e-5
    g = lambda *s: (torch.randn(*s) * 0.2).to(dtype)  # noqa: E731
    gate, up, down = g(E, ff, D), g(E, ff, D), g(E, D, ff)
    table = torch.rand(V, E).argsort(1)[:, :k].to(torch.int32).contiguous()
    part = TableRoutedGLUExperts(table.to(DEV), torch.cat([gate, up], dim=1).to(DEV), down.to(DEV))
    norm = RMSNorm((1 + 0.1 * torch.randn(D)).to(DEV), eps)
    x, toks = torch.randn(n, D), torch.randint(0, V, (n,))
    P = {"table": table}
    for e in range(E):
        P.update({f"e{e}.gate": gate[e].double(), f"e{e}.up": up[e].double(), f"e{e}.down": down[e].double()})
    h = plain.rms_norm(x.double(), norm.weight.double().cpu(), eps)
    ref = plain.table_experts(h, toks, P, "", {"router": {"experts": E, "top": k}})
    for placed in (True, False):
        ctx = _ctx(Runtime(dtype, torch.device(DEV)), [n], [0])
        ctx.token_ids = toks.to(torch.int32).to(DEV)
        part.begin_step(ctx)
        places = part.row_places(ctx, n) if placed else None
        assert (places is None) == (not placed or k > part.MAX_COPIES)
        rows, h32, _ = norm.forward(ctx, x.to(DEV), None, out_dtype=dtype, want_f32=places is None, places=places)
        assert rows.shape[0] == n * (k if isinstance(places, RowPlaces) else 1)
        y = part.forward(ctx, rows, h32, places)
        assert isinstance(y, RowSum) and y.terms[0].scale == 1.0 / k
        r = as_rows(y)
        _close(r.data, ref, tol, f"{name} placed={placed}")
        # the next norm adds the rows from where they lie
        z = torch.zeros(n, D, device=DEV)
        norm.forward(ctx, z, y, out_dtype=dtype)
        _close(z, ref, tol, f"{name}: gathered by the next norm")
        assert int(ctx.status) == 0


# --------------------------------------------------------------------------------------- whole models, by traces
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("samerax")
    return {n: SX.make_dir(root / n, n, seed=i + 1) for i, n in enumerate(SX.CONFIGS)}


def _engine(folder, dtype, max_tokens=512, page_size=16, max_slots=4, **kw):
    import jax_llm_examples_b200 as J

    return J.Engine(J.load_model(folder, dtype, DEV), max_tokens=max_tokens, page_size=page_size, max_slots=max_slots, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SX.CONFIGS))
def test_every_kind_of_cut_against_the_plain_implementation(folders, name, dtype):
    """Whole prompts; most of a prompt and then 40 tokens one by one; portions down to two tokens; up to four live
    requests mixed, in a pool too small for all of them, so that pages and slots are used again.  Every position's
    logits are compared, the first tokens of a sequence included."""
    vocab = SX.config(name)["vocab"]
    rng = random.Random(7)
    requests = H.random_requests(rng, vocab, [61, 1, 2, 33, 17, 90, 5])
    engine = _engine(folders[name], dtype, max_tokens=16 * 16)
    for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=40), H.trace_portions(requests, rng),
                  H.trace_mixed(requests, rng, max_live=4)):
        got, _ = H.run_trace(engine, steps, record_routing=False)
        assert len(got) == sum(len(t) for t in requests.values())
        SX.compare(folders[name], requests, got, dtype, stray=2 if dtype == "bfloat16" else 0)
        assert engine.manager.free_slots() == 4 and all(engine.manager.free_pages(g) == engine.num_pages for g in range(len(engine.manager.groups)))
        engine.manager.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_padded_size_128_on_pages_of_64_tokens(folders, dtype):
    """Pages of 64 tokens, as a server has them: in bfloat16 the portions of 64 tokens and more of the layers with a padded
    size of 128 run on the tcgen05 kernel (kept tokens, two maps), shorter ones on the mma.sync kernel, single tokens on the
    split-KV kernel, all in one step."""
    name = "wide"
    rng = random.Random(13)
    requests = H.random_requests(rng, SX.config(name)["vocab"], [200, 70, 131, 3])
    engine = _engine(folders[name], dtype, max_tokens=12 * 64, page_size=64)
    for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=20), H.trace_portions(requests, rng),
                  H.trace_mixed(requests, rng, max_live=4, portions=H.LONG_PORTIONS)):
        got, _ = H.run_trace(engine, steps, record_routing=False)
        SX.compare(folders[name], requests, got, dtype, stray=2 if dtype == "bfloat16" else 0)
    if dtype == "bfloat16":
        assert any("tc" in kinds for kinds in engine.attention_kernels_seen), "the tcgen05 kernel did not run"


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random_under_every_kind_of_cut(seed, tmp_path):
    """Sizes, head counts, orders of layers, repeats, windows, kept tokens, rotations and tables that nobody chose, in both
    precisions: whole prompts, a decoded tail, portions and mixed batches against the plain implementation."""
    rng = random.Random(seed)
    cfg = SX.random_config(rng)
    folder = SX.write_model(tmp_path / "m", cfg, seed)
    requests = H.random_requests(rng, cfg["vocab"], [70, 3, 130, 21, 45])
    for dtype in ("float32", "bfloat16"):
        engine = _engine(folder, dtype, max_tokens=20 * 16)
        for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=40), H.trace_portions(requests, rng),
                      H.trace_mixed(requests, rng, max_live=4)):
            got, _ = H.run_trace(engine, steps, record_routing=False)
            SX.compare(folder, requests, got, dtype, stray=4 if dtype == "bfloat16" else 0)


@pytest.mark.parametrize("seed", [0, 1, 2, 3])
def test_mid_size_configurations_on_pages_of_64_tokens(seed, tmp_path):
    """Widths of 192 to 512, maps up to 64, dozens of experts, windows of up to 300 tokens that keep up to 200, prompts of up
    to 700 tokens on pages of 64: whole prompts, a decoded tail, portions and mixed batches against the plain
    implementation.  The float32 cap is 1e-4 here: rows are sums of up to 512 terms through up to six layers."""
    rng = random.Random(1000 + seed)
    cfg = SX.mid_size_config(rng)
    folder = SX.write_model(tmp_path / "m", cfg, seed, std=0.9 / cfg["width"] ** 0.5)
    requests = H.random_requests(rng, cfg["vocab"], [700, 330, 97, 23, 1, 260])
    saved = dict(SX.TOL), dict(SX.TOL_MEAN)
    SX.TOL["float32"], SX.TOL_MEAN["float32"] = 1e-4, 2e-5
    try:
        for dtype in ("float32", "bfloat16"):
            engine = _engine(folder, dtype, max_tokens=1536, page_size=64, max_seq_len=1536)
            for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=40), H.trace_portions(requests, rng),
                          H.trace_mixed(requests, rng, max_live=4, portions=H.LONG_PORTIONS)):
                got, _ = H.run_trace(engine, steps, record_routing=False)
                SX.compare(folder, requests, got, dtype, stray=6 if dtype == "bfloat16" else 0)
    finally:
        SX.TOL.update(saved[0]), SX.TOL_MEAN.update(saved[1])


@pytest.mark.parametrize("name", list(SX.CONFIGS))
def test_logits_do_not_depend_on_the_cut_or_on_the_batch(folders, name):
    """float32: the same request whole, token by token, in portions, and beside three other requests gives the same
    logits to within rounding of a sum's order (far below the tolerance against the plain implementation)."""
    rng = random.Random(11)
    requests = H.random_requests(rng, SX.config(name)["vocab"], [70, 23, 41, 9])
    engine = _engine(folders[name], "float32")
    whole, _ = H.run_trace(engine, H.trace_whole(requests), record_routing=False)
    for steps in (H.trace_tail_decode(requests, tail=70), H.trace_portions(requests, rng), H.trace_mixed(requests, rng)):
        got, _ = H.run_trace(engine, steps, record_routing=False)
        worst = max(SX.row_err(got[k], whole[k]) for k in whole)
        assert worst < 5e-6, f"{name}: logits moved by {worst:.2e} with the cut"


@pytest.mark.parametrize("name", list(SX.CONFIGS))
def test_decoding_through_replayed_graphs_equals_decoding_without(folders, name):
    """bfloat16: decode-only steps are captured in CUDA graphs and replayed, the sort of the tables' experts on a branch of
    its own; the replayed steps must give what the same steps give launched one kernel at a time."""
    rng = random.Random(5)
    requests = H.random_requests(rng, SX.config(name)["vocab"], [50, 37])
    outs = []
    for graphs in (True, False):
        engine = _engine(folders[name], "bfloat16", use_graphs=graphs)
        got, _ = H.run_trace(engine, H.trace_tail_decode(requests, tail=30), record_routing=False)
        assert (engine.graph_replays > 0) == graphs
        outs.append(got)
    worst = max(SX.row_err(outs[0][k], outs[1][k]) for k in outs[0])
    assert worst < 2e-2, f"{name}: replayed steps differ by {worst:.2e}"


def test_the_experts_of_every_token_are_the_tables(folders):
    """The engine records the experts that ran: for every token those of its row of the table, in every run of the layer."""
    cfg, P = SX.plain_model(str(folders["small"]))
    rng = random.Random(2)
    requests = H.random_requests(rng, cfg["vocab"], [20, 9])
    engine = _engine(folders["small"], "float32")
    _, routing = H.run_trace(engine, H.trace_portions(requests, rng), record_routing=True)
    owners = [plain.owner(cfg, i) for i, L in enumerate(cfg["layers"]) if (L["mlp"] or {}).get("kind") == "moe"]
    for (rid, pos), rows in routing.items():
        for o, chosen in zip(owners, rows):
            assert list(chosen) == P[f"l{o}.mlp.table"][requests[rid][pos]].tolist()


def test_long_decoding_and_slots_used_again(folders):
    """300 tokens one by one after a short prompt, in both precisions: the window's old pages are given back on the way, the
    first ones stay; then the same slot and pages serve another request, which must not see what the first left."""
    name = "small"
    vocab = SX.config(name)["vocab"]
    rnd = random.Random(3)
    toks = [rnd.randrange(vocab) for _ in range(320)]
    other = [rnd.randrange(vocab) for _ in range(25)]
    for dtype in ("float32", "bfloat16"):
        engine = _engine(folders[name], dtype, max_tokens=320, max_slots=1)
        for req in ({"a": toks}, {"b": other}):
            got, _ = H.run_trace(engine, H.trace_tail_decode(req, tail=300), record_routing=False)
            SX.compare(folders[name], req, got, dtype, stray=3 if dtype == "bfloat16" else 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_decoding_batch_of_every_size(folders, dtype):
    """One to twenty requests decode together (the sizes at which the kernels of a decode step change), each with a context of
    its own length: every request's logits are the plain implementation's."""
    name = "wide"
    rng = random.Random(17)
    for n in (1, 3, 8, 9, 16, 17, 20):
        requests = H.random_requests(rng, SX.config(name)["vocab"], [8 + 5 * (i % 7) + i for i in range(n)])
        engine = _engine(folders[name], dtype, max_tokens=20 * 64, max_slots=20)
        heads = {"entries": [{"id": r, "tokens": t[:-3], "want": []} for r, t in requests.items()], "end": []}
        tails = [{"entries": [{"id": r, "tokens": [t[len(t) - 3 + i]], "want": [0]} for r, t in requests.items()],
                  "end": list(requests) if i == 2 else []} for i in range(3)]
        got, _ = H.run_trace(engine, [heads] + tails, record_routing=False)
        assert len(got) == 3 * n
        SX.compare(folders[name], requests, got, dtype, stray=1 if dtype == "bfloat16" else 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(SX.CONFIGS))
def test_greedy_generation_through_the_scheduler(folders, name, dtype):
    """The framework's own entry point: prompts of unequal length under a small token budget per step, so that
    prompt portions run beside decoded tokens."""
    import jax_llm_examples_b200 as J

    vocab = SX.config(name)["vocab"]
    prompts = [[(7 * i + 3 * j) % vocab for i in range(n)] for j, n in enumerate((29, 3, 12))]
    model = J.load_model(folders[name], dtype, DEV)
    got = J.generate(model, prompts, J.SamplingParams(max_new_tokens=10), page_size=16, max_tokens_per_step=16)
    for p, g in zip(prompts, got):
        assert len(g) == 10
        SX.greedy_checked(folders[name], p, g, dtype)


def test_command_line_generates_from_a_preset_and_from_a_folder(folders, capsys):
    from jax_llm_examples_b200.main import main

    assert main(["--preset", "samerax_tiny", "--random-prompts", "2", "--prompt-len", "9", "--max-new-tokens", "4"]) == 0
    assert capsys.readouterr().out.count("-" * 80) == 2
    assert main(["--model", str(folders["padded"]), "--dtype", "float32", "--prompt-ids", "1,2,3,4,5", "--max-new-tokens", "5",
                 "--page-size", "16"]) == 0
    ids = [int(t) for t in capsys.readouterr().out.splitlines()[1].split()]
    SX.greedy_checked(folders["padded"], [1, 2, 3, 4, 5], ids, "float32")


def test_models_from_tensors_keep_their_tables(folders):
    """A model made from tensors in memory is the model of the folder (a table of integers stays one)."""
    import jax_llm_examples_b200 as J

    cfg, P = SX.plain_model(str(folders["small"]))
    toks = [3, 50, 7, 7, 12, 60, 1]
    model = J.model_from_tensors(cfg, {n: t.float() if t.is_floating_point() else t for n, t in P.items()}, "float32", DEV)
    engine = J.Engine(model, max_tokens=64, page_size=16, max_slots=1)
    got, _ = H.run_trace(engine, H.trace_whole({"a": toks}), record_routing=False)
    SX.compare(folders["small"], {"a": toks}, got, "float32")


def test_trace_replay_program_on_a_samerax_folder(folders, tmp_path):
    """bin/trace_run picks the model class by config.json and writes the wanted logits."""
    name, dtype = "padded", "float32"
    vocab = SX.config(name)["vocab"]
    toks = [(5 * i + 2) % vocab for i in range(21)]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:13], "want": [0, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[13:20], "want": []}, {"id": "b", "tokens": toks[:2], "want": [1]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[20:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    p = subprocess.run([sys.executable, os.path.join(H.ROOT, "bin", "trace_run"), "--model", str(folders[name]), "--dtype", dtype,
                        "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = SX.plain_logits(folders[name], toks)
    rows = {0: [0, 12], 1: [1], 2: [20]}
    for step, places in rows.items():
        got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(places), vocab)
        for g, pl in zip(got, places):
            assert SX.row_err(g, ref[pl]) < SX.TOL[dtype]
