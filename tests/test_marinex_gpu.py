"""Marinex on the GPU against the plain implementation: each mechanism alone (kernel or part against the plain function of
the same name), inputs made so that a fault shows (a far token, a window's edge, the sink's share, the cap, a group's score),
then whole models through the engine's step function under every kind of cut, batches against requests alone, pages and
slots that are used again, long decoding, and greedy generation through the scheduler.
All configurations are this file's own (``tests/marinex_helpers.py``)."""

import json
import math
import os
import random
import subprocess
import sys

import numpy as np
import pytest
import torch

from tests import helpers as H
from tests import marinex_helpers as MX
from tests.plain import marinex_plain as plain
from tests.test_koduzen_gpu import LONG_PORTIONS, PORTIONS, _attention_in_portions
from tests.test_tebivik_gpu import _close, _ctx

pytestmark = pytest.mark.gpu
DEV = "cuda"
DTYPES = [("float32", torch.float32, 2e-5), ("bfloat16", torch.bfloat16, 3e-2)]
F64 = torch.float64


# ------------------------------------------------------------------------------------- kernels alone
@pytest.mark.parametrize("many", [False, True])
@pytest.mark.parametrize("E, k, groups, keep, D, n", [(6, 2, 3, 2, 36, 9), (18, 5, 3, 2, 192, 70), (40, 6, 8, 3, 128, 33), (5, 5, 1, 1, 30, 4),
                                                      (64, 8, 64, 20, 64, 17), (256, 3, 4, 4, 512, 20)])
def test_sigmoid_router_with_corrections_and_groups(E, k, groups, keep, D, n, many):
    """Both router kernels: sigmoid scores, the choice on score + correction (mostly negative: others of dropped groups are
    not zeros that win), groups by the sum of their two largest, weights not renormalised."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(E + k)
    h, w, corr = torch.randn(n, D, device=DEV), torch.randn(E, D, device=DEV) * D ** -0.5, torch.randn(E, device=DEV) - 1.0
    idx, wt = torch.empty(n, k, dtype=torch.int32, device=DEV), torch.empty(n, k, device=DEV)
    K.router(h, w, idx, wt, many_rows=many, weight_form="sigmoid_corrected", correction=corr, groups=groups, keep=keep, group_top=2)
    r = {"experts": E, "top": k, "groups": {"count": groups, "keep": keep}}
    own, s = plain.route(h.double().cpu(), {"router": w.double().cpu(), "correction": corr.double().cpu()}, "", r)
    got = idx.cpu().long()
    assert torch.equal(torch.sort(got, 1).values, torch.sort(own, 1).values)
    _close(wt, torch.gather(s, 1, got), 1e-5, "weights")
    choice = torch.gather(s + corr.double().cpu(), 1, got)
    assert bool((choice[:, :-1] >= choice[:, 1:] - 1e-6).all()), "the largest choice score comes first"
    # the same with the weights divided by their sum and scaled
    K.router(h, w, idx, wt, many_rows=many, weight_form="sigmoid_corrected", correction=corr, groups=groups, keep=keep, group_top=2,
             normalize=True, scale=2.5)
    g = torch.gather(s, 1, idx.cpu().long())
    _close(wt, 2.5 * g / g.sum(1, keepdim=True), 1e-5, "normalised weights")


def test_a_groups_score_is_the_sum_of_its_two_largest():
    """One large and one tiny score in a group against two middling ones, and a group of one expert; ties go to the lower
    group and the lower expert."""
    from jax_llm_examples_b200.kernels import api as K

    h, idx, wt = torch.zeros(1, 8, device=DEV), torch.empty(1, 2, dtype=torch.int32, device=DEV), torch.empty(1, 2, device=DEV)
    for many in (False, True):
        for corr, groups, keep, top2, top1 in (([2.0, -5.0, -5.0, 0.5, 0.4, 0.0], 2, 1, [3, 4], [0, 1]),
                                               ([0.0, 3.0, 1.0, 2.0, 1.5, 1.5], 3, 2, [1, 3], [1, 3]),
                                               ([-9.0, -2.0, -1.0, -8.0, -1.25, -1.25], 3, 1, [4, 5], [2, 3]),
                                               ([1.0, 1.0, 1.0, 1.0, 1.0, 1.0], 3, 1, [0, 1], [0, 1]),
                                               ([5.0, 1.0, 4.0, 2.0, 3.0, 0.0], 6, 2, [0, 2], [0, 2])):
            c = torch.tensor(corr, device=DEV)
            for group_top, want in ((2, top2), (1, top1)):
                K.router(h, torch.zeros(6, 8, device=DEV), idx, wt, many_rows=many, weight_form="sigmoid_corrected", correction=c,
                         groups=groups, keep=keep, group_top=group_top)
                assert idx[0].tolist() == want, (corr, group_top, idx[0].tolist())
                assert torch.allclose(wt, torch.full_like(wt, 0.5))  # sigmoid(0), whatever the corrections


@pytest.mark.parametrize("D, k, splits, weighted", [(36, 2, 1, True), (200, 4, 3, True), (1024, 1, 2, True), (30, 3, 2, False), (2048, 8, 1, True)])
def test_the_closing_norm_gathers_an_expert_layers_rows(D, k, splits, weighted):
    """x += w * rms_norm(sum_j weight_j * (sum of the partials of row index_j)); out = x rounded: one kernel; then the final
    norm over chosen rows, which leaves x alone."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(D)
    N, eps = 7, 1e-5
    x, y = torch.randn(N, D, device=DEV), torch.randn(splits, N * k, D, device=DEV)
    pos = torch.randperm(N * k).to(torch.int32).to(DEV)
    wt, gamma, w = torch.rand(N, k, device=DEV), torch.randn(D, device=DEV), torch.randn(D, device=DEV)
    rows = y.sum(0).double()[pos.long()].view(N, k, D).cpu()
    delta = (rows * (wt.double().cpu()[:, :, None] if weighted else 1.0)).sum(1)
    x_ref = x.double().cpu() + plain.rms_norm(delta, gamma.double().cpu(), eps)
    x2, out = x.clone(), torch.empty(N, D, device=DEV, dtype=torch.bfloat16)
    K.group_norm(x2, y, splits, None, gamma, 1, 1.0, pre_norm=False, eps=eps, out=out, delta_index=pos, delta_k=k, delta_weights=wt if weighted else None)
    _close(x2, x_ref, 3e-6, "residual")
    assert torch.equal(out, x2.to(torch.bfloat16))
    at = torch.tensor([5, 0, 6], device=DEV, dtype=torch.int32)
    x3, o3 = x.clone(), torch.empty(3, D, device=DEV)
    K.group_norm(x3, y, splits, None, gamma, 1, 1.0, w, 1, True, eps, None, o3, at, delta_index=pos, delta_k=k, delta_weights=wt if weighted else None)
    assert torch.equal(x3, x)
    _close(o3, plain.rms_norm(x_ref[[5, 0, 6]], w.double().cpu(), eps), 3e-6, "final norm")


@pytest.mark.parametrize("window", [0, 1, 5, 40, 200])
@pytest.mark.parametrize("H_, T, q_start, k_start, L", [(3, 9, 0, 0, 9), (2, 33, 50, 16, 72), (1, 2, 300, 296, 8), (2, 5, 70, 3, 77)])
def test_softmax_of_a_portion_with_a_window(window, H_, T, q_start, k_start, L):
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(T)
    s, sink = torch.randn(H_, T, L, device=DEV) * 5, torch.randn(H_, device=DEV)
    p = torch.empty(H_, T, L, device=DEV)
    K.causal_sink_softmax(s, sink, 0.7, q_start, p, k_start, window)
    i, j = torch.arange(T)[:, None] + q_start, torch.arange(L)[None, :] + k_start
    mask = (j <= i) & (i - j < (window or 1 << 30))
    for a in range(H_):
        _close(p[a], plain.softmax_with_sink(s[a].double().cpu() * 0.7, mask, float(sink[a])), 3e-6)


@pytest.mark.parametrize("P, E, extra, tile_rows, tile_groups", [(1024, 16, 0, 128, 0), (4096, 256, 0, 32, 0), (5003, 7, 0, 0, 0), (2048, 3, 100, 64, 0),
                                                                 (1500, 1, 0, 16, 0), (3000, 40, 0, 96, 33), (8192, 128, 0, 160, 0)])
def test_sort_of_many_pairs(P, E, extra, tile_rows, tile_groups):
    """The sort by expert of a prompt portion's pairs: offsets, stable order, places, and the products' row tiles."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(P)
    idx = torch.randint(0, E, (P,), dtype=torch.int32)
    idx[torch.rand(P) < 0.3] = E // 2  # one crowded expert
    groups = E + (extra > 0)
    i32 = lambda n: torch.full((n,), -7, dtype=torch.int32, device=DEV)  # noqa: E731
    off, pair, pos, st = i32(E + 2), i32(P), i32(P), torch.zeros(1, dtype=torch.int32, device=DEV)
    tiles = (i32(2 * (-(-(P + extra) // tile_rows) + groups)), i32(1)) if tile_rows else ()
    K.expert_sort(idx.to(DEV), off, pair, pos, E, st, extra, tile_rows, *tiles, **({"tile_groups": tile_groups} if tile_groups else {}))
    order = torch.sort(idx.long(), stable=True).indices
    assert torch.equal(pair.cpu().long(), order) and torch.equal(pos.cpu().long()[order], torch.arange(P))
    want = [0] + torch.cumsum(torch.bincount(idx.long(), minlength=E), 0).tolist() + ([P + extra] if extra else [])
    assert off.cpu()[:len(want)].tolist() == want and int(st) == 0
    if tile_rows:
        listed = [(g, r) for g in range(tile_groups or groups) for r in range(want[g], want[g + 1], tile_rows)]
        n = int(tiles[1])
        assert n == len(listed) and tiles[0].cpu()[:2 * n].view(n, 2).tolist() == [list(t) for t in listed]


@pytest.mark.parametrize("E, N, Kd, rows", [(16, 256, 128, 40), (4, 96, 64, 3), (3, 200, 72, 700)])
def test_activation_in_the_grouped_products_epilogue(E, N, Kd, rows):
    """gelu(a W^T) finished inside the streaming product, against float64: bfloat16 and float32 results, values far out."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(rows)
    a, w = (torch.randn(rows, Kd, device=DEV) * 1.5).bfloat16(), (torch.randn(E, N, Kd, device=DEV) * 0.3).bfloat16()
    cuts = sorted(random.Random(rows).choices(range(rows + 1), k=E - 1))
    off = torch.tensor([0] + cuts + [rows], dtype=torch.int32, device=DEV)
    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    at = off.tolist()
    ref = torch.cat([a[at[e]:at[e + 1]].double() @ w[e].double().T for e in range(E)])
    for act, fn in (("gelu", plain.gelu_exact), ("relu2", lambda z: torch.relu(z) ** 2), ("silu", lambda z: z * torch.sigmoid(z)), ("none", lambda z: z)):
        for dt, tol in ((torch.float32, 4e-6), (torch.bfloat16, 4e-3)):
            out = torch.empty(rows, N, device=DEV, dtype=dt)
            K.gemm_stream(a, w, out, st, offsets=off, rows_hint=max(rows // E, 1), mode=K.GEMM_ACT, activation=act)
            err = (out.double() - fn(ref)).abs() / (1.0 + fn(ref).abs())
            assert float(err.max()) < tol, (act, dt, float(err.max()))
    assert int(st) == 0


@pytest.mark.parametrize("E, N, Kd, u", [(16, 512, 128, 8), (3, 40, 64, 1), (5, 128, 72, 17), (2, 256, 512, 300)])
def test_equal_groups_need_no_offsets(E, N, Kd, u):
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(u)
    a, w = torch.randn(E * u, Kd, device=DEV).bfloat16(), torch.randn(E, N, Kd, device=DEV).bfloat16()
    out, st = torch.full((E * u, N), float("nan"), device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    K.gemm_stream(a, w, out, st, uniform_rows=u)
    _close(out.view(E, u, N), torch.einsum("eud,end->eun", a.double().view(E, u, Kd), w.double()), 2e-6)
    assert int(st) == 0


@pytest.mark.parametrize("N", [1, 2, 7, 8, 9, 16])
@pytest.mark.parametrize("D, E, k, groups, keep, splits, gathered", [(64, 6, 2, 3, 2, 1, False), (2048, 16, 2, 2, 1, 4, False), (512, 40, 5, 8, 3, 2, True),
                                                                     (4096, 256, 8, 1, 1, 1, False), (132, 5, 1, 1, 1, 3, True), (256, 64, 16, 64, 40, 1, False)])
def test_closing_norm_router_sort_and_gather_in_one_launch(N, D, E, k, groups, keep, splits, gathered):
    """What the one kernel of a decode step leaves is what the four kernels leave: residual rows, rounded rows, choices and
    weights, sorted pairs, tile list, gathered rows; both corrected weight forms."""
    from jax_llm_examples_b200.kernels import api as K
    from jax_llm_examples_b200.parts.base import CorrectedRouter, Dispatch

    assert K.close_route_supported(N, D, E, k)
    torch.manual_seed(N * D)
    kk = 3
    x = torch.randn(N, D, device=DEV)
    y = torch.randn(splits, N * kk if gathered else N, D, device=DEV)
    extra = dict(delta_index=torch.randperm(N * kk).to(torch.int32).to(DEV), delta_k=kk, delta_weights=torch.rand(N, kk, device=DEV)) if gathered else {}
    gamma, w, corr = torch.randn(D, device=DEV), torch.randn(E, D, device=DEV) * D ** -0.5, torch.randn(E, device=DEV) - 0.5
    i32 = lambda *s: torch.full(s, -7, dtype=torch.int32, device=DEV)  # noqa: E731
    st, tile = torch.zeros(1, dtype=torch.int32, device=DEV), 16
    for form, norm in (("sigmoid_corrected", False), ("softmax_normalized", True)):
        r = CorrectedRouter(w, None, corr, form, groups, keep, 2, norm, 1.5, k, None)
        d = Dispatch(None, i32(E + 1), i32(N * k), i32(N * k), (i32(2 * (-(-N * k // tile) + E)), i32(1)),
                     torch.zeros(N * k, D, device=DEV, dtype=torch.bfloat16), 0, tile, st)
        x1, h1, idx1, w1 = x.clone(), torch.empty(N, D, device=DEV, dtype=torch.bfloat16), i32(N, k), torch.empty(N, k, device=DEV)
        K.close_route(x1, y, splits, gamma, 0.7, 1e-5, h1, r, idx1, w1, d, **extra)
        x2, h2, idx2, w2 = x.clone(), torch.empty_like(h1), i32(N, k), torch.empty(N, k, device=DEV)
        K.group_norm(x2, y, splits, None, gamma, 1, 0.7, pre_norm=False, eps=1e-5, out=h2, **extra)
        K.router(x1, w, idx2, w2, weight_form=form, correction=corr, groups=groups, keep=keep, scale=1.5, group_top=2, normalize=norm)
        off, pair, pos, tl, nt = i32(E + 1), i32(N * k), i32(N * k), i32(2 * (-(-N * k // tile) + E)), i32(1)
        K.expert_sort(idx1, off, pair, pos, E, st, 0, tile, tl, nt)
        _close(x1, x2, 2e-6, "residual")
        assert torch.equal(h1, x1.bfloat16())
        assert torch.equal(idx1, idx2)
        _close(w1, w2, 2e-6, "weights")
        assert torch.equal(d.offsets, off) and torch.equal(d.sorted_pair, pair) and torch.equal(d.sorted_pos, pos)
        assert torch.equal(d.tiles[1], nt) and torch.equal(d.tiles[0][:2 * int(nt)], tl[:2 * int(nt)])
        assert torch.equal(d.a_sorted, h1[(pair.long() // k)])
        assert int(st) == 0


@pytest.mark.parametrize("rank, dr, heads, window", [(64, 16, 4, 0), (512, 64, 16, 100), (200, 24, 18, 33), (528, 8, 3, 0), (1024, 64, 2, 7), (16, 8, 1, 1)])
def test_latent_attention_on_the_tensor_cores_equals_the_32_bit_kernel(rank, dr, heads, window):
    """The same bfloat16 queries and cache through both kernels: contexts of one token to hundreds, whole and cut into
    ranges, all rows and listed ones (which come in the list's order)."""
    from jax_llm_examples_b200.kernels import api as K

    torch.manual_seed(rank)
    page, lens = 16, [1, 17, 32, 33, 100, 299, 300, 64]
    R = len(lens)
    width = 300 // page + 1
    pages = torch.randn(R * width, 1, 1, page, rank + dr, device=DEV).bfloat16()
    table = torch.randperm(R * width).to(torch.int32).view(R, width).to(DEV)
    if window:
        for r, n in enumerate(lens):
            table[r, :max(0, n - window) // page] = -1
    pos, req = torch.tensor([n - 1 for n in lens], dtype=torch.int32, device=DEV), torch.arange(R, dtype=torch.int32, device=DEV)
    q, qr, sink = torch.randn(heads, R, rank, device=DEV).bfloat16(), torch.randn(R, heads, dr, device=DEV).bfloat16(), torch.randn(heads, device=DEV)
    st, scale = torch.zeros(1, dtype=torch.int32, device=DEV), 2.0 * (rank + dr) ** -0.5
    want = torch.empty(heads, R, rank, device=DEV)
    K.attention_latent(q.float(), qr.float(), pages, table, req, pos, sink, want, scale, st, window=window)
    for splits, keys in ((1, 0), (5, 64), (10, 32)):
        n = R * heads * splits
        pa, pm = torch.empty(n * rank, device=DEV), torch.empty(n * 2, device=DEV)
        for single in (False, True):
            got = torch.full_like(want, float("nan"))
            K.attention_latent(q, qr, pages, table, req, pos, sink, got, scale, st, splits=splits, split_keys=keys, part_acc=pa, part_ml=pm,
                               window=window, single_tokens=single)
            _close(got, want, 6e-3, f"{splits} ranges")
        rows = torch.tensor([5, 0, 3], dtype=torch.int32, device=DEV)
        at = rows.long()
        for cast in (torch.bfloat16, torch.float32):
            got = torch.full((heads, 3, rank), float("nan"), device=DEV)
            K.attention_latent(q[:, at].to(cast).contiguous(), qr[at].to(cast).contiguous(), pages, table, req, pos, sink, got, scale, st, rows, 3,
                               splits, keys, pa, pm, window, single_tokens=True)
            _close(got, want[:, at], 6e-3, f"listed rows, {splits} ranges")
    assert int(st) == 0


# --------------------------------------------------------------------------------------------- parts alone
def _attention_part(wd, m, eps, dtype):
    from jax_llm_examples_b200.parts import GatedPagedAttention, rotary_frequencies

    c = lambda n: wd[n].to(dtype).to(DEV)  # noqa: E731
    rot = m.get("rot")
    return GatedPagedAttention(
        torch.cat([c("q"), c("k"), c("v")]), c("o"), m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps,
        q_norm_weight=c("q.norm"), k_norm_weight=c("k.norm"), norm="before", pairing="pairs", gate="none", rot_dims=rot["dims"] if rot else 0,
        inv_freq=rotary_frequencies(rot["base"], rot["dims"]).to(DEV) if rot else None, sink=torch.zeros(m["heads"], device=DEV),
        head_temperature=wd["temp"].to(DEV), softcap=m.get("softcap"), value_norm=True, window=m["mask"]["size"] if m.get("mask") else None,
        padded_dim=GatedPagedAttention.padded_size(m["dim"], m["vdim"], dtype))


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("m, portions", [
    ({"heads": 6, "kv_heads": 2, "dim": 10, "vdim": 6, "scale": 0.4, "softcap": 1.2, "rot": {"base": 60.0, "dims": 6}}, PORTIONS),
    ({"heads": 4, "kv_heads": 1, "dim": 64, "vdim": 64, "scale": 0.3, "softcap": 3.0, "rot": {"base": 10000.0, "dims": 64}}, PORTIONS),
    ({"heads": 2, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.2}, PORTIONS),
    ({"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 128, "scale": 0.09, "softcap": 25.0, "rot": {"base": 250000.0, "dims": 48}}, LONG_PORTIONS),
    ({"heads": 2, "kv_heads": 1, "dim": 128, "vdim": 128, "scale": 0.4, "softcap": 2.0, "mask": {"size": 90}}, LONG_PORTIONS),
    ({"heads": 3, "kv_heads": 3, "dim": 96, "vdim": 128, "scale": 0.2, "softcap": 9.0, "rot": {"base": 100.0, "dims": 2}}, LONG_PORTIONS),
    ({"heads": 2, "kv_heads": 1, "dim": 144, "vdim": 160, "scale": 0.2, "softcap": 5.0, "rot": {"base": 900.0, "dims": 144}}, PORTIONS),
])
def test_soft_capped_attention_in_portions(name, dtype, tol, m, portions):
    """The ``attention`` mixer as a part: weighted q/k norm, rotation in pairs, normed values, a number per head on the
    scores (one of them negative), the cap (from hardly bending to bending everything), one added to the denominator;
    portions that start inside a page, two tokens, single tokens; head size 128 on the tcgen05 kernel in bfloat16."""
    from jax_llm_examples_b200.parts import Runtime

    torch.manual_seed(m["heads"] + m["dim"])
    D, eps, T = 48, 1e-5, portions[-1][1]
    g = lambda *s: (torch.randn(*s) * 0.3).to(dtype)  # noqa: E731
    Hq, Hkv, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    temp = torch.linspace(0.4, 1.8, Hq)
    temp[-1] = -0.8
    wd = {"q": g(Hq * dk, D), "k": g(Hkv * dk, D), "v": g(Hkv * dv, D), "o": g(D, Hq * dv),
          "q.norm": (1 + g(dk)).to(dtype), "k.norm": (1 + g(dk)).to(dtype), "temp": temp}
    hs = torch.randn(T, D).to(dtype)
    page = 64 if max(dk, dv) == 128 else 16
    got, _, _ = _attention_in_portions(_attention_part(wd, m, eps, dtype), Runtime(dtype, torch.device(DEV)), hs, dtype, portions, page)
    _close(got, plain.attention_mixer(hs.double(), {"m." + k: v.double() for k, v in wd.items()}, "m.", m, eps), tol, name)


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("size", [16, 64, 128])
@pytest.mark.parametrize("cap", [1.0, 7.0, 60.0])
def test_cap_temperature_and_the_added_one_made_to_show(name, dtype, tol, size, cap):
    """All keys equal and all queries equal, so that every score of head a is one number s_a, from a tenth of the cap to far
    beyond it, positive and negative; values that name their position (after their norm: sqrt(size) in one entry).  The
    weights are then e / (1 + n e) with e = exp(cap tanh(s_a / cap)) and n keys seen: in closed form.  In a prompt and
    for tokens decoded alone."""
    from jax_llm_examples_b200.parts import GatedPagedAttention, Runtime

    T, eps, heads = 80, 1e-12, 4
    D = heads * size
    hs = torch.zeros(T, D)
    for p in range(T):
        hs[p, 1 + p % 8] = 1.0
        hs[p, 0] = 1.0
    wq, wk, wv = torch.zeros(heads * size, D), torch.zeros(size, D), torch.zeros(size, D)
    wk[:, 0] = 1.0  # every key: all ones, also after its norm
    for a in range(heads):
        wq[a * size:(a + 1) * size, 0] = 1.0
    wv[:8, 1:9] = torch.eye(8)
    temps = torch.tensor([0.1, 0.9, 4.0, -1.5])
    mixer = GatedPagedAttention(torch.cat([wq, wk, wv]).to(dtype).to(DEV), torch.eye(D).to(dtype).to(DEV), heads, 1, size, size, cap / size, eps,
                                q_norm_weight=torch.ones(size, device=DEV), k_norm_weight=torch.ones(size, device=DEV), gate="none",
                                sink=torch.zeros(heads, device=DEV), head_temperature=temps.to(DEV), softcap=cap, value_norm=True,
                                padded_dim=GatedPagedAttention.padded_size(size, size, dtype))
    page = 64 if size == 128 else 16
    for portions in (((0, T),), ((0, 64), (64, 70)) + tuple((p, p + 1) for p in range(70, T))):
        got, _, _ = _attention_in_portions(mixer, Runtime(dtype, torch.device(DEV)), hs.to(dtype), dtype, portions, page)
        for p in (0, 1, 15, 16, 63, 64, 70, 79):
            for a in range(heads):
                e = math.exp(cap * math.tanh(float(temps[a])))
                for mark in range(8):
                    seen = sum(1 for j in range(p + 1) if j % 8 == mark)
                    want = math.sqrt(size) * seen / (1.0 / e + (p + 1))
                    have = float(got[p, a * size + mark])
                    assert abs(have - want) < (2e-4 if dtype == torch.float32 else 2e-2) * math.sqrt(size), \
                        f"{name}: position {p} head {a} mark {mark}: {have:.4f} for {want:.4f}"


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("size", [16, 128])
@pytest.mark.parametrize("back", [1, 63, 64, 127, 128, 300, 390])
def test_a_key_far_back_is_found(name, dtype, tol, size, back):
    """One earlier token points where the query points, everything else points elsewhere: its value's marker comes through
    from any distance (the sequence's first tokens included), in a prompt and for a token decoded alone, also when the
    prompt came in portions."""
    from jax_llm_examples_b200.parts import GatedPagedAttention, Runtime

    torch.manual_seed(back)
    D, T = size, 392
    ones, eye = torch.ones(D, device=DEV), torch.eye(D)
    mixer = GatedPagedAttention(torch.cat([eye, eye, eye]).to(dtype).to(DEV), eye.to(dtype).to(DEV), 1, 1, D, D, 12.0 / D, 1e-6, q_norm_weight=ones,
                                k_norm_weight=ones, gate="none", sink=torch.zeros(1, device=DEV), head_temperature=torch.ones(1, device=DEV),
                                softcap=30.0, value_norm=True, padded_dim=GatedPagedAttention.padded_size(D, D, dtype))
    hs = torch.randn(T, D) * 0.3
    hs[:, 3] = hs[:, 8] = 0.0
    hs[T - 1] = 0.0
    hs[T - 1, 3] = 3.0
    hs[T - 1 - back] = 0.0
    hs[T - 1 - back, 3], hs[T - 1 - back, 8] = 3.0, 0.75
    page = 64 if size == 128 else 16
    for portions in (((0, T),), ((0, T - 1), (T - 1, T)), ((0, 130), (130, 389), (389, T - 1), (T - 1, T)), ((0, 130), (130, T - 2), (T - 2, T))):
        got, _, _ = _attention_in_portions(mixer, Runtime(dtype, torch.device(DEV)), hs.to(dtype), dtype, portions, page)
        marker = float(got[-1, 8]) / math.sqrt(D)
        assert marker > 0.1, f"{name}: the key {back} back: marker {marker:.3f} ({portions})"


def _latent_part(wd, m, eps, dtype):
    from jax_llm_examples_b200.parts import LatentAttention

    c = lambda n: wd[n].to(dtype).to(DEV)  # noqa: E731
    return LatentAttention(torch.cat([c("dq"), c("dkv"), c("g")]), c("dq.norm"), c("uq"), c("dkv.norm"), c("uk"), c("uv"), c("o"),
                           wd["sink"].to(DEV), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"],
                           m["rot"]["base"], m["rot"]["dims"], eps, window=m["mask"]["size"] if m.get("mask") else None, pairing="halves", gated=True)


def _latent_weights(m, D, dtype, spread=0.3):
    g = lambda *s: (torch.randn(*s) * spread).to(dtype)  # noqa: E731
    Hh, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    return {"dq": g(m["q_rank"], D), "dq.norm": (1 + g(m["q_rank"])).to(dtype), "uq": g(Hh * (dn + dr), m["q_rank"]), "dkv": g(rank + dr, D),
            "dkv.norm": (1 + g(rank)).to(dtype), "uk": g(Hh * dn, rank), "uv": g(Hh * dv, rank), "sink": torch.randn(Hh), "g": g(Hh, D), "o": g(D, Hh * dv)}


def _latent_in_portions(mixer, rt, hs, dtype, portions, page, gone_below=None):
    """``gone_below``: pages that hold only positions below gone_below(lo) are taken out of the table before the portion that
    starts at lo, as the manager takes back what no query can see."""
    from jax_llm_examples_b200.parts import LayerCache

    need = mixer.kv_need()
    assert need.planes == 1 and need.num_kv_heads == 1
    width = (hs.shape[0] + page - 1) // page
    pages = torch.full((width + 5, 1, 1, page, need.head_dim), float("nan"), device=DEV, dtype=dtype)  # nothing unwritten may be used
    table = torch.randperm(width + 5)[:width].reshape(1, width).to(torch.int32).to(DEV)
    outs = []
    for lo, hi in portions:
        if gone_below is not None:
            table[0, :max(0, gone_below(lo)) // page] = -1
        ctx = _ctx(rt, [hi - lo], [lo], planners=mixer.step_planners(), page_size=page)
        rows = hs[lo:hi].to(DEV)
        outs.append(H.as_rows_sum(mixer.forward(ctx, rows, LayerCache(pages, table, True, None))))
        assert int(ctx.status) == 0
    return torch.cat(outs)


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("m, portions", [
    ({"heads": 3, "dim": 5, "rot_dim": 6, "vdim": 9, "q_rank": 11, "kv_rank": 13, "scale": 0.3, "mask": {"size": 7}, "rot": {"base": 50.0, "dims": 6}}, PORTIONS),
    ({"heads": 4, "dim": 40, "rot_dim": 16, "vdim": 24, "q_rank": 48, "kv_rank": 64, "scale": 0.1, "mask": {"size": 36}, "rot": {"base": 1e4, "dims": 16}}, LONG_PORTIONS),
    ({"heads": 18, "dim": 16, "rot_dim": 8, "vdim": 16, "q_rank": 24, "kv_rank": 40, "scale": 0.15, "mask": {"size": 16}, "rot": {"base": 1e6, "dims": 8}}, LONG_PORTIONS),
    ({"heads": 2, "dim": 8, "rot_dim": 2, "vdim": 8, "q_rank": 16, "kv_rank": 24, "scale": 0.3, "mask": {"size": 1}, "rot": {"base": 1e4, "dims": 2}}, PORTIONS),
    ({"heads": 5, "dim": 16, "rot_dim": 16, "vdim": 32, "q_rank": 32, "kv_rank": 528, "scale": 0.05, "rot": {"base": 1e4, "dims": 16}}, PORTIONS),
    ({"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "q_rank": 96, "kv_rank": 512, "scale": 0.01, "mask": {"size": 100}, "rot": {"base": 1e4, "dims": 64}},
     LONG_PORTIONS),
])
def test_windowed_gated_latent_attention_in_portions(name, dtype, tol, m, portions):
    """The ``latent_attention`` mixer as a part: both latents' norms, the rotate-half rotation of the shared key part, the
    window, the learned sink, the gate per head; portions, two tokens, single tokens; pages that the window has passed
    are gone, and what was never written (or was padding) is NaN in the pool."""
    from jax_llm_examples_b200.parts import Runtime

    torch.manual_seed(m["heads"])
    D, eps, T = 48, 1e-5, portions[-1][1]
    wd = _latent_weights(m, D, dtype)
    hs = torch.randn(T, D).to(dtype)
    window = m["mask"]["size"] if m.get("mask") else None
    got = _latent_in_portions(_latent_part(wd, m, eps, dtype), Runtime(dtype, torch.device(DEV)), hs, dtype, portions, 16,
                              None if window is None else lambda lo: lo - window + 1)
    _close(got, plain.latent_attention_mixer(hs.double(), {"m." + k: v.double() for k, v in wd.items()}, "m.", m, eps), tol, name)


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("window", [None, 33, 200, 400])
def test_latent_decoding_of_unequal_requests_with_split_keys(name, dtype, tol, window):
    """Many requests decode one token each over contexts from one token to 700, beside a portion of another request: the keys
    are cut into ranges (with a window: from the first visible key's range on) and put together again."""
    from jax_llm_examples_b200.parts import LayerCache, Runtime

    torch.manual_seed(7)
    D, eps, page = 48, 1e-5, 16
    m = {"heads": 4, "dim": 16, "rot_dim": 8, "vdim": 16, "q_rank": 24, "kv_rank": 64, "scale": 0.2, "rot": {"base": 1e4, "dims": 8}}
    if window is not None:
        m["mask"] = {"size": window}
    wd = _latent_weights(m, D, dtype)
    mixer, rt = _latent_part(wd, m, eps, dtype), Runtime(dtype, torch.device(DEV))
    lens = [700, 1, 33, 34, 257, 64, 65, 400, 401, 512]
    P = {"m." + k: v.double() for k, v in wd.items()}
    seqs = [torch.randn(n + 12, D).to(dtype) for n in lens]
    refs = [plain.latent_attention_mixer(s.double(), P, "m.", m, eps) for s in seqs]
    need = mixer.kv_need()
    width = 712 // page + 1
    perm = torch.randperm(len(lens) * width).to(torch.int32).view(len(lens), width).to(DEV)
    pages = torch.full((len(lens) * width, 1, 1, page, need.head_dim), float("nan"), device=DEV, dtype=dtype)

    def step(live, q_lens, starts):
        ctx = _ctx(rt, q_lens, starts, planners=mixer.step_planners(), page_size=page)
        rows = torch.cat([seqs[r][s:s + n] for r, n, s in zip(live, q_lens, starts)]).to(DEV)
        out = H.as_rows_sum(mixer.forward(ctx, rows, LayerCache(pages, perm[live].contiguous(), True, None)))
        assert int(ctx.status) == 0
        return out

    for r, n in enumerate(lens):
        _close(step([r], [n], [0]), refs[r][:n], tol, f"{name}: prompt of {n}")
    every = list(range(len(lens)))
    got = step(every, [1] * len(lens), lens)
    for r, n in enumerate(lens):
        _close(got[r:r + 1], refs[r][n:n + 1], 2 * tol, f"{name}: token after {n}")
    q = [1, 11, 1, 2, 1, 1, 5, 1, 1, 1]
    got, at = step(every, q, [n + 1 for n in lens]), 0
    for r, n in enumerate(lens):
        _close(got[at:at + q[r]], refs[r][n + 1:n + 1 + q[r]], 2 * tol, f"{name}: mixed step, request {r}")
        at += q[r]


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("window", [5, 16, 21, 64, 90, 100])  # 100: the far key is the sequence's first token, 99 back
def test_a_key_just_inside_and_just_outside_the_latent_window(name, dtype, tol, window):
    """ONE earlier token's latent points where the query points, and its value carries a marker: window - 1 tokens back it
    shares the weight with the query itself; window tokens back it is gone.  In a prompt portion and for a token decoded
    alone; edges at and across page borders."""
    from jax_llm_examples_b200.parts import Runtime

    torch.manual_seed(window)
    D = rank = 32
    m = {"heads": 1, "dim": rank, "rot_dim": 2, "vdim": rank, "q_rank": rank, "kv_rank": rank, "scale": 12.0 / rank, "mask": {"size": window},
         "rot": {"base": 1e4, "dims": 2}}
    eye, ones = torch.eye(D), torch.ones(rank)
    down = torch.cat([eye, torch.zeros(2, D)])
    uq = torch.cat([torch.eye(rank), torch.zeros(2, rank)])
    wd = {"dq": eye, "dq.norm": ones, "uq": uq, "dkv": down, "dkv.norm": ones, "uk": torch.eye(rank), "uv": torch.eye(rank), "sink": torch.zeros(1),
          "g": torch.zeros(1, D), "o": eye}
    mixer, rt = _latent_part(wd, m, 1e-6, dtype), Runtime(dtype, torch.device(DEV))
    for qpos, decoded in ((99, False), (99, True), (70, False), (window - 1, False), (window, True)):
        for back, seen in ((window - 1, True), (window, False)):
            if qpos - back < 0 or qpos >= 100 or back == 0:
                continue
            hs = torch.randn(100, D) * 0.3
            hs[:, 3] = hs[:, 8] = 0.0
            hs[qpos] = 0.0
            hs[qpos, 3] = 4.0
            hs[qpos - back] = 0.0
            hs[qpos - back, 3], hs[qpos - back, 8] = 4.0, 1.0
            cuts = [(0, qpos), (qpos, qpos + 1)] if decoded else [(0, qpos + 1)]
            out = _latent_in_portions(mixer, rt, hs.to(dtype), dtype, [c for c in cuts if c[1] > c[0]], 16, lambda lo: lo - window + 1)
            marker = float(out[-1, 8])  # half (the gate at zero) of the key's share times about 0.25 sqrt(rank)
            assert (marker > 0.2) == seen and (seen or abs(marker) < 0.03), \
                f"{name} window {window}: query {qpos} ({'decoded' if decoded else 'prompt'}), key {back} back: marker {marker:.3f}"


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
def test_latent_sink_and_gate_made_to_show(name, dtype, tol):
    """All latents equal and no rotated part to speak of: every score is one number c, so a head's output is
    sigmoid(g_h) n e^c / (n e^c + e^sink_h) times its value, n the keys in the window, in closed form per head."""
    from jax_llm_examples_b200.parts import Runtime

    D = rank = 16
    heads, window, T = 3, 6, 40
    sink, gates = torch.tensor([-1.0, 1.0, 3.0]), torch.tensor([0.0, 2.0, -1.5])
    m = {"heads": heads, "dim": rank, "rot_dim": 2, "vdim": rank, "q_rank": rank, "kv_rank": rank, "scale": 0.125, "mask": {"size": window},
         "rot": {"base": 1e4, "dims": 2}}
    ones = torch.ones(rank)
    uq = torch.cat([torch.eye(rank), torch.zeros(2, rank)]).repeat(heads, 1)
    g = torch.zeros(heads, D)
    g[:, 0] = gates / 2.0
    wd = {"dq": torch.eye(D), "dq.norm": ones, "uq": uq, "dkv": torch.cat([torch.eye(D), torch.zeros(2, D)]), "dkv.norm": ones,
          "uk": torch.eye(rank).repeat(heads, 1), "uv": torch.eye(rank).repeat(heads, 1), "sink": sink, "g": g, "o": torch.eye(heads * rank)[:, :]}
    # the output product is the identity, so the model's width is heads * rank: widen the input with zeros
    for k in ("dq", "dkv", "g"):
        wd[k] = torch.cat([wd[k], torch.zeros(wd[k].shape[0], heads * rank - D)], dim=1)
    hs = torch.zeros(T, heads * rank)
    hs[:, :rank] = 2.0  # a latent of ones after its norm
    mixer = _latent_part(wd, m, 1e-9, dtype)
    for portions in (((0, T),), ((0, 20), (20, 22)) + tuple((p, p + 1) for p in range(22, T))):
        got = _latent_in_portions(mixer, Runtime(dtype, torch.device(DEV)), hs.to(dtype), dtype, portions, 16, lambda lo: lo - window + 1)
        for p in (0, 1, 4, 5, 6, 21, 22, 39):
            n = min(p + 1, window)
            for a in range(heads):
                e = n * math.exp(rank * 0.125)
                want = e / (e + math.exp(float(sink[a]))) / (1 + math.exp(-float(gates[a])))
                assert abs(float(got[p, a * rank + 5]) - want) < (1e-5 if dtype == torch.float32 else 8e-3), f"{name}: position {p} head {a}"


@pytest.mark.parametrize("name, dtype, tol", DTYPES)
@pytest.mark.parametrize("E, k, ff, D, groups, n", [(6, 2, 14, 36, (3, 2), 9), (8, 2, 64, 128, (4, 2), 3), (8, 3, 64, 128, (4, 2), 16), (8, 4, 64, 128, (2, 1), 17),
                                                    (12, 3, 80, 192, (3, 2), 300), (40, 1, 32, 64, (8, 8), 5), (24, 6, 2048, 64, (1, 1), 12)])
def test_experts_with_unnormalised_sigmoid_weights(name, dtype, tol, E, k, ff, D, groups, n):
    """The feed-forward as a part, from few rows (decoding) to many (a portion): exact gelu, outputs weighted."""
    from jax_llm_examples_b200.parts import RoutedMLPExperts, Runtime, as_rows

    torch.manual_seed(E + n)
    g = lambda *s: (torch.randn(*s) * 0.2).to(dtype)  # noqa: E731
    up, down, corr = g(E, ff, D), g(E, D, ff), torch.randn(E) * 0.3
    wr = torch.randn(E, D) * D ** -0.5
    ff_part = RoutedMLPExperts(wr.to(DEV), None, up.to(DEV), down.to(DEV), k, "gelu", weight_form="sigmoid_corrected", correction=corr.to(DEV),
                               groups=groups[0], keep=groups[1], group_top=2)
    x = torch.randn(n, D).to(dtype)
    ctx = _ctx(Runtime(dtype, torch.device(DEV)), [n], [0])
    ctx.scratch["record_routing"] = []
    y = as_rows(ff_part.forward(ctx, x.to(DEV), x.float().to(DEV)))
    P = {"router": wr.double(), "correction": corr.double()}
    for e in range(E):
        P[f"e{e}.up"], P[f"e{e}.down"] = up[e].double(), down[e].double()
    ml = {"router": {"experts": E, "top": k, "groups": {"count": groups[0], "keep": groups[1]}}, "expert": {"ff": ff}}
    chosen = ctx.scratch["record_routing"][0].cpu()
    ref, _, own = plain.expert_mixture(x.double(), P, "", ml, chosen)
    assert float((torch.sort(chosen.long(), 1).values != torch.sort(own, 1).values).any(1).double().mean()) <= 0.01
    _close(y.data.view(y.splits, n, D).sum(0) if y.splits > 1 else y.data, ref, tol, name)
    assert int(ctx.status) == 0


# --------------------------------------------------------------------------------------- whole models, by traces
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("marinex")
    return {n: MX.make_dir(root / n, n, seed=i + 1) for i, n in enumerate(MX.CONFIGS)}


def _engine(folder, dtype, max_tokens=512, page_size=16, max_slots=4, **kw):
    import jax_llm_examples_b200 as J

    return J.Engine(J.load_model(folder, dtype, DEV), max_tokens=max_tokens, page_size=page_size, max_slots=max_slots, **kw)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MX.CONFIGS))
def test_every_kind_of_cut_against_the_plain_implementation(folders, name, dtype):
    """Whole prompts; most of a prompt and then 40 tokens one by one; portions down to two tokens; up to four live
    requests mixed, in a pool too small for all of them, so that pages and slots are used again.  Every position's
    logits are compared, the first tokens of a sequence included."""
    vocab = MX.config(name)["vocab"]
    rng = random.Random(7)
    requests = H.random_requests(rng, vocab, [61, 1, 2, 33, 17, 90, 5])
    engine = _engine(folders[name], dtype, max_tokens=16 * 16)
    for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=40), H.trace_portions(requests, rng),
                  H.trace_mixed(requests, rng, max_live=4)):
        got, routing = H.run_trace(engine, steps, record_routing=True)
        assert len(got) == sum(len(t) for t in requests.values())
        MX.compare(folders[name], requests, got, routing, dtype, stray=2 if dtype == "bfloat16" else 0)
        assert engine.manager.free_slots() == 4 and all(engine.manager.free_pages(g) == engine.num_pages for g in range(len(engine.manager.groups)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_head_size_128_on_pages_of_64_tokens(folders, dtype):
    """Pages of 64 tokens, as a server has them: in bfloat16 the portions of 64 tokens and more of the layers with head
    size 128 run on the tcgen05 kernel (with the cap and the added one), shorter ones on the mma.sync kernel, single tokens
    on the split-KV kernel, all in one step."""
    name = "wide"
    vocab = MX.config(name)["vocab"]
    rng = random.Random(13)
    requests = H.random_requests(rng, vocab, [200, 70, 131, 3])
    engine = _engine(folders[name], dtype, max_tokens=12 * 64, page_size=64)
    for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=20), H.trace_portions(requests, rng),
                  H.trace_mixed(requests, rng, max_live=4, portions=H.LONG_PORTIONS)):
        got, routing = H.run_trace(engine, steps, record_routing=True)
        MX.compare(folders[name], requests, got, routing, dtype, stray=2 if dtype == "bfloat16" else 0)
    if dtype == "bfloat16":
        assert any("tc" in kinds for kinds in engine.attention_kernels_seen), "the tcgen05 kernel did not run"


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random_under_every_kind_of_cut(seed, tmp_path):
    """Sizes, head counts, orders of layers, windows, caps, rotations and routers that nobody chose, in both precisions: whole
    prompts, a decoded tail, portions and mixed batches against the plain implementation."""
    rng = random.Random(seed)
    cfg = MX.random_config(rng)
    folder = MX.write_model(tmp_path / "m", cfg, seed)
    requests = H.random_requests(rng, cfg["vocab"], [70, 3, 130, 21, 45])
    for dtype in ("float32", "bfloat16"):
        engine = _engine(folder, dtype, max_tokens=20 * 16)
        for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=40), H.trace_portions(requests, rng),
                      H.trace_mixed(requests, rng, max_live=4)):
            got, routing = H.run_trace(engine, steps, record_routing=True)
            MX.compare(folder, requests, got, routing, dtype, stray=4 if dtype == "bfloat16" else 0)


@pytest.mark.parametrize("seed", [0, 1, 2, 3])
def test_mid_size_configurations_on_pages_of_64_tokens(seed, tmp_path):
    """Widths of 192 to 512, head sizes up to 128, dozens of experts, windows of up to 300 tokens, prompts of up to 700
    tokens on pages of 64: whole prompts, a decoded tail, portions and mixed batches against the plain implementation.
    The float32 cap is 1e-4 here: rows are sums of up to 512 terms through up to six layers."""
    rng = random.Random(1000 + seed)
    cfg = MX.mid_size_config(rng)
    folder = MX.write_model(tmp_path / "m", cfg, seed, std=0.9 / cfg["width"] ** 0.5)
    requests = H.random_requests(rng, cfg["vocab"], [700, 330, 97, 23, 1, 260])
    saved = dict(MX.TOL), dict(MX.TOL_MEAN)
    MX.TOL["float32"], MX.TOL_MEAN["float32"] = 1e-4, 2e-5
    try:
        for dtype in ("float32", "bfloat16"):
            engine = _engine(folder, dtype, max_tokens=1536, page_size=64, max_seq_len=1536)
            for steps in (H.trace_whole(requests), H.trace_tail_decode(requests, tail=40), H.trace_portions(requests, rng),
                          H.trace_mixed(requests, rng, max_live=4, portions=H.LONG_PORTIONS)):
                got, routing = H.run_trace(engine, steps, record_routing=True)
                MX.compare(folder, requests, got, routing, dtype, stray=6 if dtype == "bfloat16" else 0)
    finally:
        MX.TOL.update(saved[0]), MX.TOL_MEAN.update(saved[1])


@pytest.mark.parametrize("name", list(MX.CONFIGS))
def test_logits_do_not_depend_on_the_cut_or_on_the_batch(folders, name):
    """float32: the same request whole, token by token, in portions, and beside three other requests gives the same
    logits to within rounding of a sum's order (far below the tolerance against the plain implementation)."""
    vocab = MX.config(name)["vocab"]
    rng = random.Random(11)
    requests = H.random_requests(rng, vocab, [70, 23, 41, 9])
    engine = _engine(folders[name], "float32")
    whole, _ = H.run_trace(engine, H.trace_whole(requests), record_routing=False)
    for steps in (H.trace_tail_decode(requests, tail=70), H.trace_portions(requests, rng), H.trace_mixed(requests, rng)):
        got, _ = H.run_trace(engine, steps, record_routing=False)
        worst = max(MX.row_err(got[k], whole[k]) for k in whole)
        assert worst < 5e-6, f"{name}: logits moved by {worst:.2e} with the cut"


@pytest.mark.parametrize("name", list(MX.CONFIGS))
def test_decoding_through_replayed_graphs_equals_decoding_without(folders, name):
    """bfloat16: decode-only steps are captured in CUDA graphs and replayed; pages are found by table on the device, so the
    replayed steps must give what the same steps give launched one kernel at a time."""
    vocab = MX.config(name)["vocab"]
    rng = random.Random(5)
    requests = H.random_requests(rng, vocab, [50, 37])
    outs = []
    for graphs in (True, False):
        engine = _engine(folders[name], "bfloat16", use_graphs=graphs)
        got, _ = H.run_trace(engine, H.trace_tail_decode(requests, tail=30), record_routing=False)
        assert (engine.graph_replays > 0) == graphs
        outs.append(got)
    worst = max(MX.row_err(outs[0][k], outs[1][k]) for k in outs[0])
    assert worst < 2e-2, f"{name}: replayed steps differ by {worst:.2e}"


def test_long_decoding_and_slots_used_again(folders):
    """300 tokens one by one after a short prompt, in both precisions: the window's old pages are given back on the way, the
    other layers' stay; then the same slot and pages serve another request, which must not see what the first left."""
    name = "small"
    vocab = MX.config(name)["vocab"]
    rnd = random.Random(3)
    toks = [rnd.randrange(vocab) for _ in range(320)]
    other = [rnd.randrange(vocab) for _ in range(25)]
    for dtype in ("float32", "bfloat16"):
        engine = _engine(folders[name], dtype, max_tokens=320, max_slots=1)
        for req in ({"a": toks}, {"b": other}):
            got, routing = H.run_trace(engine, H.trace_tail_decode(req, tail=300), record_routing=True)
            MX.compare(folders[name], req, got, routing, dtype, stray=3 if dtype == "bfloat16" else 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_decoding_batch_of_every_size(folders, dtype):
    """One to twenty requests decode together (the sizes at which the kernels of a decode step change), each with a context of
    its own length: every request's logits are the plain implementation's."""
    name = "wide"
    vocab = MX.config(name)["vocab"]
    rng = random.Random(17)
    for n in (1, 3, 8, 9, 16, 17, 20):
        requests = H.random_requests(rng, vocab, [8 + 5 * (i % 7) + i for i in range(n)])
        engine = _engine(folders[name], dtype, max_tokens=20 * 64, max_slots=20)
        heads = {"entries": [{"id": r, "tokens": t[:-3], "want": []} for r, t in requests.items()], "end": []}
        tails = [{"entries": [{"id": r, "tokens": [t[len(t) - 3 + i]], "want": [0]} for r, t in requests.items()],
                  "end": list(requests) if i == 2 else []} for i in range(3)]
        got, routing = H.run_trace(engine, [heads] + tails, record_routing=True)
        assert len(got) == 3 * n
        MX.compare(folders[name], requests, got, routing, dtype, stray=1 if dtype == "bfloat16" else 0)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MX.CONFIGS))
def test_greedy_generation_through_the_scheduler(folders, name, dtype):
    """The framework's own entry point: prompts of unequal length under a small token budget per step, so that
    prompt portions run beside decoded tokens."""
    import jax_llm_examples_b200 as J

    vocab = MX.config(name)["vocab"]
    prompts = [[(7 * i + 3 * j) % vocab for i in range(n)] for j, n in enumerate((29, 3, 12))]
    model = J.load_model(folders[name], dtype, DEV)
    got = J.generate(model, prompts, J.SamplingParams(max_new_tokens=10), page_size=16, max_tokens_per_step=16)
    for p, g in zip(prompts, got):
        assert len(g) == 10
        MX.greedy_checked(folders[name], model, p, g, dtype)


def test_command_line_generates_from_a_preset_and_from_a_folder(folders, capsys):
    from jax_llm_examples_b200.main import main

    assert main(["--preset", "marinex_tiny", "--random-prompts", "2", "--prompt-len", "9", "--max-new-tokens", "4"]) == 0
    assert capsys.readouterr().out.count("-" * 80) == 2
    assert main(["--model", str(folders["padded"]), "--dtype", "float32", "--prompt-ids", "1,2,3,4,5", "--max-new-tokens", "5",
                 "--page-size", "16"]) == 0
    ids = [int(t) for t in capsys.readouterr().out.splitlines()[1].split()]
    MX.greedy_checked(folders["padded"], None, [1, 2, 3, 4, 5], ids, "float32")


def test_trace_replay_program_on_a_marinex_folder(folders, tmp_path):
    """bin/trace_run picks the model class by config.json and writes the wanted logits."""
    name, dtype = "padded", "float32"
    vocab = MX.config(name)["vocab"]
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
    ref, _ = MX.plain_logits(folders[name], toks)
    rows = {0: [0, 12], 1: [1], 2: [20]}
    for step, places in rows.items():
        got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(len(places), vocab)
        for g, pl in zip(got, places):
            assert MX.row_err(g, ref[pl]) < MX.TOL[dtype]
