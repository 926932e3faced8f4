"""Samerax without a GPU: the configuration reader, the tensor list, random model folders, how long a layer's pages live, shared
layers, and the plain implementation against other ways of writing the same mathematics."""

import json
import math

import pytest
import torch

from tests import samerax_helpers as SX
from tests.plain import samerax_plain as plain

F64 = torch.float64


def test_config_is_read_from_the_files_own_keys():
    from jax_llm_examples_b200.config.registry import resolve
    from jax_llm_examples_b200.config.samerax import DenseSpec, SameraxConfig, TableMoeSpec

    cj = SX.config("small")
    arch = resolve(cj)
    assert arch.name == "Samerax"
    cfg = arch.parse_config(cj)
    assert isinstance(cfg, SameraxConfig)
    assert (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.embedding_scale, cfg.logit_softcap) == (61, 36, 1e-5, 1.7, 4.0)
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.keep_first, m.scale, m.diff) == (6, 2, 5, 7, 7, 3, 0.5, 0.2)
    assert (m.rot.base, m.rot.dims, m.rot.scaling.factor, m.rot.scaling.original, m.rot.scaling.fast, m.rot.scaling.slow) == (60.0, 4, 4.0, 30, 4.0, 1.0)
    assert cfg.layers[0].mlp == TableMoeSpec(5, 2, 14) and cfg.layers[1].mlp == DenseSpec(22)
    assert cfg.layers[1].mixer.rot.scaling is None and cfg.layers[4].mixer.rot is None
    assert [L.weights_of for L in cfg.layers] == [None, None, 0, 2, None]
    assert [cfg.owner(i) for i in range(5)] == [0, 1, 0, 0, 4]
    p = arch.parse_config(SX.config("padded"))
    assert p.logit_softcap is None and p.layers[0].mixer.window is None and p.layers[0].mixer.keep_first == 0


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "delta", "no mixer"),
    (("layers", 0, "mixer", "kv_heads"), 4, "no multiple"),
    (("layers", 0, "mixer", "rot", "dims"), 3, "even"),
    (("layers", 0, "mixer", "rot", "dims"), 6, "at most"),
    (("layers", 0, "mixer", "rot", "scaling", "factor"), 0.0, "scaling"),
    (("layers", 0, "mixer", "mask", "size"), 0, "mask"),
    (("layers", 0, "mixer", "mask", "keep_first"), -1, "keep_first"),
    (("layers", 0, "mixer", "vdim"), 0, "positive"),
    (("layers", 0, "mixer", "diff"), None, "diff"),
    (("layers", 1, "mlp", "kind"), "wide", "moe"),
    (("layers", 0, "mlp", "router", "top"), 6, "top-6"),
    (("layers", 2, "weights_of"), 1, "differ"),
    (("layers", 2, "weights_of"), 9, "weights_of"),
    (("layers", 0, "weights_of"), 2, "weights_of"),
    (("logit_softcap",), -1.0, "logit_softcap"),
    (("norm", "eps"), 0.0, "eps"),
])
def test_config_errors_name_the_key(path, value, word):
    from jax_llm_examples_b200.config.base import ConfigError
    from jax_llm_examples_b200.config.samerax import SameraxConfig

    cj = SX.config("small")
    d = cj
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        SameraxConfig.from_dict(cj)


def test_tensor_list_and_random_folder(tmp_path):
    from jax_llm_examples_b200.config.registry import resolve
    from jax_llm_examples_b200.weights.loader import WeightError, load_tensors

    for name in SX.CONFIGS:
        cj = SX.config(name)
        folder = SX.make_dir(tmp_path / name, name, seed=1)
        specs = resolve(cj).tensor_specs(resolve(cj).parse_config(cj))
        P = plain.read_safetensors(folder / "model.safetensors")
        assert set(P) == set(specs)
        # a layer with another's weights has none of its own; a table's rows name different experts
        for i, L in enumerate(cj["layers"]):
            own = [n for n in specs if n.startswith(f"l{i}.")]
            assert bool(own) == ("weights_of" not in L)
            if own and (L["mlp"] or {}).get("kind") == "moe":
                t, r = P[f"l{i}.mlp.table"], L["mlp"]["router"]
                assert t.dtype == torch.int32 and t.shape == (cj["vocab"], r["top"]) and int(t.min()) >= 0 and int(t.max()) < r["experts"]
                assert all(len(set(row)) == r["top"] for row in t.tolist())
        for dtype in (torch.float32, torch.bfloat16):
            got = load_tensors(folder, specs, None, dtype)
            assert all(t.dtype == (torch.int32 if n.endswith(".table") else dtype) for n, t in got.items())
    bad = {k: v for k, v in specs.items() if k != "head"}
    with pytest.raises(WeightError, match="head"):
        load_tensors(folder, bad, None, torch.float32)


def _build_cpu(name, tmp_path):
    from jax_llm_examples_b200.loading import load_model

    return load_model(SX.make_dir(tmp_path / name, name, seed=2), "float32", "cpu")


def test_what_a_layer_keeps_and_which_layers_share_a_block(tmp_path):
    from jax_llm_examples_b200.cache.manager import Retention

    model = _build_cpu("small", tmp_path)
    assert [r.block for r in model.schedule] == [0, 1, 0, 0, 2] and [r.cache for r in model.schedule] == [0, 1, 2, 3, 4]
    assert [c.retention for c in model.plan.caches] == [Retention.window(7, 3), Retention.window(11, 18), Retention.window(7, 3), Retention.window(7, 3),
                                                       Retention.window(19)]
    assert [(c.num_kv_heads, c.head_dim, c.planes) for c in model.plan.caches] == [(2, 10, 2), (3, 13, 2), (2, 10, 2), (2, 10, 2), (1, 20, 2)]
    assert len(model.plan.groups) == 3 and model.logit_softcap == 4.0 and model.embedding_scale == 1.7
    padded = _build_cpu("padded", tmp_path)
    assert [c.retention for c in padded.plan.caches] == [Retention.all(), Retention.window(1, 1), Retention.window(30, 37)]
    assert padded.logit_softcap is None


def test_bfloat16_rows_are_padded_to_the_tensor_core_sizes():
    from jax_llm_examples_b200.parts import DifferentialAttention as A

    sizes = [(A.padded_size(d, v, torch.bfloat16), A.padded_size(d, v, torch.float32)) for d, v in ((5, 7), (32, 64), (33, 8), (8, 72), (64, 128), (65, 8), (8, 144))]
    assert sizes == [(64, 10), (64, 64), (128, 66), (128, 72), (128, 128), (130, 130), (144, 144)]


def test_a_table_with_a_wrong_expert_is_refused():
    from jax_llm_examples_b200.parts import TableRoutedGLUExperts

    gu, down = torch.zeros(3, 8, 4), torch.zeros(3, 4, 4)
    for bad, word in (([[0, 3]], "there are 3"), ([[-1, 0]], "-1"), ([[1, 1]], "twice")):
        with pytest.raises(ValueError, match=word):
            TableRoutedGLUExperts(torch.tensor(bad, dtype=torch.int32), gu, down)


def test_parts_refuse_sizes_that_do_not_fit():
    from jax_llm_examples_b200.parts import DifferentialAttention, GatedPagedAttention

    ok = dict(heads=2, kv_heads=1, dim=4, value_dim=6, scale=0.5, eps=1e-6, map_weight=0.4, diff=0.4)
    w_in, w_o = torch.zeros(2 * 2 * 4 + 2 * 4 + 6, 8), torch.zeros(8, 12)
    DifferentialAttention(w_in, w_o, **ok)
    for change, word in (({"heads": 3}, "do not fit"), ({"in_bias": torch.zeros(5)}, "bias"), ({"rot_dims": 6, "inv_freq": torch.zeros(3)}, "rotated"),
                         ({"padded_dim": 7}, "padded"), ({"keep_first": -1, "window": 4}, "kept")):
        with pytest.raises(ValueError, match=word):
            DifferentialAttention(w_in, w_o, **{**ok, **change})
    with pytest.raises(ValueError, match="kept"):
        GatedPagedAttention(torch.zeros(8 + 4 + 4, 8), torch.zeros(8, 8), 2, 1, 4, 4, 0.5, 1e-6, gate="none", chunk=8, keep_first=2)


# ------------------------------------------------------------------------- the plain implementation against itself
def test_plain_mask_by_counting():
    for T, size, keep in ((12, 4, 2), (9, 1, 3), (7, 10, 0), (15, 3, 8)):
        m = plain.window_with_kept_start(T, size, keep)
        for i in range(T):
            for j in range(T):
                assert bool(m[i, j]) == (j <= i and (i - size < j or j in range(keep)))


def test_plain_rotation_is_a_turn_in_the_plane_and_its_scaling_keeps_and_stretches():
    torch.manual_seed(0)
    x, pos = torch.randn(5, 2, 10, dtype=F64), torch.tensor([0, 1, 7, 100, 3000])
    y = plain.rotate_half(x, pos, 500.0, 6)
    for i in range(3):
        z = torch.complex(x[..., i], x[..., i + 3]) * torch.polar(torch.ones(5, dtype=F64), pos.to(F64) * 500.0 ** (-i / 3))[:, None]
        assert torch.allclose(y[..., i], z.real) and torch.allclose(y[..., i + 3], z.imag)
    assert torch.equal(y[..., 6:], x[..., 6:])
    sc = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}
    f, amp = plain.stretched_frequencies(10000.0, 32, sc)
    raw, one = plain.stretched_frequencies(10000.0, 32)
    assert one == 1.0 and abs(amp - (1 + 0.1 * math.log(4.0))) < 1e-15
    assert f[0] == raw[0] and abs(f[-1] - raw[-1] / 4) < 1e-18 and all(raw[i] / 4 <= f[i] <= raw[i] for i in range(16))
    turned = plain.rotate_half(x, pos, 500.0, 6, {**sc, "factor": 8.0})
    assert torch.allclose(turned[..., :6].norm(dim=-1), x[..., :6].norm(dim=-1) * (1 + 0.1 * math.log(8.0)))


def test_plain_frequencies_are_the_products():
    from jax_llm_examples_b200.parts import yarn_frequencies

    for base, dims, sc in ((10000.0, 64, (4.0, 2048, 32.0, 1.0)), (500.0, 10, (2.0, 30, 4.0, 2.0)), (300.0, 2, (8.0, 16, 2.0, 2.0))):
        f, a = yarn_frequencies(base, dims, sc[0], sc[1], sc[2], sc[3])
        g, b = plain.stretched_frequencies(base, dims, dict(zip(("factor", "original", "fast", "slow"), sc)))
        assert torch.allclose(f.double(), torch.tensor(g, dtype=F64), rtol=1e-6) and abs(a - b) < 1e-12


def test_plain_attention_with_one_map_switched_off_is_ordinary_attention():
    """lambda = 0: the head is map 1 alone, normed; and a difference written out score by score."""
    torch.manual_seed(1)
    T, D, eps, m = 9, 6, 1e-5, {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5, "scale": 0.7, "diff": 0.25, "mask": {"size": 4, "keep_first": 1}}
    g = lambda *s: torch.randn(*s, dtype=F64)  # noqa: E731
    P = {"q": g(24, D), "q.b": g(24), "k": g(12, D), "k.b": g(12), "v": g(10, D), "v.b": g(10), "o": torch.eye(20, dtype=F64),
         "lq1": g(3), "lk1": g(3), "lq2": g(3), "lk2": g(3)}
    h = g(T, D)
    q, k, v = h @ P["q"].T + P["q.b"], h @ P["k"].T + P["k.b"], h @ P["v"].T + P["v.b"]
    lam = math.exp(float(P["lq1"] @ P["lk1"])) - math.exp(float(P["lq2"] @ P["lk2"])) + 0.25
    out = plain.differential_attention(h, P, "", m, eps)
    for i in (0, 3, 8):
        for a in range(4):
            ms = []
            for c in (0, 1):
                seen = [j for j in range(i + 1) if i - j < 4 or j < 1]
                e = [math.exp(0.7 * float(q[i, (2 * a + c) * 3:(2 * a + c + 1) * 3] @ k[j, (2 * (a // 2) + c) * 3:(2 * (a // 2) + c + 1) * 3])) for j in seen]
                ms.append(sum(w * v[j, (a // 2) * 5:(a // 2 + 1) * 5] for w, j in zip(e, seen)) / sum(e))
            o = ms[0] - lam * ms[1]
            want = 0.75 * o / math.sqrt(float(o @ o) / 5 + eps)
            assert torch.allclose(out[i, a * 5:(a + 1) * 5], want)
    zero = dict(P, lq1=torch.zeros(3, dtype=F64), lq2=torch.zeros(3, dtype=F64))
    assert float(plain.map_weight(zero, "", 0.0)) == 0.0


def test_plain_table_experts_by_hand():
    torch.manual_seed(2)
    P = {f"e{e}.{n}": torch.randn(*((4, 3) if n != "down" else (3, 4)), dtype=F64) for e in range(4) for n in ("gate", "up", "down")}
    P["table"] = torch.tensor([[0, 3], [2, 1], [1, 3]], dtype=torch.int32)
    h, toks = torch.randn(4, 3, dtype=F64), [2, 0, 2, 1]
    out = plain.table_experts(h, toks, P, "", {"router": {"experts": 4, "top": 2}})
    for t, tok in enumerate(toks):
        a, b = P["table"][tok].tolist()
        assert torch.allclose(out[t], (plain.gated_unit(h[t], P, f"e{a}.") + plain.gated_unit(h[t], P, f"e{b}.")) / 2)


def test_plain_shared_layers_equal_copies_of_their_tensors(tmp_path):
    cfg, P = SX.plain_model(str(SX.make_dir(tmp_path / "m", "small", seed=3)))
    flat = json.loads(json.dumps(cfg))
    Q = dict(P)
    for i, L in enumerate(flat["layers"]):
        if L.pop("weights_of", None) is not None:
            Q.update({n.replace("l0.", f"l{i}.", 1): t for n, t in P.items() if n.startswith("l0.")})
    toks = [3, 17, 60, 0, 5, 5, 44, 9, 31, 2, 8]
    assert torch.equal(plain.forward(cfg, P, toks), plain.forward(flat, Q, toks))
    assert float(plain.forward(cfg, P, toks).abs().max()) < 4.0  # the cap
