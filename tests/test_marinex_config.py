"""Marinex without a GPU: the configuration reader, the tensor list, random model folders, how long a layer's pages live,
and the plain implementation against other ways of writing the same mathematics."""

import itertools
import json
import math

import pytest
import torch

from tests import marinex_helpers as MX
from tests.plain import marinex_plain as plain

F64 = torch.float64


def test_config_is_read_from_the_files_own_keys():
    from jax_llm_examples_b200.config.marinex import AttentionSpec, LatentAttentionSpec, MarinexConfig
    from jax_llm_examples_b200.config.registry import resolve

    cj = MX.config("small")
    arch = resolve(cj)
    assert arch.name == "Marinex"
    cfg = arch.parse_config(cj)
    assert isinstance(cfg, MarinexConfig) and (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps) == (61, 36, 1e-5)
    assert [type(L.mixer) for L in cfg.layers] == [AttentionSpec, LatentAttentionSpec, AttentionSpec, LatentAttentionSpec]
    a, b = cfg.layers[0].mixer, cfg.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.softcap, a.rot.base, a.rot.dims, a.window) == (6, 2, 10, 7, 0.5, 1.5, 60.0, 6, None)
    assert (b.heads, b.dim, b.rot_dim, b.vdim, b.q_rank, b.kv_rank, b.window, b.scale, b.rot.base) == (3, 5, 6, 9, 11, 13, 7, 0.3, 50.0)
    m = cfg.layers[0].mlp
    assert (m.experts, m.top, m.groups, m.keep, m.ff) == (6, 2, 3, 2, 14) and cfg.layers[3].mlp is None
    plainer = cfg.layers[1].mlp
    assert (plainer.groups, plainer.keep) == (1, 1)
    p = arch.parse_config(MX.config("padded"))
    assert p.layers[0].mixer.rot is None and p.layers[2].mixer.softcap is None and p.layers[3].mixer.window is None


@pytest.mark.parametrize("path, value, word", [
    (("layers", 0, "type"), "mamba", "no mixer"),
    (("layers", 0, "mixer", "kv_heads"), 4, "no multiple"),
    (("layers", 0, "mixer", "rot", "dims"), 5, "even"),
    (("layers", 0, "mixer", "rot", "dims"), 12, "at most"),
    (("layers", 0, "mixer", "softcap"), 0.0, "softcap"),
    (("layers", 1, "mixer", "rot", "dims"), 4, "rot_dim"),
    (("layers", 1, "mixer", "mask", "size"), 0, "mask.size"),
    (("layers", 1, "mixer", "kv_rank"), 0, "positive"),
    (("layers", 0, "mlp", "kind"), "dense", "moe"),
    (("layers", 0, "mlp", "router", "top"), 5, "top-5"),
    (("layers", 0, "mlp", "router", "groups", "count"), 4, "groups"),
    (("layers", 0, "mlp", "router", "groups", "keep"), 4, "groups"),
    (("norm", "eps"), 0.0, "eps"),
])
def test_config_errors_name_the_key(path, value, word):
    from jax_llm_examples_b200.config.base import ConfigError
    from jax_llm_examples_b200.config.marinex import MarinexConfig

    cj = MX.config("small")
    d = cj
    for k in path[:-1]:
        d = d[k]
    d[path[-1]] = value
    with pytest.raises(ConfigError, match=word):
        MarinexConfig.from_dict(cj)
    cj = MX.config("small")
    del cj["layers"][0]["mixer"]["scale"]
    with pytest.raises(ConfigError, match="scale"):
        MarinexConfig.from_dict(cj)


def test_tensor_list_and_random_folder(tmp_path):
    """A folder written from a configuration holds exactly the architecture's tensors, in the shapes the sizes give."""
    from jax_llm_examples_b200.config.registry import resolve
    from jax_llm_examples_b200.weights.loader import WeightError, load_tensors

    folder = MX.make_dir(tmp_path / "m", "small", seed=3)
    cj = json.loads((folder / "config.json").read_text())
    arch = resolve(cj)
    specs = arch.tensor_specs(arch.parse_config(cj))
    P = plain.read_safetensors(folder / "model.safetensors")
    assert set(P) == set(specs)
    assert P["embed"].shape == P["head"].shape == (61, 36) and not torch.equal(P["embed"], P["head"])
    assert P["l0.mix.q"].shape == (60, 36) and P["l0.mix.v"].shape == (14, 36) and P["l0.mix.temp"].shape == (6,)
    assert P["l0.mix.q.norm"].shape == (10,) and P["l0.mix.k.norm"].shape == (10,) and P["l0.mix.o"].shape == (36, 42)
    assert P["l1.mix.dq"].shape == (11, 36) and P["l1.mix.uq"].shape == (33, 11) and P["l1.mix.dkv"].shape == (19, 36)
    assert P["l1.mix.uk"].shape == (15, 13) and P["l1.mix.uv"].shape == (27, 13) and P["l1.mix.g"].shape == (3, 36)
    assert P["l1.mix.sink"].shape == (3,) and P["l1.mix.o"].shape == (36, 27)
    assert P["l0.mlp.router"].shape == (6, 36) and P["l0.mlp.correction"].shape == (6,) and P["l0.mlp.e5.down"].shape == (36, 14)
    assert "l3.norm1" in P and "l3.norm2" not in P and "l0.mlp.e6.up" not in P
    wrong = json.loads(json.dumps(cj))
    wrong["layers"][1]["mixer"]["heads"] = 2
    with pytest.raises(WeightError, match="wrong shapes"):
        load_tensors(folder, arch.tensor_specs(arch.parse_config(wrong)), None, torch.float32)


def test_what_a_layer_keeps_and_for_how_long():
    """Attention over all positions keeps two planes for good; windowed latent attention one row per token, as long as its
    window; no layer has per-request state."""
    from jax_llm_examples_b200.cache.manager import Retention
    from jax_llm_examples_b200.config.registry import resolve
    from jax_llm_examples_b200.parts import Runtime
    from jax_llm_examples_b200.weights.random_init import random_tensors

    def built(cj):
        arch = resolve(cj)
        cfg = arch.parse_config(cj)
        return arch.build(cfg, random_tensors(arch.tensor_specs(cfg), 1), Runtime(torch.float32, torch.device("cpu")))

    model = built(MX.config("small"))
    needs = [(c.num_kv_heads, c.head_dim, c.planes, c.retention) for c in model.plan.caches]
    assert needs == [(2, 10, 2, Retention.all()), (1, 19, 1, Retention.window(7)), (2, 11, 2, Retention.all()), (1, 12, 1, Retention.window(19))]
    assert model.plan.states == () and model.lm_head is not model.embedding and model.capturable
    padded = built(MX.config("padded"))
    assert padded.plan.caches[3].retention == Retention.all() and padded.plan.caches[1].retention == Retention.window(1)


# ------------------------------------------------------------------- the plain implementation against other forms
def test_plain_rotations_are_turns_in_the_plane():
    torch.manual_seed(0)
    x, pos = torch.randn(5, 2, 10, dtype=F64), torch.tensor([0, 1, 2, 7, 500])
    for fn, pair in ((plain.rotate_pairs, lambda i: (2 * i, 2 * i + 1)), (plain.rotate_half, lambda i: (i, i + 3))):
        y = fn(x, pos, 100.0, 6)
        assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
        for i in range(3):
            a, b = pair(i)
            z = torch.complex(x[..., a], x[..., b]) * torch.exp(1j * pos.to(F64) * 100.0 ** (-2 * i / 6))[:, None]
            assert torch.allclose(torch.complex(y[..., a], y[..., b]), z)


def test_plain_softmax_sink_cap_and_mask():
    """The sink is a key without a value (an extra column that is dropped); a cap leaves small scores alone and bounds large
    ones; the window counts the query itself."""
    torch.manual_seed(1)
    s = torch.randn(6, 6, dtype=F64) * 4
    mask = plain.causal_mask(6, 3)
    assert mask.sum(1).tolist() == [1, 2, 3, 3, 3, 3] and bool(mask[5, 3]) and not bool(mask[5, 2])
    for sink in (0.0, -2.5, 9.0):
        w = plain.softmax_with_sink(s, mask, sink)
        ext = torch.cat([s.masked_fill(~mask, -math.inf), torch.full((6, 1), sink, dtype=F64)], dim=1).softmax(-1)[:, :6]
        assert torch.allclose(w, ext)
    one_added = torch.exp(s).masked_fill(~mask, 0)
    assert torch.allclose(plain.softmax_with_sink(s, mask, 0.0), one_added / (1 + one_added.sum(-1, keepdim=True)))
    c = plain.soft_cap(torch.tensor([0.01, -0.01, 50.0, -900.0], dtype=F64), 5.0)
    assert torch.allclose(c, torch.tensor([0.01, -0.01, 5.0, -5.0], dtype=F64), atol=2e-7)


def test_plain_latent_attention_equals_its_absorbed_form():
    """Scores and sums taken against the latents themselves (queries through W_uk, outputs through W_uv): the same."""
    torch.manual_seed(2)
    m = MX.config("small")["layers"][1]["mixer"]
    H, dn, dr, dv, rank, D, T = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], 36, 17
    g = lambda *s: torch.randn(*s, dtype=F64) * 0.4  # noqa: E731
    P = {"m.dq": g(m["q_rank"], D), "m.dq.norm": 1 + g(m["q_rank"]), "m.uq": g(H * (dn + dr), m["q_rank"]), "m.dkv": g(rank + dr, D),
         "m.dkv.norm": 1 + g(rank), "m.uk": g(H * dn, rank), "m.uv": g(H * dv, rank), "m.sink": g(H), "m.g": g(H, D), "m.o": g(D, H * dv)}
    h, eps, pos = g(T, D), 1e-5, torch.arange(T)
    got = plain.latent_attention_mixer(h, P, "m.", m, eps)
    q = (plain.rms_norm(h @ P["m.dq"].T, P["m.dq.norm"], eps) @ P["m.uq"].T).view(T, H, dn + dr)
    down = h @ P["m.dkv"].T
    c = plain.rms_norm(down[:, :rank], P["m.dkv.norm"], eps)
    kr = plain.rotate_half(down[:, None, rank:], pos, 50.0, dr)[:, 0]
    qr = plain.rotate_half(q[..., dn:], pos, 50.0, dr)
    rows = []
    for i in range(T):
        heads = []
        for a in range(H):
            ql = P["m.uk"].view(H, dn, rank)[a].T @ q[i, a, :dn]
            js = list(range(max(0, i - 6), i + 1))
            w = torch.exp(torch.stack([(ql @ c[j] + qr[i, a] @ kr[j]) * m["scale"] for j in js]))
            lat = (w[:, None] * c[js]).sum(0) / (w.sum() + torch.exp(P["m.sink"][a]))
            heads.append(P["m.uv"].view(H, dv, rank)[a] @ lat / (1 + torch.exp(-(P["m.g"][a] @ h[i]))))
        rows.append(torch.cat(heads))
    assert torch.allclose(got, torch.stack(rows) @ P["m.o"].T)


def test_plain_router_by_brute_force():
    """Choices by trying every set: among the kept groups' experts the set with the largest sum of choice scores; groups by
    the sum of their two best; weights are the scores without the correction, as they are."""
    torch.manual_seed(3)
    D, r = 8, {"experts": 8, "top": 2, "groups": {"count": 4, "keep": 2}}
    P = {"m.router": torch.randn(8, D, dtype=F64), "m.correction": torch.randn(8, dtype=F64) - 1.0}  # choice scores mostly negative
    h = torch.randn(40, D, dtype=F64)
    chosen, s = plain.route(h, P, "m.", r)
    for t in range(40):
        sc = torch.sigmoid(P["m.router"] @ h[t])
        c = sc + P["m.correction"]
        kept = max(itertools.combinations(range(4), 2), key=lambda g: sum(float(c[2 * i] + c[2 * i + 1]) for i in g))
        usable = [e for e in range(8) if e // 2 in kept]
        best = max(itertools.combinations(usable, 2), key=lambda es: sum(float(c[e]) for e in es))
        assert sorted(chosen[t].tolist()) == sorted(best) and torch.allclose(s[t], sc)
    # a group with one large and one tiny score loses to a group with two middling ones
    P = {"m.router": torch.zeros(6, D, dtype=F64), "m.correction": torch.tensor([2.0, -5.0, -5.0, 0.5, 0.4, 0.0], dtype=F64)}
    chosen, _ = plain.route(h[:1], P, "m.", {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}})
    assert sorted(chosen[0].tolist()) == [3, 4]


def test_plain_block_norms_the_sublayers_outputs_only():
    """Scaling the mixer's and the experts' output products changes nothing but the eps term: the norms see to that; the
    sublayers read the rows as they are (scaling the embedding does change the result)."""
    import tempfile

    with tempfile.TemporaryDirectory() as d:
        folder = MX.make_dir(d, "padded", seed=5)
        cfg, P = MX.plain_model(str(folder))
        toks = [3, 1, 4, 1, 5, 9, 2, 6]
        a = plain.forward(cfg, P, toks)
        P2 = {k: v * (1e4 if k.endswith((".o", ".down")) else 1.0) for k, v in P.items()}
        P1 = {k: v * (1e2 if k.endswith((".o", ".down")) else 1.0) for k, v in P.items()}
        assert torch.allclose(plain.forward(cfg, P1, toks), plain.forward(cfg, P2, toks), rtol=1e-4, atol=1e-6)
        P3 = dict(P, embed=P["embed"] * 2)
        assert not torch.allclose(plain.forward(cfg, P3, toks), a, rtol=1e-2)
