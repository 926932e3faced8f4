"""A plain, slow Samerax: one function per mechanism, float64 on the CPU, every score of a sequence made in full.

It shares nothing with the package: its own config reading (plain dictionaries), its own safetensors reader, its own
formulas.  ``forward`` runs whole sequences; the tests compare the engine's logits, however its steps were cut, with these.

Notation: h [T, D] rows of one sequence; W [out, in] applied as ``h @ W.T``; P maps tensor names to float64 tensors
(integer tables stay integers).
"""

from __future__ import annotations

import json
import math
import struct
from pathlib import Path

import torch

F64 = torch.float64


def read_safetensors(path) -> dict:
    """name -> float64 tensor (integers stay integers): 8 bytes of header length, a JSON header, then the data."""
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    types = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "F64": torch.float64, "I32": torch.int32,
             "I64": torch.int64}
    out = {}
    for name, meta in header.items():
        if name == "__metadata__":
            continue
        lo, hi = meta["data_offsets"]
        t = torch.frombuffer(bytearray(raw[8 + n + lo:8 + n + hi]), dtype=types[meta["dtype"]]).reshape(meta["shape"])
        out[name] = t.to(F64) if t.is_floating_point() else t
    return out


# ------------------------------------------------------------------------------------------------ small pieces
def rms_divide(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_divide(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def stretched_frequencies(base, dims, scaling=None):
    """(turn per position of every pair, factor on cosine and sine).  ``scaling``: factor, original, fast, slow; pairs
    below lo keep their frequency, pairs from hi on have it divided by the factor, a straight ramp between."""
    plain = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return plain, 1.0
    s = float(scaling["factor"])

    def place(turns):
        return dims * math.log(scaling["original"] / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(place(scaling["fast"])), 0), min(math.ceil(place(scaling["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(max((i - lo) / max(hi - lo, 1e-3), 0.0), 1.0)
        out.append(r * (f / s) + (1.0 - r) * f)
    return out, 1.0 + 0.1 * math.log(s)


def rotate_half(x, positions, base, dims, scaling=None):
    """x [T, heads, d]: entries i and i + dims/2 turn together by positions * f_i, i < dims/2; the rest pass unchanged."""
    y = x.clone()
    freqs, amp = stretched_frequencies(base, dims, scaling)
    half = dims // 2
    for i, f in enumerate(freqs):
        a = (positions.to(F64) * f)[:, None]
        u, v = x[..., i], x[..., i + half]
        y[..., i] = amp * (u * torch.cos(a) - v * torch.sin(a))
        y[..., i + half] = amp * (v * torch.cos(a) + u * torch.sin(a))
    return y


def window_with_kept_start(T, size, keep):
    """Query i sees key j <= i that is less than ``size`` back or among the sequence's first ``keep``."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def masked_softmax(s, mask):
    return torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1)


# ------------------------------------------------------------------------------------------------------- mixer
def map_weight(P, p, diff):
    """lambda: how much of the second map's output is taken off the first's."""
    return torch.exp((P[p + "lq1"] * P[p + "lk1"]).sum()) - torch.exp((P[p + "lq2"] * P[p + "lk2"]).sum()) + diff


def difference_of_maps(a1, a2, lam, diff, eps):
    """One head's output [T, vdim] from its two maps' outputs."""
    return rms_divide(a1 - lam * a2, eps) * (1.0 - diff)


def differential_attention(h, P, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ P[p + "q"].T + P[p + "q.b"]).view(T, H * 2, d)
    k = (h @ P[p + "k"].T + P[p + "k.b"]).view(T, G * 2, d)
    v = (h @ P[p + "v"].T + P[p + "v.b"]).view(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q = rotate_half(q, pos, rot["base"], rot["dims"], rot.get("scaling"))
        k = rotate_half(k, pos, rot["base"], rot["dims"], rot.get("scaling"))
    mask = window_with_kept_start(T, m["mask"]["size"], m["mask"].get("keep_first", 0)) if m.get("mask") else window_with_kept_start(T, T, 0)
    lam = map_weight(P, p, m["diff"])
    out = []
    for a in range(H):
        g = a // (H // G)
        maps = [masked_softmax(q[:, 2 * a + i] @ k[:, 2 * g + i].T * m["scale"], mask) @ v[:, g] for i in (0, 1)]
        out.append(difference_of_maps(maps[0], maps[1], lam, m["diff"], eps))
    return torch.cat(out, dim=-1) @ P[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_unit(h, P, p):
    return (silu(h @ P[p + "gate"].T) * (h @ P[p + "up"].T)) @ P[p + "down"].T


def table_experts(h, tokens, P, p, ml):
    """Every token id has its experts in a table; their outputs count alike."""
    top = ml["router"]["top"]
    chosen = P[p + "table"][torch.as_tensor(tokens, dtype=torch.long)].long()
    out = torch.zeros_like(h)
    for e in range(ml["router"]["experts"]):
        t, _ = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            out.index_add_(0, t, gated_unit(h[t], P, f"{p}e{e}.") / top)
    return out


# ------------------------------------------------------------------------------------------------- the decoder
def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg: dict, P: dict, tokens, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace``: a list that gets the residual rows after every layer."""
    eps = cfg["norm"]["eps"]
    x = P["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        x = x + differential_attention(rms_norm(x, P[p + "norm1"], eps), P, p + "mix.", L["mixer"], eps)
        ml = L.get("mlp")
        if ml:
            h = rms_norm(x, P[p + "norm2"], eps)
            x = x + (gated_unit(h, P, p + "mlp.") if ml["kind"] == "dense" else table_experts(h, tokens, P, p + "mlp.", ml))
        if trace is not None:
            trace.append(x)
    logits = rms_norm(x, P["final.norm"], eps) @ P["head"].T
    cap = cfg.get("logit_softcap")
    return logits if cap is None else soft_cap(logits, cap)
