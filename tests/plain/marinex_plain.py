"""A plain, slow Marinex: one function per mechanism, float64 on the CPU, every score of a sequence made in full.

It shares nothing with the package: its own config reading (plain dictionaries), its own safetensors reader, its own
formulas.  ``forward`` runs whole sequences; the tests compare the engine's logits, however its steps were cut, with these.

Notation: h [T, D] rows of one sequence; W [out, in] applied as ``h @ W.T``; P maps tensor names to float64 tensors.
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


def gelu_exact(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def frequencies(base, dims):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)


def turn(u, v, a):
    """The pair (u, v) turned by the angle a."""
    return u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)


def rotate_pairs(x, positions, base, dims):
    """x [T, heads, d]: entries 2i and 2i + 1 turn together, i < dims/2; entries from ``dims`` on pass unchanged."""
    y = x.clone()
    f = frequencies(base, dims)
    for i in range(dims // 2):
        a = (positions.to(F64) * f[i])[:, None]
        y[..., 2 * i], y[..., 2 * i + 1] = turn(x[..., 2 * i], x[..., 2 * i + 1], a)
    return y


def rotate_half(x, positions, base, dims):
    """x [T, heads, d]: entries i and i + dims/2 turn together, i < dims/2; entries from ``dims`` on pass unchanged."""
    y = x.clone()
    f, half = frequencies(base, dims), dims // 2
    for i in range(half):
        a = (positions.to(F64) * f[i])[:, None]
        y[..., i], y[..., i + half] = turn(x[..., i], x[..., i + half], a)
    return y


def causal_mask(T, window=None):
    """Query i sees key j <= i, with a window only the last ``window`` of them (itself included)."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    return (j <= i) if window is None else (j <= i) & (i - j < window)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_with_sink(s, mask, sink):
    """Weights exp(s_j) / (exp(sink) + sum_i exp(s_i)) over the visible j; s [T, T], ``sink`` a number."""
    s = s.masked_fill(~mask, -math.inf)
    m = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(float(sink) - m))


# ------------------------------------------------------------------------------------------------------ mixers
def attention_scores(q, k, scale, temp, cap):
    """One head's scores [T, T] before the mask: scaled, times the head's number, soft-capped (``cap`` None: not)."""
    s = (q @ k.T) * scale * temp
    return s if cap is None else soft_cap(s, cap)


def attention_mixer(h, P, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rms_norm((h @ P[p + "q"].T).view(T, H, d), P[p + "q.norm"], eps)
    k = rms_norm((h @ P[p + "k"].T).view(T, G, d), P[p + "k.norm"], eps)
    v = rms_divide((h @ P[p + "v"].T).view(T, G, dv), eps)
    rot = m.get("rot")
    if rot:
        q, k = rotate_pairs(q, pos, rot["base"], rot["dims"]), rotate_pairs(k, pos, rot["base"], rot["dims"])
    mask = causal_mask(T, m["mask"]["size"] if m.get("mask") else None)
    out = []
    for a in range(H):
        g = a // (H // G)
        s = attention_scores(q[:, a], k[:, g], m["scale"], P[p + "temp"][a], m.get("softcap"))
        out.append(softmax_with_sink(s, mask, 0.0) @ v[:, g])
    return torch.cat(out, dim=-1) @ P[p + "o"].T


def latent_attention_mixer(h, P, p, m, eps):
    T = h.shape[0]
    H, dn, dr, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    c_q = rms_norm(h @ P[p + "dq"].T, P[p + "dq.norm"], eps)
    q = (c_q @ P[p + "uq"].T).view(T, H, dn + dr)
    down = h @ P[p + "dkv"].T
    c = rms_norm(down[:, :rank], P[p + "dkv.norm"], eps)
    rot = m["rot"]
    k_rot = rotate_half(down[:, None, rank:], pos, rot["base"], rot["dims"])[:, 0]
    q_rot = rotate_half(q[..., dn:], pos, rot["base"], rot["dims"])
    k = (c @ P[p + "uk"].T).view(T, H, dn)
    v = (c @ P[p + "uv"].T).view(T, H, dv)
    mask = causal_mask(T, m["mask"]["size"] if m.get("mask") else None)
    gate = torch.sigmoid(h @ P[p + "g"].T)
    out = []
    for a in range(H):
        s = (q[:, a, :dn] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        out.append(softmax_with_sink(s, mask, P[p + "sink"][a]) @ v[:, a] * gate[:, a:a + 1])
    return torch.cat(out, dim=-1) @ P[p + "o"].T


# ------------------------------------------------------------------------------------------------ feed-forward
def route(h, P, p, r):
    """(chosen [T, top], all scores [T, experts]): sigmoid scores; the choice is made on score + correction, among the
    kept groups only (a group's score: the sum of its two largest choice scores)."""
    s = torch.sigmoid(h @ P[p + "router"].T)
    choice = s + P[p + "correction"]
    E = r["experts"]
    groups = r.get("groups")
    if groups:
        per = E // groups["count"]
        parts = choice.view(-1, groups["count"], per)
        best = parts.topk(min(2, per), dim=-1).values.sum(-1)
        keep = torch.topk(best, groups["keep"], dim=-1).indices
        allowed = torch.zeros_like(best, dtype=torch.bool).scatter_(1, keep, True)
        choice = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf)
    return torch.topk(choice, r["top"], dim=-1).indices, s


def expert(h, P, p):
    return gelu_exact(h @ P[p + "up"].T) @ P[p + "down"].T


def expert_mixture(h, P, p, ml, forced=None):
    """Returns (output, the experts used [T, top], the experts this router chose itself).  ``forced`` [T, top] replaces
    the choice (the tests hand over the engine's, where two scores nearly tie); the weights are this router's."""
    own, s = route(h, P, p, ml["router"])
    chosen = own if forced is None else forced.to(torch.int64)
    w = torch.gather(s, 1, chosen)
    out = torch.zeros_like(h)
    for e in range(ml["router"]["experts"]):
        t, j = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            out.index_add_(0, t, w[t, j][:, None] * expert(h[t], P, f"{p}e{e}."))
    return out, chosen, own


# ------------------------------------------------------------------------------------------------- the decoder
MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer}


def forward(cfg: dict, P: dict, tokens, forced_choices=None, trace=None):
    """Logits [T, vocab] of one sequence.  ``forced_choices``: {layer: chosen [T, top]}; ``trace``: a list that gets
    (the residual rows after the layer, the experts used, the experts its router chose itself) for every layer."""
    eps = cfg["norm"]["eps"]
    x = P["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + rms_norm(MIXERS[L["type"]](x, P, p + "mix.", L["mixer"], eps), P[p + "norm1"], eps)
        used = own = None
        if L.get("mlp"):
            y, used, own = expert_mixture(x, P, p + "mlp.", L["mlp"], None if forced_choices is None else forced_choices.get(i))
            x = x + rms_norm(y, P[p + "norm2"], eps)
        if trace is not None:
            trace.append((x, used, own))
    return rms_norm(x, P["final.norm"], eps) @ P["head"].T
