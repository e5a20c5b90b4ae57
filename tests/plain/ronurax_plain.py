"""A plain, slow statement of the Ronurax decoder in float64 NumPy: one function per mechanism,
whole sequences from position 0.  It shares nothing with the package: it reads the raw
``config.json`` dictionary and a dictionary of arrays by tensor name.

Notation: ``h`` [T, width] is a sublayer's input, ``W`` [out, in] is applied as ``h @ W.T``.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import numpy as np

F = np.float64


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -np.asarray(z, F)))


def centred_norm(x, w, b, eps):
    """Layer norm along the last axis: centred, over its standard deviation, gain and offset."""
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * w + b


def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


# ---- rotation ------------------------------------------------------------------------------
def plain_frequencies(dims: int, base: float):
    return np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], F)


def banded_frequencies(dims: int, base: float, factor, low, high, original):
    """Frequencies divided by ``factor`` where their wavelength is long, kept where it is short,
    and blended in between (the bands' edges are original/low and original/high)."""
    out = []
    for f in plain_frequencies(dims, base):
        length = 2.0 * math.pi / f
        if length < original / high:
            out.append(f)
        elif length > original / low:
            out.append(f / factor)
        else:
            s = (original / length - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return np.array(out, F)


def ramped_frequencies(dims: int, base: float, factor, original, fast, slow):
    """Frequencies divided by ``factor`` along a ramp over their index, and the factor on cosine
    and sine.  The ramp starts at the index that makes ``fast`` turns within ``original``
    positions and ends at the one that makes ``slow``."""
    index_of = lambda turns: dims * math.log(original / (turns * 2.0 * math.pi)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return np.array(out, F), 0.1 * math.log(factor) + 1.0


def rotate_halves(x, pos, freq, mult: float = 1.0):
    """Turn the pairs (i, i + n), i < n = len(freq), of the last axis of x [T, ..., dim] by
    pos * freq[i], cosine and sine times ``mult``; channels from 2n on pass unchanged."""
    n = len(freq)
    ang = np.asarray(pos, F)[:, None] * freq
    c, s = mult * np.cos(ang), mult * np.sin(ang)
    while c.ndim < x.ndim:
        c, s = c[:, None], s[:, None]
    out = np.array(x, F)
    u, v = x[..., :n], x[..., n:2 * n]
    out[..., :n] = u * c - v * s
    out[..., n:2 * n] = v * c + u * s
    return out


# ---- attention -----------------------------------------------------------------------------
def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def chunk_mask(T: int, size: Optional[int]):
    """[i, j]: key j is not later than query i and in the same chunk of ``size`` positions."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    seen = j <= i
    return seen if size is None else seen & (i // size == j // size)


def mixing_weight(t: Dict[str, np.ndarray], p: str, diff: float) -> float:
    """The weight of the second map: one number per layer."""
    return float(np.exp(np.sum(t[p + "lq1"] * t[p + "lk1"]))
                 - np.exp(np.sum(t[p + "lq2"] * t[p + "lk2"])) + diff)


def two_map_heads(h, t: Dict[str, np.ndarray], p: str, m: dict, eps: float):
    """Queries [T, H, 2, d] and keys [T, G, 2, d] (normed per map, rotated), values [T, G, dv]."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ t[p + "q"].T + t[p + "q.b"]).reshape(T, H, 2, d)
    k = (h @ t[p + "k"].T + t[p + "k.b"]).reshape(T, G, 2, d)
    v = (h @ t[p + "v"].T + t[p + "v.b"]).reshape(T, G, dv)
    q = unit_rms(q, eps) * t[p + "q.norm"]
    k = unit_rms(k, eps) * t[p + "k.norm"]
    rot = m.get("rot")
    if rot is not None:
        sc = rot.get("scaling")
        freq = plain_frequencies(rot["dims"], rot["base"]) if sc is None else banded_frequencies(
            rot["dims"], rot["base"], sc["factor"], sc["low"], sc["high"], sc["original"])
        q, k = rotate_halves(q, np.arange(T), freq), rotate_halves(k, np.arange(T), freq)
    return q, k, v


def two_map_combine(a1, a2, weight: float, diff: float, eps: float):
    """The heads' outputs [T, H, dv] from those of the two maps."""
    return unit_rms(a1 - weight * a2, eps) * (1.0 - diff)


def differential_attention(h, t: Dict[str, np.ndarray], p: str, m: dict, eps: float):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = two_map_heads(h, t, p, m, eps)
    k, v = np.repeat(k, H // G, axis=1), np.repeat(v, H // G, axis=1)
    seen = chunk_mask(T, None if m.get("mask") is None else int(m["mask"]["size"]))
    s = np.einsum("ihmd,jhmd->mhij", q, k) * float(m["scale"])
    a = np.einsum("mhij,jhd->mihd", softmax(np.where(seen, s, -np.inf)), v)
    o = two_map_combine(a[0], a[1], mixing_weight(t, p, float(m["diff"])), float(m["diff"]), eps)
    return o.reshape(T, -1) @ t[p + "o"].T


def latent_rotation(x, pos, m: dict):
    """The rotation of the rotated parts x [T, ..., rot_dim]."""
    rot = m.get("rot")
    if rot is None:
        return x
    sc = rot.get("scaling")
    if sc is None:
        return rotate_halves(x, pos, plain_frequencies(rot["dims"], rot["base"]))
    freq, mult = ramped_frequencies(rot["dims"], rot["base"], sc["factor"], sc["original"],
                                    sc["fast"], sc["slow"])
    return rotate_halves(x, pos, freq, mult)


def latent_keys(h, t, p, m, eps):
    """What a token leaves behind for later ones: its normed latent and its rotated key part."""
    both = h @ t[p + "dkv"].T
    c = unit_rms(both[:, :m["kv_rank"]], eps) * t[p + "dkv.norm"]
    return c, latent_rotation(both[:, m["kv_rank"]:], np.arange(h.shape[0]), m)


def latent_attention(h, t: Dict[str, np.ndarray], p: str, m: dict, eps: float):
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (h @ t[p + "q"].T).reshape(T, H, d + r)
    q_plain, q_rot = q[..., :d], latent_rotation(q[..., d:], np.arange(T), m)
    c, k_rot = latent_keys(h, t, p, m, eps)
    k_plain = (c @ t[p + "uk"].T).reshape(T, H, d)
    val = (c @ t[p + "uv"].T).reshape(T, H, dv)
    s = np.einsum("ihd,jhd->hij", q_plain, k_plain) + np.einsum("ihd,jd->hij", q_rot, k_rot)
    w = softmax(np.where(chunk_mask(T, None), s * float(m["scale"]), -np.inf))
    o = np.einsum("hij,jhd->ihd", w, val).reshape(T, H * dv)
    return (o * sigmoid(h @ t[p + "g"].T)) @ t[p + "o"].T


# ---- routed experts ------------------------------------------------------------------------
def expert(h, t, p: str):
    g = h @ t[p + "gate"].T
    return (g * sigmoid(g) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def choose(scores, top: int, count: int, keep: int):
    """Per row of scores [T, E]: the ``top`` largest among the experts of the ``keep`` best of
    ``count`` groups of neighbours, a group's score being its largest (the lowest index among
    equals)."""
    T, E = scores.shape
    best = scores.reshape(T, count, E // count).max(axis=2)
    groups = np.argsort(-best, axis=1, kind="stable")[:, :keep]
    ids = np.empty((T, top), int)
    for i in range(T):
        open_to = [e for e in range(E) if e // (E // count) in groups[i]]
        ids[i] = sorted(open_to, key=lambda e: (-scores[i, e], e))[:top]
    return ids


def choice_margin(z, top: int, count: int, keep: int):
    """Per row of router outputs, by how much they would have to change for another choice: the
    distance of the last chosen expert to the best one left out in the kept groups and, when the
    last kept group holds a chosen expert, of that group to the first one left out."""
    T, E = z.shape
    size = E // count
    best = z.reshape(T, count, size).max(axis=2)
    ids = choose(z, top, count, keep)
    least = np.full(T, np.inf)
    for i in range(T):
        order = np.argsort(-best[i], kind="stable")
        if keep < count and (ids[i] // size == order[keep - 1]).any():
            least[i] = best[i, order[keep - 1]] - best[i, order[keep]]
        left = [z[i, e] for e in range(E) if e // size in order[:keep] and e not in ids[i]]
        if left:
            least[i] = min(least[i], z[i, ids[i, -1]] - max(left))
    return least


def routed_experts(h, t, p: str, mlp: dict, margins: Optional[list] = None):
    r = mlp["router"]
    top, groups = int(r["top"]), r.get("groups") or {"count": 1, "keep": 1}
    z = h @ t[p + "router"].T
    s = softmax(z)
    ids = choose(s, top, int(groups["count"]), int(groups["keep"]))
    if margins is not None:
        margins.append(choice_margin(z, top, int(groups["count"]), int(groups["keep"])))
    out = np.zeros((h.shape[0], t[p + "e0.down"].shape[0]), F)
    for e in range(int(r["experts"])):
        rows = np.nonzero((ids == e).any(axis=1))[0]
        if len(rows):
            out[rows] += s[rows, e][:, None] * expert(h[rows], t, f"{p}e{e}.")
    return out


# --------------------------------------------------------------------------------------------
def tensors_of(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


MIXERS = {"attention": differential_attention, "latent_attention": latent_attention}


def forward(cfg: dict, tensors: Dict[str, np.ndarray], tokens,
            layers_out: Optional[List[np.ndarray]] = None, margins: Optional[list] = None):
    """Logits [T, vocab] of a whole sequence from position 0.  ``layers_out`` collects the
    residual stream behind every layer, ``margins`` the routers' margins per token."""
    t = {k: np.asarray(v, F) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    norm = lambda x, name: centred_norm(x, t[name], t[name + ".b"], eps)
    x = t["embed"][np.asarray(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{tensors_of(cfg, i)}."
        x = x + MIXERS[layer["type"]](norm(x, p + "norm1"), t, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + routed_experts(norm(x, p + "norm2"), t, p + "mlp.", layer["mlp"], margins)
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm(x, "final.norm") @ t["head"].T
