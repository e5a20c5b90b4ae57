"""A plain, slow statement of the Momuvik decoder in float64 NumPy: one function per mechanism,
whole sequences from position 0.  It shares nothing with the package: it reads the raw
``config.json`` dictionary and a dictionary of arrays by tensor name.

Notation: ``h`` [T, width] is a sublayer's input, ``W`` [out, in] is applied as ``h @ W.T``.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import numpy as np

F = np.float64
SLOPE = 1.702          # of the clamped gate's sigmoid


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -np.asarray(z, F)))


def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_around_zero(x, w, eps):
    """The layers' norm: the stored number is what the gain has beyond one."""
    return unit_rms(x, eps) * (1.0 + w)


def norm_plain(x, w, eps):
    """The latents' norm: the stored number is the gain."""
    return unit_rms(x, eps) * w


def rotate_halves(x, pos, dims: int, base: float):
    """Turn the pairs (i, i + dims/2), i < dims/2, of the last axis by pos * base^(-2i/dims);
    channels from ``dims`` on pass unchanged."""
    half = dims // 2
    ang = np.asarray(pos, F)[:, None] * F(base) ** (-2.0 * np.arange(half) / dims)
    c, s = np.cos(ang), np.sin(ang)
    while c.ndim < x.ndim:
        c, s = c[:, None], s[:, None]
    out = np.array(x, F)
    a, b = x[..., :half], x[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


def softmax_with_sink(s, sink):
    """Weights along the last axis of s [H, i, j] (-inf: not seen), with exp(sink_h) in the sum."""
    top = np.maximum(s.max(axis=-1, keepdims=True), sink[:, None, None])
    e = np.exp(s - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink[:, None, None] - top))


def latent_keys(h, t, p, m, eps):
    """What a token leaves behind for later ones: its normed latent and its rotated key part."""
    r = m["kv_rank"]
    both = h @ t[p + "dkv"].T
    k_rot = both[:, r:]
    if m.get("rot") is not None:
        k_rot = rotate_halves(k_rot, np.arange(h.shape[0]), m["rot"]["dims"], m["rot"]["base"])
    return norm_plain(both[:, :r], t[p + "dkv.norm"], eps), k_rot


def latent_queries(h, t, p, m, eps):
    T, H, d, r = h.shape[0], m["heads"], m["dim"], m.get("rot_dim") or 0
    q = norm_plain(h @ t[p + "dq"].T, t[p + "dq.norm"], eps) @ t[p + "uq"].T
    q = q.reshape(T, H, d + r)
    q_rot = q[..., d:]
    if m.get("rot") is not None:
        q_rot = rotate_halves(q_rot, np.arange(T), m["rot"]["dims"], m["rot"]["base"])
    return q[..., :d], q_rot


def latent_attention(h, t: Dict[str, np.ndarray], p: str, m: dict, eps: float):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    c, k_rot = latent_keys(h, t, p, m, eps)
    q_plain, q_rot = latent_queries(h, t, p, m, eps)
    k_plain = (c @ t[p + "uk"].T).reshape(T, H, d)
    val = (c @ t[p + "uv"].T).reshape(T, H, dv)
    s = np.einsum("ihd,jhd->hij", q_plain, k_plain) + np.einsum("ihd,jd->hij", q_rot, k_rot)
    s = s * float(m["scale"])
    s = np.where(np.tril(np.ones((T, T), bool))[None], s, -np.inf)
    w = softmax_with_sink(s, t[p + "sink"])
    return np.einsum("hij,jhd->ihd", w, val).reshape(T, H * dv) @ t[p + "o"].T


# --------------------------------------------------------------------------------------------
def gated_silu(h, t, p: str):
    g = h @ t[p + "gate"].T
    return (g * sigmoid(g) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def clamped_expert(h, t, p: str, limit: float):
    """The gate bounded above, the other half on both sides and one added to it."""
    g = np.minimum(h @ t[p + "gate"].T, limit)
    u = np.clip(h @ t[p + "up"].T, -limit, limit)
    return (g * sigmoid(SLOPE * g) * (u + 1.0)) @ t[p + "down"].T


def choose(z, top: int):
    """Per row of router outputs: the ``top`` largest (the lowest index among equals) and their
    weights, each the sigmoid of its own output."""
    ids = np.argsort(-z, axis=1, kind="stable")[:, :top]
    return ids, sigmoid(np.take_along_axis(z, ids, axis=1))


def routed_experts(h, t, p: str, mlp: dict, margins: Optional[list] = None):
    """A chosen expert sees its weight times the token's input.  ``margins`` collects, per token,
    how far the last chosen router output lies above the best one that was not chosen."""
    E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    z = h @ t[p + "router"].T
    if margins is not None and top < E:
        ordered = -np.sort(-z, axis=1)
        margins.append(ordered[:, top - 1] - ordered[:, top])
    ids, w = choose(z, top)
    out = np.zeros((h.shape[0], t[p + "e0.down"].shape[0]), F)
    for i in range(h.shape[0]):
        for e, we in zip(ids[i], w[i]):
            out[i] += clamped_expert(we * h[i:i + 1], t, f"{p}e{int(e)}.",
                                     float(mlp["expert"]["limit"]))[0]
    if mlp.get("shared") is not None:
        out += clamped_expert(h, t, p + "shared.", float(mlp["shared"]["limit"]))
    return out


def feed_forward(h, t, p: str, mlp: dict, margins: Optional[list] = None):
    if mlp["kind"] == "dense":
        return gated_silu(h, t, p)
    return routed_experts(h, t, p, mlp, margins)


# --------------------------------------------------------------------------------------------
def tensors_of(cfg: dict, i: int) -> int:
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = int(cfg["layers"][i]["weights_of"])
    return i


def forward(cfg: dict, tensors: Dict[str, np.ndarray], tokens,
            layers_out: Optional[List[np.ndarray]] = None, margins: Optional[list] = None):
    """Logits [T, vocab] of a whole sequence from position 0.  ``layers_out`` collects the
    residual stream behind every layer, ``margins`` the routers' margins per token."""
    t = {k: np.asarray(v, F) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    mult = float(cfg.get("residual_mult", 1.0))
    x = t["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{tensors_of(cfg, i)}."
        h = norm_around_zero(x, t[p + "norm1"], eps)
        x = x + mult * latent_attention(h, t, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            h = norm_around_zero(x, t[p + "norm2"], eps)
            x = x + mult * feed_forward(h, t, p + "mlp.", layer["mlp"], margins)
        if layers_out is not None:
            layers_out.append(x.copy())
    return norm_around_zero(x, t["final.norm"], eps) @ t["embed"].T
