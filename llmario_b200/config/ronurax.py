"""Typed configuration of the Ronurax decoder, read from the keys of its ``config.json``.

A Ronurax model is a list of pre-norm layers, ``x += mixer(norm1(x)); x += experts(norm2(x))``, whose
norms are layer norms with a gain and an offset.  The mixers are

* ``attention``: every head makes two attention maps over the same values and subtracts them with a
  learned weight (``diff``), grouped queries, biases, a norm per head and map, half-split rotation
  of a part of the channels with frequencies scaled by wavelength, and a mask of chunks;
* ``latent_attention``: keys and values through a low-rank latent, queries straight from the input,
  one rotated key part (half-split pairs, frequencies scaled by index) for all heads, every earlier
  key seen, a sigmoid gate per output channel.

The feed-forward is routed experts (silu-gated, softmax scores over all experts that are not
renormalised, a choice limited to the best groups) or absent.  A layer with ``weights_of: j`` runs
with layer j's tensors and a cache of its own.  Every size and constant that can differ between two
models of the design is read here and nowhere else; tensor names follow ``l<i>.<part>``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .pemolorn import _freeze_deep
from .runidra import _deep
from .spec import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec
from .vunasun import _get

MIXERS = ("attention", "latent_attention")
# the keys of rot.scaling per mixer, and the kind of the rotary part's scaling they stand for
SCALINGS = {"attention": ("bands", ("factor", "low", "high", "original")),
            "latent_attention": ("ramp", ("factor", "original", "fast", "slow"))}
# rows from which a step's kernels start in plain stream order (kernels.PAIR_MIN_ROWS)
ORDERED_ROWS = 512


@dataclass(frozen=True)
class RonuraxLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]
    mlp: Optional[Tuple[Tuple[str, Any], ...]]
    weights_of: Optional[int] = None

    def m(self) -> Dict[str, Any]:
        return _deep(dict(self.mixer))

    def f(self) -> Optional[Dict[str, Any]]:
        return None if self.mlp is None else _deep(dict(self.mlp))


@dataclass(frozen=True)
class RonuraxConfig:
    vocab: int
    width: int
    eps: float
    layers: Tuple[RonuraxLayer, ...]
    max_positions: int = 1 << 17      # the design has no limit of its own: the engine's default

    architecture = "Ronurax"
    model_type = "ronurax"

    # ---------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "RonuraxConfig":
        vocab = _get(raw, "vocab", int, "model")
        width = _get(raw, "width", int, "model")
        eps = _get(raw.get("norm"), "eps", float, "norm")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[RonuraxLayer] = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]"
            kind = e.get("type") if isinstance(e, dict) else None
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}: unsupported type {kind!r} "
                                  f"(known: {', '.join(MIXERS)})")
            m = e.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: {where}: missing 'mixer'")
            cls._check_mixer(kind, m, where + ".mixer")
            mlp = e.get("mlp")
            if mlp is not None:
                cls._check_mlp(mlp, where + ".mlp")
            of = e.get("weights_of")
            if of is not None and (isinstance(of, bool) or not isinstance(of, int)
                                   or not 0 <= of < len(entries) or of == i):
                raise ConfigError(f"config.json: {where}: weights_of {of!r} names no other layer")
            layers.append(RonuraxLayer(kind, _freeze_deep(m),
                                       None if mlp is None else _freeze_deep(mlp), of))
        max_pos = int(raw.get("max_positions") or cls.max_positions)
        out = cls(vocab, width, eps, tuple(layers), max_pos)
        for i, layer in enumerate(layers):
            owner = layers[out.owner(i)]
            if (owner.type, owner.mixer, owner.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ConfigError(f"config.json: layers[{i}] uses the weights of layer "
                                  f"{out.owner(i)}, whose sizes and constants differ from its own")
        return out

    @staticmethod
    def _check_mixer(kind: str, m: Dict[str, Any], where: str) -> None:
        sizes = ("heads", "kv_heads", "dim", "vdim") if kind == "attention" else \
            ("heads", "dim", "vdim", "kv_rank")
        for key in sizes:
            _get(m, key, int, where)
        _get(m, "scale", float, where)
        if kind == "attention":
            _get(m, "diff", float, where)
            if m["heads"] % m["kv_heads"]:
                raise ConfigError(f"config.json: {where}: {m['heads']} heads over "
                                  f"{m['kv_heads']} kv_heads")
            if m.get("mask") is not None and _get(m["mask"], "size", int, where + ".mask") < 1:
                raise ConfigError(f"config.json: {where}.mask: size must be positive")
            widest = m["dim"]
        else:
            widest = m.get("rot_dim") or 0
            if isinstance(widest, bool) or not isinstance(widest, int) or widest < 0:
                raise ConfigError(f"config.json: {where}: rot_dim {widest!r}")
        rot = m.get("rot")
        if rot is None:
            return
        dims = _get(rot, "dims", int, where + ".rot")
        _get(rot, "base", float, where + ".rot")
        if dims % 2 or dims > widest:
            raise ConfigError(f"config.json: {where}.rot: dims {dims} must be even and at most "
                              f"{widest}")
        if rot.get("scaling") is not None:
            for key in SCALINGS[kind][1]:
                if _get(rot["scaling"], key, float, where + ".rot.scaling") <= 0:
                    raise ConfigError(f"config.json: {where}.rot.scaling: {key} must be positive")

    @staticmethod
    def _check_mlp(mlp: Dict[str, Any], where: str) -> None:
        if mlp.get("kind", "moe") != "moe":
            raise ConfigError(f"config.json: {where}: unsupported mlp kind {mlp.get('kind')!r} "
                              "(known: moe)")
        r = mlp.get("router")
        n = _get(r, "experts", int, where + ".router")
        top = _get(r, "top", int, where + ".router")
        _get(mlp.get("expert"), "ff", int, where + ".expert")
        if top > n:
            raise ConfigError(f"config.json: {where}: top {top} of {n} experts")
        if r.get("groups") is not None:
            count = _get(r["groups"], "count", int, where + ".router.groups")
            keep = _get(r["groups"], "keep", int, where + ".router.groups")
            if count < 1 or n % count or not 1 <= keep <= count or keep * (n // count) < top:
                raise ConfigError(f"config.json: {where}: top {top} out of {keep} of {count} "
                                  f"groups of {n} experts")

    def to_dict(self) -> Dict[str, Any]:
        """The ``config.json`` that reads back as this configuration."""
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                               "width": self.width, "norm": {"eps": self.eps}, "layers": []}
        for layer in self.layers:
            e: Dict[str, Any] = {"type": layer.type, "mixer": layer.m(), "mlp": layer.f()}
            if layer.weights_of is not None:
                e["weights_of"] = layer.weights_of
            out["layers"].append(e)
        if self.max_positions != type(self).max_positions:
            out["max_positions"] = self.max_positions
        return out

    def owner(self, i: int) -> int:
        """The layer whose tensors layer i runs with (itself, when it names no other)."""
        seen = {i}
        while self.layers[i].weights_of is not None:
            i = self.layers[i].weights_of
            if i in seen:
                raise ConfigError(f"config.json: layers[{i}]: weights_of leads back to itself")
            seen.add(i)
        return i

    # ---------------------------------------------------------------------------------------
    def to_spec(self) -> ModelSpec:
        c = self
        W = c.width

        def norm(name: str) -> PartSpec:
            return PartSpec("layer_norm", {"width": W, "eps": c.eps, "tensors": {
                "weight": (name, (W,)), "bias": (name + ".b", (W,), 0.0)}})

        owners = [c.owner(i) for i in range(len(c.layers))]
        stored = sorted(set(owners))          # the layers with tensors of their own, in order
        layers = []
        for i in stored:
            layer = c.layers[i]
            p, x, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            m, mlp = layer.m(), layer.f()
            H, D, V = m["heads"], m["dim"], m["vdim"]
            if layer.type == "attention":
                G = m["kv_heads"]

                def head_norm(name: str) -> PartSpec:
                    return PartSpec("rms_norm", {"width": D, "eps": c.eps,
                                                 "tensors": {"weight": (x + name, (D,))}})

                t: Dict[str, Any] = {r: (x + r, (rows, W)) for r, rows in
                                     (("q", H * 2 * D), ("k", G * 2 * D), ("v", G * V))}
                t.update({r + "_bias": (x + r + ".b", (rows,), 0.0) for r, rows in
                          (("q", H * 2 * D), ("k", G * 2 * D), ("v", G * V))})
                t.update({r: (x + r, (D,), 0.0) for r in ("lq1", "lk1", "lq2", "lk2")})
                t["o"] = (x + "o", (W, H * V))
                mask = m.get("mask")
                mixer = PartSpec("attention", {
                    "hidden_size": W, "num_heads": H, "num_kv_heads": G, "head_dim": D,
                    "value_dim": V, "scale": float(m["scale"]), "eps": c.eps,
                    "two_maps": {"diff": float(m["diff"])},
                    "chunk": None if mask is None else int(mask["size"]),
                    "position": c._position(layer.type, m.get("rot")),
                    "q_norm": head_norm("q.norm"), "k_norm": head_norm("k.norm"), "tensors": t})
            else:
                R, C = int(m.get("rot_dim") or 0), m["kv_rank"]
                mixer = PartSpec("latent_attention", {
                    "hidden_size": W, "num_heads": H, "head_dim": D, "rot_dim": R, "value_dim": V,
                    "kv_rank": C, "scale": float(m["scale"]), "eps": c.eps, "window": None,
                    "position": c._position(layer.type, m.get("rot") if R else None),
                    "tensors": {
                        "q": (x + "q", (H * (D + R), W)), "dkv": (x + "dkv", (C + R, W)),
                        "dkv_norm": (x + "dkv.norm", (C,)), "uk": (x + "uk", (H * D, C)),
                        "uv": (x + "uv", (H * V, C)), "gate": (x + "g", (H * V, W)),
                        "o": (x + "o", (W, H * V))}})
            if mlp is None:
                ffn = PartSpec("none", {})
            else:
                r, ff = mlp["router"], int(mlp["expert"]["ff"])
                t = {"router": (f + "router", (int(r["experts"]), W))}
                for e in range(int(r["experts"])):
                    t.update({f"gate{e}": (f"{f}e{e}.gate", (ff, W)),
                              f"up{e}": (f"{f}e{e}.up", (ff, W)),
                              f"down{e}": (f"{f}e{e}.down", (W, ff))})
                ffn = PartSpec("moe", {
                    "hidden_size": W, "intermediate_size": ff, "experts": int(r["experts"]),
                    "top": int(r["top"]), "scores": "softmax_all", "groups": r.get("groups"),
                    "activation": "silu", "tensors": t})
            block = PartSpec("pre_norm_residual", {
                "mixer_norm": norm(p + "norm1"), "plain_order_rows": ORDERED_ROWS,
                "feed_forward_norm": norm(p + "norm2") if mlp is not None else None})
            layers.append(LayerSpec(block, mixer, ffn, p))

        spec = ModelSpec(
            architecture=c.architecture, vocab_size=c.vocab, hidden_size=W,
            max_positions=c.max_positions,
            embedding=PartSpec("token_embedding", {"vocab_size": c.vocab, "hidden_size": W,
                                                   "tensors": {"table": ("embed", (c.vocab, W))}}),
            layers=tuple(layers),
            run_order=tuple(LayerCall(stored.index(o)) for o in owners),
            final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": c.vocab, "hidden_size": W, "tied": False,
                                          "tensors": {"weight": ("head", (c.vocab, W))}}))
        spec.validate()
        return spec

    @staticmethod
    def _position(kind: str, rot: Optional[Dict[str, Any]]) -> Optional[PartSpec]:
        if rot is None:
            return None
        params: Dict[str, Any] = {"rot_dim": int(rot["dims"]), "theta": float(rot["base"])}
        if rot.get("scaling") is not None:
            name, keys = SCALINGS[kind]
            params["scaling"] = dict({k: float(rot["scaling"][k]) for k in keys}, kind=name)
        return PartSpec("rope_neox", params)


def sized_like(width: int, ff: int, heads: int, kv_heads: int, head_dim: int, layers: int,
               vocab: int, kv_rank: int = 512, rot: int = 64, experts: int = 8, top: int = 2,
               groups: Tuple[int, int] = (4, 2), chunk: int = 1024) -> RonuraxConfig:
    """A configuration for models with random weights at the sizes of a transformer: layers
    repeating (three of latent attention, one of two-map attention in chunks), all with routed
    experts.  A token leaves a latent of ``kv_rank`` and a rotated part of ``rot`` in the cache of
    a latent layer, whose heads have ``head_dim`` unrotated channels and values of ``head_dim``;
    the two maps of the other layers have half of ``head_dim`` each over values of ``head_dim``.  The
    experts are ``experts`` of width ff / top with ``top`` chosen, so that a token does the
    feed-forward work of a dense layer of width ff."""
    half = head_dim // 2
    latent = {"heads": heads, "dim": head_dim, "rot_dim": rot, "vdim": head_dim, "kv_rank": kv_rank,
              "scale": (head_dim + rot) ** -0.5,
              "rot": {"dims": rot, "base": 1e6, "scaling": {"factor": 4.0, "original": 4096,
                                                            "fast": 32.0, "slow": 1.0}}}
    maps = {"heads": heads, "kv_heads": kv_heads, "dim": half, "vdim": head_dim, "diff": 0.35,
            "scale": half ** -0.5, "mask": {"size": chunk},
            "rot": {"dims": half, "base": 5e5, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0,
                                                           "original": 4096}}}
    moe = {"kind": "moe", "expert": {"ff": max(16, ff // top // 16 * 16)},
           "router": {"experts": experts, "top": top,
                      "groups": {"count": groups[0], "keep": groups[1]}}}
    kinds = ((latent, "latent_attention"),) * 3 + ((maps, "attention"),)
    return RonuraxConfig.from_dict({
        "architecture": "Ronurax", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
        "layers": [{"type": kinds[i % 4][1], "mixer": copy.deepcopy(kinds[i % 4][0]),
                    "mlp": copy.deepcopy(moe)} for i in range(layers)]})
