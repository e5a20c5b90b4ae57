"""Typed configuration of the Momuvik decoder, read from the keys of its ``config.json``.

A Momuvik model is a list of pre-norm layers whose sublayers are added with a constant weight:
``x += residual_mult * mixer(norm1(x)); x += residual_mult * mlp(norm2(x))``.  The norms' stored
gains are what they have beyond one.  The embedding is multiplied by ``embedding.scale``; the
logits come from the embedding table itself, without that scale.  The mixer is
``latent_attention``: queries, keys and values through low-rank latents, one rotated key part
(half-split pairs) for all heads, every earlier key seen, a sink per head in the softmax.  The
feed-forward is ``dense`` (silu-gated), ``moe`` (routed experts of the clamped form, sigmoid scores
that are not renormalised and weigh the chosen expert's input; a shared expert of sizes and a
limit of its own) or absent.  A layer with ``weights_of: j`` runs with layer j's tensors and a
cache of its own.  Every size and constant that can differ between two models of the design is
read here and nowhere else; tensor names follow ``l<i>.<part>``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .pemolorn import _freeze_deep
from .runidra import _deep
from .spec import ConfigError, LayerCall, LayerSpec, ModelSpec, PartSpec
from .vunasun import _get

MIXERS = ("latent_attention",)


@dataclass(frozen=True)
class MomuvikLayer:
    type: str
    mixer: Tuple[Tuple[str, Any], ...]
    mlp: Optional[Tuple[Tuple[str, Any], ...]]
    weights_of: Optional[int] = None

    def m(self) -> Dict[str, Any]:
        return _deep(dict(self.mixer))

    def f(self) -> Optional[Dict[str, Any]]:
        return None if self.mlp is None else _deep(dict(self.mlp))


@dataclass(frozen=True)
class MomuvikConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    residual_mult: float
    layers: Tuple[MomuvikLayer, ...]
    max_positions: int = 1 << 17      # the design has no limit of its own: the engine's default

    architecture = "Momuvik"
    model_type = "momuvik"

    # ---------------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "MomuvikConfig":
        vocab = _get(raw, "vocab", int, "model")
        width = _get(raw, "width", int, "model")
        eps = _get(raw.get("norm"), "eps", float, "norm")
        scale = 1.0 if raw.get("embedding") is None else \
            _get(raw["embedding"], "scale", float, "embedding")
        mult = 1.0 if raw.get("residual_mult") is None else \
            _get(raw, "residual_mult", float, "model")
        entries = raw.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        layers: List[MomuvikLayer] = []
        for i, e in enumerate(entries):
            where = f"layers[{i}]"
            kind = e.get("type") if isinstance(e, dict) else None
            if kind not in MIXERS:
                raise ConfigError(f"config.json: {where}: unsupported type {kind!r} "
                                  f"(known: {', '.join(MIXERS)})")
            m = e.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: {where}: missing 'mixer'")
            cls._check_mixer(m, where + ".mixer")
            mlp = e.get("mlp")
            if mlp is not None:
                cls._check_mlp(mlp, where + ".mlp")
            of = e.get("weights_of")
            if of is not None and (isinstance(of, bool) or not isinstance(of, int)
                                   or not 0 <= of < len(entries) or of == i):
                raise ConfigError(f"config.json: {where}: weights_of {of!r} names no other layer")
            layers.append(MomuvikLayer(kind, _freeze_deep(m),
                                       None if mlp is None else _freeze_deep(mlp), of))
        max_pos = int(raw.get("max_positions") or cls.max_positions)
        out = cls(vocab, width, eps, scale, mult, tuple(layers), max_pos)
        for i, layer in enumerate(layers):
            owner = layers[out.owner(i)]
            if (owner.type, owner.mixer, owner.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ConfigError(f"config.json: layers[{i}] uses the weights of layer "
                                  f"{out.owner(i)}, whose sizes and constants differ from its own")
        return out

    @staticmethod
    def _check_mixer(m: Dict[str, Any], where: str) -> None:
        for key in ("heads", "dim", "vdim", "q_rank", "kv_rank"):
            _get(m, key, int, where)
        _get(m, "scale", float, where)
        rot_dim = m.get("rot_dim") or 0
        if isinstance(rot_dim, bool) or not isinstance(rot_dim, int) or rot_dim < 0:
            raise ConfigError(f"config.json: {where}: rot_dim {rot_dim!r}")
        rot = m.get("rot")
        if rot is not None:
            dims = _get(rot, "dims", int, where + ".rot")
            _get(rot, "base", float, where + ".rot")
            if dims % 2 or dims > rot_dim:
                raise ConfigError(f"config.json: {where}.rot: dims {dims} must be even and at "
                                  f"most rot_dim {rot_dim}")

    @staticmethod
    def _check_mlp(mlp: Dict[str, Any], where: str) -> None:
        kind = mlp.get("kind", "dense")
        if kind == "dense":
            _get(mlp, "ff", int, where)
        elif kind == "moe":
            n = _get(mlp.get("router"), "experts", int, where + ".router")
            top = _get(mlp.get("router"), "top", int, where + ".router")
            if top > n:
                raise ConfigError(f"config.json: {where}: top {top} of {n} experts")
            for key in ("expert", "shared"):
                if key == "shared" and mlp.get(key) is None:
                    continue
                _get(mlp.get(key), "ff", int, f"{where}.{key}")
                if _get(mlp.get(key), "limit", float, f"{where}.{key}") < 0:
                    raise ConfigError(f"config.json: {where}.{key}: limit must not be negative")
        else:
            raise ConfigError(f"config.json: {where}: unsupported mlp kind {kind!r} "
                              "(known: dense, moe)")

    def to_dict(self) -> Dict[str, Any]:
        """The ``config.json`` that reads back as this configuration."""
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab,
                               "width": self.width, "norm": {"eps": self.eps},
                               "embedding": {"scale": self.embedding_scale},
                               "residual_mult": self.residual_mult, "layers": []}
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
            return PartSpec("rms_norm", {"width": W, "eps": c.eps, "zero_centred": True,
                                         "tensors": {"weight": (name, (W,))}})

        def gated(prefix: str, ff: int) -> Dict[str, Any]:
            return {"gate": (prefix + "gate", (ff, W)), "up": (prefix + "up", (ff, W)),
                    "down": (prefix + "down", (W, ff))}

        owners = [c.owner(i) for i in range(len(c.layers))]
        stored = sorted(set(owners))          # the layers with tensors of their own, in order
        layers = []
        for i in stored:
            layer = c.layers[i]
            p, x, f = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            m, mlp = layer.m(), layer.f()
            H, D, V = m["heads"], m["dim"], m["vdim"]
            R, Rq, Rkv = int(m.get("rot_dim") or 0), m["q_rank"], m["kv_rank"]
            rot = m.get("rot")
            mixer = PartSpec("latent_attention", {
                "hidden_size": W, "num_heads": H, "head_dim": D, "rot_dim": R, "value_dim": V,
                "q_rank": Rq, "kv_rank": Rkv, "scale": float(m["scale"]), "eps": c.eps,
                "window": None,
                "position": None if rot is None or not R else PartSpec("rope_neox", {
                    "rot_dim": int(rot["dims"]), "theta": float(rot["base"]),
                    "freq_scale": 1.0, "attn_factor": 1.0}),
                "tensors": {
                    "dq": (x + "dq", (Rq, W)), "dq_norm": (x + "dq.norm", (Rq,)),
                    "uq": (x + "uq", (H * (D + R), Rq)),
                    "dkv": (x + "dkv", (Rkv + R, W)), "dkv_norm": (x + "dkv.norm", (Rkv,)),
                    "uk": (x + "uk", (H * D, Rkv)), "uv": (x + "uv", (H * V, Rkv)),
                    "sink": (x + "sink", (H,)), "o": (x + "o", (W, H * V)),
                },
            })
            if mlp is None:
                ffn = PartSpec("none", {})
            elif mlp.get("kind", "dense") == "dense":
                ff = int(mlp["ff"])
                ffn = PartSpec("swiglu", {"hidden_size": W, "intermediate_size": ff,
                                          "tensors": gated(f, ff)})
            else:
                E, ff = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
                t: Dict[str, Any] = {"router": (f + "router", (E, W))}
                for e in range(E):
                    t.update({f"{role}{e}": v for role, v in gated(f"{f}e{e}.", ff).items()})
                params: Dict[str, Any] = {
                    "hidden_size": W, "intermediate_size": ff, "experts": E,
                    "top": int(mlp["router"]["top"]), "scores": "sigmoid", "weight_on": "input",
                    "activation": "clamped_swish", "limit": float(mlp["expert"]["limit"]),
                    "tensors": t}
                if mlp.get("shared") is not None:
                    sff = int(mlp["shared"]["ff"])
                    params["shared"] = PartSpec("gated", {
                        "hidden_size": W, "intermediate_size": sff, "activation": "clamped_swish",
                        "limit": float(mlp["shared"]["limit"]),
                        "tensors": gated(f + "shared.", sff)})
                ffn = PartSpec("moe", params)
            block = PartSpec("hyper_connection", {
                "streams": 1, "residual_scale": c.residual_mult, "mixer_norm": norm(p + "norm1"),
                "feed_forward_norm": norm(p + "norm2") if mlp is not None else None})
            layers.append(LayerSpec(block, mixer, ffn, p))

        table = ("embed", (c.vocab, W))
        spec = ModelSpec(
            architecture=c.architecture, vocab_size=c.vocab, hidden_size=W,
            max_positions=c.max_positions,
            embedding=PartSpec("token_embedding", {
                "vocab_size": c.vocab, "hidden_size": W, "scale": c.embedding_scale,
                "tensors": {"table": table}}),
            layers=tuple(layers),
            run_order=tuple(LayerCall(stored.index(o)) for o in owners),
            final_norm=norm("final.norm"),
            head=PartSpec("linear_head", {"vocab_size": c.vocab, "hidden_size": W, "tied": True,
                                          "tensors": {"weight": table}}),
            residual_streams=1)
        spec.validate()
        return spec


def sized_like(width: int, ff: int, heads: int, layers: int, vocab: int, kv_rank: int = 512,
               rot: int = 64, dim: int = 128, q_rank: int = 0, experts: int = 8, top: int = 2
               ) -> MomuvikConfig:
    """A configuration for models with random weights at the sizes of a transformer: layers
    repeating (latent attention + dense, latent attention + routed experts twice, latent attention +
    dense).  A token leaves a latent of ``kv_rank`` and a rotated part of ``rot`` in the cache; heads
    have ``dim`` unrotated channels and values of ``dim``; queries pass through a latent of
    ``q_rank`` (a quarter of the width when not given).  The routed experts are ``experts`` of width
    ff / (top + 1) with ``top`` chosen, beside a shared one of that width, so that a token does the
    feed-forward work of the dense layer."""
    q_rank = q_rank or max(64, width // 4)
    att = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": dim, "q_rank": q_rank,
           "kv_rank": kv_rank, "scale": (dim + rot) ** -0.5, "rot": {"dims": rot, "base": 1e6}}
    eff = max(16, ff // (top + 1) // 16 * 16)
    dense = {"kind": "dense", "ff": ff}
    moe = {"kind": "moe", "expert": {"ff": eff, "limit": 7.0},
           "router": {"experts": experts, "top": top}, "shared": {"ff": eff, "limit": 7.0}}
    mlps = (dense, moe, moe, dense)
    return MomuvikConfig.from_dict({
        "architecture": "Momuvik", "vocab": vocab, "width": width, "norm": {"eps": 1e-6},
        "embedding": {"scale": 1.0}, "residual_mult": 0.5,
        "layers": [{"type": "latent_attention", "mixer": copy.deepcopy(att),
                    "mlp": copy.deepcopy(mlps[i % 4])} for i in range(layers)]})
