"""Small Momuvik configurations with seeded weights for the tests, the plain implementation's
logits for them, and the helpers that drive the step function.  Every configuration here is the
tests' own: one to a hundred and more heads, key rows from a few channels to several hundred, rotated
parts longer and shorter than the unrotated ones, values of other sizes than keys, routers that
choose one expert and all of them, experts with and without a shared one, layers without a
feed-forward, layers that share weights with earlier and later ones."""
from __future__ import annotations

import functools
import json
import os
import tempfile
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from plain import momuvik_plain as MP
from runidra_util import BOUND, _bf16_values, assert_close  # noqa: F401  (shared helpers)


def layer(heads=3, dim=20, rot_dim=12, vdim=28, q_rank=36, kv_rank=44, base=10000.0, scale=None,
          mlp=None, of=None, dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank,
         "kv_rank": kv_rank, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if rot_dim:
        m["rot"] = {"dims": dims or rot_dim, "base": base}
    out = {"type": "latent_attention", "mixer": m, "mlp": mlp}
    if of is not None:
        out["weights_of"] = of
    return out


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=40, limit=1.2, shared=56, shared_limit=2.0):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit},
         "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def config(layers, width=72, vocab=90, eps=1e-5, embed_scale=2.5, mult=0.8):
    return {"architecture": "Momuvik", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "residual_mult": mult, "layers": layers}


CONFIGS: Dict[str, dict] = {
    # one mechanism each
    "attn": config([layer()]),
    "dense": config([layer(mlp=dense(88))], mult=1.0, embed_scale=1.0),
    "moe": config([layer(mlp=moe())], mult=0.3),
    "moe_top1": config([layer(mlp=moe(experts=7, top=1, ff=48, limit=0.7, shared=24,
                                      shared_limit=0.6))], width=64, mult=1.4),
    "moe_all": config([layer(mlp=moe(experts=4, top=4, ff=32, shared=0))], width=64),
    "moe_many": config([layer(mlp=moe(experts=19, top=6, ff=16, limit=3.0, shared=72,
                                      shared_limit=1.0))], width=56),
    # one head; a rotated part longer than the rest; values longer than the latent
    "one_head": config([layer(heads=1, dim=8, rot_dim=24, vdim=56, kv_rank=40, q_rank=16)]),
    # more heads than a group of rows holds: 130 (token, head) pairs per token
    "many_heads": config([layer(heads=130, dim=4, rot_dim=4, vdim=6, kv_rank=28, q_rank=24)], width=40),
    # key rows that the kernels of ordinary attention take (64 and 128 channels)
    "row_64": config([layer(heads=4, dim=24, rot_dim=16, vdim=20, kv_rank=48)]),
    "row_128": config([layer(heads=8, dim=32, rot_dim=32, vdim=24, kv_rank=96, mlp=moe(4, 2, 32))],
                      width=128),
    # 128 channels with heads that do not divide 128
    "row_128_h5": config([layer(heads=5, dim=32, rot_dim=56, vdim=40, kv_rank=72)], width=96),
    # latents of several blocks of 64 channels: two, five and nine, values in one to three parts
    "row_136": config([layer(heads=7, dim=40, rot_dim=8, vdim=24, kv_rank=128, q_rank=48)], width=96),
    "row_288": config([layer(heads=10, dim=32, rot_dim=32, vdim=32, kv_rank=256, q_rank=64,
                             mlp=dense(64))], width=96),
    "row_344": config([layer(heads=3, dim=16, rot_dim=40, vdim=24, kv_rank=304, q_rank=40)], width=80),
    "row_576": config([layer(heads=16, dim=32, rot_dim=64, vdim=32, kv_rank=512, q_rank=96),
                       layer(heads=16, dim=32, rot_dim=64, vdim=32, kv_rank=512, q_rank=96, of=0)],
                      width=128),
    # a rotation of a part of the rotated part, and no rotated part at all
    "part_rot": config([layer(rot_dim=20, dims=8, base=300.0), layer(heads=2, rot_dim=0, kv_rank=40)]),
    # layers that share weights: with the first, with each other's, with a later one, in a chain
    "shared": config([layer(mlp=dense(40), of=2),
                      layer(heads=2, dim=12, rot_dim=6, mlp=moe(3, 1, 24)),
                      layer(mlp=dense(40)),
                      layer(heads=2, dim=12, rot_dim=6, mlp=moe(3, 1, 24), of=1),
                      layer(mlp=dense(40), of=0)], width=48, mult=0.6),
    # sizes that are multiples of nothing
    "odd": config([layer(heads=3, dim=11, rot_dim=6, vdim=13, q_rank=17, kv_rank=19, mlp=moe(3, 2, 9, 1.1, 11)),
                   layer(heads=5, dim=7, rot_dim=10, vdim=9, q_rank=23, kv_rank=31, mlp=dense(35))],
                  width=50, vocab=33, embed_scale=1.0),
    # experts of widths for the grouped products, without a feed-forward between them
    "mix": config([layer(heads=4, dim=24, rot_dim=8, vdim=16, kv_rank=56, mlp=moe(6, 3, 64, 1.4, 80, 0.9)),
                   layer(heads=2, dim=16, rot_dim=16, vdim=40, kv_rank=80),
                   layer(heads=4, dim=24, rot_dim=8, vdim=16, kv_rank=56, mlp=moe(6, 3, 64, 1.4, 80, 0.9), of=0),
                   layer(heads=6, dim=32, rot_dim=24, vdim=32, kv_rank=104, mlp=dense(112))],
                  width=96, vocab=120, mult=0.7),
}


def random_config(seed: int) -> str:
    """A configuration drawn from a seed: three to six layers, some of which share weights, at most
    two of them routed (so that most positions are free of close calls), sizes of the kind a small
    model has.  Registered under the returned name."""
    name = f"random{seed}"
    if name in CONFIGS:
        return name
    rng = np.random.default_rng(7000 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers: List[dict] = []
    for _ in range(int(rng.integers(3, 7))):
        routed = sum(l["mlp"] is not None and l["mlp"]["kind"] == "moe" for l in layers)
        free = [i for i, l in enumerate(layers) if "weights_of" not in l
                and (routed < 2 or l["mlp"] is None or l["mlp"]["kind"] == "dense")]
        if free and rng.random() < 0.3:
            i = pick(*free)
            layers.append(dict(json.loads(json.dumps(layers[i])), weights_of=i))
            continue
        r = rng.random()
        if r < 0.2:
            mlp = None
        elif r < 0.5 or routed >= 2:
            mlp = dense(pick(96, 160, 224))
        else:
            experts = pick(3, 4, 6)
            mlp = moe(experts, pick(1, 2, experts), pick(32, 48, 80), pick(0.8, 1.5, 4.0),
                      pick(0, 64, 96), pick(0.7, 2.0))
        rot = pick(8, 16, 32, 64)
        layers.append(layer(heads=pick(2, 4, 5, 8, 12), dim=pick(24, 32, 48), rot_dim=rot,
                            vdim=pick(24, 40, 56), q_rank=pick(48, 72, 112),
                            kv_rank=pick(64, 88, 112, 160, 192), base=pick(1e4, 5e5),
                            scale=pick(None, 0.15), mlp=mlp))
    CONFIGS[name] = config(layers, width=pick(88, 128, 160, 208), vocab=int(rng.integers(150, 500)),
                           embed_scale=pick(1.0, 3.0, 9.0), mult=pick(0.4, 1.0, 1.3))
    return name


def _weights(cfg: dict, seed: int) -> Dict[str, np.ndarray]:
    """Seeded weights, already rounded to bfloat16 values so that both precisions and the
    plain implementation compute with the same numbers."""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
    t: Dict[str, np.ndarray] = {}

    def mat(name, out, inn, gain=1.0):
        t[name] = rng.standard_normal((out, inn)) * gain / np.sqrt(inn)

    def vec(name, n, mean=0.0, std=1.0):
        t[name] = mean + std * rng.standard_normal(n)

    def expert(p, ff):
        mat(p + "gate", ff, W, 1.5), mat(p + "up", ff, W, 1.5), mat(p + "down", W, ff)

    t["embed"] = rng.standard_normal((cfg["vocab"], W)) / cfg["embedding"]["scale"]
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, x, f, m, mlp = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", l["mixer"], l["mlp"]
        H, d, r, dv, q, c = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
        vec(p + "norm1", W, 0.0, 0.2)
        mat(x + "dq", q, W), vec(x + "dq.norm", q, 1.0, 0.2), mat(x + "uq", H * (d + r), q, 1.5)
        mat(x + "dkv", c + r, W), vec(x + "dkv.norm", c, 1.0, 0.2)
        mat(x + "uk", H * d, c, 1.5), mat(x + "uv", H * dv, c), vec(x + "sink", H, 0.0, 1.5)
        mat(x + "o", W, H * dv)
        if mlp is None:
            continue
        vec(p + "norm2", W, 0.0, 0.2)
        if mlp["kind"] == "dense":
            expert(f, mlp["ff"])
        else:
            # logits far enough apart that rounding seldom changes who is chosen
            mat(f + "router", mlp["router"]["experts"], W, 4.0)
            for e in range(mlp["router"]["experts"]):
                expert(f"{f}e{e}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                expert(f + "shared.", mlp["shared"]["ff"])
    vec("final.norm", W, 0.0, 0.2)
    return _bf16_values(t)


CUSTOM: Dict[str, Dict[str, np.ndarray]] = {}     # configurations whose weights a test has made


@functools.lru_cache(maxsize=None)
def weights(name: str, seed: int = 0) -> Dict[str, np.ndarray]:
    return CUSTOM[name] if name in CUSTOM else _weights(CONFIGS[name], seed)


_dirs: Dict[tuple, str] = {}


def model_dir(name: str, seed: int = 0) -> str:
    """A folder with config.json and model.safetensors (bfloat16) of the configuration."""
    from llmario_b200.weights.safetensors_io import write_safetensors

    key = (name, seed)
    if key not in _dirs:
        d = tempfile.mkdtemp(prefix=f"momuvik_{name}_")
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(CONFIGS[name], f)
        write_safetensors(os.path.join(d, "model.safetensors"),
                          {n: torch.from_numpy(np.asarray(a)).to(torch.bfloat16)
                           for n, a in weights(name, seed).items()})
        _dirs[key] = d
    return _dirs[key]


# A router's choice between two experts whose outputs lie closer than this can fall either way
# once the router's input is rounded to 16 bits; the 16-bit tests leave such positions out.
CLOSE_CALL = 0.1


@functools.lru_cache(maxsize=None)
def _plain(name: str, seed: int, tokens: tuple):
    margins: list = []
    z = MP.forward(CONFIGS[name], weights(name, seed), list(tokens), margins=margins)
    # (what rounding moves a router's outputs by grows with every routed layer in front of it)
    scaled = [m / 2.5 ** i for i, m in enumerate(margins)]
    least = np.min(np.stack(scaled), axis=0) if scaled else np.full(len(tokens), np.inf)
    return z, least


def plain_logits(name: str, tokens: Sequence[int], seed: int = 0) -> np.ndarray:
    return _plain(name, seed, tuple(int(t) for t in tokens))[0]


def router_margins(name: str, tokens: Sequence[int], seed: int = 0) -> np.ndarray:
    """Per position, the smallest margin of any router's choice there (those of later routers
    scaled down)."""
    return _plain(name, seed, tuple(int(t) for t in tokens))[1]


@functools.lru_cache(maxsize=None)
def _sensitivity(name: str, seed: int, tokens: tuple) -> np.ndarray:
    """Per position, how far the logits move when the inputs move by about one bfloat16
    rounding or two: the plain implementation run again with the embedding rows scaled by
    1 + 2^-7 N(0, 1) (the largest of three such moves)."""
    w = dict(weights(name, seed))
    rng = np.random.default_rng(99)
    embed, ref = w["embed"], _plain(name, seed, tokens)[0]
    worst = np.zeros(len(tokens))
    for _ in range(3):
        # (the table is the output matrix as well: the move is a layer's, not the head's)
        moved = dict(w, embed=embed * (1 + 2.0 ** -7 * rng.standard_normal(embed.shape)))
        worst = np.maximum(worst, np.abs(MP.forward(CONFIGS[name], moved, list(tokens)) - ref).max(axis=1))
    return worst


def tokens_for(name: str, n: int, seed: int) -> List[int]:
    rng = np.random.default_rng(1000 + seed)
    return [int(t) for t in rng.integers(0, CONFIGS[name]["vocab"], n)]


def slack_for(name: str, tokens: Sequence[int], dtype: str, seed: int = 0) -> Optional[np.ndarray]:
    """What a position is allowed on top of the bound.  float32: nothing.  bfloat16: twice what a
    move of the inputs by a rounding or two does to it in the plain implementation, and
    everything from a position on where a router makes a close call (another expert may run)."""
    if dtype != "bfloat16":
        return None
    toks = tuple(int(t) for t in tokens)
    slack = 2.0 * _sensitivity(name, seed, toks)
    slack[router_margins(name, toks, seed) < CLOSE_CALL] = np.inf
    return slack


def runner_for(name: str, dtype: str, page_size: int = 16, cache_tokens: int = 1024,
               max_requests: int = 4, seed: int = 0, use_graphs: bool = True,
               max_context: int = 0):
    from llmario_b200.engine.model import Model
    from llmario_b200.engine.step import ModelRunner

    model = Model.from_folder(model_dir(name, seed), dtype, "cuda:0")
    return ModelRunner(model, page_size=page_size, n_pages=-(-cache_tokens // page_size),
                       max_requests=max_requests, max_context=max_context or cache_tokens,
                       token_budget=cache_tokens, use_graphs=use_graphs)


def run_steps(runner, steps):
    """``steps``: lists of (request, tokens, wanted places).  Returns request -> {position: logits}."""
    from llmario_b200.engine.step import StepEntry

    got = {}
    for step in steps:
        entries = [StepEntry(r, list(t), list(w)) for r, t, w in step]
        starts = {r: (runner.length(r) if runner.cache.has(r) else 0) for r, _, _ in step}
        logits = runner.step(entries).cpu().numpy()
        i = 0
        for r, _, want in step:
            for wpos in want:
                got.setdefault(r, {})[starts[r] + wpos] = logits[i].copy()
                i += 1
    return got


def check_request(got, name, tokens, dtype, what, seed=0):
    ref = plain_logits(name, tokens, seed)
    pos = sorted(got)
    slack = slack_for(name, tokens, dtype, seed)
    assert_close(np.stack([got[p] for p in pos]), ref[pos], dtype, what,
                 slack=None if slack is None else slack[pos])
