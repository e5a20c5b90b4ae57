"""Small Ronurax configurations with seeded weights for the tests, the plain implementation's
logits for them, and the helpers that drive the step function.  Every configuration here is the
tests' own: one to many heads in groups of one to sixteen, the two maps' keys longer and shorter than
their value, cache rows for every attention kernel, chunks of one to hundreds of positions and no
chunks, latents of a few to several hundred channels, routers with one to all groups kept and one
to all experts chosen, layers without a feed-forward, layers that share weights with earlier and
later ones."""
from __future__ import annotations

import functools
import json
import os
import tempfile
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from plain import ronurax_plain as RP
from momuvik_util import run_steps  # noqa: F401  (shared helpers)
from runidra_util import BOUND, _bf16_values, assert_close  # noqa: F401


def latent(heads=3, dim=20, rot_dim=12, vdim=28, kv_rank=44, base=10000.0, scale=None, mlp=None,
           of=None, scaling=(3.0, 64, 20.0, 1.5)):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return _entry("latent_attention", m, mlp, of)


def maps(heads=4, kv=2, dim=20, vdim=28, chunk=23, rot=8, base=5000.0, scale=None, diff=0.25,
         mlp=None, of=None, scaling=(4.0, 1.0, 4.0, 128)):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "diff": diff,
         "scale": scale if scale is not None else dim ** -0.5}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"dims": rot, "base": base}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return _entry("attention", m, mlp, of)


def _entry(kind, m, mlp, of):
    out = {"type": kind, "mixer": m, "mlp": mlp}
    if of is not None:
        out["weights_of"] = of
    return out


def moe(experts=6, top=2, count=3, keep=2, ff=40):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def config(layers, width=72, vocab=90, eps=1e-5):
    return {"architecture": "Ronurax", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": layers}


CONFIGS: Dict[str, dict] = {
    # one mechanism each
    "latent": config([latent()]),
    "maps": config([maps()]),
    "moe": config([latent(mlp=moe())]),
    "moe_one_group": config([maps(mlp=moe(8, 2, 4, 1, 32))], width=64),
    "moe_top1": config([latent(mlp=moe(9, 1, 3, 1, 48))], width=64),
    "moe_all": config([latent(mlp=moe(4, 4, 2, 2, 32))], width=64),
    "moe_single": config([maps(mlp=moe(1, 1, 1, 1, 24))], width=56),
    "moe_groups_of_one": config([latent(mlp=moe(7, 3, 7, 4, 16))], width=56),
    "moe_many": config([latent(mlp=moe(44, 5, 11, 3, 16))], width=56),
    # cache rows of 64 and 128 channels (the tensor-core kernels), groups of 2 to 16 query rows
    "map_64": config([maps(heads=4, kv=4, dim=32, vdim=64, chunk=19)]),
    "map_128": config([maps(heads=8, kv=2, dim=64, vdim=128, chunk=50, rot=32)], width=96),
    "map_128_wide_keys": config([maps(heads=4, kv=1, dim=64, vdim=40, chunk=64, rot=64)], width=96),
    "map_64_wide_value": config([maps(heads=8, kv=1, dim=16, vdim=64, chunk=33, rot=16)], width=64),
    # rows that are brought to such a size by padding: 48 to 64, 112 to 128
    "map_48": config([maps(heads=6, kv=3, dim=24, vdim=40, chunk=29, mlp=moe())], width=80),
    "map_112": config([maps(heads=2, kv=2, dim=56, vdim=96, chunk=41, rot=24)]),
    # more query rows to a key row than these kernels take, a row of 32, a long row, one head
    "map_many": config([maps(heads=24, kv=1, dim=32, vdim=64, chunk=37)]),
    "map_32": config([maps(heads=4, kv=2, dim=16, vdim=32, chunk=26)]),
    "map_200": config([maps(heads=2, kv=1, dim=100, vdim=72, chunk=31, rot=100)]),
    "map_one": config([maps(heads=1, kv=1, dim=8, vdim=12, chunk=5, rot=2, diff=0.8)], width=40),
    # chunks of one position, chunks longer than a prompt, no chunks; no rotation, no scaling
    "chunk_1": config([maps(chunk=1), latent()]),
    "chunk_long": config([maps(heads=6, kv=2, dim=32, vdim=64, chunk=700, rot=32)]),
    "chunk_none": config([maps(heads=3, kv=3, chunk=0, dim=32, vdim=64), maps(chunk=0, rot=0)]),
    "no_scaling": config([maps(scaling=None), latent(scaling=None), latent(rot_dim=0, kv_rank=40)]),
    # key rows of latents for every kernel: 64 and 128 channels (with and without fitting heads),
    # several blocks of 64, values in parts
    "row_64": config([latent(heads=4, dim=24, rot_dim=16, vdim=20, kv_rank=48)]),
    "row_128": config([latent(heads=8, dim=32, rot_dim=32, vdim=24, kv_rank=96, mlp=moe(4, 2, 2, 1, 32))],
                      width=128),
    "row_128_h5": config([latent(heads=5, dim=32, rot_dim=56, vdim=40, kv_rank=72)], width=96),
    "row_288": config([latent(heads=10, dim=32, rot_dim=32, vdim=32, kv_rank=256, mlp=moe(6, 3, 3, 2, 64))],
                      width=96),
    "row_576": config([latent(heads=16, dim=32, rot_dim=64, vdim=32, kv_rank=512),
                       latent(heads=16, dim=32, rot_dim=64, vdim=32, kv_rank=512, of=0)], width=128),
    "many_heads": config([latent(heads=130, dim=4, rot_dim=4, vdim=6, kv_rank=28)], width=40),
    "one_head": config([latent(heads=1, dim=8, rot_dim=24, vdim=56, kv_rank=40)]),
    # layers that share weights: with an earlier and a later one, in a chain; two kinds of mixer
    "shared": config([maps(mlp=moe(3, 1, 3, 2, 24), of=2), latent(heads=2, dim=12, rot_dim=6),
                      maps(mlp=moe(3, 1, 3, 2, 24)), latent(heads=2, dim=12, rot_dim=6, of=1),
                      maps(mlp=moe(3, 1, 3, 2, 24), of=0)], width=48),
    # sizes that are multiples of nothing
    "odd": config([latent(heads=3, dim=11, rot_dim=6, vdim=13, kv_rank=19, mlp=moe(3, 2, 1, 1, 9)),
                   maps(heads=5, kv=5, dim=7, vdim=9, rot=6, chunk=11, mlp=moe(5, 2, 5, 3, 35)),
                   maps(heads=3, kv=1, dim=13, vdim=31, rot=10, chunk=17)], width=50, vocab=33),
    "mix": config([latent(heads=4, dim=24, rot_dim=8, vdim=16, kv_rank=56, mlp=moe(6, 2, 3, 1, 64)),
                   maps(heads=6, kv=3, dim=32, vdim=64, chunk=27, rot=24),
                   latent(heads=4, dim=24, rot_dim=8, vdim=16, kv_rank=56, mlp=moe(6, 2, 3, 1, 64), of=0),
                   maps(heads=4, kv=1, dim=24, vdim=48, chunk=40, rot=8, mlp=moe(6, 3, 3, 2, 48))],
                  width=96, vocab=120),
}


def random_config(seed: int) -> str:
    """A configuration drawn from a seed: three to six layers, some of which share weights, at most
    two of them routed (so that most positions are free of close calls), sizes of the kind a small
    model has.  Registered under the returned name."""
    name = f"random{seed}"
    if name in CONFIGS:
        return name
    rng = np.random.default_rng(8100 + seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]
    layers: List[dict] = []
    for _ in range(int(rng.integers(3, 7))):
        routed = sum(l["mlp"] is not None for l in layers)
        free = [i for i, l in enumerate(layers) if "weights_of" not in l
                and (routed < 2 or l["mlp"] is None)]
        if free and rng.random() < 0.3:
            i = pick(*free)
            layers.append(dict(json.loads(json.dumps(layers[i])), weights_of=i))
            continue
        mlp = None
        if routed < 2 and rng.random() < 0.7:
            count, size = pick(1, 2, 3, 4), pick(1, 2, 3)
            keep = int(rng.integers(1, count + 1))
            mlp = moe(count * size, int(rng.integers(1, min(4, keep * size) + 1)), count, keep,
                      pick(32, 48, 80))
        if rng.random() < 0.5:
            kv = pick(1, 2, 3)
            dim = pick(24, 32, 48, 64)
            layers.append(maps(heads=kv * pick(1, 2, 4), kv=kv, dim=dim, vdim=pick(dim, 2 * dim, 40),
                               chunk=pick(13, 60, 64, 100, 171), rot=pick(8, 16, 24), base=pick(1e4, 5e5),
                               scale=pick(None, 0.2), diff=pick(0.2, 0.45, 0.7), mlp=mlp,
                               scaling=pick((4.0, 1.0, 4.0, 128), (8.0, 1.0, 2.0, 512), (2.0, 2.0, 8.0, 96))))
        else:
            layers.append(latent(heads=pick(2, 4, 5, 8, 12), dim=pick(24, 32, 48), rot_dim=pick(8, 16, 32),
                                 vdim=pick(24, 40, 56), kv_rank=pick(48, 64, 88, 112, 160), mlp=mlp,
                                 base=pick(1e4, 5e5), scale=pick(None, 0.15),
                                 scaling=pick((3.0, 64, 20.0, 1.5), (2.5, 400, 24.0, 1.0), (6.0, 100, 8.0, 2.0))))
    CONFIGS[name] = config(layers, width=pick(88, 128, 160, 208), vocab=int(rng.integers(150, 500)),
                           eps=pick(1e-6, 1e-5))
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

    def norm(name):
        vec(name, W, 1.0, 0.2), vec(name + ".b", W, 0.0, 0.2)

    t["embed"] = rng.standard_normal((cfg["vocab"], W)) + 0.3      # (the rows have a mean)
    for i, l in enumerate(cfg["layers"]):
        if l.get("weights_of") is not None:
            continue
        p, x, f, m, mlp = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp.", l["mixer"], l["mlp"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        if l["type"] == "attention":
            G = m["kv_heads"]
            for r, n in (("q", H * 2 * d), ("k", G * 2 * d), ("v", G * dv)):
                mat(x + r, n, W), vec(x + r + ".b", n, 0.0, 0.4)
            for r in ("q", "k"):
                vec(x + r + ".norm", d, 1.3, 0.2)
            for r in ("lq1", "lk1", "lq2", "lk2"):
                vec(x + r, d, 0.0, 0.6 / np.sqrt(d) ** 0.5)
        else:
            r, c = m["rot_dim"], m["kv_rank"]
            mat(x + "q", H * (d + r), W, 1.5)
            mat(x + "dkv", c + r, W), vec(x + "dkv.norm", c, 1.0, 0.2)
            mat(x + "uk", H * d, c, 1.5), mat(x + "uv", H * dv, c), mat(x + "g", H * dv, W, 1.5)
        mat(x + "o", W, H * dv)
        if mlp is None:
            continue
        norm(p + "norm2")
        # logits far enough apart that rounding seldom changes who is chosen
        mat(f + "router", mlp["router"]["experts"], W, 4.0)
        for e in range(mlp["router"]["experts"]):
            q = f"{f}e{e}."
            mat(q + "gate", mlp["expert"]["ff"], W, 1.5), mat(q + "up", mlp["expert"]["ff"], W, 1.5)
            mat(q + "down", W, mlp["expert"]["ff"])
    norm("final.norm")
    mat("head", cfg["vocab"], W)
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
        d = tempfile.mkdtemp(prefix=f"ronurax_{name}_")
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(CONFIGS[name], f)
        write_safetensors(os.path.join(d, "model.safetensors"),
                          {n: torch.from_numpy(np.asarray(a)).to(torch.bfloat16)
                           for n, a in weights(name, seed).items()})
        _dirs[key] = d
    return _dirs[key]


# A router's choice between two experts (or two groups) whose outputs lie closer than this can fall
# either way once the router's input is rounded to 16 bits; the 16-bit tests leave such positions out.
CLOSE_CALL = 0.08


@functools.lru_cache(maxsize=None)
def _plain(name: str, seed: int, tokens: tuple):
    margins: list = []
    z = RP.forward(CONFIGS[name], weights(name, seed), list(tokens), margins=margins)
    # (what rounding moves a router's outputs by grows with every routed layer in front of it)
    scaled = [m / 2.0 ** i for i, m in enumerate(margins)]
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
        moved = dict(w, embed=embed * (1 + 2.0 ** -7 * rng.standard_normal(embed.shape)))
        worst = np.maximum(worst, np.abs(RP.forward(CONFIGS[name], moved, list(tokens)) - ref).max(axis=1))
    return worst


def tokens_for(name: str, n: int, seed: int) -> List[int]:
    rng = np.random.default_rng(1000 + seed)
    return [int(t) for t in rng.integers(0, CONFIGS[name]["vocab"], n)]


def slack_for(name: str, tokens: Sequence[int], dtype: str, seed: int = 0) -> Optional[np.ndarray]:
    """What a position is allowed on top of the bound.  float32: nothing.  bfloat16: twice what a
    move of the inputs by a rounding or two does to it in the plain implementation, and
    everything where a router makes a close call (another expert may run)."""
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


def check_request(got, name, tokens, dtype, what, seed=0):
    ref = plain_logits(name, tokens, seed)
    pos = sorted(got)
    slack = slack_for(name, tokens, dtype, seed)
    assert_close(np.stack([got[p] for p in pos]), ref[pos], dtype, what,
                 slack=None if slack is None else slack[pos])
