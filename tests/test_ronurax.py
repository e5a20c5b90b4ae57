"""The Ronurax decoder against the plain float64 implementation (tests/plain/ronurax_plain.py):
every mechanism alone and together, in whole prompts, portions, single decoded tokens, mixed
batches, reused slots and pages, and through the engine's own entry point."""
from __future__ import annotations

import json
import math

import numpy as np
import pytest
import torch

from plain import ronurax_plain as RP
from ronurax_util import (CLOSE_CALL, CONFIGS, CUSTOM, _bf16_values, _weights, assert_close,
                          check_request, config, latent, maps, model_dir, moe, plain_logits,
                          random_config, router_margins, run_steps, runner_for, slack_for,
                          tokens_for, weights)

DTYPES = ("float32", "bfloat16")


# --------------------------------------------------------------------------------------------
# no GPU: configuration, and the plain implementation against its own definitions
# --------------------------------------------------------------------------------------------
def test_configuration_round_trip_and_tensor_names():
    from llmario_b200.config import ConfigError, RonuraxConfig, resolve_architecture
    from llmario_b200.weights.loader import check_tensors, expected_tensors

    for seed in range(4):
        random_config(seed)
    for name, raw in CONFIGS.items():
        assert resolve_architecture(raw) == "Ronurax"
        cfg = RonuraxConfig.from_dict(raw)
        assert RonuraxConfig.from_dict(cfg.to_dict()) == cfg
        assert cfg.to_dict() == raw, name
        spec = cfg.to_spec()
        have = {n: a.shape for n, a in weights(name).items()}
        assert set(expected_tensors(spec)) == set(have), name
        check_tensors(spec, have)
        assert len(spec.run_order) == len(raw["layers"])
        for i, call in enumerate(spec.run_order):
            assert spec.layers[call.layer].weight_prefix == f"l{RP.tensors_of(raw, i)}."
            assert call.reads_cache_of is None            # a cache of its own for every layer
        assert len(spec.layers) == sum("weights_of" not in l for l in raw["layers"])
    shared = RonuraxConfig.from_dict(CONFIGS["shared"]).to_spec()
    assert [shared.layers[c.layer].weight_prefix for c in shared.run_order] == \
        ["l2.", "l1.", "l2.", "l1.", "l2."]

    def broken(change, match):
        raw = json.loads(json.dumps(CONFIGS["mix"]))
        change(raw)
        with pytest.raises(ConfigError, match=match):
            RonuraxConfig.from_dict(raw)

    layers = lambda r: r["layers"]
    broken(lambda r: layers(r)[0].update(type="conv"), "unsupported type")
    broken(lambda r: layers(r)[0]["mlp"].update(kind="dense"), "mlp kind")
    broken(lambda r: layers(r)[0]["mlp"]["router"].update(top=3), "top")
    broken(lambda r: layers(r)[0]["mlp"]["router"]["groups"].update(count=4), "groups")
    broken(lambda r: layers(r)[0]["mlp"]["router"]["groups"].update(keep=4), "groups")
    broken(lambda r: layers(r)[0]["mlp"]["router"]["groups"].pop("keep"), "keep")
    broken(lambda r: layers(r)[1]["mixer"]["rot"].update(dims=34), "dims")
    broken(lambda r: layers(r)[1]["mixer"]["rot"]["scaling"].pop("low"), "low")
    broken(lambda r: layers(r)[0]["mixer"]["rot"]["scaling"].update(fast=0), "fast")
    broken(lambda r: layers(r)[1]["mixer"].update(kv_heads=4), "kv_heads")
    broken(lambda r: layers(r)[1]["mixer"].pop("diff"), "diff")
    broken(lambda r: layers(r)[1]["mixer"]["mask"].update(size=0), "size")
    broken(lambda r: layers(r)[2].update(weights_of=9), "weights_of")
    broken(lambda r: layers(r)[2]["mixer"].update(vdim=17), "differ")
    broken(lambda r: (layers(r)[2].update(weights_of=0), layers(r)[0].update(weights_of=2)), "itself")
    broken(lambda r: r.pop("norm"), "eps")


def test_a_sized_configuration_reads_back():
    from llmario_b200.config import RonuraxConfig
    from llmario_b200.config.ronurax import sized_like

    cfg = sized_like(256, 512, 4, 2, 64, 6, 500, kv_rank=96, rot=32)
    assert RonuraxConfig.from_dict(cfg.to_dict()) == cfg
    assert [l.type for l in cfg.layers] == ["latent_attention"] * 3 + ["attention"] + ["latent_attention"] * 2


def test_random_weights_have_offsets_around_zero():
    """The tensors that are offsets (norms, projections, the maps' weight) are drawn around zero,
    gains around one."""
    from llmario_b200.config import RonuraxConfig
    from llmario_b200.weights import random_tensors

    t = random_tensors(RonuraxConfig.from_dict(CONFIGS["mix"]).to_spec(), 3, torch.float32)
    for name, mean in (("l0.norm1", 1.0), ("l0.norm1.b", 0.0), ("l1.mix.q.b", 0.0), ("l1.mix.lk2", 0.0),
                       ("l1.mix.k.norm", 1.0), ("final.norm.b", 0.0)):
        assert abs(float(t[name].mean()) - mean) < 0.02, name


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, dict(factor=4.0, low=1.0, high=4.0, original=128)),
    (64, 500000.0, dict(factor=8.0, low=1.0, high=4.0, original=8192)),
    (6, 30.0, dict(factor=2.5, low=2.0, high=3.0, original=40)),
    (2, 7.0, dict(factor=2.0, low=1.0, high=2.0, original=4)),
    (10, 100.0, dict(factor=3.0, low=1.0, high=50.0, original=300))])
def test_frequencies_scaled_by_wavelength(dims, base, scaling):
    from llmario_b200.config import PartSpec
    from llmario_b200.parts.position import RotaryHalfSplit

    p = RotaryHalfSplit(PartSpec("rope_neox", {"rot_dim": dims, "theta": base,
                                               "scaling": dict(scaling, kind="bands")}), {}, None, "cpu")
    want = RP.banded_frequencies(dims, base, **scaling)
    np.testing.assert_allclose(p.inv_freq.numpy(), want, rtol=3e-7)
    assert p.attn_factor == 1.0
    plain = RP.plain_frequencies(dims, base)
    # short waves stay, long ones are stretched by the factor, and nothing leaves that range
    assert (want <= plain * (1 + 1e-12)).all() and (want >= plain / scaling["factor"] * (1 - 1e-12)).all()


@pytest.mark.parametrize("dims,base,scaling", [
    (16, 10000.0, dict(factor=3.0, original=64, fast=20.0, slow=1.5)),
    (64, 1e6, dict(factor=40.0, original=4096, fast=32.0, slow=1.0)),
    (8, 50.0, dict(factor=2.0, original=100, fast=8.0, slow=7.0)),       # a ramp within one index
    (12, 20.0, dict(factor=5.0, original=30, fast=100.0, slow=0.001)),   # beyond both ends
    (2, 9.0, dict(factor=1.5, original=16, fast=2.0, slow=1.0))])
def test_frequencies_scaled_by_index(dims, base, scaling):
    from llmario_b200.config import PartSpec
    from llmario_b200.parts.position import RotaryHalfSplit

    p = RotaryHalfSplit(PartSpec("rope_neox", {"rot_dim": dims, "theta": base,
                                               "scaling": dict(scaling, kind="ramp")}), {}, None, "cpu")
    want, mult = RP.ramped_frequencies(dims, base, **scaling)
    np.testing.assert_allclose(p.inv_freq.numpy(), want, rtol=3e-7)
    assert abs(p.attn_factor - mult) < 1e-12 and mult == 0.1 * math.log(scaling["factor"]) + 1.0
    assert p.constants() != RotaryHalfSplit(PartSpec("rope_neox", {"rot_dim": dims, "theta": base}),
                                            {}, None, "cpu").constants()


def test_plain_mechanisms():
    """The plain statement against its own definitions."""
    rng = np.random.default_rng(1)
    x = rng.standard_normal((5, 12)) + 3.0
    # the layer norm: centred, a mean square of one, then gain and offset
    y = RP.centred_norm(x, np.ones(12), np.zeros(12), 0.0)
    np.testing.assert_allclose(y.mean(1), 0.0, atol=1e-12)
    np.testing.assert_allclose((y * y).mean(1), 1.0)
    np.testing.assert_allclose(RP.centred_norm(x, np.full(12, 2.0), np.full(12, 0.5), 0.0), 2 * y + 0.5)
    # rotation: lengths of pairs stay (times the factor), scores depend on the distance alone
    f = RP.plain_frequencies(8, 50.0)
    r = RP.rotate_halves(x, np.arange(5), f)
    np.testing.assert_allclose(r[0], x[0])
    np.testing.assert_allclose(r[:, :4] ** 2 + r[:, 4:8] ** 2, x[:, :4] ** 2 + x[:, 4:8] ** 2)
    np.testing.assert_allclose(r[:, 8:], x[:, 8:])
    np.testing.assert_allclose(RP.rotate_halves(x, np.arange(5), f, 1.3)[:, :8], 1.3 * r[:, :8])
    a, b = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    dot = lambda p, q: float(RP.rotate_halves(a, [p], f)[0] @ RP.rotate_halves(b, [q], f)[0])
    assert abs(dot(9, 4) - dot(105, 100)) < 1e-9 and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    # chunks: counted from position 0, the own token always seen
    m = RP.chunk_mask(7, 3)
    assert [int(v.sum()) for v in m] == [1, 2, 3, 1, 2, 3, 1] and m.diagonal().all()
    assert RP.chunk_mask(4, None).sum() == 10 and RP.chunk_mask(4, 1).sum() == 4
    # the maps: one that is subtracted from itself with weight one leaves nothing to divide
    a1 = rng.standard_normal((2, 3, 8))
    assert np.abs(RP.two_map_combine(a1, a1, 1.0, 0.2, 1e-5)).max() < 1e-9
    o = RP.two_map_combine(a1, rng.standard_normal((2, 3, 8)), 0.4, 0.25, 0.0)
    np.testing.assert_allclose((o * o).mean(-1), 0.75 ** 2)
    t = {"lq1": np.array([1.0, 2.0]), "lk1": np.array([0.5, 0.1]), "lq2": np.array([0.0, 1.0]),
         "lk2": np.array([3.0, -1.0])}
    assert abs(RP.mixing_weight(t, "", 0.3) - (math.exp(0.7) - math.exp(-1.0) + 0.3)) < 1e-12
    # groups: the best of a left-out group is not chosen however good it is among the rest
    s = np.array([[0.30, 0.01, 0.02, 0.25, 0.20, 0.22]])
    assert RP.choose(s, 2, 3, 1).tolist() == [[0, 1]]
    assert RP.choose(s, 3, 3, 2).tolist() == [[0, 3, 2]]
    assert RP.choose(s, 3, 3, 3).tolist() == [[0, 3, 5]] and RP.choose(s, 3, 1, 1).tolist() == [[0, 3, 5]]
    assert RP.choose(np.ones((1, 6)), 3, 3, 2).tolist() == [[0, 1, 2]]      # equal: the lowest indices
    np.testing.assert_allclose(RP.choice_margin(np.log(s), 3, 3, 2), [np.log(0.25 / 0.22)])
    np.testing.assert_allclose(RP.choice_margin(np.log(s), 1, 3, 2), [np.log(0.30 / 0.25)])


def test_plain_constants_matter():
    """Each constant and branch of the configuration moves the plain logits."""
    raw, toks = CONFIGS["mix"], tokens_for("mix", 60, 3)
    w = weights("mix")
    ref = RP.forward(raw, w, toks)

    def moved(change):
        other = json.loads(json.dumps(raw))
        change(other)
        return np.abs(RP.forward(other, w, toks) - ref).max() / np.abs(ref).max()

    assert moved(lambda r: r["norm"].update(eps=1e-2)) > 1e-4
    for l in (0, 1, 2, 3):
        mix = lambda r: r["layers"][l]["mixer"]
        assert moved(lambda r: mix(r).update(scale=0.3)) > 1e-3
        assert moved(lambda r: mix(r)["rot"].update(base=500.0)) > 1e-4
        assert moved(lambda r: mix(r)["rot"].pop("scaling")) > 1e-5
        assert moved(lambda r: mix(r)["rot"]["scaling"].update(factor=9.0)) > 1e-5
        assert moved(lambda r: mix(r)["rot"]["scaling"].update(original=3000)) > 1e-5
    for l in (1, 3):
        mix = lambda r: r["layers"][l]["mixer"]
        assert moved(lambda r: mix(r).update(diff=0.5)) > 1e-2
        for step in (-1, 1):
            assert moved(lambda r: mix(r)["mask"].update(size=mix(r)["mask"]["size"] + step)) > 1e-2
        assert moved(lambda r: mix(r)["rot"].update(dims=4)) > 1e-3
    for l in (0, 3):
        router = lambda r: r["layers"][l]["mlp"]["router"]
        assert moved(lambda r: router(r).update(top=1)) > 1e-3
        assert moved(lambda r: router(r)["groups"].update(keep=router(r)["groups"]["keep"] + 1)) > 1e-3
        assert moved(lambda r: router(r).update(groups={"count": 2, "keep": 1})) > 1e-3


# --------------------------------------------------------------------------------------------
# kernels of the mechanisms, each against a few lines of NumPy
# --------------------------------------------------------------------------------------------
def _dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device="cuda")


def _np(t):
    return t.double().cpu().numpy()


@pytest.mark.gpu
@pytest.mark.parametrize("width", [1, 3, 50, 72, 256, 1000, 1024, 2048, 4096, 5000, 8192, 9000])
@pytest.mark.parametrize("rows", [1, 7, 600])
def test_layer_norm_kernel(rows, width):
    """Rows with a mean far from zero (the deviations are summed behind the mean), and the rows of an
    index."""
    from llmario_b200 import kernels

    rng = np.random.default_rng(rows + width)
    x = rng.standard_normal((rows, width)) + 10.0 * rng.standard_normal((rows, 1))
    x = _dev(x)
    w, b = _dev(1 + rng.standard_normal(width)), _dev(rng.standard_normal(width))
    ref = RP.centred_norm(_np(x), _np(w), _np(b), 1e-4)
    for dtype, tol in ((torch.float32, 1e-4), (torch.bfloat16, 1e-2)):
        out = torch.full((rows, width), float("nan"), dtype=dtype, device="cuda")
        kernels.layer_norm(x, w, b, out, 1e-4)
        np.testing.assert_allclose(_np(out), ref, rtol=tol, atol=tol)
        index = _dev(rng.integers(0, rows, 5), torch.int32)
        some = torch.full((5, width), float("nan"), dtype=dtype, device="cuda")
        kernels.layer_norm(x, w, b, some, 1e-4, index)
        np.testing.assert_allclose(_np(some), ref[index.cpu().numpy()], rtol=tol, atol=tol)


@pytest.mark.gpu
@pytest.mark.parametrize("E,top,count,keep", [(8, 3, 4, 2), (6, 2, 3, 1), (12, 5, 2, 1), (9, 4, 9, 5), (70, 6, 35, 7),
                                              (128, 8, 64, 20), (66, 1, 2, 2), (5, 5, 1, 1), (300, 16, 100, 9)])
@pytest.mark.parametrize("scores", ["softmax_all", "softmax_chosen", "softmax_all_renormed", "sigmoid"])
def test_router_with_groups(E, top, count, keep, scores):
    from llmario_b200 import kernels

    rng = np.random.default_rng(E + keep)
    rows = 41
    z = rng.standard_normal((rows, E)) * 2
    z[3] = 0.5                        # all equal: the lowest groups and experts win
    z[4] = np.arange(E) * 0.05        # the last groups win
    z[5, :] = -5.0 - np.arange(E) * 0.01
    z[5, E - 1] = 4.0                 # one good expert opens the group of its poor neighbours
    z_d = _dev(z)
    ids = torch.empty(rows, top, dtype=torch.int32, device="cuda")
    wts = torch.empty(rows, top, dtype=torch.float32, device="cuda")

    def check(zz, i, w):
        zz = _np(zz)
        want = RP.choose(RP.softmax(zz), top, count, keep)
        assert i.cpu().numpy().tolist() == want.tolist()
        s = np.take_along_axis(RP.softmax(zz), want, axis=1)
        if scores in ("softmax_chosen", "softmax_all_renormed"):
            s = s / s.sum(1, keepdims=True)
        elif scores == "sigmoid":
            s = RP.sigmoid(np.take_along_axis(zz, want, axis=1))
        np.testing.assert_allclose(_np(w), s, rtol=2e-5)

    kernels.moe_route(z_d, E, top, ids, wts, scores, groups=(count, keep))
    check(z_d, ids, wts)
    for dtype, width, n in ((torch.float32, 50, rows), (torch.bfloat16, 256, rows), (torch.bfloat16, 72, 300)):
        h = _dev(rng.standard_normal((n, width)), dtype)
        w = _dev(rng.standard_normal((E, width)) / 8)
        z2 = torch.empty(n, E, dtype=torch.float32, device="cuda")
        ids2 = torch.empty(n, top, dtype=torch.int32, device="cuda")
        wts2 = torch.empty(n, top, dtype=torch.float32, device="cuda")
        kernels.moe_router(h, w, None, E, top, z2, ids2, wts2, scores, groups=(count, keep))
        np.testing.assert_allclose(_np(z2), _np(h) @ _np(w).T, rtol=1e-4, atol=1e-4)
        check(z2, ids2, wts2)
    if E % 7:
        with pytest.raises(kernels.KernelError):
            kernels.moe_route(z_d, E, top, ids, wts, scores, groups=(7, 1))


def _cache(rows, page, heads, hd, dtype, planes=2):
    """Pages of a cache whose block table is shuffled, for rows of several requests; everything in it
    is NaN.  Returns view, row_slot, row_pos and the place of every row."""
    from llmario_b200.cache.manager import CacheView

    rng = np.random.default_rng(rows)
    n_req = 3
    slot = rng.integers(0, n_req, rows)
    pos = np.zeros(rows, int)
    for s in range(n_req):
        mine = np.nonzero(slot == s)[0]
        pos[mine] = np.arange(len(mine)) + 5 * s
    per = int(pos.max()) // page + 1
    pages = rng.permutation(n_req * per).reshape(n_req, per)
    st = torch.full((n_req * per, 2, planes, heads, page, hd), float("nan"), dtype=dtype, device="cuda")
    table = _dev(pages, torch.int32)
    view = CacheView(st[0, 1, 0], st[0, 1, -1], st.stride(0), table, page, 0, st, 1)

    def rows_of(plane):
        return np.stack([_np(st[pages[s, p // page], 1, plane, :, p % page]) for s, p in zip(slot, pos)])
    return view, _dev(slot, torch.int32), _dev(pos, torch.int32), pos, rows_of


@pytest.mark.gpu
@pytest.mark.parametrize("rows", [1, 9, 1100])
@pytest.mark.parametrize("H,G,d,dv,hd,rot", [(4, 2, 16, 32, 32, 8), (3, 1, 20, 28, 40, 20), (5, 5, 7, 9, 14, 6),
                                             (8, 2, 64, 128, 128, 64), (6, 3, 24, 40, 64, 0), (2, 1, 100, 72, 200, 36)])
def test_two_map_store_kernel(rows, H, G, d, dv, hd, rot):
    """Biases, norm per map, rotation, the queries' rows and the keys side by side in the cache; the
    projections are zeroed behind it."""
    from llmario_b200 import kernels

    rng = np.random.default_rng(rows + d)
    cols = [H * 2 * d, G * 2 * d, G * dv]
    pad = 4
    proj_np = rng.standard_normal((rows, sum(cols) + pad))
    biases = [rng.standard_normal(n) for n in cols]
    qw, kw = 1 + 0.3 * rng.standard_normal(d), 1 + 0.3 * rng.standard_normal(d)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        for clear in (False, True):
            proj = _dev(proj_np)
            view, slot, pos_d, pos, rows_of = _cache(rows, 16, G, hd, dtype)
            q_out = torch.full((rows, H * 2 * hd), float("nan"), dtype=dtype, device="cuda")
            cs = None
            if rot:
                ang = pos[:, None] * RP.plain_frequencies(rot, 300.0)
                cs = _dev(np.stack([np.cos(ang), np.sin(ang)], axis=-1))
            a, b = cols[0], cols[0] + cols[1]
            bias = [_dev(x) for x in biases]
            kernels.qkv_store(proj[:, :a], proj[:, a:b], proj[:, b:b + cols[2]], q_out, view, slot, pos_d, H, G, d,
                              dv, hd, kernels.NORM_PER_HEAD, _dev(qw), _dev(kw), 1e-5, rot, cs, maps=2,
                              biases=tuple(bias), clear=clear)
            f = _np(_dev(proj_np))
            # the kernel turns adjacent pairs: the same as half-split pairs of reordered channels
            order = [i for i in range(0, rot, 2)] + [i for i in range(1, rot, 2)] + list(range(rot, d))
            back = np.argsort(order)

            def turned(x):
                if not rot:
                    return x
                return RP.rotate_halves(x[..., order], pos, RP.plain_frequencies(rot, 300.0))[..., back]
            q = turned(RP.unit_rms((f[:, :a] + biases[0]).reshape(rows, H, 2, d), 1e-5) * qw)
            k = turned(RP.unit_rms((f[:, a:b] + biases[1]).reshape(rows, G, 2, d), 1e-5) * kw)
            v = (f[:, b:b + cols[2]] + biases[2]).reshape(rows, G, dv)
            got = _np(q_out).reshape(rows, H, 2, hd)
            want = np.zeros((rows, H, 2, hd))
            want[:, :, 0, :d], want[:, :, 1, d:2 * d] = q[:, :, 0], q[:, :, 1]
            np.testing.assert_allclose(got, want, rtol=tol, atol=tol)
            keys, vals = np.zeros((rows, G, hd)), np.zeros((rows, G, hd))
            keys[..., :2 * d], vals[..., :dv] = k.reshape(rows, G, 2 * d), v
            np.testing.assert_allclose(rows_of(0), keys, rtol=tol, atol=tol)
            np.testing.assert_allclose(rows_of(1), vals, rtol=tol, atol=tol)
            left = _np(proj)[:, :sum(cols)]
            assert (left == 0).all() if clear else (left == f[:, :sum(cols)]).all()


@pytest.mark.gpu
@pytest.mark.parametrize("H,dv,n", [(1, 1, 1), (3, 28, 28), (8, 128, 128), (5, 40, 128), (2, 300, 304), (7, 9, 14),
                                    (40, 64, 64), (1, 640, 640), (4, 264, 264)])
@pytest.mark.parametrize("rows", [1, 77])
def test_two_map_heads_kernel(rows, H, dv, n):
    from llmario_b200 import kernels

    rng = np.random.default_rng(rows + dv)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
        a = _dev(rng.standard_normal((rows, H * 2 * n)), dtype)
        a.view(rows, H, 2, n)[..., dv:] = float("nan")        # behind the value: not read
        out = torch.full((rows, H * dv), float("nan"), dtype=dtype, device="cuda")
        kernels.two_map_heads(a, out, H, dv, 0.85, 0.3, 1e-3)
        f = _np(a).reshape(rows, H, 2, n)[..., :dv]
        ref = RP.two_map_combine(f[:, :, 0], f[:, :, 1], 0.85, 0.3, 1e-3)
        np.testing.assert_allclose(_np(out).reshape(ref.shape), ref, rtol=tol, atol=tol)


@pytest.mark.gpu
@pytest.mark.parametrize("H,d,r,c,extra", [(3, 20, 12, 44, 0), (4, 24, 16, 48, 8), (5, 7, 6, 19, 3), (130, 4, 4, 28, 4),
                                           (2, 16, 0, 40, 2), (32, 128, 64, 512, 16), (3, 9, 5, 8, 1)])
@pytest.mark.parametrize("rows", [1, 30, 600])
def test_latent_prepare_kernel(rows, H, d, r, c, extra):
    """Queries and key rows from one matrix with other columns between them; one plane and two; the
    columns that were read are zeroed, the others stay."""
    from llmario_b200 import kernels

    rng = np.random.default_rng(rows + c)
    nq = H * (d + r)
    proj_np = rng.standard_normal((rows, nq + extra + c + r))
    gain, half = 1 + 0.3 * rng.standard_normal(c), (r // 2)
    for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
        for clear, planes in ((False, 1), (True, 2)):
            proj = _dev(proj_np)
            view, slot, pos_d, pos, rows_of = _cache(rows, 8, 1, c + r, dtype, planes)
            q_plain = torch.full((rows, H * d), float("nan"), dtype=dtype, device="cuda")
            q_full = torch.full((rows, H * (c + r)), float("nan"), dtype=dtype, device="cuda")
            cs = None
            if half:
                ang = pos[:, None] * RP.plain_frequencies(2 * half, 300.0)
                cs = _dev(1.2 * np.stack([np.cos(ang), np.sin(ang)], axis=-1))
            kernels.latent_prepare(proj, 0, nq + extra, _dev(gain), cs, q_plain, q_full, view, slot, pos_d, H, d, r,
                                   c, 1e-5, clear=clear)
            f = _np(_dev(proj_np))
            order = list(range(0, 2 * half, 2)) + list(range(1, 2 * half, 2)) + list(range(2 * half, r))
            back = np.argsort(order)

            def turned(x):
                if not half:
                    return x
                return RP.rotate_halves(x[..., order], pos, RP.plain_frequencies(2 * half, 300.0), 1.2)[..., back]
            q = f[:, :nq].reshape(rows, H, d + r)
            np.testing.assert_allclose(_np(q_plain).reshape(rows, H, d), q[..., :d], rtol=tol, atol=tol)
            np.testing.assert_allclose(_np(q_full).reshape(rows, H, c + r)[..., c:], turned(q[..., d:]), rtol=tol,
                                       atol=tol)
            both = f[:, nq + extra:]
            key = np.concatenate([RP.unit_rms(both[:, :c], 1e-5) * gain, turned(both[:, c:])], axis=1)
            np.testing.assert_allclose(rows_of(0)[:, 0], key, rtol=tol, atol=tol)
            if planes == 2:
                np.testing.assert_allclose(rows_of(1)[:, 0, :c], key[:, :c], rtol=tol, atol=tol)
            left = _np(proj)
            np.testing.assert_array_equal(left[:, nq:nq + extra], f[:, nq:nq + extra])
            read = np.concatenate([left[:, :nq], left[:, nq + extra:]], axis=1)
            assert (read == 0).all() if clear else (left == f).all()


@pytest.mark.gpu
@pytest.mark.parametrize("rows,cols,first,extra", [(1, 8, 0, 0), (5, 128, 4, 12), (33, 84, 16, 4), (700, 256, 8, 8),
                                                   (3, 40, 3, 5), (9, 17, 0, 2)])
@pytest.mark.parametrize("dtype", (torch.float32, torch.bfloat16))
@pytest.mark.parametrize("clear", (False, True))
def test_channel_gate_kernel(rows, cols, first, extra, dtype, clear):
    """A gate per channel from a column range of a wider matrix, of any alignment."""
    from llmario_b200 import kernels

    rng = np.random.default_rng(rows + cols)
    wide = _dev(rng.standard_normal((rows, first + cols + extra)) * 4)
    out = _dev(rng.standard_normal((rows, cols)), dtype)
    f, o = _np(wide), _np(out)
    kernels.channel_gate(out, wide[:, first:first + cols], clear=clear)
    tol = 1e-6 if dtype == torch.float32 else 8e-3
    np.testing.assert_allclose(_np(out), o * RP.sigmoid(f[:, first:first + cols]), rtol=tol, atol=tol)
    left = _np(wide)
    np.testing.assert_array_equal(left[:, :first], f[:, :first])
    np.testing.assert_array_equal(left[:, first + cols:], f[:, first + cols:])
    np.testing.assert_array_equal(left[:, first:first + cols], 0.0 if clear else f[:, first:first + cols])


# --------------------------------------------------------------------------------------------
# whole models through the step function
# --------------------------------------------------------------------------------------------
NAMES = sorted(n for n in CONFIGS if not n.startswith(("random", "needle")))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(name, dtype):
    """Every position of a prompt that spans several pages and chunks, the first tokens included."""
    toks = tokens_for(name, 110, 1)
    runner = runner_for(name, dtype)
    got = run_steps(runner, [[("a", toks, range(len(toks)))]])
    check_request(got["a"], name, toks, dtype, "whole prompt")
    runner.cache.check_invariants()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_single_tokens(name, dtype):
    """A prompt, then tokens one by one through recorded steps, across borders of pages and chunks."""
    toks = tokens_for(name, 90, 2)
    n = 21
    runner = runner_for(name, dtype)
    steps = [[("a", toks[:n], [0, n - 1])]] + [[("a", [t], [0])] for t in toks[n:]]
    got = run_steps(runner, steps)
    check_request(got["a"], name, toks, dtype, "prompt, then single tokens")
    assert runner.counters["graph_replays"] > 40


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_many_sizes(name, dtype):
    """Portions cut in the middle of pages and chunks, down to two tokens; then single tokens."""
    toks = tokens_for(name, 120, 3)
    cuts = [2, 3, 2, 17, 2, 31, 5, 2, 29, 1, 2, 1, 1, 16, 2, 4]
    assert sum(cuts) == len(toks)
    steps, at = [], 0
    for c in cuts:
        steps.append([("a", toks[at:at + c], range(c))])
        at += c
    runner = runner_for(name, dtype)
    got = run_steps(runner, steps)
    check_request(got["a"], name, toks, dtype, "portions")
    # and the cut does not matter beyond rounding: the same prompt whole
    whole = run_steps(runner_for(name, dtype), [[("a", toks, range(len(toks)))]])
    a = np.stack([got["a"][p] for p in range(len(toks))])
    b = np.stack([whole["a"][p] for p in range(len(toks))])
    assert_close(a, b.astype(np.float64), dtype, "portions against whole",
                 1e-5 if dtype == "float32" else 2e-2, slack=slack_for(name, toks, dtype))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("mix", "shared", "odd", "moe_top1", "map_128", "map_48", "row_288", "chunk_1"))
def test_mixed_batches_and_reused_slots(name, dtype):
    """Four request slots, six requests of unequal lengths: portions of some beside single tokens
    of others, requests that pause, requests that end and whose slot and pages the next one
    takes.  Every request must get what it gets alone (the plain implementation's logits)."""
    lengths = {"a": 70, "b": 9, "c": 41, "d": 33, "e": 52, "f": 2}
    toks = {r: tokens_for(name, n, 10 + i) for i, (r, n) in enumerate(lengths.items())}
    runner = runner_for(name, dtype, page_size=8, cache_tokens=208, max_requests=4)
    at = {r: 0 for r in toks}

    def take(r, n):
        n = min(n, lengths[r] - at[r])
        part = toks[r][at[r]:at[r] + n]
        at[r] += n
        return (r, part, range(n))

    plan = [[("a", 30), ("b", 2)], [("a", 1), ("b", 1), ("c", 17)], [("b", 6), ("c", 1), ("d", 2)],
            [("a", 1), ("c", 23), ("d", 1)], [("a", 38)], [("d", 30), ("e", 3)],
            [("e", 1), ("f", 2)], [("e", 48)]]
    got = {}
    for step in plan:
        entries = [take(r, n) for r, n in step]
        for r, res in run_steps(runner, [entries]).items():
            got.setdefault(r, {}).update(res)
        for r, _ in step:
            if at[r] == lengths[r]:
                runner.close(r)
        runner.cache.check_invariants()
    assert all(at[r] == lengths[r] for r in toks)
    for r in toks:
        assert sorted(got[r]) == list(range(lengths[r]))
        check_request(got[r], name, toks[r], dtype, f"request {r}", seed=0)
    assert runner.cache.free_slots() == 4


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("mix", "moe", "map_128", "chunk_long", "row_576"))
def test_a_long_prompt_over_the_engine_page(name, dtype):
    """A prompt of several hundred tokens with the engine's default page of 64 (in plain stream
    order: 512 rows and more), then a second portion that starts inside a page, then single tokens."""
    toks = tokens_for(name, 620, 6)
    runner = runner_for(name, dtype, page_size=64, cache_tokens=1024)
    steps = [[("a", toks[:533], range(533))], [("a", toks[533:610], range(77))]] \
        + [[("a", [t], [0])] for t in toks[610:]]
    got = run_steps(runner, steps)
    check_request(got["a"], name, toks, dtype, "long prompt")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_from_a_seed(seed, dtype):
    """Layers with sizes drawn from a seed, the engine's page of 64: a prompt in portions, then
    single tokens, against the plain implementation."""
    name = random_config(seed)
    toks = tokens_for(name, 230, 7)
    runner = runner_for(name, dtype, page_size=64, cache_tokens=512)
    steps = [[("a", toks[:150], range(150))], [("a", toks[150:153], range(3))],
             [("a", toks[153:200], range(47))]] + [[("a", [t], [0])] for t in toks[200:]]
    got = run_steps(runner, steps)
    check_request(got["a"], name, toks, dtype, f"{name} {CONFIGS[name]['layers']}")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ("mix", "shared", "map_64"))
def test_long_decoding(name, dtype):
    """Hundreds of single tokens behind a one-token prompt; a layer with chunks gives back the pages
    behind them."""
    toks = tokens_for(name, 260, 4)
    runner = runner_for(name, dtype, page_size=32, cache_tokens=512)
    got = run_steps(runner, [[("a", [t], [0])] for t in toks])
    check_request(got["a"], name, toks, dtype, "long decoding")
    if name == "map_64":
        assert min(runner.cache.free_pages()) >= 512 // 32 - 3


@pytest.mark.gpu
def test_a_request_alone_and_in_a_batch_gives_the_same_values():
    """32-bit: what else is in the batch, and which slot and pages a request has, changes nothing."""
    name = "mix"
    a, b = tokens_for(name, 50, 30), tokens_for(name, 37, 31)
    alone = run_steps(runner_for(name, "float32"), [[("a", a[:40], range(40))]] + [[("a", [t], [0])] for t in a[40:]])
    runner = runner_for(name, "float32")
    both = run_steps(runner, [[("b", b[:9], [8])], [("b", b[9:30], [20]), ("a", a[:40], range(40))]]
                     + [[("a", [t], [0]), ("b", [b[30]], [0])] if i == 0 else [("a", [t], [0])]
                        for i, t in enumerate(a[40:])])
    x = np.stack([alone["a"][p] for p in range(50)])
    y = np.stack([both["a"][p] for p in range(50)])
    assert np.abs(x - y).max() <= 1e-6 * np.abs(x).max()


@pytest.mark.gpu
def test_which_kernels_run():
    """Cache rows of 64 and 128 channels, padded ones included, run on the tensor-core attention
    kernels, others on the generic one; latents on theirs."""
    from llmario_b200 import driver

    for name, kinds, never in (("map_64", ("tcgen05", "decode_tma"), "generic"),
                               ("map_128", ("tcgen05", "decode_tma"), "generic"),
                               ("map_48", ("tcgen05", "decode_tma"), "generic"),
                               ("map_112", ("tcgen05", "decode_tma"), "generic"),
                               ("map_128_wide_keys", ("tcgen05", "decode_tma"), "generic"),
                               ("map_many", ("generic",), "tcgen05"), ("map_200", ("generic",), "tcgen05"),
                               ("row_288", ("latent",), "generic")):
        before = driver.kernel_counts()
        toks = tokens_for(name, 60, 1)
        runner = runner_for(name, "bfloat16")
        run_steps(runner, [[("a", toks[:59], [0])], [("a", toks[59:], [0])]])
        ran = {k: v - before[k] for k, v in driver.kernel_counts().items()}
        assert all(ran[k] > 0 for k in kinds) and ran[never] == 0, (name, ran)


# --------------------------------------------------------------------------------------------
# keys that stand out
# --------------------------------------------------------------------------------------------
def _mark_two_tokens(w) -> None:
    """Channels 0 and 1 of layer 0's normed input: about zero for every token but 0 (channel 0) and
    1 (channel 1)."""
    w["embed"][:, :2] = w["embed"][:, 2:].mean(axis=1, keepdims=True)
    w["embed"][0, 0] += 4.0
    w["embed"][1, 1] += 4.0
    w["l0.norm1"][:], w["l0.norm1.b"][:] = 1.0, 0.0


def latent_needle(kv_rank: int, rot: int, heads: int) -> str:
    """A layer whose weights make one score stand out.  Token 0 is the needle: its latent is one
    large direction, which head 0's key map turns into a key that the probe's (token 1's) query
    points along; every other token has neither.  A probe's output is then decided by whether it
    finds the needle, however far back."""
    name = f"needle_latent{kv_rank}_{rot}_{heads}"
    if name not in CONFIGS:
        CONFIGS[name] = config([latent(heads=heads, dim=16, rot_dim=rot, vdim=24, kv_rank=kv_rank, scale=1.0)],
                               width=64, vocab=64)
        w = {n: a.copy() for n, a in _weights(CONFIGS[name], 7).items()}
        _mark_two_tokens(w)
        x = "l0.mix."
        for m in ("q", "dkv"):
            w[x + m] *= 0.15
            w[x + m][:, :2] = 0.0
        w[x + "dkv"][5, 0] = 20.0                       # the needle's latent: channel 5
        w[x + "uk"] *= 0.15
        w[x + "uk"][7, 5] = 1.0                         # head 0, key channel 7 <- latent channel 5
        w[x + "q"][7, 1] = 5.0 / np.sqrt(kv_rank)       # head 0, plain query channel 7 <- the probe
        w[x + "uv"][:24, 5] *= 6.0                      # head 0's value of the needle
        w[x + "g"][:24] *= 0.3                          # head 0's gates stay open
        CUSTOM[name] = _bf16_values(w)
    return name


def map_needle(which: int, chunk: int, dim: int, vdim: int, heads: int, kv: int) -> str:
    """The same for one map (``which``) of head 0 of a layer with chunks: the needle's key and the
    probe's query of that map point along channel dim - 1, which the rotation leaves alone."""
    name = f"needle_map{which}_{chunk}_{dim}_{vdim}_{heads}_{kv}"
    if name not in CONFIGS:
        CONFIGS[name] = config([maps(heads=heads, kv=kv, dim=dim, vdim=vdim, chunk=chunk, rot=dim // 2 // 2 * 2,
                                     scale=14.0 / dim, diff=0.5)], width=64, vocab=64)
        w = {n: a.copy() for n, a in _weights(CONFIGS[name], 9).items()}
        _mark_two_tokens(w)
        x = "l0.mix."
        for r in ("q", "k", "v"):
            w[x + r][:, :2] = 0.0
            w[x + r + ".b"] *= 0.1
        at = which * dim + dim - 1                      # head 0 (and key head 0), this map, last channel
        for r, col in (("q", 1), ("k", 0)):
            w[x + r][at] *= 0.05
            w[x + r + ".b"][at] = 0.0
            w[x + r][at, col] = 15.0
            w[x + r + ".norm"][:] = 0.4                 # the other channels' scores stay small
            w[x + r + ".norm"][dim - 1] = 1.0
        w[x + "v"][:vdim, 0] = 4.0 * np.sign(w[x + "v"][:vdim, 5])      # the needle's value
        for r in ("lq1", "lk1", "lq2", "lk2"):
            w[x + r][:] = 0.0                           # the second map's weight is diff
        CUSTOM[name] = _bf16_values(w)
    return name


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page", (16, 64))
@pytest.mark.parametrize("kv_rank,rot,heads", [(40, 16, 3), (48, 16, 2), (112, 24, 4), (256, 40, 6)])
def test_a_key_that_stands_out_far_back(dtype, page, kv_rank, rot, heads):
    """Needles at the very start, on the last and the first place of a page, and just before the
    probe; the probes in the prompt, in a later portion and decoded one by one.  Leaving the needle
    out moves the probe's logits visibly."""
    name = latent_needle(kv_rank, rot, heads)
    rng = np.random.default_rng(5)
    n = 330
    probes = [40, 150, 200, 201, 280, 320, 329]
    for at in (0, page - 1, page, 2 * page - 1):
        toks = [int(t) for t in rng.integers(2, 64, n)]
        toks[at] = 0
        for p in probes:
            if p > at:
                toks[p] = 1
        seen = [p for p in probes if p > at]
        runner = runner_for(name, dtype, page_size=page, cache_tokens=1024)
        got = run_steps(runner, [[("a", toks, range(n))]])
        check_request(got["a"], name, toks, dtype, f"needle at {at}, whole prompt")
        steps = [[("b", toks[:190], [150])], [("b", toks[190:192], [0, 1])], [("b", toks[192:270], range(78))]] \
            + [[("b", [t], [0])] for t in toks[270:]]
        got = run_steps(runner, steps)
        check_request(got["b"], name, toks, dtype, f"needle at {at}, portions and single tokens")
        ref = plain_logits(name, toks)
        other = list(toks)
        other[at] = 2
        d = np.abs(plain_logits(name, other) - ref).max(axis=1)
        assert d[seen].min() > 0.1 * np.abs(ref).max()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("which", (0, 1))
@pytest.mark.parametrize("page,chunk,dim,vdim,heads,kv", [
    (16, 50, 32, 64, 6, 3), (64, 96, 64, 128, 8, 2), (16, 41, 20, 28, 4, 1), (32, 32, 24, 40, 2, 2), (64, 200, 16, 64, 8, 1)])
def test_a_key_that_stands_out_at_a_chunk_edge(dtype, which, page, chunk, dim, vdim, heads, kv):
    """A needle on the last place of a chunk (no probe of the next chunk sees it) and one on the first
    place (every probe of its chunk does), in a prompt, in portions cut around the edge, and decoded
    across it.  In the plain implementation moving the needle across the edge moves the logits."""
    name = map_needle(which, chunk, dim, vdim, heads, kv)
    rng = np.random.default_rng(6)
    n = 2 * chunk + 30
    edge = chunk
    for at in (edge - 1, edge, 2 * chunk - 1):
        toks = [int(t) for t in rng.integers(2, 64, n)]
        probes = [p for p in (edge - 2, edge, edge + 1, edge + 2, edge + chunk // 2, 2 * chunk - 1, 2 * chunk, n - 1)
                  if p != at]
        for p in probes:
            toks[p] = 1
        toks[at] = 0
        runner = runner_for(name, dtype, page_size=page, cache_tokens=1024)
        got = run_steps(runner, [[("a", toks, range(n))]])
        check_request(got["a"], name, toks, dtype, f"needle at {at}, whole prompt")
        cuts = [edge - 3, 2, 2, 2, chunk // 2]
        steps, start = [], 0
        for c in cuts:
            steps.append([("b", toks[start:start + c], range(c))])
            start += c
        steps += [[("b", [t], [0])] for t in toks[start:]]
        got = run_steps(runner, steps)
        check_request(got["b"], name, toks, dtype, f"needle at {at}, portions and single tokens")
        got = run_steps(runner, [[("c", toks[:edge - 2], [0])]] + [[("c", [t], [0])] for t in toks[edge - 2:edge + 5]])
        check_request(got["c"], name, toks[:edge + 5], dtype, f"needle at {at}, decoded across the edge")
        ref = plain_logits(name, toks)
        other = list(toks)
        other[at] = 2
        d = np.abs(plain_logits(name, other) - ref).max(axis=1)
        inside = [p for p in probes if p > at and p // chunk == at // chunk]
        outside = [p for p in probes if p // chunk != at // chunk]
        assert not inside or d[inside].min() > 0.06 * np.abs(ref).max()
        assert d[outside].max() < 1e-9


# --------------------------------------------------------------------------------------------
# the engine's own entry point, the command line, the trace runner
# --------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_engine(dtype):
    """The engine's own entry point and scheduler: prompts of unequal lengths, more requests than
    slots, greedy tokens.  The plain implementation, reading the engine's sequence, must choose
    the same token wherever its two best logits are clearly apart."""
    from llmario_b200.engine.engine import Engine
    from llmario_b200.sampling import SamplingParams

    for name in ("mix", "shared", "map_128"):
        eng = Engine(model_dir(name), dtype=dtype, page_size=16, cache_tokens=1024, max_requests=2,
                     token_budget=48, context=256)
        prompts = [tokens_for(name, n, 20 + i) for i, n in enumerate((5, 70, 33, 1, 18))]
        outs = eng.generate(prompts, SamplingParams.greedy_params(max_tokens=24, ignore_eos=True))
        margin = 1e-3 if dtype == "float32" else 8e-2
        clear = 0
        for p, o in zip(prompts, outs):
            assert len(o) == 24
            ref = plain_logits(name, list(p) + list(o))
            close = np.nonzero(router_margins(name, list(p) + list(o)) < CLOSE_CALL)[0]
            until = int(close[0]) if len(close) and dtype == "bfloat16" else len(ref)
            for j, tok in enumerate(o):
                if len(p) - 1 + j >= until:
                    break
                l = ref[len(p) - 1 + j]
                top = np.sort(l)[-2:]
                if top[1] - top[0] > margin * np.abs(l).max():
                    clear += 1
                    assert tok == int(np.argmax(l)), f"{name}: token {j} of a request"
        assert clear > (60 if dtype == "float32" else 3)
        assert eng.stats()["graph_replays"] > 0
        eng.runner.cache.check_invariants()


@pytest.mark.gpu
def test_command_line_and_trace_runner(tmp_path):
    """The two programs a user starts: ``llmario-b200 run`` on a Ronurax model folder (greedy ids
    against the plain implementation) and on a preset, and ``bin/trace_run`` (given tokens in steps,
    logits in files), which choose the model class by ``config.json``."""
    import os
    import subprocess
    import sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    name = "mix"
    prompt = tokens_for(name, 19, 40)
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "llmario-b200"), "run",
                        model_dir(name), "--tokens", ",".join(map(str, prompt)), "--max-tokens", "6",
                        "--dtype", "float32", "--page-size", "16", "--context", "128"],
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    out = [int(t) for t in p.stdout.strip().splitlines()[-1].split(",")]
    assert len(out) == 6
    ref = plain_logits(name, prompt + out)
    for j, tok in enumerate(out):
        l = ref[len(prompt) - 1 + j]
        top = np.sort(l)[-2:]
        if top[1] - top[0] > 1e-3 * np.abs(l).max():
            assert tok == int(np.argmax(l))
    # a preset name gives a model with random weights
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "llmario-b200"), "run", "ronurax-tiny",
                        "--prompt-len", "5", "--n", "6", "--dtype", "bfloat16", "--page-size", "16",
                        "--context", "64"], capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert len(p.stdout.strip().splitlines()[-1].split(",")) == 6
    # the trace runner: three requests, portions beside single tokens, a slot given back and taken
    a, b, c = (tokens_for(name, n, 50 + i) for i, n in enumerate((40, 7, 12)))
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:25], "want": [0, 24]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[25:26], "want": [0]},
                                {"id": "b", "tokens": b, "want": [6]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[26:], "want": [13]},
                                {"id": "c", "tokens": c[:2], "want": []}], "end": ["a"]},
        {"step": 3, "entries": [{"id": "c", "tokens": c[2:], "want": [0, 9]}], "end": ["c"]},
    ]
    out_dir = tmp_path / "out"
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", model_dir(name), "--dtype",
                        "float32", "--out", str(out_dir), "--max-tokens", "192"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True,
                       text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb, rc = plain_logits(name, a), plain_logits(name, b), plain_logits(name, c)
    want = {0: np.stack([ra[0], ra[24]]), 1: np.stack([ra[25], rb[6]]), 2: ra[39:40],
            3: np.stack([rc[2], rc[11]])}
    for i, ref in want.items():
        got = np.fromfile(out_dir / f"{i}.f32", dtype="<f4").reshape(ref.shape)
        assert_close(got, ref, "float32", f"trace step {i}")
