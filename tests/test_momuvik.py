"""The Momuvik decoder against the plain float64 implementation (tests/plain/momuvik_plain.py):
every mechanism alone and together, in whole prompts, portions, single decoded tokens, mixed
batches, reused slots and pages, and through the engine's own entry point."""
from __future__ import annotations

import json
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from plain import momuvik_plain as MP
from momuvik_util import (CLOSE_CALL, CONFIGS, CUSTOM, _bf16_values, _weights, assert_close,
                          check_request, config, dense, layer, model_dir, moe, plain_logits,
                          random_config, router_margins, run_steps, runner_for, slack_for,
                          tokens_for, weights)

DTYPES = ("float32", "bfloat16")


# --------------------------------------------------------------------------------------------
# no GPU: configuration, and the plain implementation against itself
# --------------------------------------------------------------------------------------------
def test_configuration_round_trip_and_tensor_names():
    from llmario_b200.config import ConfigError, MomuvikConfig, resolve_architecture
    from llmario_b200.weights.loader import check_tensors, expected_tensors

    for seed in range(4):
        random_config(seed)
    for name, raw in CONFIGS.items():
        assert resolve_architecture(raw) == "Momuvik"
        cfg = MomuvikConfig.from_dict(raw)
        assert MomuvikConfig.from_dict(cfg.to_dict()) == cfg
        assert cfg.to_dict() == raw, name
        spec = cfg.to_spec()
        want = expected_tensors(spec)
        have = {n: a.shape for n, a in weights(name).items()}
        assert set(want) == set(have), name
        check_tensors(spec, have)
        assert len(spec.run_order) == len(raw["layers"])
        for i, call in enumerate(spec.run_order):
            assert spec.layers[call.layer].weight_prefix == f"l{MP.tensors_of(raw, i)}."
            assert call.reads_cache_of is None            # a cache of its own for every layer
        assert len(spec.layers) == sum("weights_of" not in l for l in raw["layers"])
    shared = MomuvikConfig.from_dict(CONFIGS["shared"]).to_spec()
    assert [shared.layers[c.layer].weight_prefix for c in shared.run_order] == \
        ["l2.", "l1.", "l2.", "l1.", "l2."]

    def broken(change, match):
        raw = json.loads(json.dumps(CONFIGS["mix"]))
        change(raw)
        with pytest.raises(ConfigError, match=match):
            MomuvikConfig.from_dict(raw)

    broken(lambda r: r["layers"][0].update(type="conv"), "unsupported type")
    broken(lambda r: r["layers"][0]["mlp"].update(kind="routed"), "mlp kind")
    broken(lambda r: r["layers"][0]["mlp"]["router"].update(top=7), "top")
    broken(lambda r: r["layers"][0]["mlp"]["expert"].pop("limit"), "limit")
    broken(lambda r: r["layers"][1]["mixer"]["rot"].update(dims=18), "dims")
    broken(lambda r: r["layers"][2].update(weights_of=9), "weights_of")
    broken(lambda r: r["layers"][2]["mixer"].update(vdim=17), "differ")
    broken(lambda r: (r["layers"][2].update(weights_of=0), r["layers"][0].update(weights_of=2)), "itself")
    broken(lambda r: r.pop("norm"), "eps")


def test_a_sized_configuration_reads_back():
    from llmario_b200.config import MomuvikConfig
    from llmario_b200.config.momuvik import sized_like

    cfg = sized_like(256, 512, 4, 6, 500, kv_rank=96, rot=32, dim=48)
    assert MomuvikConfig.from_dict(cfg.to_dict()) == cfg
    assert [l.f()["kind"] for l in cfg.layers] == ["dense", "moe", "moe", "dense", "dense", "moe"]


def test_plain_mechanisms():
    """The plain statement against its own definitions."""
    rng = np.random.default_rng(1)
    x = rng.standard_normal((5, 12))
    # rotation: lengths of pairs stay, scores depend on the distance alone, position 0 is identity
    r = MP.rotate_halves(x, np.arange(5), 8, 50.0)
    np.testing.assert_allclose(r[0], x[0])
    np.testing.assert_allclose(r[:, :4] ** 2 + r[:, 4:8] ** 2, x[:, :4] ** 2 + x[:, 4:8] ** 2)
    np.testing.assert_allclose(r[:, 8:], x[:, 8:])
    a, b = rng.standard_normal((1, 8)), rng.standard_normal((1, 8))
    dot = lambda p, q: float(MP.rotate_halves(a, [p], 8, 50.0)[0] @ MP.rotate_halves(b, [q], 8, 50.0)[0])
    assert abs(dot(9, 4) - dot(105, 100)) < 1e-9 and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    # the norm around zero: a stored zero leaves the row at a root mean square of one
    y = MP.norm_around_zero(x, np.zeros(12), 0.0)
    np.testing.assert_allclose(np.mean(y * y, axis=1), 1.0)
    np.testing.assert_allclose(MP.norm_around_zero(x, np.full(12, 0.5), 0.0), 1.5 * y)
    # the sink takes its share of the weights and nothing else
    s = rng.standard_normal((2, 3, 3))
    w = MP.softmax_with_sink(s, np.array([0.3, -80.0]))
    np.testing.assert_allclose(w[1].sum(-1), 1.0)
    np.testing.assert_allclose(w[0].sum(-1), np.exp(s[0]).sum(-1) / (np.exp(s[0]).sum(-1) + np.exp(0.3)))
    # the router: order of the logits, sigmoid weights that are not renormalised
    ids, wt = MP.choose(np.array([[0.1, 2.0, -1.0, 2.0]]), 3)
    assert ids.tolist() == [[1, 3, 0]]
    np.testing.assert_allclose(wt[0], MP.sigmoid(np.array([2.0, 2.0, 0.1])))
    # an expert that is not linear tells a weight on its input from one on its output
    t = {"gate": rng.standard_normal((6, 12)), "up": rng.standard_normal((6, 12)),
         "down": rng.standard_normal((12, 6))}
    on_input, on_output = MP.clamped_expert(0.4 * x, t, "", 1.1), 0.4 * MP.clamped_expert(x, t, "", 1.1)
    assert np.abs(on_input - on_output).max() > 0.1
    big = MP.clamped_expert(100 * x, t, "", 1.1)     # every half at its bound
    assert np.abs(big).max() < 6 * 1.1 * 2.1 * np.abs(t["down"]).max()


def test_plain_constants_matter():
    """Each constant and branch of the configuration moves the plain logits."""
    raw, toks = CONFIGS["mix"], tokens_for("mix", 40, 3)
    w = weights("mix")
    ref = MP.forward(raw, w, toks)

    def moved(change):
        other = json.loads(json.dumps(raw))
        change(other)
        return np.abs(MP.forward(other, w, toks) - ref).max() / np.abs(ref).max()

    assert moved(lambda r: r.update(residual_mult=0.71)) > 1e-3
    assert moved(lambda r: r["embedding"].update(scale=2.6)) > 1e-3
    assert moved(lambda r: r["norm"].update(eps=1e-2)) > 1e-4
    for l in (0, 2):
        assert moved(lambda r: r["layers"][l]["mlp"]["expert"].update(limit=1.5)) > 1e-4
        assert moved(lambda r: r["layers"][l]["mlp"]["shared"].update(limit=1.0)) > 1e-4
        assert moved(lambda r: r["layers"][l]["mlp"].update(shared=None)) > 1e-2
        assert moved(lambda r: r["layers"][l]["mixer"]["rot"].update(base=9000.0)) > 1e-5
        assert moved(lambda r: r["layers"][l]["mixer"].update(scale=0.2)) > 1e-3
    without = dict(w, **{"l0.mix.sink": np.full_like(w["l0.mix.sink"], -80.0)})
    assert np.abs(MP.forward(raw, without, toks) - ref).max() > 1e-2 * np.abs(ref).max()


# --------------------------------------------------------------------------------------------
# kernels of the mechanisms, each against a few lines of NumPy
# --------------------------------------------------------------------------------------------
@pytest.mark.gpu
@pytest.mark.parametrize("E,top", [(3, 1), (6, 2), (16, 4), (70, 8), (5, 5)])
def test_sigmoid_router_kernel(E, top):
    from llmario_b200 import kernels

    rng = np.random.default_rng(E)
    rows = 37
    z = rng.standard_normal((rows, E)) * 3
    z[3] = 0.5                        # all equal: the lowest indices win
    z[4] = 60.0 + np.arange(E)        # every sigmoid rounds to one: the order is still the logits'
    z_d = torch.tensor(z, dtype=torch.float32, device="cuda")
    ids = torch.empty(rows, top, dtype=torch.int32, device="cuda")
    wts = torch.empty(rows, top, dtype=torch.float32, device="cuda")

    def check(zz):
        want, w = MP.choose(zz.double().cpu().numpy(), top)
        assert ids.cpu().numpy().tolist() == want.tolist()
        np.testing.assert_allclose(wts.cpu().numpy(), w, rtol=1e-5)

    kernels.moe_route(z_d, E, top, ids, wts, "sigmoid")
    check(z_d)
    for dtype, width in ((torch.float32, 50), (torch.bfloat16, 256)):
        h = torch.tensor(rng.standard_normal((rows, width)), dtype=dtype, device="cuda")
        w = torch.tensor(rng.standard_normal((E, width)) / 8, dtype=torch.float32, device="cuda")
        z2 = torch.empty(rows, E, dtype=torch.float32, device="cuda")
        kernels.moe_router(h, w, None, E, top, z2, ids, wts, "sigmoid")
        np.testing.assert_allclose(z2.cpu().numpy(), h.double().cpu().numpy() @ w.double().cpu().numpy().T,
                                   rtol=1e-4, atol=1e-4)
        check(z2)
    with pytest.raises(AssertionError):
        kernels.moe_route(z_d, E, top, ids, wts, "sigmoid", torch.zeros(E, device="cuda"))


@pytest.mark.gpu
@pytest.mark.parametrize("rows,E,top,width,ff,limit", [(3, 4, 2, 64, 32, 0.8), (70, 6, 3, 96, 48, 1.5),
                                                       (700, 8, 2, 128, 80, 0.6), (40, 16, 1, 64, 16, 9.0),
                                                       (9, 1, 1, 72, 176, 1.0)])
def test_weighted_input_experts_against_numpy(rows, E, top, width, ff, limit):
    """The clamped form with weights on the inputs: grouped tensor-core products, row-wise kernels
    with either order of an expert's rows, against NumPy; then the silu form with interleaved rows."""
    from llmario_b200 import kernels
    from llmario_b200.parts.feed_forward import interleaved_gate_up

    rng = np.random.default_rng(rows + E)
    b16 = lambda a: torch.tensor(a, dtype=torch.bfloat16, device="cuda")
    h = b16(rng.standard_normal((rows, width)))
    gate, up = b16(rng.standard_normal((E, ff, width)) / 6), b16(rng.standard_normal((E, ff, width)) / 6)
    dn = b16(rng.standard_normal((E, width, ff)) / 8)
    ids = torch.tensor(np.stack([rng.permutation(E)[:top] for _ in range(rows)]), dtype=torch.int32,
                       device="cuda")
    wts = torch.tensor(rng.random((rows, top)) + 0.05, dtype=torch.float32, device="cuda")
    hf, gf, uf, dnf = (a.double().cpu().numpy() for a in (h, gate, up, dn))
    wf, idf = wts.double().cpu().numpy(), ids.cpu().numpy()
    rounded = lambda a: torch.tensor(a).to(torch.bfloat16).double().numpy()

    def reference(silu):
        ref = np.zeros((rows, width))
        for r in range(rows):
            for k in range(top):
                e = idf[r, k]
                s = 1.0 if silu else wf[r, k]
                g, u = s * (gf[e] @ hf[r]), s * (uf[e] @ hf[r])
                if silu:
                    a = g * MP.sigmoid(g) * u
                else:
                    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
                    a = g * MP.sigmoid(1.702 * g) * (u + 1)
                ref[r] += (wf[r, k] if silu else 1.0) * (dnf[e] @ rounded(a))
        return ref

    both = interleaved_gate_up(gate, up)
    plain = torch.cat([gate, up], dim=1).contiguous()
    pairs = rows * top
    bn = kernels.moe_tile(pairs, E)
    tiles = -(-pairs // bn) + E
    pos = torch.empty(pairs, dtype=torch.int32, device="cuda")
    tile_group = torch.empty(tiles, dtype=torch.int32, device="cuda")
    kernels.moe_align(ids, E, bn, pos, tile_group)
    xp = torch.full((tiles * bn, width), float("nan"), dtype=torch.bfloat16, device="cuda")
    scale = torch.full((tiles * bn,), float("nan"), dtype=torch.float32, device="cuda")
    kernels.moe_gather(h, pos, xp, top, wts=wts, row_scale=scale)
    np.testing.assert_array_equal(scale.cpu().numpy()[pos.cpu().numpy()], wts.cpu().numpy().reshape(-1))
    act = torch.empty(tiles * bn, ff, dtype=torch.bfloat16, device="cuda")
    d = torch.empty(tiles * bn, width, dtype=torch.float32, device="cuda")
    for silu in (False, True):
        ref = reference(silu)
        tol = 0.02 * np.abs(ref).max()
        if silu:
            kernels.gemm_grouped(xp, both, act, tile_group, bn, gated=True, interleaved=True)
        else:
            kernels.gemm_grouped(xp, both, act, tile_group, bn, gated=True, interleaved=True,
                                 activation="clamped_swish", limit=limit, row_scale=scale)
        kernels.gemm_grouped(act, dn, d, tile_group, bn, gated=False)
        y = torch.ones(rows, width, dtype=torch.float32, device="cuda")
        kernels.moe_combine(d, pos, wts if silu else None, y, True)
        np.testing.assert_allclose(y.cpu().numpy() - 1.0, ref, atol=tol)
        for w, interleaved in ((both, True), (plain, False)):
            act2 = torch.empty(rows, top, ff, dtype=torch.bfloat16, device="cuda")
            y2 = torch.empty(rows, width, dtype=torch.float32, device="cuda")
            kernels.moe_gate_up_rows(h, w, ids, act2, "silu" if silu else "clamped_swish", limit,
                                     None if silu else wts, interleaved)
            kernels.moe_down_rows(act2, dn, ids, wts if silu else None, y2, False)
            np.testing.assert_allclose(y2.cpu().numpy(), ref, atol=tol)
    kernels.check_tc_status(h.device)


@pytest.mark.gpu
@pytest.mark.parametrize("rows", [1, 5, 17, 60, 200, 700])
@pytest.mark.parametrize("ff,width,limit", [(48, 64, 0.9), (176, 136, 1.7), (320, 96, 30.0)])
def test_clamped_product(rows, ff, width, limit):
    """The gated product with the clamped form in its epilogue: one tile of tokens, several, and the
    CTA-pair kernel."""
    from llmario_b200 import kernels
    from llmario_b200.parts.feed_forward import interleaved_gate_up

    g = torch.Generator(device="cuda").manual_seed(rows + ff)
    rnd = lambda *s: torch.randn(*s, generator=g, device="cuda").to(torch.bfloat16)
    h, gate, up = rnd(rows, width), rnd(ff, width) / 5, rnd(ff, width) / 5
    out = torch.empty(rows, ff, dtype=torch.bfloat16, device="cuda")
    kernels.gate_up_clamped(h, interleaved_gate_up(gate, up), out, limit)
    zg = torch.clamp(h.double() @ gate.double().T, max=limit)
    zu = torch.clamp(h.double() @ up.double().T, -limit, limit)
    ref = zg * torch.sigmoid(1.702 * zg) * (zu + 1)
    assert float((out.double() - ref).abs().max()) < 1e-2 * float(ref.abs().max())
    kernels.check_tc_status(h.device)


def _paged(total, page_size, kd, lengths, rng, entries=2):
    """Key rows of several requests in pages handed out in a shuffled order.  Returns the view and
    a list of float64 key rows per request."""
    n_pages = total // page_size + len(lengths) + 3
    storage = torch.zeros(n_pages, entries, 1, 1, page_size, kd, dtype=torch.bfloat16, device="cuda")
    table = torch.full((len(lengths), n_pages), -1, dtype=torch.int32)
    free = list(rng.permutation(n_pages))
    keys = []
    for r, n in enumerate(lengths):
        rows = torch.tensor(rng.standard_normal((n, kd)), dtype=torch.float32).to(torch.bfloat16)
        keys.append(rows.double().numpy())
        for p in range(-(-n // page_size)):
            page = int(free.pop())
            table[r, p] = page
            part = rows[p * page_size:(p + 1) * page_size]
            storage[page, 1, 0, 0, :len(part)] = part.cuda()
    from llmario_b200.cache.manager import CacheView

    st = storage
    return CacheView(st[0, 1, 0], st[0, 1, -1], st.stride(0), table.cuda(), page_size, 0, st, 1), keys


@pytest.mark.gpu
@pytest.mark.parametrize("kd,vd,H", [(16, 8, 3), (112, 88, 5), (128, 64, 16), (136, 128, 130), (200, 192, 9),
                                     (288, 256, 40), (344, 304, 3), (576, 512, 16), (576, 512, 128), (640, 640, 7)])
@pytest.mark.parametrize("page", [8, 16, 64, 128])
def test_latent_attention_kernel(kd, vd, H, page):
    """Rows of any number of heads over one key row per token: single tokens (keys cut into parts and
    merged), portions that start anywhere, both beside each other, with a sink and with a window."""
    from llmario_b200 import driver, kernels
    from llmario_b200.parts.base import Segment

    rng = np.random.default_rng(kd + H + page)
    lengths = [1, 64, 65, 200, 333]
    view, keys = _paged(sum(lengths), page, kd, lengths, rng)
    sink = torch.tensor(rng.standard_normal(H) * 2, dtype=torch.float32, device="cuda")
    scale = float(1.5 / np.sqrt(kd))
    # (request, tokens of the step): the last ones of the request
    for plan in ([(0, 1), (1, 1), (2, 1), (3, 1), (4, 1)], [(4, 150)], [(3, 2), (4, 1), (2, 65), (1, 30), (0, 1)]):
        for window in (None, 37):
            pos, slot, segments, at = [], [], [], 0
            for r, n in plan:
                start = lengths[r] - n
                segments.append(Segment(r, r, at, n, start))
                pos += list(range(start, start + n))
                slot += [r] * n
                at += n
            ctx = SimpleNamespace(rows=at, max_pos=max(pos), segments=segments, dtype=torch.bfloat16,
                                  tokens=None, shared={},
                                  row_pos=torch.tensor(pos, dtype=torch.int32, device="cuda"),
                                  row_slot=torch.tensor(slot, dtype=torch.int32, device="cuda"))
            q = torch.tensor(rng.standard_normal((at, H * kd)), dtype=torch.float32).to(torch.bfloat16).cuda()
            out = torch.full((at, H * vd), float("nan"), dtype=torch.bfloat16, device="cuda")
            assert kernels.attention_latent_ok(torch.bfloat16, kd, vd, page)
            driver.latent_attention(ctx, q, out, view, H, kd, vd, scale, window, sink if window is None else None)
            kernels.check_tc_status("cuda:0")
            qf = q.double().cpu().numpy().reshape(at, H, kd)
            got = out.double().cpu().numpy().reshape(at, H, vd)
            assert np.isfinite(got).all()
            for t in rng.choice(at, size=min(at, 24), replace=False):
                lo = 0 if window is None else max(0, pos[t] + 1 - window)
                k = keys[slot[t]][lo:pos[t] + 1]
                s = qf[t] @ k.T * scale
                z = sink.double().cpu().numpy() if window is None else np.full(H, -np.inf)
                m = np.maximum(s.max(1), z)
                e = np.exp(s - m[:, None])
                ref = (e / (e.sum(1) + np.exp(z - m))[:, None]) @ k[:, :vd]
                np.testing.assert_allclose(got[t], ref, atol=0.02 * max(1.0, np.abs(ref).max()),
                                           err_msg=f"row {t} of {plan}, window {window}")


# --------------------------------------------------------------------------------------------
# whole models through the step function
# --------------------------------------------------------------------------------------------
NAMES = sorted(n for n in CONFIGS if not n.startswith("random"))


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(name, dtype):
    """Every position of a prompt that spans several pages, the first tokens included."""
    toks = tokens_for(name, 110, 1)
    runner = runner_for(name, dtype)
    got = run_steps(runner, [[("a", toks, range(len(toks)))]])
    check_request(got["a"], name, toks, dtype, "whole prompt")
    runner.cache.check_invariants()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompt_then_single_tokens(name, dtype):
    """A prompt, then tokens one by one through recorded steps, across page borders."""
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
    """Portions cut in the middle of pages, down to two tokens; then single tokens."""
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
@pytest.mark.parametrize("name", ("mix", "shared", "odd", "moe_top1", "row_128", "row_288", "many_heads"))
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
@pytest.mark.parametrize("name", ("mix", "moe", "row_128", "row_344", "row_576"))
def test_a_long_prompt_over_the_engine_page(name, dtype):
    """A prompt of several hundred tokens with the engine's default page of 64, then a second
    portion that starts inside a page, then single tokens."""
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
@pytest.mark.parametrize("name", ("mix", "shared", "row_288"))
def test_long_decoding(name, dtype):
    """Hundreds of single tokens behind a one-token prompt."""
    toks = tokens_for(name, 260, 4)
    runner = runner_for(name, dtype, page_size=32, cache_tokens=512)
    got = run_steps(runner, [[("a", [t], [0])] for t in toks])
    check_request(got["a"], name, toks, dtype, "long decoding")


@pytest.mark.gpu
def test_a_request_alone_and_in_a_batch_gives_the_same_bits():
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


# --------------------------------------------------------------------------------------------
# a key that stands out
# --------------------------------------------------------------------------------------------
def needle_model(kv_rank: int, rot: int, heads: int) -> str:
    """A layer whose weights make one score stand out.  Token 0 is the needle: its latent is one
    large direction, which head 0's key map turns into a key that the probe's (token 1's) query
    points along; every other token has neither.  A probe's output is then decided by whether it
    finds the needle, however far back.  The sinks take visible weight where no needle is."""
    name = f"needle{kv_rank}_{rot}_{heads}"
    if name not in CONFIGS:
        CONFIGS[name] = config([layer(heads=heads, dim=16, rot_dim=rot, vdim=24, q_rank=24, kv_rank=kv_rank,
                                      scale=1.0, mlp=dense(40))], width=64, vocab=64, embed_scale=1.5, mult=0.9)
        w = {n: a.copy() for n, a in _weights(CONFIGS[name], 7).items()}
        w["embed"][:, :2] = 0.0
        w["embed"][0, 0] = 2.0
        w["embed"][1, 1] = 2.0
        x = "l0.mix."
        for m in ("dq", "dkv"):
            w[x + m] *= 0.25
            w[x + m][:, :2] = 0.0
        w[x + "dkv"][5, 0] = 20.0       # the needle's latent: channel 5
        w[x + "dq"][3, 1] = 20.0        # the probe's query latent: channel 3
        w[x + "uv"][:24, 5] *= 4.0      # head 0's value of the needle
        w[x + "uk"] *= 0.15
        w[x + "uq"] *= 0.15
        peak = 12.0 / np.sqrt(kv_rank * 24)
        w[x + "uk"][7, 5] = 1.0         # head 0, key channel 7 <- latent channel 5
        w[x + "uq"][7, 3] = peak        # head 0, plain query channel 7 <- query latent channel 3
        w[x + "sink"][:] = 3.0
        CUSTOM[name] = _bf16_values(w)
    return name


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("page", (16, 64))
@pytest.mark.parametrize("kv_rank,rot,heads", [(40, 16, 3), (48, 16, 2), (112, 24, 4), (256, 40, 6)])
def test_a_key_that_stands_out_far_back(dtype, page, kv_rank, rot, heads):
    """Needles at the very start, on the last and the first place of a page, and just before the
    probe; the probes in the prompt, in a later portion and decoded one by one.  Leaving the needle
    out moves the probe's logits visibly (so does leaving the sink out where there is no needle)."""
    from llmario_b200 import driver

    name = needle_model(kv_rank, rot, heads)
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
        before = driver.kernel_counts()
        runner = runner_for(name, dtype, page_size=page, cache_tokens=1024)
        got = run_steps(runner, [[("a", toks, range(n))]])
        check_request(got["a"], name, toks, dtype, f"needle at {at}, whole prompt")
        after = driver.kernel_counts()
        if dtype == "bfloat16" and kv_rank != 48:
            assert after["latent"] > before["latent"]      # the kernel for latents ran
        steps = [[("b", toks[:190], [150])], [("b", toks[190:192], [0, 1])], [("b", toks[192:270], range(78))]] \
            + [[("b", [t], [0])] for t in toks[270:]]
        got = run_steps(runner, steps)
        check_request(got["b"], name, toks, dtype, f"needle at {at}, portions and single tokens")
        ref = plain_logits(name, toks)
        other = list(toks)
        other[at] = 2
        d = np.abs(plain_logits(name, other) - ref).max(axis=1)
        assert d[seen].min() > 0.1 * np.abs(ref).max()
    w2 = dict(weights(name), **{"l0.mix.sink": np.full(heads, -80.0)})
    assert np.abs(MP.forward(CONFIGS[name], w2, toks) - ref).max() > 0.05 * np.abs(ref).max()


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

    for name in ("mix", "shared"):
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
        assert clear > (60 if dtype == "float32" else 5)
        assert eng.stats()["graph_replays"] > 0
        eng.runner.cache.check_invariants()


@pytest.mark.gpu
def test_command_line_and_trace_runner(tmp_path):
    """The two programs a user starts: ``llmario-b200 run`` on a Momuvik model folder (greedy ids
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
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "llmario-b200"), "run", "momuvik-tiny",
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
