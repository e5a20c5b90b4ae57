"""Momuvik beside Runidra (the closest of the other designs: attention through latents with a sink,
routed experts beside a shared one) and Qwen3 at equal sizes: prompt and decode rates of whole
models with random weights, and the design's own kernels one by one against the memory or tensor
roofline, each beside the like kernel of another design.

    python -m llmario_b200.benchmarks.momuvik [--sizes 0.6b,8b] [--layers 8] [--kernels]

A Momuvik model of a size has the width, feed-forward width, attention heads and number of layers
of the Qwen3 preset of that name; a token leaves a latent of 512 and a rotated part of 64 in the
cache, heads have 128 unrotated channels and values of 128; the feed-forwards repeat (dense, routed
experts twice, dense), a token using two of eight experts and a shared one, each a third of the
dense width (``config.momuvik.sized_like``).  ``bench.py --workload momuvik`` prints the same record
as its JSON line.
"""
from __future__ import annotations

import argparse
import json
import sys
from types import SimpleNamespace
from typing import Any, Dict, List

from .runidra import runidra_config
from .vunasun import SIZES, _rates, _time


def momuvik_config(preset: Dict[str, Any], layers: int, vocab: int = 32768):
    """The Momuvik configuration with the sizes of a Qwen3 preset."""
    from ..config.momuvik import sized_like

    return sized_like(preset["hidden_size"], preset["intermediate_size"],
                      preset["num_attention_heads"], layers, vocab)


def compare(sizes: List[str], layers: int, batch: int = 8, prompt_len: int = 1024,
            prefill_tokens: int = 2048, steps: int = 64, warmup: int = 24,
            page_size: int = 64) -> Dict[str, Any]:
    import torch

    from ..cli import PRESETS
    from ..engine.model import Model
    from .roofline import peaks

    pk = peaks()
    out: Dict[str, Any] = {}
    for size in sizes:
        preset = dict(PRESETS[SIZES[size]], vocab_size=32768)
        rec: Dict[str, Any] = {}
        for which in ("qwen3", "runidra", "momuvik"):
            if which == "qwen3":
                from ..config import Qwen3Config

                cfg = Qwen3Config.from_dict(dict(preset, num_hidden_layers=layers,
                                                 tie_word_embeddings=False,
                                                 architectures=["Qwen3ForCausalLM"]))
            elif which == "runidra":
                cfg = runidra_config(preset, layers)
            else:
                cfg = momuvik_config(preset, layers)
            model = Model.random(cfg, seed=0, dtype="bfloat16", device="cuda:0")
            r = _rates(model, page_size, batch, prompt_len, prefill_tokens, steps, warmup)
            # a decode step streams the weights once (all experts counted) and every live
            # request's recurrent state twice
            moved = r["weight_bytes"] + 2 * batch * r["state_bytes_per_request"]
            r["decode_frac_of_copy_peak"] = round(moved / (r["decode_ms"] / 1e3) / (pk["hbm_gbs"] * 1e9), 3)
            rec[which] = r
            del model
            torch.cuda.empty_cache()
        out[size] = rec
    return {"layers": layers, "batch": batch, "prompt_len": prompt_len,
            "prefill_tokens": prefill_tokens, "page_size": page_size, "peaks": pk["source"],
            "sizes": out}


class _View:
    """A paged cache of one layer call as the kernels take it (one or two planes)."""

    def __init__(self, storage, table, page):
        self.storage, self.slot = storage, 0
        self.k, self.v = storage[0, 0, 0], storage[0, 0, -1]
        self.page_stride, self.block_table, self.page_size = storage.stride(0), table, page


def kernel_table(width: int = 4096, ff: int = 12288, tokens: int = 2048, batch: int = 64,
                 heads: int = 32, context: int = 4096, attention_only: bool = False
                 ) -> List[Dict[str, Any]]:
    """The design's own kernels, each alone at the sizes of ``momuvik_config`` for ``width``, with
    the bytes they must move (or the operations they must do) and the fraction of the measured
    copy (or tensor) rate; beside each the like kernel of another design.  The prompt case is a
    portion of ``tokens`` rows of one request that starts at position 0; the decode case is
    ``batch`` requests at position ``context`` - 1."""
    import torch

    from .. import driver, kernels
    from ..parts.base import Segment
    from ..parts.feed_forward import interleaved_gate_up
    from .roofline import peaks

    dev = "cuda:0"
    pk = peaks()
    flush = torch.empty(160 << 20, dtype=torch.uint8, device=dev)
    rows_out: List[Dict[str, Any]] = []

    def rec(name, us, nbytes, flops=0, note=""):
        r = {"kernel": name, "us": round(us, 2), "bytes": int(nbytes),
             "gb_s": round(nbytes / us / 1e3, 1),
             "frac_of_copy_peak": round(nbytes / (us * 1e-6) / (pk["hbm_gbs"] * 1e9), 3), "note": note}
        if flops:
            r["tflops"] = round(flops / us / 1e6, 1)
            r["frac_of_tensor_peak"] = round(flops / (us * 1e-6) / (pk["bf16_tflops"] * 1e12), 3)
        rows_out.append(r)

    f32 = lambda *s: torch.randn(*s, dtype=torch.float32, device=dev)
    b16 = lambda *s: torch.randn(*s, dtype=torch.bfloat16, device=dev)
    ints = lambda a: torch.tensor(a, dtype=torch.int32, device=dev)
    C, R, D, Vd, Rq, page = 512, 64, 128, 128, max(64, width // 4), 64
    kd = C + R
    for label, rows, single in ((f"prompt of {tokens}", tokens, False),
                                (f"decode, batch {batch} at position {context - 1}", batch, True)):
        live = rows if single else 1
        length = context if single else tokens
        pos = [context - 1] * rows if single else list(range(rows))
        slot = list(range(rows)) if single else [0] * rows
        segments = [Segment(i, i, i, 1, context - 1) for i in range(rows)] if single \
            else [Segment(0, 0, 0, rows, 0)]

        def ctx():
            return SimpleNamespace(rows=rows, max_pos=max(pos), segments=segments, shared={},
                                   dtype=torch.bfloat16, tokens=None, row_pos=ints(pos),
                                   row_slot=ints(slot))

        per = -(-length // page)
        # ---- attention: over latents, and the Qwen3 path's at the same number of heads
        table = torch.arange(live * per, dtype=torch.int32, device=dev).view(live, per)
        pairs = sum(p + 1 for p in pos)
        c = ctx()
        for name, H, key_dim, vd, ph in ((f"attention over latents, {heads} heads on key rows of {kd}", heads, kd, C, 1),
                                         (f"attention over latents, 16 heads on key rows of {kd}", 16, kd, C, 1),
                                         ("attention over latents, 16 heads on key rows of 128", 16, 128, 64, 1),
                                         ("attention over latents, 16 heads on key rows of 288", 16, 288, 256, 1),
                                         (f"attention of the Qwen3 path, {heads} on 8 key heads of 128", heads, 128, 128, 8),
                                         ("attention of Runidra, 16 heads on key rows of 128 with a sink", 16, 128, 64, 0)):
            planes = 1 if ph == 1 else 2
            kv = max(1, ph)
            storage = b16(live * per, 1, planes, kv, page, key_dim) * 0.3
            view = _View(storage, table, page)
            whole = vd if ph == 1 else key_dim
            q = b16(rows, H * key_dim) * 0.3
            out = torch.empty(rows, H * whole, dtype=torch.bfloat16, device=dev)
            sink = f32(H) if ph != 8 else None
            if ph == 1:
                fn = lambda: driver.latent_attention(c, q, out, view, H, key_dim, vd, key_dim ** -0.5, None, sink)
            else:
                fn = lambda: driver.attention(c, q, out, view, H, kv, key_dim, key_dim ** -0.5, None, sink=sink)
            us = _time(fn, flush=flush)
            moved = live * length * kv * key_dim * planes * 2 + rows * H * (key_dim + whole) * 2
            rec(f"{name} ({label})", us, moved, flops=2.0 * pairs * H * (key_dim + (vd if ph == 1 else key_dim)))
            del storage, view, q, out
        if attention_only:
            continue
        # ---- around it
        row_pos, row_slot = ints(pos), ints(slot)
        storage = torch.zeros(live * per, 1, 1, 1, page, kd, dtype=torch.bfloat16, device=dev)
        view = _View(storage, table, page)
        down, angles = f32(rows, Rq + kd), f32(rows, R // 2, 2)
        cq = torch.empty(rows, Rq, dtype=torch.bfloat16, device=dev)
        gq, gc = f32(Rq), f32(C)
        us = _time(lambda: kernels.latent_store(down, gq, gc, angles, cq, view, row_slot, row_pos, Rq, C, R, 1e-6),
                   flush=flush)
        rec(f"latent_store: two norms, rotation, cache write ({label})", us, rows * ((Rq + kd) * 4 + (Rq + kd) * 2))
        q32 = f32(rows, heads * (D + R))
        q_plain = torch.empty(rows, heads * D, dtype=torch.bfloat16, device=dev)
        q_full = torch.empty(rows, heads * kd, dtype=torch.bfloat16, device=dev)
        us = _time(lambda: kernels.latent_query(q32, angles, q_plain, q_full, heads, D, R, C), flush=flush)
        rec(f"latent_query: rounding and rotation ({label})", us, rows * heads * (D + R) * 6)
        kmap, vmap = b16(heads, C, D) * 0.1, b16(heads, Vd, C) * 0.1
        us = _time(lambda: kernels.head_linear(q_plain.view(rows, heads, D), kmap,
                                               q_full.view(rows, heads, kd)[:, :, :C]), flush=flush)
        rec(f"head_linear: the heads' key maps on the queries ({label})", us,
            rows * heads * (D + C) * 2 + heads * C * D * 2, flops=2.0 * rows * heads * C * D)
        mixed, out = b16(rows, heads * C), torch.empty(rows, heads * Vd, dtype=torch.bfloat16, device=dev)
        us = _time(lambda: kernels.head_linear(mixed.view(rows, heads, C), vmap, out.view(rows, heads, Vd)), flush=flush)
        rec(f"head_linear: the heads' value maps on the output ({label})", us,
            rows * heads * (Vd + C) * 2 + heads * C * Vd * 2, flops=2.0 * rows * heads * C * Vd)
        del storage, view, q32, q_plain, q_full, mixed, out
        # ---- the residual with its constant, and the norm that follows
        h16 = torch.empty(rows, width, dtype=torch.bfloat16, device=dev)
        wn, y = f32(width), f32(rows, width)
        for S in (1, 2):
            xs, one = f32(S, rows, width), torch.ones(S, dtype=torch.float32, device=dev)
            mix = torch.eye(S, dtype=torch.float32, device=dev)
            us = _time(lambda: kernels.stream_step(xs, y=y, mix=mix, out_coef=one * 0.5, in_coef=one, weight=wn,
                                                   eps=1e-6, out=h16), flush=flush)
            rec(f"stream_step: write + read + norm, {S} stream{'s' * (S > 1)} ({label})", us,
                rows * width * (8 * S + 4 + 2), note="" if S == 1 else "Runidra's")
        x1 = f32(rows, width)
        us = _time(lambda: kernels.rms_norm(x1, wn, h16, 1e-6), flush=flush)
        rec(f"rms_norm, the Qwen3 path's ({label})", us, rows * width * 6)
        # ---- routed experts
        E, top, eff = 8, 2, max(16, ff // 3 // 16 * 16)
        h = b16(rows, width)
        wr, z = f32(E, width), torch.empty(rows, E, dtype=torch.float32, device=dev)
        ids = torch.empty(rows, top, dtype=torch.int32, device=dev)
        wts = torch.empty(rows, top, dtype=torch.float32, device=dev)
        for name, mode in (("softmax over the chosen (Runidra)", "softmax_chosen"), ("sigmoid", "sigmoid")):
            us = _time(lambda: kernels.moe_router(h, wr, None, E, top, z, ids, wts, mode), flush=flush)
            rec(f"moe_router, {name} ({label})", us, rows * (width * 2 + E * 4 + top * 8) + E * width * 4)
        bn = kernels.moe_tile(rows * top, E)
        tiles = -(-rows * top // bn) + E
        ppos, tgroup = torch.empty(rows * top, dtype=torch.int32, device=dev), torch.empty(tiles, dtype=torch.int32, device=dev)
        us = _time(lambda: kernels.moe_align(ids, E, bn, ppos, tgroup), flush=flush)
        rec(f"moe_align ({label})", us, rows * top * 8)
        xp = torch.zeros(tiles * bn, width, dtype=torch.bfloat16, device=dev)
        scale = torch.ones(tiles * bn, dtype=torch.float32, device=dev)
        us = _time(lambda: kernels.moe_gather(h, ppos, xp, top, wts=wts, row_scale=scale), flush=flush)
        rec(f"moe_gather with the weights ({label})", us, rows * top * width * 2 + rows * width * 2)
        gate, up, dn = b16(E, eff, width) * 0.02, b16(E, eff, width) * 0.02, b16(E, width, eff) * 0.02
        both, stacked = interleaved_gate_up(gate, up), torch.cat([gate, up], dim=1).contiguous()
        used = len(set(ids.flatten().tolist()))
        act = torch.empty(tiles * bn, eff, dtype=torch.bfloat16, device=dev)
        work = dict(flops=2.0 * rows * top * 2 * eff * width)
        moved = used * 2 * eff * width * 2 + rows * top * (width + eff) * 2
        us = _time(lambda: kernels.gemm_grouped(xp, both, act, tgroup, bn, gated=True, interleaved=True,
                                                activation="clamped_swish", limit=7.0, row_scale=scale), flush=flush)
        rec(f"grouped gate/up, clamped, weights on the input ({label})", us, moved, **work)
        us = _time(lambda: kernels.gemm_grouped(xp, both, act, tgroup, bn, gated=True, interleaved=True), flush=flush)
        rec(f"grouped gate/up, silu ({label})", us, moved, note="Runidra's", **work)
        us = _time(lambda: kernels.gemm_grouped(xp, stacked, act, tgroup, bn, gated=True), flush=flush)
        rec(f"grouped gate/up, silu, rows not interleaved ({label})", us, moved, note="as before", **work)
        d = torch.empty(tiles * bn, width, dtype=torch.float32, device=dev)
        us = _time(lambda: kernels.gemm_grouped(act, dn, d, tgroup, bn, gated=False), flush=flush)
        rec(f"grouped down ({label})", us, used * eff * width * 2 + rows * top * (eff * 2 + width * 4),
            flops=2.0 * rows * top * eff * width)
        for name, w in (("weights one", None), ("with weights (Runidra)", wts)):
            us = _time(lambda: kernels.moe_combine(d, ppos, w, y, True), flush=flush)
            rec(f"moe_combine, {name} ({label})", us, rows * width * (top * 4 + 8))
        act1 = torch.empty(rows, eff, dtype=torch.bfloat16, device=dev)
        for name, fn in (("clamped", lambda: kernels.gate_up_clamped(h, both[0], act1, 7.0)),
                         ("silu (the Qwen3 path's)", lambda: kernels.gemm_tcgen05(h, both[0], act1, 3, eff))):
            us = _time(fn, flush=flush)
            rec(f"gate/up product, {name} ({label})", us, 2 * eff * width * 2 + rows * (width + eff) * 2,
                flops=2.0 * rows * 2 * eff * width)
        del gate, up, dn, both, stacked, xp, act, d
    return rows_out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--sizes", default="0.6b,8b")
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--kernels", action="store_true", help="only the table of kernels")
    ap.add_argument("--attention", action="store_true", help="only the attention kernels of the table")
    ap.add_argument("--tokens", type=int, default=2048, help="tokens of the table's prompt portion")
    a = ap.parse_args(argv)
    rec: Dict[str, Any] = {}
    if not (a.kernels or a.attention):
        rec = compare([s for s in a.sizes.split(",") if s], a.layers, batch=a.batch)
    rec["kernels"] = kernel_table(tokens=a.tokens, attention_only=a.attention)
    json.dump(rec, sys.stdout, indent=1)
    print()
    return 0


if __name__ == "__main__":
    sys.exit(main())
