"""Ronurax beside Momuvik (the closest of the other designs: attention through latents, routed
experts) and Qwen3 at equal sizes: prompt and decode rates of whole models with random weights, and
the design's own kernels one by one against the memory or tensor roofline, each beside the like
kernel of another design.

    python -m llmario_b200.benchmarks.ronurax [--sizes 0.6b,8b] [--layers 8] [--kernels]

A Ronurax model of a size has the width, feed-forward width, heads and number of layers of the
Qwen3 preset of that name; layers repeat (latent attention three times, attention with two maps in
chunks of 1,024); a token leaves a latent of 512 and a rotated part of 64 in the cache of a latent
layer and the Qwen3 preset's key and value rows in the others; every layer has eight routed experts in
four groups of which two are kept, a token using two experts of half the feed-forward width
(``config.ronurax.sized_like``).  ``bench.py --workload ronurax`` prints the same record as its JSON
line.
"""
from __future__ import annotations

import argparse
import json
import sys
from types import SimpleNamespace
from typing import Any, Dict, List

from .momuvik import _View, momuvik_config
from .vunasun import SIZES, _rates, _time


def ronurax_config(preset: Dict[str, Any], layers: int, vocab: int = 32768):
    """The Ronurax configuration with the sizes of a Qwen3 preset."""
    from ..config.ronurax import sized_like

    return sized_like(preset["hidden_size"], preset["intermediate_size"],
                      preset["num_attention_heads"], preset["num_key_value_heads"],
                      preset["head_dim"], layers, vocab)


def compare(sizes: List[str], layers: int, batch: int = 8, prompt_len: int = 1024,
            prefill_tokens: int = 2048, steps: int = 64, warmup: int = 24,
            page_size: int = 64) -> Dict[str, Any]:
    import torch

    from ..cli import PRESETS
    from ..config import Qwen3Config
    from ..engine.model import Model
    from .roofline import peaks

    pk = peaks()
    out: Dict[str, Any] = {}
    for size in sizes:
        preset = dict(PRESETS[SIZES[size]], vocab_size=32768)
        rec: Dict[str, Any] = {}
        for which in ("qwen3", "momuvik", "ronurax"):
            if which == "qwen3":
                cfg = Qwen3Config.from_dict(dict(preset, num_hidden_layers=layers,
                                                 tie_word_embeddings=False,
                                                 architectures=["Qwen3ForCausalLM"]))
            else:
                cfg = (momuvik_config if which == "momuvik" else ronurax_config)(preset, layers)
            model = Model.random(cfg, seed=0, dtype="bfloat16", device="cuda:0")
            r = _rates(model, page_size, batch, prompt_len, prefill_tokens, steps, warmup)
            # a decode step streams the weights once (all experts counted)
            r["decode_frac_of_copy_peak"] = round(
                r["weight_bytes"] / (r["decode_ms"] / 1e3) / (pk["hbm_gbs"] * 1e9), 3)
            rec[which] = r
            del model
            torch.cuda.empty_cache()
        out[size] = rec
    return {"layers": layers, "batch": batch, "prompt_len": prompt_len,
            "prefill_tokens": prefill_tokens, "page_size": page_size, "peaks": pk["source"],
            "sizes": out}


def kernel_table(width: int = 4096, ff: int = 12288, tokens: int = 2048, batch: int = 64,
                 heads: int = 32, kv_heads: int = 8, context: int = 4096, chunk: int = 1024
                 ) -> List[Dict[str, Any]]:
    """The design's own kernels, each alone at the sizes of ``ronurax_config`` for ``width``, with
    the bytes they must move (or the operations they must do) and the fraction of the measured
    copy (or tensor) rate; beside each the like kernel of another design.  The prompt case is a
    portion of ``tokens`` rows of one request that starts at position 0; the decode case is
    ``batch`` requests at position ``context`` - 1, the last of a chunk."""
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
    C, R, D, V, page, hd = 512, 64, 128, 128, 64, 128
    kd, Rq, half = C + R, max(64, width // 4), hd // 2
    for label, rows, single in ((f"prompt of {tokens}", tokens, False),
                                (f"decode, batch {batch} at position {context - 1}", batch, True)):
        live, length = (rows, context) if single else (1, tokens)
        pos = [context - 1] * rows if single else list(range(rows))
        slot = list(range(rows)) if single else [0] * rows
        segments = [Segment(i, i, i, 1, context - 1) for i in range(rows)] if single \
            else [Segment(0, 0, 0, rows, 0)]
        row_pos, row_slot = ints(pos), ints(slot)
        c = SimpleNamespace(rows=rows, max_pos=max(pos), segments=segments, shared={}, tokens=None,
                            dtype=torch.bfloat16, row_pos=row_pos, row_slot=row_slot)
        per = -(-length // page)
        table = torch.arange(live * per, dtype=torch.int32, device=dev).view(live, per)
        # ---- attention with two maps in chunks, and the Qwen3 path's with the same mask and without
        storage = b16(live * per, 1, 2, kv_heads, page, hd) * 0.3
        view = _View(storage, table, page)
        seen = {n: [p % n + 1 if n else p + 1 for p in pos] for n in (chunk, 0)}
        for name, H, mask, need in (
                (f"attention with two maps in chunks of {chunk}, {heads} heads", 2 * heads, chunk, half + V),
                (f"attention of the Qwen3 path in chunks of {chunk}, {heads} heads", heads, chunk, 2 * hd),
                (f"attention of the Qwen3 path, {heads} heads", heads, 0, 2 * hd)):
            q, out = b16(rows, H * hd) * 0.3, torch.empty(rows, H * hd, dtype=torch.bfloat16, device=dev)
            us = _time(lambda: driver.attention(c, q, out, view, H, kv_heads, hd, hd ** -0.5, -mask if mask else None),
                       flush=flush)
            keys = sum(seen[mask]) if single else length
            rec(f"{name} ({label})", us, keys * kv_heads * hd * 4 + rows * H * hd * 4,
                flops=2.0 * sum(seen[mask]) * H * need,
                note="operations of the design (the zeros of a map's query row not counted)" if H > heads else "")
            del q, out
        # ---- what makes its queries and keys, and what follows
        angles = f32(rows, half // 2, 2)
        qw, kw = f32(half), f32(half)
        proj = f32(rows, 2 * heads * half + 2 * kv_heads * half + kv_heads * hd)
        bias = [f32(n) for n in (2 * heads * half, 2 * kv_heads * half, kv_heads * hd)]
        q_out = torch.empty(rows, 2 * heads * hd, dtype=torch.bfloat16, device=dev)
        a, b = 2 * heads * half, 2 * heads * half + 2 * kv_heads * half
        us = _time(lambda: kernels.qkv_store(proj[:, :a], proj[:, a:b], proj[:, b:], q_out, view, row_slot, row_pos,
                                             heads, kv_heads, half, V, hd, kernels.NORM_PER_HEAD, qw, kw, 1e-6, half,
                                             angles, maps=2, biases=tuple(bias)), flush=flush)
        rec(f"qkv_store, two maps: biases, norms, rotation, stores ({label})", us,
            rows * (proj.shape[1] * 4 + 2 * heads * hd * 2 + 2 * kv_heads * hd * 2))
        wide, q1 = f32(rows, (heads + 2 * kv_heads) * hd), torch.empty(rows, heads * hd, dtype=torch.bfloat16, device=dev)
        an1, w1 = f32(rows, hd // 2, 2), f32(hd)
        a1, b1 = heads * hd, (heads + kv_heads) * hd
        us = _time(lambda: kernels.qkv_store(wide[:, :a1], wide[:, a1:b1], wide[:, b1:], q1, view, row_slot, row_pos,
                                             heads, kv_heads, hd, hd, hd, kernels.NORM_PER_HEAD, w1, w1, 1e-6, hd, an1),
                   flush=flush)
        rec(f"qkv_store, one map (Pavatar's) ({label})", us, rows * (wide.shape[1] * 4 + (heads + 2 * kv_heads) * hd * 2))
        maps, out = b16(rows, 2 * heads * hd), torch.empty(rows, heads * V, dtype=torch.bfloat16, device=dev)
        us = _time(lambda: kernels.two_map_heads(maps, out, heads, V, 0.4, 0.3, 1e-6), flush=flush)
        rec(f"two_map_heads: difference and norm per head ({label})", us, rows * heads * V * 6)
        o32, g32, wv = f32(rows, heads * V), f32(rows, heads * V), f32(V)
        us = _time(lambda: kernels.gated_group_norm(o32, g32, wv, out, V, 1e-6, False), flush=flush)
        rec(f"gated_group_norm (Vunasun's) ({label})", us, rows * heads * V * 10)
        del storage, view, proj, q_out, wide, q1, maps, o32, g32
        # ---- attention through latents
        storage = b16(live * per, 1, 1, 1, page, kd) * 0.3
        view = _View(storage, table, page)
        q, mixed = b16(rows, heads * kd) * 0.3, torch.empty(rows, heads * C, dtype=torch.bfloat16, device=dev)
        sink = f32(heads)
        for name, s in (("attention over latents", None), ("attention over latents with a sink (Momuvik's)", sink)):
            us = _time(lambda: driver.latent_attention(c, q, mixed, view, heads, kd, C, kd ** -0.5, None, s), flush=flush)
            rec(f"{name}, {heads} heads on key rows of {kd} ({label})", us,
                live * length * kd * 2 + rows * heads * (kd + C) * 2, flops=2.0 * sum(seen[0]) * heads * (kd + C))
        angles = f32(rows, R // 2, 2)
        nq = heads * (D + R)
        proj = f32(rows, nq + heads * V + kd)
        gain = f32(C)
        q_plain = torch.empty(rows, heads * D, dtype=torch.bfloat16, device=dev)
        us = _time(lambda: kernels.latent_prepare(proj, 0, nq + heads * V, gain, angles, q_plain, q, view, row_slot,
                                                  row_pos, heads, D, R, C, 1e-6), flush=flush)
        rec(f"latent_prepare: queries and key row in one launch ({label})", us, rows * (nq + kd) * 6)
        down, cq, gq = f32(rows, Rq + kd), torch.empty(rows, Rq, dtype=torch.bfloat16, device=dev), f32(Rq)
        us = _time(lambda: kernels.latent_store(down, gq, gain, angles, cq, view, row_slot, row_pos, Rq, C, R, 1e-6),
                   flush=flush)
        rec(f"latent_store (Momuvik's) ({label})", us, rows * (Rq + kd) * 6)
        q32 = f32(rows, nq)
        us = _time(lambda: kernels.latent_query(q32, angles, q_plain, q, heads, D, R, C), flush=flush)
        rec(f"latent_query (Momuvik's) ({label})", us, rows * nq * 6)
        kmap, vmap = b16(heads, C, D) * 0.1, b16(heads, V, C) * 0.1
        us = _time(lambda: kernels.head_linear(q_plain.view(rows, heads, D), kmap,
                                               q.view(rows, heads, kd)[:, :, :C]), flush=flush)
        rec(f"head_linear: the heads' key maps, as Momuvik's ({label})", us,
            rows * heads * (D + C) * 2 + heads * C * D * 2, flops=2.0 * rows * heads * C * D)
        us = _time(lambda: kernels.head_linear(mixed.view(rows, heads, C), vmap, out.view(rows, heads, V)), flush=flush)
        rec(f"head_linear: the heads' value maps, as Momuvik's ({label})", us,
            rows * heads * (V + C) * 2 + heads * C * V * 2, flops=2.0 * rows * heads * C * V)
        us = _time(lambda: kernels.channel_gate(out, proj[:, nq:nq + heads * V]), flush=flush)
        rec(f"channel_gate (as Pavatar's) ({label})", us, rows * heads * V * 8)
        del storage, view, q, mixed, proj, q_plain, q32
        # ---- norms
        h = torch.empty(rows, width, dtype=torch.bfloat16, device=dev)
        x1, wn, bn_ = f32(rows, width), f32(width), f32(width)
        us = _time(lambda: kernels.layer_norm(x1, wn, bn_, h, 1e-6), flush=flush)
        rec(f"layer_norm ({label})", us, rows * width * 6)
        us = _time(lambda: kernels.rms_norm(x1, wn, h, 1e-6), flush=flush)
        rec(f"rms_norm, the Qwen3 path's ({label})", us, rows * width * 6)
        # ---- routed experts
        E, top, eff = 8, 2, max(16, ff // 2 // 16 * 16)
        wr, z = f32(E, width), torch.empty(rows, E, dtype=torch.float32, device=dev)
        ids = torch.empty(rows, top, dtype=torch.int32, device=dev)
        wts = torch.empty(rows, top, dtype=torch.float32, device=dev)
        for name, mode, groups in (("sigmoid (Momuvik's)", "sigmoid", None),
                                   ("softmax over all, two of four groups", "softmax_all", (4, 2))):
            us = _time(lambda: kernels.moe_router(h, wr, None, E, top, z, ids, wts, mode, groups=groups), flush=flush)
            rec(f"moe_router, {name} ({label})", us, rows * (width * 2 + E * 4 + top * 8) + E * width * 4)
        bn = kernels.moe_tile(rows * top, E)
        tiles = -(-rows * top // bn) + E
        ppos, tgroup = (torch.empty(n, dtype=torch.int32, device=dev) for n in (rows * top, tiles))
        us = _time(lambda: kernels.moe_align(ids, E, bn, ppos, tgroup), flush=flush)
        rec(f"moe_align ({label})", us, rows * top * 8)
        xp = torch.zeros(tiles * bn, width, dtype=torch.bfloat16, device=dev)
        us = _time(lambda: kernels.moe_gather(h, ppos, xp, top), flush=flush)
        rec(f"moe_gather ({label})", us, rows * top * width * 2 + rows * width * 2)
        both = interleaved_gate_up(b16(E, eff, width) * 0.02, b16(E, eff, width) * 0.02)
        dn = b16(E, width, eff) * 0.02
        scale = torch.ones(tiles * bn, dtype=torch.float32, device=dev)
        used = len(set(ids.flatten().tolist()))
        act = torch.empty(tiles * bn, eff, dtype=torch.bfloat16, device=dev)
        for name, kw in (("silu", {}), ("clamped (Momuvik's)", dict(activation="clamped_swish", limit=7.0, row_scale=scale))):
            us = _time(lambda: kernels.gemm_grouped(xp, both, act, tgroup, bn, gated=True, interleaved=True, **kw), flush=flush)
            rec(f"grouped gate/up, {name} ({label})", us, used * 2 * eff * width * 2 + rows * top * (width + eff) * 2,
                flops=2.0 * rows * top * 2 * eff * width)
        d, y = torch.empty(tiles * bn, width, dtype=torch.float32, device=dev), f32(rows, width)
        us = _time(lambda: kernels.gemm_grouped(act, dn, d, tgroup, bn, gated=False), flush=flush)
        rec(f"grouped down ({label})", us, used * eff * width * 2 + rows * top * (eff * 2 + width * 4),
            flops=2.0 * rows * top * eff * width)
        for name, w in (("with weights", wts), ("weights one (Momuvik's)", None)):
            us = _time(lambda: kernels.moe_combine(d, ppos, w, y, True), flush=flush)
            rec(f"moe_combine, {name} ({label})", us, rows * width * (top * 4 + 8))
        del both, dn, xp, act, d
    return rows_out


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(description=__doc__.split("\n\n")[0])
    ap.add_argument("--sizes", default="0.6b,8b")
    ap.add_argument("--layers", type=int, default=8)
    ap.add_argument("--batch", type=int, default=8)
    ap.add_argument("--kernels", action="store_true", help="only the table of kernels")
    ap.add_argument("--tokens", type=int, default=2048, help="tokens of the table's prompt portion")
    a = ap.parse_args(argv)
    rec: Dict[str, Any] = {}
    if not a.kernels:
        rec = compare([s for s in a.sizes.split(",") if s], a.layers, batch=a.batch)
    rec["kernels"] = kernel_table(tokens=a.tokens)
    json.dump(rec, sys.stdout, indent=1)
    print()
    return 0


if __name__ == "__main__":
    sys.exit(main())
