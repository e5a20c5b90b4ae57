"""Rotary position encoding: ``freq_i = theta^(-2i/rot_dim)``, ``angle = pos * freq_scale *
freq_i``, all in 32-bit (crates/engine/cpu/src/ops.rs:46-66).  The pair that angle i turns is
(i, i + rot_dim/2) for ``rope_neox`` (``RopeKind::Neox``) and (2i, 2i + 1) for ``rope_normal``
(``RopeKind::Normal``, ops.rs:57-60).  The rotation itself is applied by the kernel that also
norms the heads and writes the cache; this part owns the constants.

``scaling`` (a dictionary, absent by default) changes the frequencies for sequences longer than
``original`` positions; both forms are made in 64-bit and rounded once:

* ``kind: "bands"`` (``factor``, ``low``, ``high``, ``original``), by wavelength ``2 pi / f``: below
  ``original / high`` f stays, above ``original / low`` it becomes ``f / factor``, between them the
  two are blended linearly in ``original / wavelength``;
* ``kind: "ramp"`` (``factor``, ``original``, ``fast``, ``slow``), by index: from f at the index
  that turns ``fast`` times within ``original`` positions (rounded down) to ``f / factor`` at the
  one that turns ``slow`` times (rounded up), linearly between; cosine and sine are multiplied by
  ``0.1 ln(factor) + 1``."""
from __future__ import annotations

import math
from typing import Any, Dict, Mapping, Optional, Tuple

import numpy as np
import torch

from ..config.spec import ConfigError, PartSpec
from .base import register_part


def scaled_frequencies(freq: np.ndarray, rot_dim: int, theta: float, scaling: Mapping[str, Any]
                       ) -> Tuple[np.ndarray, float]:
    """The frequencies (float64) under ``scaling``, and the factor on cosine and sine."""
    kind = scaling.get("kind")
    factor, original = float(scaling["factor"]), float(scaling["original"])
    if kind == "bands":
        low, high = float(scaling["low"]), float(scaling["high"])
        turns = original * freq / (2.0 * math.pi)            # original / wavelength
        share = np.clip((turns - low) / (high - low), 0.0, 1.0) if high != low else \
            (turns > high).astype(np.float64)
        return (1.0 - share) * freq / factor + share * freq, 1.0
    if kind == "ramp":
        def index(t: float) -> float:
            return rot_dim * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(theta))

        lo = max(math.floor(index(float(scaling["fast"]))), 0)
        hi = min(math.ceil(index(float(scaling["slow"]))), rot_dim - 1)
        ramp = np.clip((np.arange(len(freq)) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
        return freq / factor * ramp + freq * (1.0 - ramp), 0.1 * math.log(factor) + 1.0
    raise ConfigError(f"rotary scaling of kind {kind!r} (known: bands, ramp)")


class RotaryHalfSplit:
    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], dtype, device):
        self.rot_dim = int(spec["rot_dim"])
        self.theta = float(spec["theta"])
        self.freq_scale = float(spec.get("freq_scale", 1.0))
        self.attn_factor = float(spec.get("attn_factor", 1.0))
        if self.rot_dim % 2:
            raise ValueError("rot_dim must be even")
        i = np.arange(self.rot_dim // 2, dtype=np.float32)
        exponent = (-(np.float32(2.0) * i) / np.float32(self.rot_dim)).astype(np.float32)
        freq = np.power(np.float32(self.theta), exponent).astype(np.float32)
        freq = (np.float32(self.freq_scale) * freq).astype(np.float32)
        scaling = spec.get("scaling")
        self.scaling = None if scaling is None else tuple(sorted(scaling.items()))
        if scaling is not None:
            plain = self.freq_scale * self.theta ** (-2.0 * np.arange(self.rot_dim // 2)
                                                     / self.rot_dim)
            freq, mult = scaled_frequencies(plain, self.rot_dim, self.theta, scaling)
            freq = freq.astype(np.float32)
            self.attn_factor *= mult
        self.inv_freq = torch.from_numpy(freq).to(device)

    def rotary_tables(self) -> Optional[Tuple[torch.Tensor, int, float]]:
        return self.inv_freq, self.rot_dim, self.attn_factor

    def constants(self) -> Tuple:
        """What the table of a step's angles depends on."""
        return self.rot_dim, self.theta, self.freq_scale, self.attn_factor, self.scaling

    def step_angles(self, ctx) -> torch.Tensor:
        """cos and sin of every row's angles, float32 [rows, rot_dim / 2, 2]: made once per
        step and shared by all layers whose rotation has the same constants."""
        key = ("rope",) + self.constants()
        table = ctx.shared.get(key)
        if table is None:
            from .. import kernels
            table = ctx.buffer("rope.%r" % (key,),
                               (ctx.rows, self.rot_dim // 2, 2), torch.float32)
            kernels.rope_table(ctx.row_pos, self.inv_freq, table, self.attn_factor)
            ctx.shared[key] = table
        return table


class RotaryAdjacentPairs(RotaryHalfSplit):
    """Angle i turns the pair (2i, 2i + 1).  The kernels turn (i, i + rot_dim/2); the mixer
    therefore orders each head of its query and key projections by :meth:`head_permutation`
    when it is built (scores do not depend on the order in which a head's values stand, as long
    as queries and keys stand alike), and nothing else changes."""

    def head_permutation(self, head_dim: int) -> torch.Tensor:
        """``perm`` with ``stored[j] = original[perm[j]]``: the even members of the rotated
        pairs first, then the odd ones, then what is not rotated."""
        half = self.rot_dim // 2
        perm = list(range(0, self.rot_dim, 2)) + list(range(1, self.rot_dim, 2)) \
            + list(range(self.rot_dim, head_dim))
        assert len(perm) == head_dim and perm[half] == 1
        return torch.tensor(perm, dtype=torch.long)


register_part("position", "rope_neox", RotaryHalfSplit, replace=True)
register_part("position", "rope_normal", RotaryAdjacentPairs, replace=True)
