"""RMS norm: ``y = x * 1/sqrt(mean(x^2) + eps) * w`` with sums and scale in 32-bit; the weight is
the plain gain (crates/engine/cpu/src/ops.rs:18-29) or, with ``zero_centred``, what the gain has
beyond one (``1 + w``, added once in 32-bit when the part is built).

Layer norm: ``y = d * 1/sqrt(mean(d^2) + eps) * w + b`` with ``d = x - mean(x)``, in 32-bit."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .. import kernels
from ..config.spec import PartSpec
from .base import StepContext, register_part, tensor_of


class RmsNorm:
    graph_safe = True

    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], dtype, device):
        self.width = int(spec["width"])
        self.eps = float(spec["eps"])
        self.weight = tensor_of(spec, "weight", weights).to(device=device, dtype=torch.float32)
        assert self.weight.numel() == self.width
        if spec.get("zero_centred"):
            self.weight = 1.0 + self.weight

    def apply(self, ctx: Optional[StepContext], x: torch.Tensor, out: torch.Tensor,
              rows_index: Optional[torch.Tensor] = None) -> None:
        kernels.rms_norm(x, self.weight, out, self.eps, rows_index)


class ScalarRmsNorm(RmsNorm):
    """RMS norm whose gain is one stored number for all coordinates (a tensor without
    dimensions).  It is spread over the width once, so every kernel that takes a gain per
    channel takes this norm as well."""

    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], dtype, device):
        self.width = int(spec["width"])
        self.eps = float(spec["eps"])
        gain = tensor_of(spec, "weight", weights).to(device=device, dtype=torch.float32)
        assert gain.numel() == 1
        self.weight = gain.reshape(1).expand(self.width).contiguous()


class LayerNorm:
    """Centred norm with a gain and an offset per channel (tensor roles ``weight``, ``bias``)."""

    graph_safe = True

    def __init__(self, spec: PartSpec, weights: Dict[str, torch.Tensor], dtype, device):
        self.width = int(spec["width"])
        self.eps = float(spec["eps"])
        self.weight, self.bias = (tensor_of(spec, r, weights).to(device=device, dtype=torch.float32)
                                  .contiguous() for r in ("weight", "bias"))
        assert self.weight.numel() == self.bias.numel() == self.width

    def apply(self, ctx: Optional[StepContext], x: torch.Tensor, out: torch.Tensor,
              rows_index: Optional[torch.Tensor] = None) -> None:
        kernels.layer_norm(x, self.weight, self.bias, out, self.eps, rows_index)


register_part("norm", "rms_norm", RmsNorm, replace=True)
register_part("norm", "rms_norm_scalar", ScalarRmsNorm, replace=True)
register_part("norm", "layer_norm", LayerNorm, replace=True)
