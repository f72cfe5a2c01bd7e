"""RMSNorm, fused with the residual addition that precedes it."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..config.registry import register_part
from ..kernels import ops
from .base import Part, WeightSlot


class RMSNorm(Part):
    """y = x * rsqrt(mean(x^2) + eps) * gain, statistics in FP32
    (src/op/kernels/cuda/rmsnorm_kernel.cu:49-104; eps inside the root, :79)."""

    # What a kernel that runs this norm inside itself computes (with ``gain`` and ``eps``): the
    # skinny products fuse norms of this kind only.
    fused_kind = "rmsnorm"

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        return {"weight": WeightSlot((hidden_size,), init="ones")}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        super().__init__(spec, hidden_size, weights, rt)
        self.eps = float(spec.eps)
        self.gain = rt.gain(weights["weight"])

    def forward(self, h: torch.Tensor, delta: Optional[torch.Tensor],
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        n = h.shape[0] if rows is None else rows.numel()
        out = self.rt.empty(n, self.hidden_size)
        ops.add_rmsnorm(h, delta, self.gain, self.eps, out, rows)
        return out


class ScalarRMSNorm(RMSNorm):
    """y = x * rsqrt(mean(x^2) + eps) * g with ONE gain g for all coordinates (stored as a tensor without
    axes).  On the device the gain is spread over the width, so every kernel that takes an RMSNorm - the
    fused ones included - takes this one unchanged."""

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        return {"weight": WeightSlot((), init="ones")}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        Part.__init__(self, spec, hidden_size, weights, rt)
        self.eps = float(spec.eps)
        self.gain = rt.gain(weights["weight"]).reshape(1).expand(hidden_size).contiguous()


class RMSNormOnePlus(RMSNorm):
    """y = x * rsqrt(mean(x^2) + eps) * (1 + w): the weight is stored around zero.  On the device the gain is 1 + w in
    FP32, so every kernel that takes an RMSNorm - the fused ones included - takes this one unchanged."""

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        return {"weight": WeightSlot((hidden_size,), init="zeros")}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        Part.__init__(self, spec, hidden_size, weights, rt)
        self.eps = float(spec.eps)
        self.gain = rt.gain(weights["weight"]) + 1.0


class DynamicTanh(Part):
    """y = tanh(alpha x) * w + b, coordinate by coordinate: one learned scalar ``alpha``, a weight and a bias ("weight",
    "alpha", "b").  It has no statistics (the spec's eps is not read), so whatever forms x in registers can norm it on
    the spot: ``tanh_norm`` is the triple (alpha, weight, bias), FP32 on the device."""

    kernel_modules = ("hyper",)       # libraries of csrc that this part's kernels live in

    @staticmethod
    def weight_slots(spec, hidden_size: int) -> Dict[str, WeightSlot]:
        return {"weight": WeightSlot((hidden_size,), init="ones"), "b": WeightSlot((hidden_size,), init="zeros"),
                "alpha": WeightSlot((), init="ones")}

    def __init__(self, spec, hidden_size, weights, rt) -> None:
        super().__init__(spec, hidden_size, weights, rt)
        self.tanh_norm = (rt.gain(weights["alpha"]).reshape(1), rt.gain(weights["weight"]), rt.gain(weights["b"]))

    def forward(self, h: torch.Tensor, delta: Optional[torch.Tensor],
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        if delta is not None and delta.dtype != torch.float32:
            ops.residual_add(h, delta)
            delta = None
        out = self.rt.empty(h.shape[0] if rows is None else rows.numel(), self.hidden_size)
        ops.tanh_norm(h, delta, *self.tanh_norm, out, rows)
        return out


register_part("norm", "dynamic_tanh", DynamicTanh, replace=True)
register_part("norm", "rmsnorm", RMSNorm, replace=True)
register_part("norm", "rmsnorm_one_plus", RMSNormOnePlus, replace=True)
register_part("norm", "rmsnorm_scalar", ScalarRMSNorm, replace=True)
