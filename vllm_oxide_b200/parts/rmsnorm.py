"""RMSNorm with the residual add folded in.

out = weight * (x * 1/sqrt(mean(x^2) + eps)), weight last, sums in float32
(crates/engine/src/backend/cpu/mod.rs:182-197). The block hands the norm the float32 residual
and the delta its previous part produced; the kernel adds the delta into the residual (the
reference's `add`, :351-358) and normalises the sum in one pass over the row. A delta in parts
([parts, T, width], what sub-layers that ran side by side returned) is added part by part, and
with `extra` / `vec` a float32 row per token and one vector join the residual in the same pass.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from .base import Norm, StepContext, aligned


class RMSNorm(Norm):
    several_parts = True          # `forward` takes a delta in parts, and `extra` and `vec`
    scale_and_weight = True       # out = weight * (x * scale(x)): folds into the products around it

    def __init__(self, weight: torch.Tensor, eps: float, device, unit_offset: bool = False):
        """`unit_offset`: the stored weight lies around zero and the factor is 1 + weight (the sum is
        taken once, here, in float32)."""
        if weight.dim() != 1:
            raise ValueError(f"RMSNorm weight must be a vector, got {list(weight.shape)}")
        # The weight is read as float32 whatever it was stored as (widening is exact).
        self.weight = weight.to(device=device, dtype=torch.float32).contiguous()
        if unit_offset:
            self.weight = (self.weight + 1.0).contiguous()
        self.eps = float(eps)
        self.width = weight.shape[0]

    def weight_bytes(self) -> int:
        return self.weight.numel() * 4

    def workspace_bytes(self, rows: int, act_bytes: int) -> int:
        return aligned(rows * self.width * act_bytes)

    def kernel_modules(self, dtype, max_rows):
        return ("elementwise",)

    def forward(self, resid: torch.Tensor, delta: Optional[torch.Tensor], ctx: StepContext,
                rows: Optional[torch.Tensor] = None, num_rows: Optional[int] = None,
                delta_scale: Optional[torch.Tensor] = None, extra: Optional[torch.Tensor] = None,
                vec: Optional[torch.Tensor] = None) -> torch.Tensor:
        n = resid.shape[0] if rows is None else (num_rows if num_rows is not None else rows.numel())
        out = ctx.alloc((n, self.width))
        kernels.add_rmsnorm(resid, delta, self.weight, self.eps, out, rows[:n] if rows is not None else None,
                            delta_scale if delta is not None else None, extra, vec)
        return out
