"""RMSNorm: ``x * rsqrt(mean(x^2) + eps) * w`` computed in float32, multiplication
order ``(x * r) * w``, the weight a plain multiplier (no ``1 + w``), as the reference
computes it (src/kernel/cuda/norm.cu:31-48; built by ModelCreatorBase::build_norm,
src/core/model/base/ModelCreatorBase.cpp:198-221)."""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..registry import register_part
from .base import Norm, WeightSpec, VECTOR


@register_part("norm", "rms_norm")
class RMSNorm(Norm):
    def __init__(self, dim: int, eps: float, name: str = "weight", weight_offset: float = 0.0, one_number: bool = False,
                 prefix: str = ""):
        super().__init__(prefix)
        self.dim = int(dim)
        self.eps = float(eps)
        self.name = name                  # the weight's tensor name relative to the prefix
        # a weight stored around zero: the multiplier is weight_offset + w (1 + w in the designs that do this); the sum
        # is taken once, in float32, when the tensor is loaded
        self.weight_offset = float(weight_offset)
        self.one_number = bool(one_number)        # the weight is a single number (a tensor of no dimensions) for all columns
        self.weight: Optional[torch.Tensor] = None

    def weight_specs(self) -> Dict[str, WeightSpec]:
        shape = () if self.one_number else (self.dim,)
        if self.weight_offset != 0.0:
            return {self.name: WeightSpec(shape, VECTOR, init="normal", init_scale=0.1)}
        return {self.name: WeightSpec(shape, VECTOR, init="one_plus_normal")}

    def load(self, tensors, ops, act_dtype) -> None:
        self.weight = tensors[self.name]
        if self.weight_offset != 0.0:
            self.weight = (self.weight.to(torch.float32) + self.weight_offset).contiguous()
        if self.one_number:
            self.weight = self.weight.reshape(1).expand(self.dim).contiguous()

    def deferred(self, x, ops, out_dtype):
        """The norm of ``x`` as an object that the kernel library's products can fold in, or None when the
        library cannot (then ``forward`` runs the norm kernel)."""
        can = getattr(ops, "can_fold_norm", None)
        if can is None or not can(x, self.weight, out_dtype):
            return None
        from ..kernels.library import DeferredNorm
        return DeferredNorm(x, self.weight, self.eps, out_dtype, ops)

    def forward(self, x, ops, out_dtype, row_index=None):
        rows = x.shape[0] if row_index is None else row_index.shape[0]
        out = torch.empty((rows, self.dim), dtype=out_dtype, device=x.device)
        ops.rmsnorm(x, self.weight, self.eps, out, row_index)
        return out
