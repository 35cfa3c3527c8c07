"""RMSNorm: y = x * rsqrt(mean(x^2) + eps) * w; eps inside the root, added after the mean; no mean
subtraction, no bias, the weight multiplies as it is (src/forward.cpp:21-31, kernels/ops/rmsnorm.cu:9-28).
``weight_name`` in the spec renames the one tensor (default "weight") under the part's prefix. ``weight_offset``
(default 0) is added to the stored weight when it is loaded: a design whose norms multiply by (1 + w) stores w around zero.
``groups`` (default 1) splits the row into that many equal consecutive parts, each divided by its own root mean square."""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config.specs import PartSpec
from .base import Norm, register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    # Kernels that take (float32 rows, weight, eps) can apply this norm themselves: the streaming product of a
    # decode step normalises its lanes' fragments of the rows in registers, once per CTA, which saves the norm
    # kernel and its round trip through memory.
    fusable = True

    def __init__(self, spec: PartSpec, runtime):
        super().__init__(spec, runtime)
        self.size, self.eps = int(spec["size"]), float(spec["eps"])
        self.offset = float(spec.get("weight_offset") or 0.0)
        self.groups = int(spec.get("groups") or 1)
        if self.size <= 0 or self.eps <= 0:
            raise ValueError("rmsnorm needs a positive size and eps")
        if self.groups < 1 or self.size % self.groups:
            raise ValueError(f"rmsnorm: a row of {self.size} does not split into {self.groups} equal groups")
        if self.groups > 1:
            self.fusable = False         # those kernels take one root mean square per row
        self.weight = None

    @classmethod
    def param_shapes(cls, spec):
        return {str(spec.get("weight_name", "weight")): (int(spec["size"]),)}

    @classmethod
    def init_params(cls, spec, name, shape, gen):
        return 1.0 - float(spec.get("weight_offset") or 0.0) + 0.1 * torch.randn(shape, generator=gen, dtype=torch.float32, device=gen.device)

    def load(self, params):
        self.weight = params[str(self.spec.get("weight_name", "weight"))].to(device=self.rt.device, dtype=torch.float32).contiguous()
        if self.offset:
            self.weight = (self.weight + self.offset).contiguous()

    def forward(self, x: torch.Tensor, out_dtype: Optional[torch.dtype] = None,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        if self.groups > 1:
            return ops.stream_link(x, 1, out_dtype or self.rt.dtype, norm_w=self.weight, eps=self.eps, groups=self.groups, rows=rows)[1]
        return ops.rmsnorm(x, self.weight, self.eps, out_dtype or self.rt.dtype, rows)
