"""RMSNorm: y = x * 1/sqrt(mean(x^2) + eps) * w (crates/backend-cpu/src/kernels/norm.rs:6-39).

'rmsnorm_groups': the row in `groups` equal consecutive parts, each divided by its own root mean square, then the
weight over the whole row.

`offset` (rmsnorm): the weight is stored around zero and the norm multiplies by offset + w (added once, in float32, when
the tensors are bound: every kernel that norms reads the sum).  `add_normed_then(x, y, norm)`: x += this norm of y, and the
norm that reads x next, in one kernel."""
from __future__ import annotations

import torch

from .. import ops
from ..config.errors import ConfigError
from .base import Norm, ParamDecl, register_part


@register_part("norm", "rmsnorm")
class RMSNorm(Norm):
    def __init__(self, *, dtype: str, size: int, eps: float, offset: float = 0.0):
        super().__init__()
        self.size, self.eps, self.dtype, self.offset = int(size), float(eps), dtype, float(offset)
        self.decls = {"weight": ParamDecl((self.size,), role="vector",
                                          init=("uniform", 0.5 - self.offset, 1.5 - self.offset) if self.offset else ("ones",))}

    def prepare(self):
        if self.offset:
            self.w["weight"] = self.w["weight"] + self.offset

    def forward(self, x, out_dtype, rows=None):
        return ops.rmsnorm(x, self.w["weight"], self.eps, out_dtype, rows=rows)

    def reserve(self, device, max_rows, n_ctx):
        if self.w["weight"].dtype == torch.float32 and self.dtype == "bfloat16":
            ops.reserve_norm_handoff(device, self.size)

    def expect(self, x):
        ops.expect_norm(x, self.w["weight"])

    def add_normed_then(self, x, y, norm, act_dtype):
        """x float32 [T, d] += RMSNorm(y) in place; returns `norm` of the new rows in act_dtype, or None where norm is None
        or not an RMSNorm over the whole row (the caller then norms x itself)."""
        fused = getattr(norm, "kind", None) == "rmsnorm"
        return ops.add_rmsnorm(x, y, self.w["weight"], self.eps, norm.w["weight"] if fused else None,
                               norm.eps if fused else 0.0, out_dtype=act_dtype)

    def kernel_modules(self, dtype):
        return [("elementwise", None), ("sublayer", None)] if self.offset else [("elementwise", None)]


@register_part("norm", "rmsnorm_groups")
class GroupedRMSNorm(Norm):
    def __init__(self, *, dtype: str, size: int, eps: float, groups: int):
        super().__init__()
        self.size, self.eps, self.groups, self.dtype = int(size), float(eps), int(groups), dtype
        if self.groups < 1 or self.size % self.groups:
            raise ConfigError(f"rmsnorm_groups: {self.groups} groups do not divide a row of {self.size}")
        self.decls = {"weight": ParamDecl((self.size,), role="vector", init=("ones",))}

    def forward(self, x, out_dtype, rows=None):
        return ops.rmsnorm_groups(x, self.w["weight"], self.eps, self.groups, out_dtype, rows=rows)

    def kernel_modules(self, dtype):
        return [("elementwise", None)]
