"""Plain (ungated) feed-forward: f = W_down act(W_up h (+ b)) (+ b'), act(z) = max(z, 0)^2.

The activation is the up product's epilogue on every path (tensor cores and the 32-bit engine's), so the up product's
result is stored once, activated, in the activation dtype."""
from __future__ import annotations

import torch

from ..config.errors import ConfigError
from .base import FeedForward, ParamDecl, register_part
from .linear import linear, linear_modules

ACTS = ("relu2",)


@register_part("feed_forward", "plain")
class PlainFeedForward(FeedForward):
    def __init__(self, *, dtype: str, size: int, ff: int, act: str = "relu2", bias: bool = False):
        super().__init__()
        self.size, self.ff, self.act, self.bias = int(size), int(ff), str(act), bool(bias)
        if self.act not in ACTS:
            raise ConfigError(f"plain feed-forward: unknown activation {act!r} ({', '.join(ACTS)})")
        self.decls = {"up.weight": ParamDecl((self.ff, self.size)), "down.weight": ParamDecl((self.size, self.ff))}
        if self.bias:
            self.decls["up.bias"] = ParamDecl((self.ff,), role="vector", init=("normal", 0.1))
            self.decls["down.bias"] = ParamDecl((self.size,), role="vector", init=("normal", 0.1))

    takes_lazy_norm = True
    can_store = True          # forward(store=True) writes the float32 rows `out` instead of adding into them

    def forward(self, hn, ctx, out, store=False):
        w = self.w
        z = linear(hn, w["up.weight"], w.get("up.bias"), act=self.act)
        if store:
            linear(z, w["down.weight"], w.get("down.bias"), out=out, out_dtype=torch.float32)
        else:
            linear(z, w["down.weight"], w.get("down.bias"), out=out, accumulate=True)
        return out

    def weight_order(self):
        return [self.w["up.weight"], self.w["down.weight"]]

    def kernel_modules(self, dtype):
        return linear_modules(dtype)
