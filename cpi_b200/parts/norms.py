"""Norms.

"rmsnorm"        y = x * rsqrt(mean(x^2) + eps) * w  (src/engine/llama4_cpu_engine.cpp:47-62); with `weight_offset` o the
                 stored weight is a distance from o: y = x * rsqrt(mean(x^2) + eps) * (o + w).
"dynamic_tanh"   y = tanh(alpha x) * w + b with one scalar alpha, a weight and an offset per element: no statistics of the
                 row, so the norms on both sides of a residual sum, and the sum, are one pass (`csrc/norm_step.cu`).

Both know how to let a sublayer's output enter the residual: `enter(y, x, following, h_out)` does x += norm(y) and, with
`following` (another norm), h_out = following(x).  y is a float32 row per token or an `ExpertSum`.
"""
from __future__ import annotations

import torch

from ..csrc import lib as K
from ..weights.store import TensorReq
from .base import ExpertSum, Norm, register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    """params: size, eps, weight (tensor name relative to the prefix, or None for a weightless norm),
    weight_offset (0 by default; 1 for a weight stored around zero)."""
    graph_safe = True

    def __init__(self, spec, prefix="", workspace=None, tag="norm"):
        super().__init__(spec, prefix)
        self.size, self.eps = int(spec["size"]), float(spec["eps"])
        self.weight_name = None if spec.get("weight") is None else prefix + spec["weight"]
        self.weight = None
        self.weight_offset = float(spec.get("weight_offset", 0.0))
        self.ws, self.tag = workspace, tag

    def requirements(self):
        if self.weight_name is None:
            return []
        return [TensorReq(self.weight_name, (self.size,), init="normal" if self.weight_offset else "ones")]

    def load(self, source, device):
        if self.weight_name is not None:
            self.weight = source.get(self.weight_name, device).contiguous()

    def __call__(self, x, out_dtype, rows=None, out=None):
        n = x.shape[0] if rows is None else rows.numel()
        if out is None:
            out = self.ws.get(self.tag, (n, self.size), out_dtype)
        K.rmsnorm(x, self.weight, self.eps, out, rows, self.weight_offset)
        return out

    def enter(self, y, x, following=None, h_out=None):
        together = isinstance(following, RMSNorm) and following.weight is not None
        if self.weight is not None:            # both norms, the sum and the combination of experts: one kernel
            kw = {"experts": y.lists()} if isinstance(y, ExpertSum) else {"y": y}
            K.rms_step(x, post=(self.weight, self.weight_offset, self.eps), h_out=h_out if together else None,
                       pre=(following.weight, following.weight_offset, following.eps) if together else None, **kw)
        else:
            together = False
            y = y.rows(self.ws) if isinstance(y, ExpertSum) else y
            K.sum_norm_add([y], [1.0], None, x, eps=self.eps, add=True)
        if following is not None and not together:
            following(x, h_out.dtype, out=h_out)


@register_norm("dynamic_tanh")
class DynamicTanh(Norm):
    """params: size, weight, alpha, offset (tensor names relative to the prefix)."""
    graph_safe = True

    def __init__(self, spec, prefix="", workspace=None, tag="norm"):
        super().__init__(spec, prefix)
        self.size = int(spec["size"])
        self.names = {k: prefix + spec[k] for k in ("weight", "alpha", "offset")}
        self.ws, self.tag = workspace, tag
        self.norm = None                       # (alpha, weight, offset): a float and two float32 vectors

    def requirements(self):
        n = self.names
        return [TensorReq(n["weight"], (self.size,), init="ones+normal"), TensorReq(n["alpha"], (), init="const:0.5"),
                TensorReq(n["offset"], (self.size,))]

    def load(self, source, device):
        f32 = lambda k: source.get(self.names[k], device).to(torch.float32).contiguous()
        self.norm = (float(source.get(self.names["alpha"], "cpu").to(torch.float32)), f32("weight"), f32("offset"))

    def __call__(self, x, out_dtype, rows=None, out=None):
        n = x.shape[0] if rows is None else rows.numel()
        if out is None:
            out = self.ws.get(self.tag, (n, self.size), out_dtype)
        K.norm_step(x, pre=self.norm, h_out=out, rows=rows)
        return out

    def enter(self, y, x, following=None, h_out=None):
        together = isinstance(following, DynamicTanh)
        kw = {"experts": y.lists()} if isinstance(y, ExpertSum) else {"y": y}
        K.norm_step(x, post=self.norm, pre=following.norm if together else None, h_out=h_out if together else None, **kw)
        if following is not None and not together:
            following(x, h_out.dtype, out=h_out)
