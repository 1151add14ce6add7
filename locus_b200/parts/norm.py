"""Norms.  RMSNorm(eps): out = x * rsqrt(mean(x^2) + eps) * w, statistics in float32; with ``offset`` the stored
weight is taken as w + offset (a weight stored around zero: offset 1).
LayerNorm(eps): out = (x - mean) / sqrt(var + eps) * w + b (below).
DynamicTanh: out = tanh(alpha x) * w + b, elementwise, no statistics (below).

Formula and multiplication order of the reference's ``rmsnorm``
(src/locus/backend/cpu_ops.cpp:1687-1699): no mean subtraction, no bias, the weight used
as stored (not 1 + w).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels as K
from .base import Norm, PendingAdd, PendingNorm, PendingRows, TensorSource, register_norm


class RMSNorm(Norm):
    def __init__(self, prefix: str, *, width: int, eps: float, tensor: str = "", offset: float = 0.0) -> None:
        """``tensor``: the checkpoint tensor's name where it is not ``<prefix>.weight``.  ``offset``: added to the
        stored weight, in float32 (at bind, so that 1 + w is not rounded to the weight's 16 bits)."""
        super().__init__(prefix)
        self.width = int(width)
        self.eps = float(eps)
        self.offset = float(offset)
        self.tensor = str(tensor or prefix + ".weight")

    def bind(self, rt) -> None:
        if self.offset != 0.0 and not getattr(self, "_offset_done", False):
            self.params["weight"] = (self.params["weight"].float() + self.offset).contiguous()
            self._offset_done = True

    def param_shapes(self):
        return {"weight": (self.width,)}

    def sources(self):
        return [TensorSource(self.tensor, (self.width,), "weight", 0, "norm")]

    def kernel_modules(self, dtype):
        return ["elementwise"]

    def forward(self, x: torch.Tensor, out: torch.Tensor, rows: Optional[torch.Tensor] = None, add=None) -> None:
        # the experts' sum of the block in front, rows added between two layer calls, or both: folded into the norm's pass
        extra = {}
        if isinstance(add, PendingRows) and K.rmsnorm_adds(x) and (add.before is None or isinstance(add.before, PendingAdd)):
            extra["add_rows"], add = add.y, add.before
        if add is not None and not (isinstance(add, PendingAdd) and K.rmsnorm_adds(x)):
            add.apply(x)
            add = None
        K.rmsnorm(x, self.params["weight"], self.eps, out, rows,
                  add=None if add is None else (add.pair_out, add.pair_pos, add.top_k), **extra)

    def forward_add(self, y: torch.Tensor, x: torch.Tensor, scale: Optional[torch.Tensor] = None) -> None:
        """x += norm(y): the norm of a sublayer's output (float32 rows) added to the residual stream."""
        w = self.params["weight"]
        if scale is not None:
            # the scale multiplies the weight, once, in float32
            if getattr(self, "_scaled", None) is None or self._scaled[0] is not scale:
                self._scaled = (scale, (w.float() * scale.float()).contiguous())
            w = self._scaled[1]
        K.rmsnorm_add(y, w, self.eps, x)


class LayerNorm(Norm):
    """Layer norm with weight and bias, mean and variance (the mean of the squared deviations) in float32.  With
    ``streams`` > 1 a row of x holds that many copies of the residual stream, one behind the other, and the norm
    reads their weighted sum (``coef`` [streams] float32 on the device; None: the plain sum)."""

    def __init__(self, prefix: str, *, width: int, eps: float, streams: int = 1, tensor: str = "",
                 bias_tensor: str = "") -> None:
        """``tensor`` / ``bias_tensor``: the checkpoint tensors' names where they are not ``<prefix>.weight`` and
        ``<prefix>.bias``."""
        super().__init__(prefix)
        self.width, self.eps, self.streams = int(width), float(eps), int(streams)
        self.tensor = str(tensor or prefix + ".weight")
        self.bias_tensor = str(bias_tensor or prefix + ".bias")

    def param_shapes(self):
        return {"weight": (self.width,), "bias": (self.width,)}

    def sources(self):
        return [TensorSource(self.tensor, (self.width,), "weight", 0, "norm"),
                TensorSource(self.bias_tensor, (self.width,), "bias", 0, "bias")]

    def kernel_modules(self, dtype):
        return ["elementwise"]

    def forward(self, x: torch.Tensor, out: torch.Tensor, rows: Optional[torch.Tensor] = None, add=None,
                coef: Optional[torch.Tensor] = None) -> None:
        if add is not None:
            add.apply(x)   # nothing is folded into this norm's pass
        K.layernorm(x, self.params["weight"], self.params["bias"], self.eps, out, rows, n_streams=self.streams, coef=coef)

    def forward_post(self, x: torch.Tensor, y: torch.Tensor, alpha: float, cast: Optional[torch.Tensor] = None) -> None:
        """x <- norm(alpha x + y) in place on the float32 residual stream (the norm behind a sublayer's sum); ``cast``:
        the new rows once more in that buffer's element type."""
        if self.streams != 1:
            raise ValueError("layernorm: the norm behind a sum works on one residual stream")
        K.layernorm_post(x, y, alpha, self.params["weight"], self.params["bias"], self.eps, cast)


class DynamicTanh(Norm):
    """Dynamic Tanh: D(z) = tanh(alpha z) * w + b elementwise with a stored scalar alpha, all of it in float32.  It has no
    statistics, so what was left pending in the same form (x += scale * D'(y), the norm behind the sublayer in front)
    is folded into its pass over the rows."""

    def __init__(self, prefix: str, *, width: int, tensor: str = "", bias_tensor: str = "", alpha_tensor: str = "") -> None:
        """``tensor`` / ``bias_tensor`` / ``alpha_tensor``: the checkpoint tensors' names where they are not
        ``<prefix>.weight``, ``<prefix>.bias`` and ``<prefix>.alpha``."""
        super().__init__(prefix)
        self.width = int(width)
        self.names = {"alpha": str(alpha_tensor or prefix + ".alpha"), "weight": str(tensor or prefix + ".weight"),
                      "bias": str(bias_tensor or prefix + ".bias")}

    def param_shapes(self):
        return {"alpha": (), "weight": (self.width,), "bias": (self.width,)}

    def sources(self):
        inits = {"alpha": "norm", "weight": "norm", "bias": "bias"}
        return [TensorSource(self.names[p], shape, p, 0, inits[p]) for p, shape in self.param_shapes().items()]

    def kernel_modules(self, dtype):
        return ["elementwise"]

    def bind(self, rt) -> None:
        if len({t.dtype for t in self.params.values()}) > 1:   # the kernel takes the three in one element type
            self.params.update({n: t.float().contiguous() for n, t in self.params.items()})

    def tensors(self):
        """(alpha, weight, bias) as the kernels take them."""
        return self.params["alpha"], self.params["weight"], self.params["bias"]

    def forward(self, x: torch.Tensor, out: torch.Tensor, rows: Optional[torch.Tensor] = None, add=None) -> None:
        fold = None
        if isinstance(add, PendingNorm) and isinstance(add.norm, DynamicTanh):
            fold = (add.y, add.norm.tensors(), add.scale)
        elif add is not None:
            add.apply(x)
        K.dyt(x, self.tensors(), out, rows, add=fold)

    def forward_add(self, y: torch.Tensor, x: torch.Tensor, scale: Optional[torch.Tensor] = None) -> None:
        K.dyt(x, add=(y, self.tensors(), scale))


register_norm("rmsnorm", RMSNorm)
register_norm("dynamic_tanh", DynamicTanh)
register_norm("layernorm", LayerNorm)
