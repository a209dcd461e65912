"""RMSNorm over the residual stream, and a norm without statistics (``dynamic_tanh``, at its class).

y = gain * x * rsqrt(mean(x^2) + eps), in 32-bit, with the preceding residual add folded
in when there is one (engine/ek_kernels.py:89-123; gain is a plain factor, no +1, no
bias).  Parameters: ``size``, ``eps``, and optionally ``one_plus``: the stored weight w lies
around zero and the factor is 1 + w (formed once at load, in 32-bit).  Tensor: ``gain`` [size].
"""

from __future__ import annotations

import torch

from ..ops import kernels
from ..registry import register_part
from .base import Norm
from .spec import TensorSpec


@register_part("norm", "rms_norm")
class RMSNorm(Norm):
    @classmethod
    def tensors(cls, spec):
        return [TensorSpec(spec.weights["gain"], (spec.params["size"],),
                           "around_zero" if spec.params.get("one_plus") else "gain")]

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        self.size, self.eps = int(self.param("size")), float(self.param("eps"))
        self.one_plus = bool(spec.params.get("one_plus"))
        self.gain = None

    def load(self, tensors):
        self.gain = tensors[self.spec.weights["gain"]].to(torch.float32).contiguous()
        if self.one_plus:
            self.gain = (self.gain + 1.0).contiguous()

    def bytes_read_per_step(self, n_tokens):
        return self.gain.numel() * self.gain.element_size()

    def deferrable(self):
        return self.gain, self.eps

    def forward(self, stream, ctx, add=None, rows=None, n_rows=None, write_back=True):
        if n_rows is None:
            n_rows = rows.numel() if rows is not None else ctx.n_tokens
        y = ctx.workspace.get("normed" if rows is None else "normed_rows", (n_rows, self.size),
                              self.dtype)
        kernels.rmsnorm(y, stream, self.gain, self.eps, add=add, rows=rows, n_rows=n_rows,
                        write_back=write_back)
        return y


@register_part("norm", "dynamic_tanh")
class DynamicTanh(Norm):
    """y = tanh(alpha x) * weight + shift, element by element, in 32-bit: no mean, no variance, so it can ride in
    whatever kernel writes the stream (``Norm.pointwise``).  Parameter: ``size``.  Tensors: ``alpha`` [] (one
    number), ``gain`` [size], ``shift`` [size]."""

    @classmethod
    def tensors(cls, spec):
        size = spec.params["size"]
        return [TensorSpec(spec.weights["alpha"], (), "gain"), TensorSpec(spec.weights["gain"], (size,), "gain"),
                TensorSpec(spec.weights["shift"], (size,), "around_zero")]

    def __init__(self, spec, dtype, device):
        super().__init__(spec, dtype, device)
        self.size = int(self.param("size"))
        self.alpha = self.gain = self.shift = None

    def load(self, tensors):
        w, f32 = self.spec.weights, torch.float32
        self.alpha = tensors[w["alpha"]].to(f32).reshape(1).contiguous()
        self.gain = tensors[w["gain"]].to(f32).contiguous()
        self.shift = tensors[w["shift"]].to(f32).contiguous()

    def pointwise(self):
        return self.alpha, self.gain, self.shift

    def forward(self, stream, ctx, add=None, rows=None, n_rows=None, write_back=True):
        if n_rows is None:
            n_rows = rows.numel() if rows is not None else ctx.n_tokens
        y = ctx.workspace.get("normed" if rows is None else "normed_rows", (n_rows, self.size), self.dtype)
        kernels.dynamic_tanh(y, stream, self.pointwise(), add=add, rows=rows, n_rows=n_rows, write_back=write_back)
        return y
