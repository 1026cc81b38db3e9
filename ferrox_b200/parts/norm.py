"""RMSNorm: x * (1 / sqrt(mean(x^2) + eps)) * w, statistics in 32 bits
(reference: crates/ferrox-core/src/matmul.rs:62-69,121-123)."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorDecl
from .base import Norm, register_part


class RmsNorm(Norm):
    """``one_plus``: the stored weight lies around zero and the norm multiplies by 1 + w (added once, in 32 bits,
    when the weights are loaded).  ``scale_name``: the result is multiplied by one more vector; both factors are one
    32-bit weight from the loading on.  ``scalar``: the stored weight is one number, spread over the row when it is
    loaded, so that every kernel finds a vector."""

    graph_safe = True

    def _name(self):
        return getattr(self.spec, "name", None) or self.spec.prefix + "weight"

    def _scalar(self):
        return bool(getattr(self.spec, "scalar", False))

    def tensor_decls(self):
        one_plus = getattr(self.spec, "one_plus", False)
        d = [TensorDecl(self._name(), () if self._scalar() else (self.spec.size,), init="normal" if one_plus else "ones")]
        if getattr(self.spec, "scale_name", None):
            d.append(TensorDecl(self.spec.scale_name, (self.spec.size,), init="ones"))
        return d

    def load(self, src, rt):
        super().load(src, rt)
        self.weight = src.get(self._name())
        if self._scalar():
            self.weight = self.weight.to(torch.float32).reshape(1).expand(self.spec.size).contiguous()
        if getattr(self.spec, "one_plus", False):
            self.weight = (1.0 + self.weight.to(torch.float32)).contiguous()
        if getattr(self.spec, "scale_name", None):
            self.weight = (self.weight.to(torch.float32) * src.get(self.spec.scale_name).to(torch.float32)).contiguous()

    def forward(self, h, rows=None):
        n = h.shape[0] if rows is None else rows.numel()
        out = self.rt.empty(n, self.spec.size)
        return ops.rmsnorm(h, self.weight, self.spec.eps, out, rows=rows)

    def forward_in_place(self, h):
        """The 32-bit stream normed where it lies."""
        normed = self.rt.empty(h.shape[0], h.shape[1], dtype=torch.float32)
        h.copy_(ops.rmsnorm(h, self.weight, self.spec.eps, normed))
        return h

    def as_rms(self):
        return self.weight, self.spec.eps


class LayerNorm(Norm):
    """(x - mean) / sqrt(variance + eps) * w (+ b), the variance being the mean of the squared deviations; a weight
    and, where the spec names one, a bias; statistics in 32 bits."""

    graph_safe = True

    def _bias_name(self):
        return getattr(self.spec, "bias_name", None)

    def tensor_decls(self):
        d = [TensorDecl(self.spec.name, (self.spec.size,), init="ones")]
        if self._bias_name():
            d.append(TensorDecl(self._bias_name(), (self.spec.size,)))
        return d

    def load(self, src, rt):
        super().load(src, rt)
        self.weight = src.get(self.spec.name)
        self.bias = src.get(self._bias_name()) if self._bias_name() else None

    def forward(self, h, rows=None):
        n = h.shape[0] if rows is None else rows.numel()
        out = self.rt.empty(n, self.spec.size)
        return ops.layernorm(h, self.weight, self.spec.eps, out, rows=rows, bias=self.bias)

    def forward_in_place(self, h):
        """The 32-bit stream normed where it lies."""
        return ops.layernorm(h, self.weight, self.spec.eps, h, bias=self.bias)

    def as_layer_norm(self):
        """(weight, eps) for a kernel that applies the norm itself; None with a bias, which those kernels lack."""
        return (self.weight, self.spec.eps) if self.bias is None else None


register_part("rms_norm", RmsNorm, replace=True)
register_part("layer_norm", LayerNorm, replace=True)
