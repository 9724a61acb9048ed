"""Norms of rows: RMSNorm, alone or fused with the residual sum; LayerNorm; a tanh norm without statistics.

ullm/layers/layernorm.py:20-34: everything in 32-bit; with a residual the sum
x + residual is normed unrounded and its rounded value becomes the new
residual; the weight multiplies before the cast back.
"""

from __future__ import annotations

from ..csrc import kernels
from .base import Norm, ParamDecl
from .registry import register_norm


@register_norm("rmsnorm")
class RMSNorm(Norm):
    def __init__(self, size: int, eps: float, param: str = "weight", around_zero: bool = False):
        """`param`: the name of the weight behind the norm's prefix (may be empty: the prefix is the name).
        `around_zero`: the checkpoint stores the weight minus one; 1 + w is formed once, in 32-bit, when the weights are
        there."""
        super().__init__()
        self.size = size
        self.eps = eps
        self.param = param
        self.around_zero = bool(around_zero)
        self._one_plus = None

    def param_decls(self):
        return {self.param: ParamDecl((self.size,), "bias32" if self.around_zero else "norm")}

    def weights_loaded(self):
        if self.around_zero:
            self._one_plus = self.tensors[self.param] + 1.0

    @property
    def weight(self):
        if self.around_zero:
            if self._one_plus is None:
                raise RuntimeError("a norm's weights are used before they were loaded (Part.weights_loaded)")
            return self._one_plus
        return self.tensors[self.param]

    def rms_params(self):
        return self.weight, self.eps

    def row_params(self):
        return self.weight, self.eps, 0

    def scale_add(self, a, stream, mult: float, copy=None):
        kernels().norm_scale_add(a, stream, self.weight, self.eps, mult, copy)
        return stream

    def forward_rows(self, stream, rows, out):
        kernels().rmsnorm_rows_f32(stream, rows, self.weight, self.eps, out)
        return out

    def forward(self, x, residual=None, out=None):
        """x [T, size].  residual (same shape), if given, is updated in place
        to x + residual.  Returns the normed rows (in `out` if given; `out`
        may be `x`)."""
        if out is None:
            out = x
        kernels().add_rmsnorm(x, residual, self.weight, self.eps, out)
        return out


@register_norm("layernorm")
class LayerNorm(Norm):
    """(x - mean) / sqrt(variance + eps) * weight over the row, the variance being the mean of the squared
    deviations; a weight and no bias.  It reads and writes a 32-bit residual stream (`forward_rows`, `scale_add`)
    or norms plain rows (`forward`); sums are 32-bit, one rounding at the store."""

    def __init__(self, size: int, eps: float, param: str = "weight"):
        super().__init__()
        self.size = size
        self.eps = eps
        self.param = param

    def param_decls(self):
        return {self.param: ParamDecl((self.size,), "norm")}

    @property
    def weight(self):
        return self.tensors[self.param]

    def row_params(self):
        return self.weight, self.eps, 1

    def scale_add(self, a, stream, mult: float, copy=None):
        if copy is not None:
            raise NotImplementedError("a rounded copy of the stream beside a centred norm")
        kernels().norm_add_norm(stream, a, self.weight, self.eps, mult, center=True)
        return stream

    def forward_rows(self, stream, rows, out):
        kernels().norm_rows(stream, rows, self.weight, self.eps, out, center=True)
        return out


@register_norm("dynamic_tanh")
class DynamicTanh(Norm):
    """tanh(alpha * x) * weight + bias, element by element: one learned slope for the whole row, no mean and no
    variance (`eps` is accepted and unused).  32-bit arithmetic on a 32-bit residual stream, one rounding at the store."""

    def __init__(self, size: int, eps: float = 0.0, param: str = "weight", bias_param: str = "bias",
                 alpha_param: str = "alpha"):
        super().__init__()
        self.size = size
        self.eps = eps
        self.names = dict(weight=param, bias=bias_param, alpha=alpha_param)

    def param_decls(self):
        n = self.names
        return {n["weight"]: ParamDecl((self.size,), "norm"), n["bias"]: ParamDecl((self.size,), "bias32"),
                n["alpha"]: ParamDecl((), "norm")}

    def row_params(self):
        n = self.names
        return self.tensors[n["weight"]], self.eps, 2, self.tensors[n["alpha"]], self.tensors[n["bias"]]

    def forward_rows(self, stream, rows, out):
        w, eps, _kind, alpha, bias = self.row_params()
        kernels().norm_rows(stream, rows, w, eps, out, alpha=alpha, bias=bias)
        return out
