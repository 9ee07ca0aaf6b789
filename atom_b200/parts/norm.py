"""Norms, fused with the residual add.  RMSNorm (atom/model_ops/layernorm.py:57-75):
   r = x + r;  y = r * rsqrt(mean(r^2) + eps) * w,  computed in 32-bit on a 32-bit residual.

In a step of few rows the norm can do without a kernel of its own.  If what is to be added comes as
a product still to run (``PendingProduct``) and the receiver of the normalised rows takes
``ScaledRows``, the product runs with the residual epilogue (r += x W^T in 32-bit, bf16(r * w) and the
sums of r^2 written beside it) and the receiver's first product multiplies its rows by rstd:
   RMSNorm(r; w) V^T = rstd(r) * ((r * w) V^T).
The sums and rstd stay 32-bit; what differs from the kernel of its own is where bf16 rounds."""
from __future__ import annotations

from typing import Dict

import torch

from .. import native
from . import linear as _linear
from .base import Norm
from .linear import NormedDelta, PendingProduct, ScaledRows, SumDelta
from .registry import register
from .spec import ParamSpec


@register("norm", "rmsnorm")
class RMSNorm(Norm):
    graph_safe = True

    def __init__(self, size: int, eps: float, weight_offset: float = 0.0):
        """weight_offset: the stored weight lies around zero and the factor is weight_offset + w (1 + w for a
        design that stores its norm weights so); the sum is formed once after loading, in 32-bit."""
        self.size, self.eps, self.weight_offset = size, eps, float(weight_offset)

    def params(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.size,), role="vector", init="normal" if self.weight_offset else "norm")}

    def after_load(self) -> None:
        super().after_load()
        if self.weight_offset:
            self.w_weight = (self.w_weight.float() + self.weight_offset).contiguous()

    fuses_products = True      # add_norm takes a PendingProduct as delta and the keyword scaled_ok

    def add_norm(self, residual, delta, tag, rows=None, n_rows=None, scaled_ok=False, delta_scale=1.0):
        """delta_scale: what is added to the residual is delta_scale * delta (a design whose sub-blocks enter the
        residual stream times a constant); the product's residual epilogue takes the factor too."""
        if isinstance(delta, NormedDelta):
            if isinstance(delta.norm, RMSNorm) and delta.x_bias is None:
                # what is added passes a norm of its own first: both norms and the add in one kernel
                n = residual.shape[0] if rows is None else (rows.numel() if n_rows is None else n_rows)
                out = self.rt.workspace.get(tag, (n, self.size), self.rt.dtype)
                native.normed_add_rmsnorm(out, residual, delta.x, delta.norm.w_weight, delta.norm.eps, self.w_weight,
                                          self.eps, rows, n, delta_scale)
                return out
            delta = delta.run()
        if isinstance(delta, PendingProduct):
            if scaled_ok and rows is None and self._folds(residual, delta):
                M, ws = residual.shape[0], self.rt.workspace
                xw = ws.get(tag + ".scaled", (M, self.size), torch.bfloat16)
                ssq = ws.get(tag + ".ssq", (native.gemm_rows_grid(), 16), torch.float32)
                native.gemm_rows(delta.x, delta.weight, residual=residual, norm_w=self.w_weight, xout=xw, ssq_out=ssq,
                                 res_scale=delta_scale)
                return ScaledRows(xw, ssq, self.size, self.eps)
            delta = delta.run()
        n = residual.shape[0] if rows is None else (rows.numel() if n_rows is None else n_rows)
        out = self.rt.workspace.get(tag, (n, self.size), self.rt.dtype)
        native.add_rmsnorm(out, residual, delta, self.w_weight, self.eps, rows, n, delta_scale)
        return out

    def normalise(self, x, out, x_bias=None):
        """out = norm(x (+ x_bias)) of rows that are no part of the stream."""
        if x_bias is not None:
            native.add_bias(x, x_bias)
        native.rmsnorm(out, x, self.w_weight, self.eps)
        return out

    def _folds(self, residual, p: PendingProduct) -> bool:
        """The pending product can run with the residual epilogue, and a product over this norm's
        ``size`` columns can take the rows' factors."""
        M = residual.shape[0]
        return (_linear.FOLD_NORMS and p.bias is None and self.rt.dtype == torch.bfloat16
                and residual.dtype == torch.float32 and residual.is_contiguous()
                and p.weight.shape[0] == self.size and _linear.may_defer(p.x, p.weight)
                and M <= native.ROWS_M and native.gemm_rows_supports(M, 1, self.size, self.size))


@register("norm", "layernorm")
class LayerNorm(Norm):
    """(x - mean) / sqrt(variance + eps) * w + b, with the variance as the mean of squared deviations; the add in front
    of it, and the norm that what is added passes first (a ``NormedDelta`` with a LayerNorm), are the same kernel."""
    graph_safe = True
    fuses_products = True

    def __init__(self, size: int, eps: float):
        self.size, self.eps = size, eps

    def params(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.size,), role="vector", init="norm"),
                "bias": ParamSpec((self.size,), role="vector", init="normal")}

    def add_norm(self, residual, delta, tag, rows=None, n_rows=None, scaled_ok=False, delta_scale=1.0):
        """delta_scale: what is added to the residual is delta_scale * delta (after the delta's own norm)."""
        own, x_bias = None, None
        if isinstance(delta, NormedDelta) and isinstance(delta.norm, LayerNorm):
            own, x_bias = (delta.norm.w_weight, delta.norm.w_bias, delta.norm.eps), delta.x_bias
            delta = delta.x
        delta = _linear.resolve(delta)
        n = residual.shape[0] if rows is None else (rows.numel() if n_rows is None else n_rows)
        out = self.rt.workspace.get(tag, (n, self.size), self.rt.dtype)
        native.add_layernorm(out, residual, delta, self.w_weight, self.w_bias, self.eps, rows, n, delta_scale, x_bias, own)
        return out

    def normalise(self, x, out, x_bias=None):
        """out = norm(x (+ x_bias)) of rows that are no part of the stream."""
        native.layernorm(out, x, self.w_weight, self.w_bias, self.eps, x_bias)
        return out


@register("norm", "dynamic_tanh")
class DynamicTanh(Norm):
    """tanh(alpha * r) * w + b with a number alpha of the norm's own, no mean and no variance; the add in front of it, of one
    sub-block's output or of two that run side by side (``SumDelta``), is the same kernel."""
    graph_safe = True
    fuses_sums = True

    def __init__(self, size: int):
        self.size = size

    def params(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.size,), role="vector", init="norm"),
                "bias": ParamSpec((self.size,), role="vector", init="normal"),
                "alpha": ParamSpec((1,), role="vector", init="norm", rows=(1,), members_lack_axis=True)}

    def after_load(self) -> None:
        self._alpha = float(self.w_alpha.float().cpu()[0])

    def add_norm(self, residual, delta, tag, rows=None, n_rows=None):
        a, b = (delta.a, delta.b) if isinstance(delta, SumDelta) else (_linear.resolve(delta), None)
        n = residual.shape[0] if rows is None else (rows.numel() if n_rows is None else n_rows)
        out = self.rt.workspace.get(tag, (n, self.size), self.rt.dtype)
        native.add_dynamic_tanh(out, residual, a, b, self.w_weight, self.w_bias, self._alpha, rows, n)
        return out
