"""A weight matrix with an optional bias and the product against it; the helper parts build
their projections from.  Not a part itself.

y[t, o] = sum_i W[o, i] x[t, i] (+ b[o])  (src/kernels.rs:54-57).  The product is written in the
activation precision, in float32 (logits), or added into the float32 residual stream.  A factor per
output feature on what is added (``out_scale``, float32 [out]) is applied in float32 after the product.
``stores``: ``add_into`` writes its rows instead of adding to them (rows that are the product's alone).
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels


class Linear:
    def __init__(self, weight: torch.Tensor, bias: Optional[torch.Tensor] = None):
        self.weight = weight.contiguous()
        self.bias = None if bias is None else bias.to(torch.float32).contiguous()
        self.out_features, self.in_features = weight.shape
        self.out_scale: Optional[torch.Tensor] = None
        self.stores = False

    @classmethod
    def stacked(cls, matrices, bias: Optional[torch.Tensor] = None, multiple: int = 1) -> "Linear":
        """One product for several matrices of the same input, their rows one after the other, with rows
        of zeros up to a multiple of ``multiple`` (results whose rows TMA can address)."""
        rows = sum(m.shape[0] for m in matrices)
        pad = -rows % multiple
        first = matrices[0]
        if pad:
            matrices = list(matrices) + [torch.zeros((pad, first.shape[1]), dtype=first.dtype, device=first.device)]
            if bias is not None:
                bias = torch.cat([bias, torch.zeros(pad, dtype=bias.dtype, device=bias.device)])
        return cls(torch.cat(list(matrices), dim=0), bias)

    def __call__(self, x, out_dtype: Optional[torch.dtype] = None, out: Optional[torch.Tensor] = None,
                 act: Optional[str] = None) -> torch.Tensor:
        """x @ W.T (+ b); ``x`` a tensor, or kernels.UnscaledRows (a norm taken into this product).
        ``act``: one of kernels.PLAIN_ACTS, applied before the results are rounded."""
        rows = x.rows if isinstance(x, kernels.UnscaledRows) else x
        if out is None:
            out = torch.empty((rows.shape[0], self.out_features), dtype=out_dtype or rows.dtype, device=rows.device)
        kernels.gemm(x, self.weight, out, self.bias, accumulate=False, act=act)
        return out

    def add_into(self, x: torch.Tensor, residual: torch.Tensor, then_norm=None):
        """residual += (x @ W.T (+ b)) * out_scale; residual is float32.  ``then_norm``: the RMSNorm part that
        reads the residual next, if any; where the kernel can it leaves that norm's input
        (kernels.UnscaledRows), which is returned, else None and the norm runs by itself."""
        if self.stores:
            if self.out_scale is not None or then_norm is not None:
                raise ValueError("a product that stores its rows takes no factor on them and leaves nothing for a norm")
            kernels.gemm(x, self.weight, residual, self.bias)
            return None
        link = (then_norm.weight, then_norm.eps) if then_norm is not None else None
        return kernels.gemm(x, self.weight, residual, self.bias, accumulate=True, then_norm=link, col_scale=self.out_scale)

    def bytes(self) -> int:
        b = 0 if self.bias is None else self.bias.numel() * self.bias.element_size()
        return self.weight.numel() * self.weight.element_size() + b
