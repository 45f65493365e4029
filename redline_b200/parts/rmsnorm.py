"""RMSNorm fused with the residual add: y = x * rsqrt(mean(x^2) + eps) * w with the
weight multiplying directly, sums in float32
(reference: src/cuda/kernels/elementwise.cu:29-64); designs that store the weight around
zero (``zero_centred``) multiply by 1 + w, formed in float32 when the weights are loaded, and
so is a constant factor on the normed rows (``scale``: a factor on the logits, say).
``rmsnorm_sum`` norms the weighted sum of the stream and a sublayer's output, for blocks
that norm after the sum."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional

import torch

from ..ops import kernels
from .base import Norm, WeightedTerms, register
from .spec import TensorSpec


@dataclass(frozen=True)
class RMSNormParams:
    size: int
    eps: float
    zero_centred: bool = False
    scale: float = 1.0             # the normed rows are multiplied by this


@register("norm", "rmsnorm")
class RMSNorm(Norm):
    def tensors(self) -> Dict[str, TensorSpec]:
        return {"weight": TensorSpec((self.params.size,))}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors["weight"]
        if self.params.zero_centred:
            self.weight = (1.0 + self.weight.float()).contiguous()
        if self.params.scale != 1.0:
            self.weight = (self.weight.float() * self.params.scale).contiguous()

    def nbytes(self) -> int:
        return self.weight.numel() * self.weight.element_size()

    def add_norm(self, residual, delta, out, rows_idx=None, rows=None) -> None:
        kernels.add_rmsnorm(residual, delta, self.weight, out, self.params.eps, rows_idx, rows)

    def rms_params(self):
        return self.weight, self.params.eps


@dataclass(frozen=True)
class RMSNormSumParams:
    size: int
    eps: float
    alpha: float = 1.0             # factor on the stream
    zero_centred: bool = False
    scaled: bool = False           # the sublayer's output is multiplied by a vector first


@register("norm", "rmsnorm_sum")
class RMSNormSum(Norm):
    """stream = rmsnorm(alpha * stream + scale * delta) * weight: the norm after the sum ("postnorm" blocks)."""

    sums_terms = True

    def tensors(self) -> Dict[str, TensorSpec]:
        t = {"weight": TensorSpec((self.params.size,))}
        if self.params.scaled:
            t["scale"] = TensorSpec((self.params.size,))
        return t

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors["weight"].float()
        if self.params.zero_centred:
            self.weight = 1.0 + self.weight
        self.weight = self.weight.contiguous()
        self.scale = tensors["scale"].float().contiguous() if self.params.scaled else None

    def nbytes(self) -> int:
        return self.weight.numel() * 4 * (2 if self.params.scaled else 1)

    def add_post_cast(self, residual: torch.Tensor, delta: torch.Tensor, out: Optional[torch.Tensor],
                      rows: Optional[int] = None) -> None:
        """The norm of the sum in place on the stream; with ``out`` also out = the new stream rows in out's type.
        ``delta`` may be ``WeightedTerms``: the same kernel then forms their sum."""
        p = self.params
        terms = {}
        if isinstance(delta, WeightedTerms):
            terms = dict(top=delta.top, mix_weight=delta.weight, shared=delta.shared, shared_gate=delta.shared_gate)
            delta = delta.rows
        kernels.sum_norm(residual, delta, self.weight, self.scale, p.alpha, p.eps, out, rows=rows, **terms)
