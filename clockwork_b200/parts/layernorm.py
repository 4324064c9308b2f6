"""Layer norm with a weight and no bias over the float32 residual stream, fused with the pending residual add:
``(x - mean) / sqrt(mean of the squared deviations + eps) * weight``.

Parameters as ``rmsnorm``'s (``size``, ``eps``, optional ``offset`` and ``weight_suffix``), whose kernels it runs with the
row's mean taken off first.  A product cannot begin this norm (the mean is known only when the whole row is), so it has
no ``split_weight``, and the products that read it get plain tensors.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import ResidualStream
from .registry import register_norm
from .rmsnorm import WeightedNorm


class LayerNorm(WeightedNorm):
    def forward(self, stream: ResidualStream, status: torch.Tensor, lazy: bool = False):
        stream.half_norm = stream.normed = None
        delta, stream.pending = stream.pending, None
        return ops.add_rmsnorm(stream.residual, delta, self.weight, self.eps, self.dtype, status, center=True)

    def forward_rows(self, stream: ResidualStream, rows: torch.Tensor, status: torch.Tensor) -> torch.Tensor:
        stream.flush()
        return ops.rmsnorm_rows(stream.residual, rows, self.weight, self.eps, self.dtype, status, center=True)


register_norm("layernorm", LayerNorm, replace=True)
