"""Group-wise RMS norm: a vector is cut into ``groups`` runs of equal length, every run is brought to unit mean square by itself
(``eps`` inside the root), and a weight scales element by element (``groups`` 1: the ordinary RMS norm).  Sums and scaling in 32-bit on the device, the result in the
dtype the next matrix product reads.

As a norm that sits BEHIND the sum of the residual stream and a sublayer's result (``norm_sum``) it writes the stream itself:
``x = norm(alpha * x + sigmoid(gate) * y)``, in one pass over the row, and leaves a copy of the new row in the products'
dtype when asked.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import NORMS, Norm, ParamSpec


@NORMS.register("group_rmsnorm")
class GroupRMSNorm(Norm):
    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.size = int(spec.params["size"])
        self.eps = float(spec.params["eps"])
        self.groups = int(spec.params.get("groups", 1))
        if self.groups < 1 or self.size % self.groups:
            raise ValueError(f"group_rmsnorm: {self.groups} groups do not divide a vector of {self.size}")
        self.tensor_name = spec.get("tensor_name", "weight")     # below the part's prefix ("": the prefix itself)
        self.weight = None

    def params(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor_name, (self.size,), kind="vector", init="ones")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors[self.tensor_name].reshape(self.size).to(torch.float32).contiguous()

    def weight_bytes(self) -> int:
        return self.size * 4

    def forward(self, x, out, rows=None) -> None:
        """``out[i] = norm(x[rows[i]])`` (``rows`` None: every row of ``x``)."""
        self.ctx.ops.group_rmsnorm(x, self.weight, self.eps, self.groups, out, rows)

    def norm_sum(self, x, alpha: float, y, gate=None, gate_bias=None, n_sum: int = 1, copy=None) -> None:
        """``x = norm(alpha * x + sigmoid(gate + gate_bias) * y)`` in place (``Ops.gated_sum_norm``)."""
        self.ctx.ops.gated_sum_norm(x, alpha, y, self.weight, self.eps, self.groups, gate=gate, gate_bias=gate_bias, n_sum=n_sum, copy=copy)
