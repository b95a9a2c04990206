"""A gate on a sublayer's result: ``sigmoid(W h + b)`` per element, ``h`` being what the sublayer reads.

The part makes the 32-bit logits ``W h`` only; whoever adds the sublayer's result to the stream applies bias, sigmoid and
product in the kernel that reads the result anyway.  Its matrix reads the same input as the sublayer's first product, so a
mixer that can take a guest (``Mixer.takes_guest``) computes the logits as further rows of that product.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import RESIDUAL_GATES, ParamSpec, Part


@RESIDUAL_GATES.register("sigmoid")
class SigmoidGate(Part):
    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.size = int(spec.params["size"])
        # below the part's prefix ("": the prefix itself); the bias is the weight's name with a suffix
        self.tensor_name = spec.get("tensor_name", "weight")
        self.bias_name = self.tensor_name + spec.get("bias_suffix", ".b")
        self.matrix = self.weight = self.bias = None
        self.lends = False                # the block has found a mixer that may take the matrix (set before weights are bound)
        self.hosted = False               # a mixer's first product makes the logits
        self._logits = None

    def params(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor_name, (self.size, self.size)), ParamSpec(self.bias_name, (self.size,), kind="vector", init="zeros")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.matrix = tensors[self.tensor_name].contiguous()
        self.bias = tensors[self.bias_name].reshape(-1).to(torch.float32).contiguous()
        if not self.lends:
            self._keep()

    def _keep(self) -> None:
        self.weight, self.matrix = self.ctx.ops.pack_weight(self.matrix), None

    def host_rows(self, dtype: torch.dtype):
        """The matrix, for a mixer that appends it to its first product (which then owns the only copy), or None when its
        dtype is another."""
        if self.matrix is None:
            return None
        if self.matrix.dtype != dtype:
            self._keep()
            return None
        rows, self.matrix, self.hosted = self.matrix, None, True
        return rows

    def receive(self, logits) -> None:
        """What the host's product computed for this step: ``[tokens, size]``, 32-bit, a column range of its result."""
        self._logits = logits

    def weight_bytes(self) -> int:
        return (0 if self.hosted else self.weight.numel() * self.weight.element_size()) + self.size * 4

    def logits(self, h, step):
        """``W h`` of the step's tokens, ``[tokens, size]`` in 32-bit, without the bias."""
        if self.hosted:
            out, self._logits = self._logits, None
            if out is None:
                raise RuntimeError("residual gate: the mixer that makes the logits has not run")
            return out
        out = self.ctx.workspace.buffer("residual_gate.logits", (self.ctx.max_step_tokens, self.size), torch.float32)[: step.num_tokens]
        self.ctx.ops.linear(h, self.weight, out)
        return out
