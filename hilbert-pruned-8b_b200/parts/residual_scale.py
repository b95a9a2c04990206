"""A learned factor per channel on a sublayer's result, ``x += factors * sublayer(h)``.

The part only holds the vector, widened to 32-bit at load; the kernel that adds the result to the stream multiplies.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import RESIDUAL_SCALES, ParamSpec, Part


@RESIDUAL_SCALES.register("channel")
class ChannelScale(Part):
    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.size = int(spec.params["size"])
        self.tensor_name = spec.get("tensor_name", "weight")     # below the part's prefix ("": the prefix itself)
        self.factors = None

    def params(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor_name, (self.size,), kind="vector", init="ones")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.factors = tensors[self.tensor_name].reshape(self.size).to(torch.float32).contiguous()

    def weight_bytes(self) -> int:
        return self.size * 4
