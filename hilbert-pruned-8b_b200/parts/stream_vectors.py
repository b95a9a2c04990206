"""Vectors that plan entries add to every token's stream in front of themselves (``PlanEntry.adds``): a model that goes through
a run of layers several times with the same weights tells the passes apart by them.

The part holds the table, widened to 32-bit at load.  A block with ``adds_vector`` adds the next entry's vector in the kernel
that forms its own sum; in front of other entries the model adds it by a kernel of its own.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import STREAM_VECTORS, ParamSpec, Part


@STREAM_VECTORS.register("stream_vectors")
class StreamVectors(Part):
    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.size = int(spec.params["size"])
        self.count = int(spec.params["count"])
        self.tensor_name = spec.get("tensor_name", "weight")
        self.table = None

    def params(self) -> List[ParamSpec]:
        return [ParamSpec(self.tensor_name, (self.count, self.size))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.table = tensors[self.tensor_name].to(torch.float32).contiguous()
        self._rows = [self.table[i].clone() for i in range(self.count)]      # every row on an allocation's (16-byte) boundary

    def weight_bytes(self) -> int:
        return self.count * self.size * 4

    def vector(self, i: int) -> torch.Tensor:
        return self._rows[i]
