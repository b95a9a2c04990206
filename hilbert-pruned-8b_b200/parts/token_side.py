"""A layer's own input per token: every token has a vector of ``dim`` numbers for every layer, which enters behind the
layer's sublayers, modulated by the stream.

With ``e`` the token's vector for this layer (the columns ``[offset, offset + dim)`` of its row of a table that all layers
share and the embedding part owns: ``embedding_with_side``), ``g = gelu_tanh(W_gate x) * e``, ``y = W_proj g`` and
``x <- x + y / sqrt(mean(y^2) + eps) * w``.  32-bit: both products' results, the gelu, the product with e, the norm and the sum.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import TOKEN_SIDES, ParamSpec, Part

SIDE_TABLE = "token_side.table"           # key of ``StepBatch.shared`` under which the embedding leaves the table


@TOKEN_SIDES.register("gelu_side")
class GeluTokenSide(Part):
    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        self.size = int(spec.params["size"])
        self.dim = int(spec.params["dim"])
        self.offset = int(spec.params["offset"])
        self.eps = float(spec.params["eps"])
        self.padded = (self.dim + 7) // 8 * 8        # the projection's inner size as the tensor-core product reads it
        self.w_gate = self.w_proj = self.norm_weight = None

    def params(self) -> List[ParamSpec]:
        return [ParamSpec("gate", (self.dim, self.size)), ParamSpec("proj", (self.size, self.dim)),
                ParamSpec("norm", (self.size,), kind="vector", init="ones")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        pack, proj = self.ctx.ops.pack_weight, tensors["proj"]
        self.w_gate = pack(tensors["gate"].contiguous())
        if self.padded > self.dim:
            wide = torch.zeros(self.size, self.padded, dtype=proj.dtype, device=proj.device)
            wide[:, : self.dim] = proj
            proj = wide
        self.w_proj = pack(proj.contiguous())
        self.norm_weight = tensors["norm"].reshape(-1).to(torch.float32).contiguous()

    def weight_bytes(self) -> int:
        return sum(w.numel() * w.element_size() for w in (self.w_gate, self.w_proj)) + self.size * 4

    def forward(self, h, x, step, copy=None) -> None:
        """``h`` the stream as products read it, ``x`` the 32-bit stream; ``copy`` receives the new rows."""
        ops, ws, T, cap = self.ctx.ops, self.ctx.workspace, step.num_tokens, self.ctx.max_step_tokens
        table = step.shared.get(SIDE_TABLE)
        if table is None:
            raise ValueError("token_side: the model's embedding has left no side table (embedding_with_side does)")
        s = ws.buffer("token_side.gate", (cap, self.padded), torch.float32)[:T, : self.dim]
        ops.linear(h, self.w_gate, s)
        g = ws.buffer("token_side.unit", (cap, self.padded), self.ctx.dtype)[:T]
        ops.side_unit(s, step.tokens, table, self.offset, g, self.dim)
        y = ws.buffer("token_side.proj", (cap, self.size), torch.float32)[:T]
        ops.linear(g, self.w_proj, y)
        ops.rmsnorm_add(y, self.norm_weight, self.eps, 0.0, x, copy=copy)
