"""Mixture of experts with a clamped gated unit, and an optional shared expert.

Router: ``z = W_router h`` in 32-bit; the ``top`` experts with the largest logits are chosen per
token and weighted by the softmax over the chosen logits alone.  Expert (no biases):
``g = min(W_gate h, limit)``, ``u = clamp(W_up h, -limit, limit)``, ``y = g sigmoid(alpha g) (u + 1)``,
output ``W_down y``; ``alpha`` is 1.702 unless the spec says otherwise.  The layer's result is the
weighted sum of the chosen experts' outputs, plus the shared expert's (same form, own sizes and
limit), which runs for every token.

Options beside that form.  ``router`` "scores": scores are the softmax over ALL router outputs; the choice goes by
``score + correction`` (tensor ``correction``), only among the outputs of the ``keep`` best of ``groups`` equal runs of
neighbours (a run's score: its largest choice score; the others count as minus infinity); the weights are the chosen
outputs' scores, without the correction, divided by their sum ``+ 1e-20``.  ``identity`` n: the router's last n outputs are
identity experts, which hand the token's input back (times the weight) and have no tensors.  ``unit`` "gelu": an expert is
``W_down gelu(W_up h)`` with the exact (erf) gelu, no gate matrix.  ``shared_gate``: the shared expert's result is multiplied
by ``sigmoid(W_sg h)``, one number per token (tensor ``shared.sg`` ``[1, width]``).  ``router`` "sigmoid": the ``top`` largest
logits as in the plain form, weighted by their sigmoids, not divided by anything.  ``unit`` "silu_glu": an expert is
``W_down (silu(W_gate h) * (W_up h))``.  ``weigh`` "input": an expert is fed ``weight * h`` and its result is added as it is
(evaluated as ``W (w h) = w (W h)`` in front of the activation, in 32-bit).  ``router_bias``: the router's logits have a bias (tensor
``router.b``), which counts for the choice and for the weights; for the routers "top_logits" and "sigmoid".

Tensors below the part's prefix: ``router``, ``e<i>.gate|up|down``, ``shared.gate|up|down``.  The
experts' matrices are stacked at load time (and packed for the tensor cores where those take them); the routed products gather their rows on the device
from a plan that a kernel makes, so a step reads nothing back and decode steps can be captured.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from .base import FEED_FORWARDS, FeedForward, ParamSpec


@FEED_FORWARDS.register("moe")
class MixtureOfExperts(FeedForward):
    can_overwrite = True

    def __init__(self, spec, ctx):
        super().__init__(spec, ctx)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.n_experts = int(p["num_experts"])
        self.top = int(p["top"])
        self.ff = int(p["expert_size"])
        self.limit = float(p.get("limit", 0.0))
        self.alpha = float(p.get("alpha", 1.702))
        self.shared_ff = int(p.get("shared_size") or 0)
        self.shared_limit = float(p.get("shared_limit", self.limit))
        self.router = p.get("router", "top_logits")
        self.unit = p.get("unit", "clamped_glu")
        self.weigh = p.get("weigh", "output")
        if self.router not in ("top_logits", "scores", "sigmoid") or self.unit not in ("clamped_glu", "gelu", "silu_glu") \
                or self.weigh not in ("output", "input"):
            raise ValueError(f"moe: router {self.router!r} ('top_logits', 'scores' or 'sigmoid'), unit {self.unit!r} ('clamped_glu', 'gelu' or "
                             f"'silu_glu'), weigh {self.weigh!r} ('output' or 'input')")
        self.identity = int(p.get("identity") or 0)
        self.groups, self.keep = int(p.get("groups") or 1), int(p.get("keep") or 1)
        self.shared_gate = bool(p.get("shared_gate", False))
        self.n_outputs = self.n_experts + self.identity
        if (self.identity or self.groups > 1) and self.router != "scores":
            raise ValueError("moe: identity experts and groups belong to the router 'scores'")
        if self.n_outputs % self.groups or not 1 <= self.keep <= self.groups or self.top > self.n_outputs // self.groups * self.keep:
            raise ValueError(f"moe: {self.n_outputs} router outputs in {self.groups} groups, {self.keep} kept, top {self.top}")
        if not 1 <= self.top <= self.n_outputs:
            raise ValueError(f"moe: top {self.top} of {self.n_outputs} experts")
        if self.weigh == "input" and self.identity:
            raise ValueError("moe: identity experts have their results weighted")
        self.router_bias = bool(p.get("router_bias", False))
        if self.router_bias and self.router == "scores":
            raise ValueError("moe: the router 'scores' has a correction, not a bias")
        if self.unit == "silu_glu" and self.shared_gate:
            raise ValueError("moe: the gate on the shared expert belongs to the unit 'gelu'")
        self.glu = self.unit != "gelu"                        # two matrices in front of the activation
        # the experts' results can be handed on unsummed (one row per token and chosen expert)
        self.sums_entries = self.weigh == "input" and not self.shared_ff
        # or with their weights and the shared expert's result beside them
        self.weighs_entries = not self.identity
        self.b_router = None
        self.first = None                     # both products' weights packed for the tensor cores (then w_gate and w_up are not kept)
        self.correction = None
        self.gate_col = None
        self.w_router = self.w_gate = self.w_up = self.w_down = self.ws_gate_up = self.ws_down = None

    def params(self) -> List[ParamSpec]:
        W, F = self.hidden, self.ff
        glu = self.glu
        out = [ParamSpec("router", (self.n_outputs, W))]
        if self.router_bias:
            out.append(ParamSpec("router.b", (self.n_outputs,), kind="vector", init="zeros"))
        if self.router == "scores":
            out.append(ParamSpec("correction", (self.n_outputs,), kind="vector", init="zeros"))
        for e in range(self.n_experts):
            out += ([ParamSpec(f"e{e}.gate", (F, W))] if glu else []) + [ParamSpec(f"e{e}.up", (F, W)), ParamSpec(f"e{e}.down", (W, F))]
        if self.shared_ff:
            S = self.shared_ff
            out += ([ParamSpec("shared.gate", (S, W))] if glu else []) + [ParamSpec("shared.up", (S, W)), ParamSpec("shared.down", (W, S))]
            if self.shared_gate:
                out.append(ParamSpec("shared.sg", (1, W)))
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        t, E = tensors, self.n_experts
        self.w_router = t["router"].to(torch.float32).contiguous()
        if self.router_bias:
            self.b_router = t["router.b"].reshape(-1).to(torch.float32).contiguous()
        glu = self.glu
        self.w_gate = torch.stack([t[f"e{e}.gate"] for e in range(E)]).contiguous() if glu else None
        self.w_up = torch.stack([t[f"e{e}.up"] for e in range(E)]).contiguous()
        self.w_down = torch.stack([t[f"e{e}.down"] for e in range(E)]).contiguous()
        packed = self.ctx.ops.pack_experts(self.w_gate if glu else self.w_up, self.w_up if glu else None, self.w_down)
        if packed is not None:
            self.first, self.w_down = packed
            self.w_gate = self.w_up = None
        if self.router == "scores":
            self.correction = t["correction"].reshape(-1).to(torch.float32).contiguous()
        if self.shared_ff:
            pack = self.ctx.ops.pack_weight
            rows = ([t["shared.gate"]] if glu else []) + [t["shared.up"]]
            if self.shared_gate:
                # the per-token gate is one more row of the shared expert's first product (zero rows up to 16 bytes)
                self.gate_col = sum(r.shape[0] for r in rows)
                rows.append(t["shared.sg"].reshape(1, self.hidden))
                pad = (-(self.gate_col + 1)) % 8
                if pad:
                    rows.append(torch.zeros(pad, self.hidden, dtype=rows[0].dtype, device=rows[0].device))
            # (the plain gated unit is the epilogue of its first product: linear_swiglu)
            self.ws_gate_up = pack(torch.cat(rows, dim=0).contiguous(), swiglu=self.unit == "silu_glu")
            self.ws_down = pack(t["shared.down"].contiguous())

    def weight_bytes(self) -> int:
        # what a decode step of one token reads: the router, `top` experts, the shared expert
        per = (3 if self.glu else 2) * self.ff * self.hidden * self.w_down.element_size()
        shared = sum(w.numel() * w.element_size() for w in (self.ws_gate_up, self.ws_down)) if self.shared_ff else 0
        return self.w_router.numel() * 4 + self.top * per + shared

    def forward_entries(self, h, step):
        """``(rows, top)``: the chosen experts' results, 32-bit ``[tokens * top, width]``, whose sum per token is the result."""
        return self._experts(h, step, None, False)[0], self.top

    def forward_weighted(self, h, step):
        rows, weights = self._experts(h, step, None, False)
        base = None
        if self.shared_ff:
            base = self.ctx.workspace.buffer("moe.shared_out", (self.ctx.max_step_tokens, self.hidden), torch.float32)[: step.num_tokens]
            self._shared(h, base, step, accumulate=False)
        return rows, self.top, weights if self.weigh == "output" else None, base

    def _experts(self, h, step, residual, accumulate: bool):
        ops, ws, T, cap = self.ctx.ops, self.ctx.workspace, step.num_tokens, self.ctx.max_step_tokens
        experts = ws.buffer("moe.experts", (cap, self.top), torch.int32)[:T]
        weights = ws.buffer("moe.weights", (cap, self.top), torch.float32)[:T]
        if self.router == "scores":
            ops.moe_route_scores(h, self.w_router, self.correction, self.top, self.groups, self.keep, experts, weights)
        else:
            ops.moe_route(h, self.w_router, self.top, experts, weights, scoring="sigmoid" if self.router == "sigmoid" else "softmax_chosen",
                          bias=self.b_router)
        if self.unit == "gelu":
            rows = ops.moe_experts(h, experts, weights, self.first if self.first is not None else self.w_up, None, self.w_down, 0.0, 0.0, residual,
                                   accumulate, ws, cap, tag=".gelu", identity=self.identity > 0, unit="gelu", weigh=self.weigh)
        else:
            rows = ops.moe_experts(h, experts, weights, self.first if self.first is not None else self.w_gate, self.w_up, self.w_down, self.limit,
                                   self.alpha, residual, accumulate, ws, cap, unit=self.unit, weigh=self.weigh)
        return rows, weights

    def forward(self, h, residual, step, accumulate: bool = True):
        ops, ws, T, cap = self.ctx.ops, self.ctx.workspace, step.num_tokens, self.ctx.max_step_tokens
        self._experts(h, step, residual, accumulate)
        if self.shared_ff:
            self._shared(h, residual, step, accumulate=True)

    def _shared(self, h, out, step, accumulate: bool) -> None:
        """The shared expert's result, added to ``out`` or written there."""
        ops, ws, T, cap = self.ctx.ops, self.ctx.workspace, step.num_tokens, self.ctx.max_step_tokens
        S = self.shared_ff
        act = ws.buffer("moe.shared_act", (cap, S), self.ctx.dtype)[:T]
        if self.unit == "silu_glu":
            ops.linear_swiglu(h, self.ws_gate_up, act, ws, cap)
        else:
            first = self.ws_gate_up.shape[0]
            gu = ws.buffer(f"moe.shared_first.{first}", (cap, first), torch.float32)[:T]
            ops.linear(h, self.ws_gate_up, gu)
            if self.unit == "gelu":
                # sigmoid(W_sg h) * (W_down act) = W_down (sigmoid(W_sg h) * act): the gate multiplies the rows the product reads
                ops.gelu_unit(gu, act, "erf", row_gate=self.gate_col)
            else:
                ops.glu_clamp(gu[:, : 2 * S], act, self.shared_limit, self.alpha)
        ops.linear(act, self.ws_down, out, accumulate=accumulate)
