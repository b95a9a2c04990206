"""The generic decoder: embedding, blocks in plan order, final norm, head.

Built from a ``ModelSpec`` through the part registries; it holds no architecture-specific
code.  The order of the reference's forward pass (cleanroom-transformer/src/cpu_backend.c:218-263):
embed, then per layer norm -> mixer -> residual, norm -> feed-forward -> residual, then the
final norm and the head only at the positions whose logits are wanted (the reference reads
out the last position only, cpu_backend.c:253-259).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from ..config.spec import ModelSpec
from ..parts.base import BLOCKS, EMBEDDINGS, HEADS, NORMS, STREAM_VECTORS, BuildContext, CacheNeed, ParamSpec, StateNeed
from ..parts.block import NORMED, NormAhead


class _NullOps:
    """Stands in for the kernel library where a model is only described, not run."""

    def __getattr__(self, name):
        raise RuntimeError("this model was built without kernels (description only)")


def describe_context() -> BuildContext:
    return BuildContext(device=torch.device("cpu"), dtype=torch.float32, ops=_NullOps(), workspace=None,
                        max_step_tokens=1)


class DecoderModel:
    def __init__(self, spec: ModelSpec, ctx: BuildContext):
        spec.validate()
        self.spec = spec
        self.ctx = ctx
        self.embedding = EMBEDDINGS.build(spec.embedding, ctx)
        self.blocks = [BLOCKS.get(ls.block)(ls, ctx) for ls in spec.layers]
        self.final_norm = NORMS.build(spec.final_norm, ctx)
        self.head = HEADS.build(spec.head, ctx)
        self.stream_vectors = STREAM_VECTORS.build(spec.stream_vectors, ctx) if spec.stream_vectors is not None else None
        self.prefix = spec.weight_prefixes[-1]
        self.graph_safe = (all(getattr(part, "graph_safe", True) for _, part in self.named_parts())
                           and all(getattr(b, "graph_safe", True) for b in self.blocks))

    # ------------------------------------------------------------------ weights
    def named_parts(self) -> List[Tuple[str, object]]:
        """(prefix below the decoder's prefix, part) of every part that may own weights."""
        out: List[Tuple[str, object]] = [(self.spec.embedding_prefix, self.embedding)]
        for ls, block in zip(self.spec.layers, self.blocks):
            for sub, part in block.named_parts():
                out.append((ls.prefix + sub, part))
        out.append((self.spec.final_norm_prefix, self.final_norm))
        out.append((self.spec.head_prefix, self.head))
        if self.stream_vectors is not None:
            out.append((self.spec.stream_vectors_prefix, self.stream_vectors))
        return out

    def weight_table(self, prefix: Optional[str] = None) -> Dict[str, ParamSpec]:
        prefix = self.prefix if prefix is None else prefix
        table: Dict[str, ParamSpec] = {}
        for sub, part in self.named_parts():
            for p in part.params():
                full = (sub + p.name) if p.absolute else (prefix + sub + p.name)
                if full in table:
                    raise ValueError(f"weights: two parts name the tensor {full}")
                table[full] = p
        return table

    def bind(self, tensors: Dict[str, torch.Tensor], prefix: Optional[str] = None) -> None:
        prefix = self.prefix if prefix is None else prefix
        for sub, part in self.named_parts():
            local = {}
            for p in part.params():
                full = (sub + p.name) if p.absolute else (prefix + sub + p.name)
                if full in tensors:
                    local[p.name] = tensors[full]
            part.bind(local)
        if getattr(self.head, "tied", False):
            stored = self.head.tie(self.embedding.weight)
            if stored is not None and stored is not self.embedding.weight and hasattr(self.embedding, "share"):
                self.embedding.share(stored)       # one copy of the table for both

    def first_weight_name(self) -> str:
        return self.spec.embedding_prefix + self.embedding.params()[0].name

    # ------------------------------------------------------------------ cache needs
    def cache_needs(self) -> Dict[int, CacheNeed]:
        out = {}
        for i, e in enumerate(self.spec.plan):
            need = self.blocks[e.layer].cache_need()
            if need is not None and e.cache_of is None:
                out[i] = need
        return out

    EMBEDDING_STATE = -1        # the key of the embedding's per-sequence state beside the plan entries'

    def state_needs(self) -> Dict[int, StateNeed]:
        out = {}
        if getattr(self.embedding, "state_need", None) is not None and self.embedding.state_need() is not None:
            out[self.EMBEDDING_STATE] = self.embedding.state_need()
        for i, e in enumerate(self.spec.plan):
            need = self.blocks[e.layer].state_need()
            if need is not None:
                out[i] = need
        return out

    # ------------------------------------------------------------------ accounting
    def step_weight_bytes(self) -> int:
        """Bytes of weights one decode step reads: every plan entry's matrices once, the
        norms, and the head (the embedding table is only gathered from)."""
        total = 0
        for e in self.spec.plan:
            b = self.blocks[e.layer]
            total += sum(p.weight_bytes() for _, p in b.named_parts())
        total += self.final_norm.weight_bytes() + self.head.weight_bytes()
        if self.stream_vectors is not None:
            total += self.stream_vectors.weight_bytes()
        return total

    def num_parameters(self) -> int:
        n = 0
        for p in self.weight_table().values():
            if p.optional:
                continue
            c = 1
            for s in p.shape:
                c *= s
            n += c
        return n

    # ------------------------------------------------------------------ forward
    def _add_vector(self, x, entry, block, step):
        """Adds the entry's vector to the stream, and in the same pass makes the block's first norm output where its request is
        of that form; returns what the block then finds prepared."""
        request = block.fold_request(step) if getattr(block, "folds_norms", False) else None
        vector = self.stream_vectors.vector(entry.adds)
        if isinstance(request, NormAhead) and tuple(request[3].shape) == tuple(x.shape):
            self.ctx.ops.parallel_sum(x, vector=vector, then=(request[0], request[2], request[1]), then_out=request[3])
            return NORMED
        self.ctx.ops.parallel_sum(x, vector=vector)
        return None

    def forward(self, step, cache) -> Optional[torch.Tensor]:
        """Runs the step's tokens through the decoder; returns ``[wanted, vocab]`` 32-bit
        logits (None when nothing is wanted)."""
        ws, cap, T = self.ctx.workspace, self.ctx.max_step_tokens, step.num_tokens
        H, V = self.spec.hidden_size, self.spec.vocab_size
        x = ws.buffer("model.x", (cap, H), torch.float32)[:T]
        if getattr(self.embedding, "state_need", None) is not None:
            self.embedding.forward(step.tokens, x, step=step, state=cache.state_view(self.EMBEDDING_STATE))
        elif getattr(self.embedding, "takes_step", False):
            self.embedding.forward(step.tokens, x, step=step)      # it leaves something in step.shared for the layers
        else:
            self.embedding.forward(step.tokens, x)
        # Norms at the seam between two blocks may be folded into the products around them: a block
        # that can says what it needs (fold_request), the block in front prepares it and hands on
        # what it prepared.
        # A vector that the next entry adds goes with the request to a block that can add it to its own sum (adds_vector).
        plan, prepared, added = self.spec.plan, None, False
        for i, e in enumerate(plan):
            owner = i if e.cache_of is None else e.cache_of
            block = self.blocks[e.layer]
            if e.adds is not None and not added:
                prepared = self._add_vector(x, e, block, step)
            args = (x, step, cache.view(owner), cache.state_view(i), e.cache_of is None)
            after = plan[i + 1] if i + 1 < len(plan) else None
            added = False
            if getattr(block, "folds_norms", False):
                nxt = self.blocks[after.layer] if after is not None else None
                request = nxt.fold_request(step) if nxt is not None and getattr(nxt, "folds_norms", False) else None
                kw = {}
                if after is not None and after.adds is not None:
                    if getattr(block, "adds_vector", False):
                        kw["vector"], added = self.stream_vectors.vector(after.adds), True
                    else:
                        request = None              # the norm in front of the next entry reads the stream behind the vector
                prepared = block.forward(*args, prepared=prepared, prepare_next=request, **kw)
            else:
                block.forward(*args)
                prepared = None
        n = step.num_wanted
        if n == 0:
            return None
        hn = ws.buffer("model.head_in" + step.tag, (n, H), self.ctx.dtype)
        self.final_norm.forward(x, hn, rows=step.want_rows)
        logits = ws.buffer("model.logits" + step.tag, (n, V), torch.float32)
        self.head.forward(hn, logits)
        return logits


def weight_table(spec: ModelSpec, prefix: Optional[str] = None) -> Dict[str, ParamSpec]:
    """The weight table of ``spec`` without building anything on a device."""
    return DecoderModel(spec, describe_context()).weight_table(prefix)
