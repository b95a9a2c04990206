"""Typed configuration of the Mirorax decoder: a pre-norm stack whose two sublayers stand side by side, ``h = norm(x)``, ``x +=
s_a * mixer(h) + s_b * ff(h)``, with a learned factor per channel on each result, and in which a run of neighbouring layers may
be gone through several times with the same weights (every pass with caches of its own, and a learned vector of its own added
to the stream in front of it).  Two kinds of mixer: a causal grouped attention without positions, with biases and a sigmoid
gate on every element of the heads' results; and an attention over a sliding window with a sink per head whose keys and
values come from one small cached latent per token, a separate part of queries and keys rotated by position.  The feed-forward
is a clamped gated unit, or a mixture of experts (silu units, the largest biased logits, softmax over the chosen) with a
shared expert, or absent.  The head has a matrix of its own.

config.json keys (every size and every constant that may differ between models comes from here): ``architecture``
("Mirorax"), ``vocab``, ``width``, ``norm {eps}``, ``loop {start, stop, times}`` (absent or null: every layer runs once) and ``layers``: a
list of ``{"type", "mixer", "mlp"}`` with ``type``

* "attention": ``mixer`` = ``heads, kv_heads, dim, vdim, scale``;
* "latent_attention": ``mixer`` = ``heads, dim, rot_dim, vdim, kv_rank, scale, mask {size}, rot {base, dims}``;

and ``mlp`` null, ``{"kind": "dense", "ff", "limit"}`` or ``{"kind": "moe", "router {experts, top}", "expert {ff}", "shared {ff}" | absent}``.
Tensor names: ``embed``, ``loop.step``, ``l<i>.norm1``, ``l<i>.ls1|ls2``, ``l<i>.mix.*`` (bias: ``.b`` added), ``l<i>.mlp.*``, ``final.norm``,
``head``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError
from .ridotar import _sizes
from .spec import LayerSpec, ModelSpec, PartSpec, PlanEntry
from .tonovik import _float, _int, _number, _rot


def _mixer(kind: str, m: Any, where: str) -> Dict[str, Any]:
    if not isinstance(m, dict):
        raise ConfigError(f"config: missing {where[:-1]}")
    mixer: Dict[str, Any] = _sizes(m, ("heads", "dim", "vdim"), where)
    mixer["scale"] = _float(m, "scale", where)
    if kind == "attention":
        mixer["kv_heads"] = _int(m, "kv_heads", where)
        if mixer["heads"] % mixer["kv_heads"]:
            raise ConfigError(f"config: {where}heads is no multiple of kv_heads")
        return mixer
    mixer["kv_rank"], mixer["rot_dim"] = _int(m, "kv_rank", where), _int(m, "rot_dim", where, least=0)
    mixer["mask"] = {"size": _int(m.get("mask"), "size", where + "mask.")}
    mixer["rot"] = _rot(m, where, mixer["rot_dim"], scaling=False) if mixer["rot_dim"] or m.get("rot") is not None else {"base": 1.0, "dims": 0}
    return mixer


def _mlp(mlp: Any, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    kind = mlp.get("kind") if isinstance(mlp, dict) else None
    if kind == "dense":
        limit = _float(mlp, "limit", where)
        if limit < 0.0:
            raise ConfigError(f"config: {where}limit is negative")
        return {"kind": "dense", "ff": _int(mlp, "ff", where), "limit": limit}
    if kind != "moe":
        raise ConfigError(f"config: {where}kind must be dense or moe (or mlp null)")
    router = _sizes(mlp.get("router"), ("experts", "top"), where + "router.")
    if router["top"] > router["experts"]:
        raise ConfigError(f"config: {where}router.top is larger than the number of experts")
    out = {"kind": "moe", "router": router, "expert": _sizes(mlp.get("expert"), ("ff",), where + "expert.")}
    if mlp.get("shared") is not None:
        out["shared"] = _sizes(mlp["shared"], ("ff",), where + "shared.")
    return out


@dataclass(frozen=True)
class MiroraxConfig:
    vocab: int
    width: int
    eps: float
    loop: Optional[Dict[str, int]] = None                            # start, stop (one past the last layer), times
    layers: List[Dict[str, Any]] = field(default_factory=list)       # the validated entries of config.json
    eos_token_ids: List[int] = field(default_factory=list)
    max_position_embeddings: Optional[int] = None

    architecture = "Mirorax"
    model_type = "mirorax"

    # llama-style names that the generic entry points and the benchmark read
    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, root: Dict[str, Any]) -> "MiroraxConfig":
        if not isinstance(root, dict):
            raise ConfigError("config: config.json is not an object")
        vocab, width = _int(root, "vocab", ""), _int(root, "width", "")
        eps = _float(root.get("norm"), "eps", "norm.")
        raw = root.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config: layers must be a list with at least one entry")
        layers: List[Dict[str, Any]] = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]."
            kind = entry.get("type") if isinstance(entry, dict) else None
            if kind not in ("attention", "latent_attention"):
                raise ConfigError(f"config: {where}type must be attention or latent_attention")
            layers.append({"type": kind, "mixer": _mixer(kind, entry.get("mixer"), where + "mixer."), "mlp": _mlp(entry.get("mlp"), where + "mlp.")})
        loop = root.get("loop")
        if loop is not None:
            loop = {"start": _int(loop, "start", "loop.", least=0), "stop": _int(loop, "stop", "loop."), "times": _int(loop, "times", "loop.")}
            if not loop["start"] < loop["stop"] <= len(layers):
                raise ConfigError(f"config: loop runs layers {loop['start']} .. {loop['stop'] - 1} of {len(layers)}")
        eos = root.get("eos_token_id")
        eos_ids = [int(eos)] if _number(eos) else [int(e) for e in eos if _number(e)] if isinstance(eos, list) else []
        for e in eos_ids:
            if not 0 <= e < vocab:
                raise ConfigError(f"config: eos_token_id {e} is outside the vocabulary")
        max_pos = root.get("max_position_embeddings")
        return cls(vocab=vocab, width=width, eps=eps, loop=loop, layers=layers, eos_token_ids=eos_ids,
                   max_position_embeddings=int(max_pos) if _number(max_pos) and max_pos >= 1 else None)

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "layers": copy.deepcopy(self.layers), "norm": {"eps": self.eps},
                             "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            d["loop"] = dict(self.loop)
        if self.eos_token_ids:
            d["eos_token_id"] = self.eos_token_ids[0] if len(self.eos_token_ids) == 1 else list(self.eos_token_ids)
        if self.max_position_embeddings is not None:
            d["max_position_embeddings"] = self.max_position_embeddings
        return d

    # ------------------------------------------------------------------ model description
    def _mixer_spec(self, layer: Dict[str, Any]) -> PartSpec:
        m = layer["mixer"]
        common = {"hidden_size": self.width, "num_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "scale": m["scale"],
                  "eps": self.eps}
        if layer["type"] == "attention":
            return PartSpec("sink_attention", {**common, "num_kv_heads": m["kv_heads"], "bias": True, "out_bias": True, "element_gate": True})
        position = None
        if m["rot"]["dims"]:
            position = PartSpec("rotary", {"head_dim": m["rot_dim"], "rotary_dim": m["rot"]["dims"], "theta": m["rot"]["base"],
                                           "frequencies_in_64_bit": True})
        return PartSpec("latent_attention", {**common, "rotary_head_dim": m["rot_dim"], "kv_rank": m["kv_rank"], "window": m["mask"]["size"],
                                             "sink": True, "position": position})

    def _feed_forward_spec(self, mlp: Dict[str, Any]) -> PartSpec:
        if mlp["kind"] == "dense":
            return PartSpec("clamped_glu", {"hidden_size": self.width, "intermediate_size": mlp["ff"], "limit": mlp["limit"]})
        return PartSpec("moe", {"hidden_size": self.width, "num_experts": mlp["router"]["experts"], "top": mlp["router"]["top"],
                                "expert_size": mlp["expert"]["ff"], "shared_size": mlp["shared"]["ff"] if mlp.get("shared") else 0,
                                "router": "top_logits", "router_bias": True, "unit": "silu_glu"})

    def plan(self) -> List[PlanEntry]:
        """The order in which the layers run; the first layer of a pass adds the pass's vector to the stream."""
        n, loop = len(self.layers), self.loop or {"start": 0, "stop": 0, "times": 0}
        entries = [PlanEntry(i) for i in range(loop["start"])]
        for t in range(loop["times"]):
            entries += [PlanEntry(i, adds=t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
        return entries + [PlanEntry(i) for i in range(loop["stop"], n)]

    def model_spec(self) -> ModelSpec:
        W = self.width
        norm = PartSpec("rmsnorm", {"size": W, "eps": self.eps, "tensor_name": ""})
        scale = PartSpec("channel", {"size": W, "tensor_name": ""})
        layers: List[LayerSpec] = []
        for i, l in enumerate(self.layers):
            parts = {"norm": norm, "mixer": self._mixer_spec(l), "mixer_scale": scale}
            prefixes = {"norm": "norm1", "mixer": "mix.", "mixer_scale": "ls1"}
            if l["mlp"] is not None:
                parts.update({"feed_forward": self._feed_forward_spec(l["mlp"]), "feed_forward_scale": scale})
                prefixes.update({"feed_forward": "mlp.", "feed_forward_scale": "ls2"})
            layers.append(LayerSpec(prefix=f"l{i}.", block="parallel_prenorm", parts=parts, part_prefixes=prefixes))
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=W, vocab_size=self.vocab, layers=layers, plan=self.plan(),
            embedding=PartSpec("embedding", {"vocab_size": self.vocab, "hidden_size": W, "tensor_name": "embed"}), final_norm=norm,
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": W, "tied": False, "tensor_name": "head"}),
            weight_prefixes=[""], embedding_prefix="", final_norm_prefix="final.norm", head_prefix="",
            stop_token_ids=list(self.eos_token_ids), max_position=self.max_position_embeddings,
            stream_vectors=PartSpec("stream_vectors", {"size": W, "count": self.loop["times"], "tensor_name": "step"}) if self.loop else None,
            stream_vectors_prefix="loop.")
        spec.validate()
        return spec
