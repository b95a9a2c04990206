"""Typed configuration of the Ridotar decoder: a stack whose sublayers read the residual stream itself and whose norm sits behind
the sum, ``x = norm(alpha x + sigmoid(W x + b) * sublayer(x))``, the norm being an RMS norm over equal parts of the row; behind
the sublayers every layer adds an input that belongs to the token alone.  Three kinds of mixer: a matrix memory with a fixed
decay per head; a matrix memory whose forget gate doubles as its input gate; an attention over one small cached latent per
token whose queries come through a latent of their own, and which may read an earlier layer's cached latents instead of
keeping its own.  The feed-forward is a mixture of experts (the largest sigmoids, which multiply the experts' inputs), or
absent.  The head is the embedding table.

config.json keys (every size and every constant that may differ between models comes from here): ``architecture``
("Ridotar"), ``vocab``, ``width``, ``norm {eps, groups}``, ``postln_alpha``, ``token_side {dim}`` (absent or null: no such input) and
``layers``: a list of ``{"type", "mixer", "mlp"}`` with ``type``

* "lightning": ``mixer`` = ``heads, dim, vdim, decay [per head]``;
* "hgrn2": ``mixer`` = ``heads, dim, vdim``;
* "latent_attention": ``mixer`` = ``heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot {base, dims}`` and optionally ``kv_from``, the
  number of the earlier layer whose latents it reads (``q_rank`` and ``kv_rank`` may be left to the shapes of ``l<i>.mix.dq`` and
  ``l<i>.mix.uk``, which ``with_tensor_shapes`` reads);

and ``mlp`` null or ``{"kind": "moe", "router {experts, top}", "expert {ff}"}``.  Tensor names: ``embed``, ``side.embed``,
``l<i>.norm1|norm2``, ``l<i>.rg1|rg2`` (bias: ``.b`` added), ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.gate|proj|norm``, ``final.norm``.
"""
from __future__ import annotations

import copy
import dataclasses
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional

from .base import ConfigError
from .spec import LayerSpec, ModelSpec, PartSpec, PlanEntry
from .tonovik import _float, _int, _number, _rot


def _sizes(m: Any, keys, where: str) -> Dict[str, int]:
    return {k: _int(m, k, where) for k in keys}


def _mlp(mlp: Any, where: str) -> Optional[Dict[str, Any]]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config: {where}kind must be moe (or mlp null)")
    router = _sizes(mlp.get("router"), ("experts", "top"), where + "router.")
    if router["top"] > router["experts"]:
        raise ConfigError(f"config: {where}router.top is larger than the number of experts")
    return {"kind": "moe", "router": router, "expert": _sizes(mlp.get("expert"), ("ff",), where + "expert.")}


@dataclass(frozen=True)
class RidotarConfig:
    vocab: int
    width: int
    eps: float
    groups: int = 1
    alpha: float = 1.0
    side_dim: int = 0
    layers: List[Dict[str, Any]] = field(default_factory=list)       # the validated entries of config.json
    eos_token_ids: List[int] = field(default_factory=list)
    max_position_embeddings: Optional[int] = None

    architecture = "Ridotar"
    model_type = "ridotar"

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
    def from_dict(cls, root: Dict[str, Any]) -> "RidotarConfig":
        if not isinstance(root, dict):
            raise ConfigError("config: config.json is not an object")
        vocab, width = _int(root, "vocab", ""), _int(root, "width", "")
        norm = root.get("norm")
        eps = _float(norm, "eps", "norm.")
        groups = _int(norm, "groups", "norm.") if norm.get("groups") is not None else 1
        if width % groups:
            raise ConfigError(f"config: norm.groups {groups} does not divide the width {width}")
        alpha = _float(root, "postln_alpha", "") if root.get("postln_alpha") is not None else 1.0
        side = root.get("token_side")
        side_dim = _int(side, "dim", "token_side.") if side is not None else 0
        raw = root.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config: layers must be a list with at least one entry")
        layers: List[Dict[str, Any]] = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]."
            kind = entry.get("type") if isinstance(entry, dict) else None
            if kind not in ("lightning", "hgrn2", "latent_attention"):
                raise ConfigError(f"config: {where}type must be lightning, hgrn2 or latent_attention")
            m, mw = entry.get("mixer"), where + "mixer."
            if not isinstance(m, dict):
                raise ConfigError(f"config: missing {where}mixer")
            mixer: Dict[str, Any] = _sizes(m, ("heads", "dim", "vdim"), mw)
            if kind == "lightning":
                decay = m.get("decay")
                if not isinstance(decay, list) or len(decay) != mixer["heads"] or not all(_number(x) and 0.0 <= x <= 1.0 for x in decay):
                    raise ConfigError(f"config: {mw}decay must give a number in [0, 1] per head")
                mixer["decay"] = [float(x) for x in decay]
            elif kind == "latent_attention":
                mixer["rot_dim"] = _int(m, "rot_dim", mw, least=0)
                mixer["scale"] = _float(m, "scale", mw)
                for k in ("q_rank", "kv_rank"):
                    if m.get(k) is not None:
                        mixer[k] = _int(m, k, mw)
                mixer["rot"] = _rot(m, mw, mixer["rot_dim"], scaling=False) if mixer["rot_dim"] or m.get("rot") is not None else {"base": 1.0, "dims": 0}
                if m.get("kv_from") is not None:
                    mixer["kv_from"] = j = _int(m, "kv_from", mw, least=0)
                    if j >= i or layers[j]["type"] != "latent_attention" or "kv_from" in layers[j]["mixer"]:
                        raise ConfigError(f"config: {mw}kv_from must name an earlier latent_attention layer that keeps latents of its own")
                    other = layers[j]["mixer"]
                    if any(other.get(k) != mixer.get(k) and None not in (other.get(k), mixer.get(k)) for k in ("kv_rank", "rot_dim", "rot")):
                        raise ConfigError(f"config: {mw}kv_from names a layer whose kv_rank, rot_dim or rotation differ")
            layers.append({"type": kind, "mixer": mixer, "mlp": _mlp(entry.get("mlp"), where + "mlp.")})
        eos = root.get("eos_token_id")
        eos_ids = [int(eos)] if _number(eos) else [int(e) for e in eos if _number(e)] if isinstance(eos, list) else []
        for e in eos_ids:
            if not 0 <= e < vocab:
                raise ConfigError(f"config: eos_token_id {e} is outside the vocabulary")
        max_pos = root.get("max_position_embeddings")
        return cls(vocab=vocab, width=width, eps=eps, groups=groups, alpha=alpha, side_dim=side_dim, layers=layers, eos_token_ids=eos_ids,
                   max_position_embeddings=int(max_pos) if _number(max_pos) and max_pos >= 1 else None)

    def with_tensor_shapes(self, shapes: Dict[str, Any]) -> "RidotarConfig":
        """The configuration with the latent sizes that config.json leaves to a tensor's shape (``shapes``: tensor name ->
        shape); a stated size that a shape contradicts is an error."""
        layers = copy.deepcopy(self.layers)
        for i, l in enumerate(layers):
            if l["type"] != "latent_attention":
                continue
            for key, name, axis in (("q_rank", f"l{i}.mix.dq", 0), ("kv_rank", f"l{i}.mix.uk", 1)):
                shape = shapes.get(name)
                if shape is None or len(shape) != 2:
                    continue
                stated = l["mixer"].get(key)
                if stated is not None and stated != int(shape[axis]):
                    raise ConfigError(f"config: layers[{i}].mixer.{key} is {stated}, but {name} has the shape {list(shape)}")
                l["mixer"][key] = int(shape[axis])
        return dataclasses.replace(self, layers=layers)

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"architecture": self.architecture, "layers": copy.deepcopy(self.layers), "norm": {"eps": self.eps, "groups": self.groups},
                             "postln_alpha": self.alpha, "vocab": self.vocab, "width": self.width}
        if self.side_dim:
            d["token_side"] = {"dim": self.side_dim}
        if self.eos_token_ids:
            d["eos_token_id"] = self.eos_token_ids[0] if len(self.eos_token_ids) == 1 else list(self.eos_token_ids)
        if self.max_position_embeddings is not None:
            d["max_position_embeddings"] = self.max_position_embeddings
        return d

    # ------------------------------------------------------------------ model description
    def _mixer(self, i: int, layer: Dict[str, Any]) -> PartSpec:
        m = layer["mixer"]
        common = {"hidden_size": self.width, "num_heads": m["heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"], "eps": self.eps}
        if layer["type"] == "lightning":
            return PartSpec("decay_memory", {**common, "decay": tuple(m["decay"]), "activation": "silu", "norm": "row", "gate": "sigmoid"})
        if layer["type"] == "hgrn2":
            return PartSpec("forget_gate_memory", common)
        for key in ("q_rank", "kv_rank"):
            if m.get(key) is None:
                raise ConfigError(f"config: layers[{i}].mixer.{key} is neither stated nor known from a tensor's shape")
        position = None
        if m["rot"]["dims"]:
            position = PartSpec("rotary", {"head_dim": m["rot_dim"], "rotary_dim": m["rot"]["dims"], "theta": m["rot"]["base"],
                                           "frequencies_in_64_bit": True})
        return PartSpec("latent_attention", {**common, "rotary_head_dim": m["rot_dim"], "kv_rank": m["kv_rank"], "q_rank": m["q_rank"],
                                             "scale": m["scale"], "shares_cache": m.get("kv_from") is not None, "position": position})

    def model_spec(self) -> ModelSpec:
        W = self.width
        norm = PartSpec("group_rmsnorm", {"size": W, "eps": self.eps, "groups": self.groups, "tensor_name": ""})
        gate = PartSpec("sigmoid", {"size": W, "tensor_name": ""})
        layers: List[LayerSpec] = []
        for i, l in enumerate(self.layers):
            parts = {"mixer_gate": gate, "mixer": self._mixer(i, l), "mixer_norm": norm}
            prefixes = {"mixer_gate": "rg1", "mixer": "mix.", "mixer_norm": "norm1"}
            if l["mlp"] is not None:
                r = l["mlp"]["router"]
                parts.update({"feed_forward_gate": gate, "feed_forward_norm": norm, "feed_forward": PartSpec("moe", {
                    "hidden_size": W, "num_experts": r["experts"], "top": r["top"], "expert_size": l["mlp"]["expert"]["ff"], "router": "sigmoid",
                    "unit": "silu_glu", "weigh": "input"})})
                prefixes.update({"feed_forward_gate": "rg2", "feed_forward": "mlp.", "feed_forward_norm": "norm2"})
            if self.side_dim:
                parts["token_side"] = PartSpec("gelu_side", {"size": W, "dim": self.side_dim, "offset": i * self.side_dim, "eps": self.eps})
                prefixes["token_side"] = "side."
            layers.append(LayerSpec(prefix=f"l{i}.", block="postnorm_sum", parts=parts, part_prefixes=prefixes,
                                    block_params={"residual_scale": self.alpha}))
        embedding = {"vocab_size": self.vocab, "hidden_size": W, "tensor_name": "embed"}
        if self.side_dim:
            embedding.update({"side_columns": self.side_dim * len(layers), "side_tensor_name": "side.embed"})
        spec = ModelSpec(
            architecture=self.architecture, hidden_size=W, vocab_size=self.vocab, layers=layers,
            plan=[PlanEntry(i, l["mixer"].get("kv_from")) for i, l in enumerate(self.layers)],
            embedding=PartSpec("embedding_with_side" if self.side_dim else "embedding", embedding), final_norm=norm,
            head=PartSpec("lm_head", {"vocab_size": self.vocab, "hidden_size": W, "tied": True}),
            weight_prefixes=[""], embedding_prefix="", final_norm_prefix="final.norm", head_prefix="lm_head.",
            stop_token_ids=list(self.eos_token_ids), max_position=self.max_position_embeddings)
        spec.validate()
        return spec
