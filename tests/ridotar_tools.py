"""Small Ridotar configurations and weights for the tests.

The weights are drawn so that every mechanism moves the logits: norm weights far from one, gates that are neither open nor
shut, decays and lower bounds spread over their range, routers whose scores differ, side inputs of the stream's size.  Stored
in bfloat16, so that a 32-bit engine and the 64-bit plain model read the same numbers.
"""
import json
import os

import torch


def lightning(heads, dim, vdim, decay):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)}}


def hgrn2(heads, dim, vdim):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=1000.0, kv_from=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": 1.4 * (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def with_mlp(layer, mlp):
    return dict(layer, mlp=mlp)


def config(width, vocab, layers, groups=4, eps=1e-5, alpha=1.6, side=12):
    c = {"architecture": "Ridotar", "layers": layers, "norm": {"eps": eps, "groups": groups}, "postln_alpha": alpha, "vocab": vocab, "width": width}
    if side:
        c["token_side"] = {"dim": side}
    return c


# every kind of layer, several latent layers: two that keep latents of their own (different ranks, so two cache groups), one
# reader right behind its source, two readers of one source with other layers between; layers without a feed-forward
MIXED = config(64, 200, [
    with_mlp(latent(4, 16, 8, 12, 24, 40), moe(6, 2, 24)),
    with_mlp(hgrn2(3, 8, 12), moe(5, 1, 16)),
    with_mlp(latent(6, 12, 8, 20, 16, 40, kv_from=0), None),
    with_mlp(lightning(4, 12, 8, (0.5, 0.9, 0.97, 0.998)), moe(3, 3, 20)),
    with_mlp(latent(2, 24, 16, 16, 40, 32, base=50.0), moe(4, 3, 8)),
    with_mlp(latent(3, 8, 16, 24, 8, 32, base=50.0, kv_from=4), moe(1, 1, 12)),
    with_mlp(hgrn2(2, 20, 10), None),
    with_mlp(latent(5, 4, 8, 4, 12, 40, kv_from=0), moe(2, 2, 8))])
# sizes that are equal or 1 where the others differ: one head, two state rows, small and odd ranks (but no single state row
# and no norm over one or two numbers, which leave little more than signs: the mixers' own tests have those), two rotated dimensions, decays of zero and one, one expert, every expert chosen, one group or a number of groups that is no
# power of two, a factor of one, side vectors of one number; a large eps, which tames the norms over so few numbers
EDGES = config(48, 130, [
    with_mlp(lightning(1, 2, 5, (1.0,)), moe(1, 1, 8)),
    with_mlp(latent(1, 8, 2, 5, 7, 9, base=20.0), moe(3, 3, 5)),
    with_mlp(hgrn2(1, 2, 6), moe(2, 1, 1)),
    with_mlp(lightning(3, 5, 7, (0.0, 1.0, 0.75)), None),
    with_mlp(latent(3, 3, 4, 3, 5, 8, base=20.0), moe(4, 1, 8)),
    with_mlp(latent(3, 3, 4, 3, 8, 8, base=20.0, kv_from=4), moe(1, 1, 16))], groups=3, eps=2e-2, alpha=1.0, side=1)
ONE_GROUP = config(40, 90, [
    with_mlp(hgrn2(2, 4, 4), None), with_mlp(latent(2, 4, 4, 4, 8, 8), None), with_mlp(lightning(2, 4, 4, (0.9, 0.9)), moe(2, 1, 8))],
    groups=1, eps=1e-3, alpha=0.5, side=0)
# widths the tensor-core products take; heads whose written-out sizes the tensor-core prompt kernel is built for (64 to 192
# numbers a key); sixteen heads; states of 64 x 128 and more; experts whose sizes the tensor-core tiles take
WIDE = config(256, 300, [
    with_mlp(lightning(4, 64, 32, (0.4, 0.95, 0.99, 0.9995)), moe(8, 2, 64)),
    with_mlp(latent(16, 32, 32, 64, 96, 64), moe(6, 2, 32)),
    with_mlp(hgrn2(2, 128, 64), moe(4, 1, 96)),
    with_mlp(latent(4, 96, 32, 96, 48, 64, kv_from=1), moe(6, 3, 64)),
    with_mlp(latent(2, 128, 64, 128, 64, 192, base=10000.0), None),
    with_mlp(hgrn2(3, 40, 96), moe(5, 2, 32))], groups=16, side=40, alpha=2.2)

CONFIGS = {"mixed": MIXED, "edges": EDGES, "one_group": ONE_GROUP, "wide": WIDE}


def draw(name, shape, g):
    """A tensor for the local or full name ``name``."""
    leaf = name.split(".")[-1]
    n = lambda std=1.0, mean=0.0: torch.randn(shape, generator=g) * std + mean
    if leaf in ("norm", "norm1", "norm2") and len(shape) == 1:
        return n(0.2, 1.0)
    if name.endswith("f.b"):
        return n(1.5, 1.0)
    if leaf == "b":
        return n(0.7, 0.3)
    if leaf == "lower":
        return torch.rand(shape, generator=g) * 0.95
    if leaf == "router":
        return n(2.0 / shape[1] ** 0.5)
    if leaf in ("rg1", "rg2"):
        return n(1.5 / shape[1] ** 0.5)
    if leaf == "embed":                                   # embed and side.embed
        return n(1.0)
    return n(1.0 / shape[1] ** 0.5) if len(shape) == 2 else n(1.0)


def draw_tensors(cfg, seed):
    """name -> bfloat16 tensor for every tensor the configuration's model reads."""
    import hilbert_pruned_8b_b200 as hb
    from hilbert_pruned_8b_b200.engine.model import weight_table
    table = weight_table(hb.RidotarConfig.from_dict(cfg).model_spec(), "")
    g = torch.Generator().manual_seed(seed)
    return {name: draw(name, tuple(spec.shape), g).to(torch.bfloat16) for name, spec in table.items() if not spec.optional}


def write_model(folder, cfg, seed, state_ranks=True):
    """Writes config.json and model.safetensors; ``state_ranks`` False leaves the ranks out of config.json, so that a reader
    must take them from the tensors' shapes."""
    import copy
    from hilbert_pruned_8b_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    tensors = draw_tensors(cfg, seed)
    stored = copy.deepcopy(cfg)
    if not state_ranks:
        for layer in stored["layers"]:
            for key in ("q_rank", "kv_rank"):
                layer["mixer"].pop(key, None)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(stored, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return tensors
