"""Small Mirorax configurations and weights for the tests.

The weights are drawn so that every mechanism moves the logits: norm weights and the factors on the results far from one, gates
that are neither open nor shut, sinks of the scores' size, routers whose scores differ, pass vectors of the stream's size.
Stored in bfloat16, so that a 32-bit engine and the 64-bit plain model read the same numbers.
"""
import json
import os

import torch


def attention(heads, kv_heads, dim, vdim, scale=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                           "scale": 1.4 * dim ** -0.5 if scale is None else scale}}


def latent(heads, dim, rot_dim, vdim, kv_rank, window, base=1000.0, scale=None, rotated=None):
    return {"type": "latent_attention", "mixer": {
        "heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "mask": {"size": window},
        "scale": 1.4 * (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot_dim if rotated is None else rotated}}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def with_mlp(layer, mlp):
    return dict(layer, mlp=mlp)


def config(width, vocab, layers, loop=None, eps=1e-5):
    c = {"architecture": "Mirorax", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if loop is not None:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


# both mixers with every kind of feed-forward; a loop in the middle that is gone through three times and opens with a latent
# layer; grouped, single and as many key/value heads as heads; two windows and two latent ranks, so two windowed cache groups
MIXED = config(64, 200, [
    with_mlp(attention(4, 2, 16, 12), moe(6, 2, 24, 40)),
    with_mlp(latent(4, 16, 8, 12, 40, 30), dense(72, 0.9)),
    with_mlp(attention(3, 1, 20, 28), None),
    with_mlp(latent(6, 12, 8, 20, 24, 70, base=50.0), moe(5, 3, 16, 8)),
    with_mlp(attention(2, 2, 24, 24), dense(40, 3.0)),
    with_mlp(latent(3, 8, 16, 24, 40, 30, base=50.0), moe(4, 1, 12))], loop=(1, 4, 3))
# sizes that are equal or 1 where the others differ: one head, windows of one and two tokens, one expert, every expert chosen, no
# rotated part and a partly rotated one, a loop over the whole stack, a loop of one pass's worth of one layer is in ONE_PASS
EDGES = config(40, 130, [
    with_mlp(latent(1, 8, 2, 5, 9, 1, base=20.0), moe(1, 1, 8, 1)),
    with_mlp(attention(1, 1, 3, 7), dense(1, 0.5)),
    with_mlp(latent(3, 3, 4, 3, 8, 64, base=20.0, rotated=2), moe(3, 3, 5, 24)),
    with_mlp(latent(2, 8, 0, 8, 16, 2), None),
    with_mlp(attention(5, 5, 8, 8), moe(2, 1, 8))], loop=(0, 5, 2), eps=1e-2)
ONE_PASS = config(48, 90, [
    with_mlp(attention(2, 1, 8, 16), dense(24, 100.0)), with_mlp(latent(2, 8, 8, 8, 16, 65), dense(24, 0.0))], loop=(1, 2, 1), eps=1e-3)
NO_LOOP = config(56, 96, [
    with_mlp(latent(2, 16, 8, 8, 24, 33), moe(4, 2, 16, 16)), with_mlp(attention(4, 4, 8, 8), dense(32, 1.5))])
# widths the tensor-core products take; head sizes for the tcgen05 prompt kernel with and without padding, and for the kernel of few tokens with one
# and two tiles of query heads; windows that straddle pages; the loop runs to the stack's end
WIDE = config(192, 300, [
    with_mlp(attention(8, 2, 64, 64), dense(320, 1.1)),
    with_mlp(latent(16, 64, 32, 96, 128, 127), moe(8, 2, 64, 128)),
    with_mlp(attention(20, 1, 40, 48), moe(6, 3, 40, 56)),
    with_mlp(latent(20, 24, 8, 72, 64, 100), dense(128, 0.7)),
    with_mlp(attention(4, 4, 128, 104), moe(5, 2, 32, 72)),
    with_mlp(latent(4, 128, 64, 128, 192, 65, base=10000.0), None)], loop=(2, 6, 2))

CONFIGS = {"mixed": MIXED, "edges": EDGES, "one_pass": ONE_PASS, "no_loop": NO_LOOP, "wide": WIDE}


def draw(name, shape, g):
    """A tensor for the local or full name ``name``."""
    leaf = name.split(".")[-1]
    n = lambda std=1.0, mean=0.0: torch.randn(shape, generator=g) * std + mean
    if leaf in ("norm", "norm1") and len(shape) == 1:
        return n(0.2, 1.0)
    if leaf in ("ls1", "ls2"):
        return n(0.4, 0.5)
    if leaf == "sink":
        return n(1.5, 1.0)
    if leaf == "b":
        return n(0.5)
    if leaf == "router":
        return n(2.0 / shape[1] ** 0.5)
    if leaf == "embed":
        return n(1.0)
    if leaf == "step":
        return n(0.8)
    if leaf in ("gate", "up") and "mlp" in name:
        return n(1.6 / shape[1] ** 0.5)                   # the clamped unit is clamped at many places
    return n(1.0 / shape[1] ** 0.5) if len(shape) == 2 else n(1.0)


def draw_tensors(cfg, seed):
    """name -> bfloat16 tensor for every tensor the configuration's model reads."""
    import hilbert_pruned_8b_b200 as hb
    from hilbert_pruned_8b_b200.engine.model import weight_table
    table = weight_table(hb.MiroraxConfig.from_dict(cfg).model_spec(), "")
    g = torch.Generator().manual_seed(seed)
    return {name: draw(name, tuple(spec.shape), g).to(torch.bfloat16) for name, spec in table.items() if not spec.optional}


def write_model(folder, cfg, seed):
    from hilbert_pruned_8b_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    tensors = draw_tensors(cfg, seed)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors)
    return tensors
