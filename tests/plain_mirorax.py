"""A plain, slow Mirorax decoder: the oracle of the tests.

One function per mechanism, written from the design's equations in torch on the CPU (float64 unless another dtype is asked
for); it shares no code with the library.  ``PlainMirorax`` feeds a whole sequence at once and recomputes everything from the
first token: attention goes through an explicit mask with every head's keys and values written out, the experts are evaluated
token by token, and a run of layers that is gone through several times is a loop in the program.

Notation: ``x`` residual stream, ``h`` what both sublayers of a layer read, ``a`` and ``b`` the layer's two scales: ``x <- x + a *
mixer(h) + b * ff(h)``.  ``rnd`` rounds a tensor where the library rounds in bfloat16 (what a matrix product reads, queries,
cached keys, values, latents and key parts); the identity by default.
"""
from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional

import torch


# ------------------------------------------------------------------------------------------------ small pieces
def same(t):
    return t


def to_bf16(t):
    return t.to(torch.bfloat16).to(t.dtype)


def silu(z):
    return z * torch.sigmoid(z)


def rms_norm(x, w, eps: float):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def parallel_sum(x, mixed, a, fed=None, b=None):
    """x + a * mixed + b * fed: both sublayers' results on their way into the stream, each times a factor per channel."""
    x = x + a * mixed
    return x if fed is None else x + b * fed


def layer_runs(n_layers: int, loop: Optional[dict]):
    """[(layer, pass or None, whether the layer opens that pass)] in the order in which the layers run."""
    if loop is None:
        return [(i, None, False) for i in range(n_layers)]
    first, behind, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    runs = [(i, None, False) for i in range(first)]
    for t in range(times):
        runs += [(i, t, i == first) for i in range(first, behind)]
    return runs + [(i, None, False) for i in range(behind, n_layers)]


# ------------------------------------------------------------------------------------------------ attention
def visible(T: int, window: Optional[int] = None):
    """[T, T] of booleans: query i (row) sees key j when j <= i and, with a window, i - j < window."""
    back = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (back >= 0) if window is None else (back >= 0) & (back < window)


def softmax_attention(q, k, v, scale: float, mask, sink=None):
    """q [T, H, n], k [T, G, n], v [T, G, dv] -> [T, H, dv]; query head h reads key/value head h // (H / G).  ``sink`` [H]: one more
    term exp(sink_h) in the sum the weights are divided by."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    own = torch.arange(H) // (H // G)
    s = (torch.einsum("ihn,jhn->hij", q, k[:, own]) * scale).masked_fill(~mask, -math.inf)
    if sink is not None:
        s = torch.cat([s, sink.to(s.dtype)[:, None, None].expand(H, T, 1)], dim=-1)
    p = torch.softmax(s, dim=-1)[..., :T]
    return torch.einsum("hij,jhd->ihd", p, v[:, own])


def attention_mixer(h, w: Dict[str, torch.Tensor], c: dict, rnd=same):
    """Causal grouped attention without positions, biases on q, k, v and o, every element of the heads' results times a sigmoid."""
    H, G, d, dv, T = int(c["heads"]), int(c["kv_heads"]), int(c["dim"]), int(c["vdim"]), h.shape[0]
    q = rnd(h @ w["q"].T + w["q.b"]).reshape(T, H, d)
    k = rnd(h @ w["k"].T + w["k.b"]).reshape(T, G, d)
    v = rnd(h @ w["v"].T + w["v.b"]).reshape(T, G, dv)
    o = softmax_attention(q, k, v, float(c["scale"]), visible(T)).reshape(T, H * dv)
    return rnd(o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T + w["o.b"]


def rotate_pairs(t, positions, dims: int, base: float):
    """t [T, heads, n]: the pairs (2i, 2i + 1), i < dims / 2, turned by positions * base^(-2i/dims)."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    a = positions.to(torch.float64)[:, None] * torch.pow(torch.tensor(float(base), dtype=torch.float64), -2.0 * i / max(dims, 1))[None, :]
    cos, sin = torch.cos(a).to(t.dtype)[:, None, :], torch.sin(a).to(t.dtype)[:, None, :]
    out = t.clone()
    u, v = t[..., 0:dims:2], t[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def latent_mixer(h, w: Dict[str, torch.Tensor], c: dict, eps: float, positions, rnd=same):
    """Attention over a window whose keys and values come from one latent per token, with a sink per head."""
    H, d, dr, dv, rank, T = int(c["heads"]), int(c["dim"]), int(c["rot_dim"]), int(c["vdim"]), int(c["kv_rank"]), h.shape[0]
    dims, base = int(c["rot"]["dims"]), float(c["rot"]["base"])
    q, down = (h @ w["q"].T).reshape(T, H, d + dr), h @ w["dkv"].T
    q_r = rotate_pairs(q[..., d:], positions, dims, base)
    k_r = rotate_pairs(down[:, None, rank:], positions, dims, base)
    lat = rnd(rms_norm(down[:, :rank], w["dkv.norm"], eps))
    k_u, v = rnd(lat @ w["uk"].T).reshape(T, H, d), rnd(lat @ w["uv"].T).reshape(T, H, dv)
    qq = torch.cat([rnd(q[..., :d]), rnd(q_r)], dim=-1)
    kk = torch.cat([k_u, rnd(k_r).expand(T, H, dr)], dim=-1)
    o = softmax_attention(qq, kk, v, float(c["scale"]), visible(T, int(c["mask"]["size"])), w["sink"]).reshape(T, H * dv)
    return rnd(o) @ w["o"].T


# ------------------------------------------------------------------------------------------------ feed-forwards
def clamped_unit(g, u, limit: float):
    """g' sigmoid(1.702 g') (u' + 1): g' is g cut off above ``limit``, u' is u cut off at both ends."""
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w: Dict[str, torch.Tensor], c: dict, rnd=same):
    return rnd(clamped_unit(h @ w["gate"].T, h @ w["up"].T, float(c["limit"]))) @ w["down"].T


def route(h, w_router, bias, top: int):
    """-> (chosen [T, top], weights [T, top]): the ``top`` largest of z = W_router h + bias; the softmax over those alone."""
    best = torch.topk(h @ w_router.T + bias, top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


def regret(h, w_router, bias, chosen):
    """Per token, how far the best router logit left out is above the worst one chosen (negative: the choice is the best)."""
    z = h @ w_router.T + bias
    left = z.scatter(1, chosen, -math.inf).max(-1).values
    return left - torch.gather(z, 1, chosen).min(-1).values


def moe_ff(h, w: Dict[str, torch.Tensor], c: dict, rnd=same, chosen=None):
    """The weighted sum of the chosen experts' results, and the shared expert's.  ``chosen`` [T, top]: a choice made elsewhere
    (of experts whose logits are nearly tied, say), weighted by this input's logits."""
    if chosen is None:
        chosen, weights = route(h, w["router"], w["router.b"], int(c["router"]["top"]))
    else:
        weights = torch.softmax(torch.gather(h @ w["router"].T + w["router.b"], 1, chosen), dim=-1)
    unit = lambda z, name: rnd(silu(z @ w[name + ".gate"].T) * (z @ w[name + ".up"].T)) @ w[name + ".down"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), weights[t]):
            out[t] += s * unit(h[t], f"e{e}")
    return out + unit(h, "shared") if c.get("shared") is not None else out


# ------------------------------------------------------------------------------------------------ the model
def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        meta = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    out = {}
    for name, m in meta.items():
        if name == "__metadata__":
            continue
        a, b = m["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[m["dtype"]]).reshape(m["shape"]).clone()
    return out


class PlainMirorax:
    def __init__(self, cfg, tensors=None, dtype=torch.float64, round_to=None):
        """``cfg``: the configuration (a dict) with ``tensors`` (name -> tensor), or a model folder."""
        if tensors is None:
            folder = cfg
            with open(os.path.join(folder, "config.json")) as f:
                cfg = json.load(f)
            tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
        self.cfg = cfg
        self.rnd = to_bf16 if round_to == torch.bfloat16 else same
        self.w = {n: t.to(dtype) for n, t in tensors.items()}

    def _sub(self, prefix: str) -> Dict[str, torch.Tensor]:
        return {n[len(prefix):]: t for n, t in self.w.items() if n.startswith(prefix)}

    def logits(self, tokens: List[int], layers_out: Optional[list] = None, choices: Optional[list] = None, regrets_out: Optional[list] = None):
        """[T, vocab] for the whole sequence; ``layers_out`` collects the stream after every layer run.  ``choices``: per run of a
        mixture of experts a choice [T, top] to be taken as made, whose ``regret`` ``regrets_out`` collects."""
        c, w, rnd = self.cfg, self.w, self.rnd
        eps, positions = float(c["norm"]["eps"]), torch.arange(len(tokens))
        x = w["embed"][torch.tensor(tokens)]
        made = iter(choices) if choices is not None else None
        for i, turn, opens in layer_runs(len(c["layers"]), c.get("loop")):
            p, layer = f"l{i}.", c["layers"][i]
            if opens:
                x = x + w["loop.step"][turn]
            h = rnd(rms_norm(x, w[p + "norm1"], eps))
            mw, m = self._sub(p + "mix."), layer["mixer"]
            mixed = attention_mixer(h, mw, m, rnd) if layer["type"] == "attention" else latent_mixer(h, mw, m, eps, positions, rnd)
            fed, mlp = None, layer.get("mlp")
            if mlp is not None and mlp["kind"] == "dense":
                fed = dense_ff(h, self._sub(p + "mlp."), mlp, rnd)
            elif mlp is not None:
                chosen = next(made) if made is not None else None
                if regrets_out is not None:
                    regrets_out.append(regret(h, w[p + "mlp.router"], w[p + "mlp.router.b"], chosen))
                fed = moe_ff(h, self._sub(p + "mlp."), mlp, rnd, chosen)
            x = parallel_sum(x, mixed, w[p + "ls1"], fed, w.get(p + "ls2"))
            if layers_out is not None:
                layers_out.append(x.clone())
        return rnd(rms_norm(x, w["final.norm"], eps)) @ w["head"].T
