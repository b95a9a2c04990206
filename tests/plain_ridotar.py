"""A plain, slow Ridotar decoder: the oracle of the tests.

One function per mechanism, written from the design's equations in torch on the CPU (float64 unless another dtype is asked
for); it shares no code with the library.  ``PlainRidotar`` feeds a whole sequence at once and recomputes everything from
the first token: the recurrences are token-by-token loops, attention goes through an explicit mask with every head's keys
and values written out, the experts are evaluated token by token.

Notation: ``x`` residual stream (which the sublayers read as it is), ``S`` a recurrent state, ``a`` the factor on the stream
in ``x <- norm(a x + gate * sublayer(x))``.  ``rnd`` rounds a tensor where the library rounds in bfloat16 (what a matrix
product reads, queries, cached latents and key parts); the identity by default.
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


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(x, w, eps: float):
    """x / sqrt(mean(x^2) + eps) * w over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def group_rms_norm(x, w, eps: float, groups: int):
    """A row cut into ``groups`` runs of equal length, every run brought to unit mean square by itself, then scaled by w."""
    parts = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    return (parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)).reshape(x.shape) * w


def gated_sum_norm(x, y, gate_logits, alpha: float, w, eps: float, groups: int):
    """norm(alpha x + sigmoid(gate_logits) y): a sublayer's result on its way into the stream."""
    return group_rms_norm(alpha * x + torch.sigmoid(gate_logits) * y, w, eps, groups)


def token_side(x, h, e, w_gate, w_proj, w_norm, eps: float, rnd=same):
    """x + rmsnorm(W_proj (gelu(W_gate h) * e)): ``e`` [T, dim] the tokens' own vectors for this layer, ``h`` the stream as a
    product reads it."""
    g = gelu_tanh(h @ w_gate.T) * e
    return x + rms_norm(rnd(g) @ w_proj.T, w_norm, eps)


# ------------------------------------------------------------------------------------------------ recurrent memories
def forget_gate_memory(q, v, f):
    """q, f [T, H, d], v [T, H, dv] -> [T, H, dv]: S <- diag(f_t) S + (1 - f_t) v_t^T, o_t = S^T q_t."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for hd in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = f[t, hd][:, None] * S + torch.outer(1.0 - f[t, hd], v[t, hd])
            out[t, hd] = S.T @ q[t, hd]
    return out


def hgrn2_mixer(h, w: Dict[str, torch.Tensor], c: dict, eps: float, rnd=same):
    H, d, dv, T = int(c["heads"]), int(c["dim"]), int(c["vdim"]), h.shape[0]
    q = silu(h @ w["q"].T).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, dv)
    low = w["lower"]
    f = (low + (1.0 - low) * torch.sigmoid(h @ w["f"].T + w["f.b"])).reshape(T, H, d)
    o = rms_norm(forget_gate_memory(q, v, f), w["norm"], eps).reshape(T, H * dv)
    return rnd(o) @ w["o"].T


def fixed_decay_memory(q, k, v, decay):
    """q, k [T, H, d], v [T, H, dv], decay [H] -> [T, H, dv]: S <- decay_h S + k_t v_t^T, o_t = S^T q_t."""
    T, H, d = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for hd in range(H):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = decay[hd] * S + torch.outer(k[t, hd], v[t, hd])
            out[t, hd] = S.T @ q[t, hd]
    return out


def lightning_mixer(h, w: Dict[str, torch.Tensor], c: dict, eps: float, rnd=same):
    H, d, dv, T = int(c["heads"]), int(c["dim"]), int(c["vdim"]), h.shape[0]
    q, k = silu(h @ w["q"].T).reshape(T, H, d), silu(h @ w["k"].T).reshape(T, H, d)
    v = silu(h @ w["v"].T).reshape(T, H, dv)
    o = fixed_decay_memory(q, k, v, [float(x) for x in c["decay"]]).reshape(T, H * dv)
    return rnd(rms_norm(o, w["norm"], eps) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------------------------ latent attention
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


def causal_softmax(q, k, v, scale: float):
    """q, k [T, H, n], v [T, H, dv] -> [T, H, dv], position i over every j <= i."""
    T = q.shape[0]
    mask = torch.arange(T)[None, :] <= torch.arange(T)[:, None]
    s = torch.einsum("ihn,jhn->hij", q, k) * scale
    return torch.einsum("hij,jhd->ihd", torch.softmax(s.masked_fill(~mask, -math.inf), dim=-1), v)


def latents(h, w: Dict[str, torch.Tensor], c: dict, eps: float, positions, rnd=same):
    """What a layer with a down projection caches per token: the normed latent [T, rank] and the rotated key part [T, dr]."""
    rank, rot = int(c["kv_rank"]), c["rot"]
    down = h @ w["dkv"].T
    k_r = rotate_pairs(down[:, None, rank:], positions, int(rot["dims"]), float(rot["base"]))[:, 0]
    return rnd(rms_norm(down[:, :rank], w["dkv.norm"], eps)), rnd(k_r)


def latent_mixer(h, w: Dict[str, torch.Tensor], c: dict, eps: float, positions, cached=None, rnd=same):
    """-> (result, (latent, key part)); ``cached``: another layer's pair, read instead of this layer's own."""
    H, d, dr, dv, T = int(c["heads"]), int(c["dim"]), int(c["rot_dim"]), int(c["vdim"]), h.shape[0]
    rot = c["rot"]
    q = (rnd(rms_norm(h @ w["dq"].T, w["dq.norm"], eps)) @ w["uq"].T).reshape(T, H, d + dr)
    q_r = rotate_pairs(q[..., d:], positions, int(rot["dims"]), float(rot["base"]))
    lat, k_r = cached if cached is not None else latents(h, w, c, eps, positions, rnd)
    k_u, v = rnd(lat @ w["uk"].T).reshape(T, H, d), rnd(lat @ w["uv"].T).reshape(T, H, dv)
    qq = torch.cat([rnd(q[..., :d]), rnd(q_r)], dim=-1)
    kk = torch.cat([k_u, k_r[:, None, :].expand(T, H, dr)], dim=-1)
    o = causal_softmax(qq, kk, v, float(c["scale"])).reshape(T, H * dv)
    return rnd(o) @ w["o"].T, (lat, k_r)


# ------------------------------------------------------------------------------------------------ mixture of experts
def route(h, w_router, top: int):
    """-> (chosen [T, top], scores [T, top]): the ``top`` largest of s = sigmoid(W_router h), and those scores themselves."""
    s = torch.sigmoid(h @ w_router.T)
    best = torch.topk(s, top, dim=-1)
    return best.indices, best.values


def regret(h, w_router, chosen):
    """Per token, how far the best router logit left out is above the worst one chosen (negative: the choice is the best)."""
    z = h @ w_router.T
    left = z.scatter(1, chosen, -math.inf).max(-1).values
    return left - torch.gather(z, 1, chosen).min(-1).values


def moe_ff(h, w: Dict[str, torch.Tensor], c: dict, rnd=same, chosen=None):
    """The sum of the chosen experts' results, an expert being fed the token's input TIMES its score.  ``chosen`` [T, top]: a
    choice made elsewhere (of experts whose logits are nearly tied, say), with the scores of this input."""
    if chosen is None:
        chosen, scores = route(h, w["router"], int(c["router"]["top"]))
    else:
        scores = torch.gather(torch.sigmoid(h @ w["router"].T), 1, chosen)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t].tolist(), scores[t]):
            z = s * h[t]
            out[t] += rnd(silu(z @ w[f"e{e}.gate"].T) * (z @ w[f"e{e}.up"].T)) @ w[f"e{e}.down"].T
    return out


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


class PlainRidotar:
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
        """[T, vocab] for the whole sequence; ``layers_out`` collects the stream after every layer.  ``choices``: per
        mixture of experts a choice [T, top] to be taken as made, whose ``regret`` ``regrets_out`` collects."""
        c, w, rnd = self.cfg, self.w, self.rnd
        eps, groups, alpha = float(c["norm"]["eps"]), int(c["norm"]["groups"]), float(c["postln_alpha"])
        ids, positions = torch.tensor(tokens), torch.arange(len(tokens))
        x = w["embed"][ids]
        cached = {}
        made = iter(choices) if choices is not None else None
        for i, layer in enumerate(c["layers"]):
            p, m = f"l{i}.", layer["mixer"]
            mw, h = self._sub(p + "mix."), rnd(x)
            if layer["type"] == "lightning":
                y = lightning_mixer(h, mw, m, eps, rnd)
            elif layer["type"] == "hgrn2":
                y = hgrn2_mixer(h, mw, m, eps, rnd)
            else:
                source = m.get("kv_from")
                y, cached[i] = latent_mixer(h, mw, m, eps, positions, None if source is None else cached[source], rnd)
            x = gated_sum_norm(x, y, h @ w[p + "rg1"].T + w[p + "rg1.b"], alpha, w[p + "norm1"], eps, groups)
            if layer.get("mlp") is not None:
                h = rnd(x)
                chosen = next(made) if made is not None else None
                if regrets_out is not None:
                    regrets_out.append(regret(h, w[p + "mlp.router"], chosen))
                y = moe_ff(h, self._sub(p + "mlp."), layer["mlp"], rnd, chosen)
                x = gated_sum_norm(x, y, h @ w[p + "rg2"].T + w[p + "rg2.b"], alpha, w[p + "norm2"], eps, groups)
            if c.get("token_side") is not None:
                n = int(c["token_side"]["dim"])
                x = token_side(x, rnd(x), w["side.embed"][ids][:, i * n: (i + 1) * n], w[p + "side.gate"], w[p + "side.proj"], w[p + "side.norm"],
                               eps, rnd)
            if layers_out is not None:
                layers_out.append(x.clone())
        return rnd(group_rms_norm(x, w["final.norm"], eps, groups)) @ w["embed"].T
