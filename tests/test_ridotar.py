"""The Ridotar decoder against the plain implementation (tests/plain_ridotar.py): every mechanism alone (the group-wise norm, the
norm behind a gated sum, the token side input, the sigmoid router with weighted expert inputs, the two matrix memories, the
attention over latents with a query latent and with another layer's latents), then the engine: whole prompts, token-by-token
decoding, prompts in portions down to two tokens, unequal batches with slots and pages used again, long decoding, greedy
generation through the library's entry point and the replay program."""
import copy
import math

import pytest
import torch

import ridotar_tools as rt
import trace_tools as tt
from conftest import require_gpu
from plain_ridotar import (PlainRidotar, causal_softmax, fixed_decay_memory, forget_gate_memory, gated_sum_norm, gelu_tanh, group_rms_norm,
                           hgrn2_mixer, latent_mixer, lightning_mixer, moe_ff, rms_norm, rotate_pairs, route, silu, to_bf16, token_side)
from test_tonovik import _MixerRun, _compare, _context, _reference, _requests

DTYPES = ["float32", "bfloat16"]
NAMES = list(rt.CONFIGS)
DEV = "cuda:0"


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (folder, config, {"exact" | dtype: plain model})"""
    out = {}
    for i, (name, cfg) in enumerate(rt.CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("ridotar_" + name))
        tensors = rt.write_model(d, cfg, 90 + i, state_ranks=(name != "mixed"))
        out[name] = (d, cfg, {"exact": PlainRidotar(cfg, tensors), "float32": PlainRidotar(cfg, tensors, dtype=torch.float32),
                              "bfloat16": PlainRidotar(cfg, tensors, round_to=torch.bfloat16)})
    return out


def _engine(folder, dtype, max_tokens, **kw):
    from hilbert_pruned_8b_b200.engine.step import Engine
    return Engine.from_folder(folder, dtype, max_tokens=max_tokens, **kw)


class _Choices:
    """Runs an engine's steps and notes which experts every router chose for every token (without captured graphs, which
    replay kernels only): two experts whose logits are nearly tied may be chosen either way once the router's input is rounded
    to bfloat16, and a comparison of logits has to follow the choice that was made."""

    def __init__(self, eng):
        eng.use_graphs = False
        self.tokens, self.rows = {}, {}                   # seq id -> tokens fed, choices per token [[top] per router]
        noted, route, step = [], eng.ctx.ops.moe_route, eng.step

        def moe_route(h, w_router, top, experts, weights, **kw):
            route(h, w_router, top, experts, weights, **kw)
            noted.append(experts.cpu().long())

        def noted_step(entries, **kw):
            noted.clear()
            logits = step(entries, **kw)
            at = 0
            for e in entries:
                for t in e.tokens:
                    self.tokens.setdefault(e.seq.seq_id, []).append(t)
                    self.rows.setdefault(e.seq.seq_id, []).append([n[at] for n in noted])
                    at += 1
            return logits
        eng.ctx.ops.moe_route, eng.step = moe_route, noted_step

    def of(self, tokens):
        """The choices made for a request of these tokens the last time it ran: one [T, top] tensor per router."""
        seq = max(s for s, t in self.tokens.items() if t == tokens)
        return [torch.stack(r) for r in zip(*self.rows[seq])]


CLOSE_CALL = 0.3        # a choice may differ from the exact model's by so much of a logit (rounding moves logits by hundredths)


def _check(eng, steps, plain, requests, dtype, what):
    """Runs the steps and compares every wanted position with the plain models (test_tonovik's bounds)."""
    if dtype == "float32":
        _compare(tt.run_in_process(eng, steps), _reference(plain, requests, dtype), dtype, what)
        return
    choices = _Choices(eng)
    got = tt.run_in_process(eng, steps)

    class Followed:
        """A plain model that takes the library's choices as made."""

        def __init__(self, model, exact):
            self.model, self.exact = model, exact

        def logits(self, toks):
            made, regrets = choices.of(toks), []
            out = self.model.logits(toks, choices=made, regrets_out=regrets)
            if self.exact and regrets:
                worst = torch.stack(regrets).max().item()
                assert worst < CLOSE_CALL, f"{what}: an expert was chosen whose logit is {worst:.3f} below one left out"
            return out
    follow = {k: Followed(m, k == "exact") for k, m in plain.items()}
    _compare(got, _reference(follow, requests, dtype), dtype, what)


def _rnd(dtype):
    return to_bf16 if dtype == torch.bfloat16 else (lambda z: z)


# --------------------------------------------------------------------------- without a GPU
def test_config_round_trip_weight_table_and_cache_plan(tmp_path):
    import hilbert_pruned_8b_b200 as hb
    from hilbert_pruned_8b_b200.config import ConfigError, config_class_for
    from hilbert_pruned_8b_b200.engine.model import DecoderModel, describe_context, weight_table
    for cfg in rt.CONFIGS.values():
        assert config_class_for(cfg) is hb.RidotarConfig
        c = hb.RidotarConfig.from_dict(cfg)
        assert hb.RidotarConfig.from_dict(c.to_dict()) == c
        table = weight_table(c.model_spec(), "")
        side = cfg.get("token_side")
        assert ("side.embed" in table) == (side is not None)
        if side:
            assert table["side.embed"].shape == (cfg["vocab"], side["dim"] * len(cfg["layers"]))
        for i, layer in enumerate(cfg["layers"]):
            m, has = layer["mixer"], lambda n: f"l{i}.{n}" in table
            assert has("norm1") and has("rg1") and has("rg1.b")
            assert has("norm2") == has("rg2") == has("rg2.b") == has("mlp.router") == (layer["mlp"] is not None)
            assert has("side.gate") == has("side.proj") == has("side.norm") == (side is not None)
            assert has("mix.lower") == has("mix.f.b") == (layer["type"] == "hgrn2") and has("mix.g") == (layer["type"] == "lightning")
            assert has("mix.dq") == has("mix.uq") == has("mix.uk") == (layer["type"] == "latent_attention")
            assert has("mix.dkv") == has("mix.dkv.norm") == (layer["type"] == "latent_attention" and "kv_from" not in m)
            if layer["mlp"]:
                E = layer["mlp"]["router"]["experts"]
                assert has(f"mlp.e{E - 1}.gate") and not has(f"mlp.e{E}.gate") and table[f"l{i}.mlp.e0.down"].shape == (cfg["width"], layer["mlp"]["expert"]["ff"])
    c = hb.RidotarConfig.from_dict(rt.MIXED)
    table = weight_table(c.model_spec(), "")
    assert table["l0.mix.uq"].shape == (4 * 24, 24) and table["l0.mix.dkv"].shape == (48, 64) and table["l2.mix.uv"].shape == (6 * 20, 40)
    assert table["l1.mix.norm"].shape == (12,) and table["l3.mix.norm"].shape == (32,) and table["l1.mix.lower"].shape == (24,)
    # readers keep no latents of their own; two ranks are two needs; a memory per memory layer
    model = DecoderModel(c.model_spec(), describe_context())
    needs = model.cache_needs()
    assert sorted(needs) == [0, 4] and needs[0].head_dim == 48 and needs[0].value_dim == 40 and needs[4].head_dim == 48 and needs[4].value_dim == 32
    assert sorted(model.state_needs()) == [1, 3, 6] and model.state_needs()[3].shape == (4 * 12 * 8,)
    assert [e.cache_of for e in model.spec.plan] == [None, None, 0, None, None, 4, None, 0]
    # ranks that only the tensors' shapes give
    bare = copy.deepcopy(rt.MIXED)
    for layer in bare["layers"]:
        for key in ("q_rank", "kv_rank"):
            layer["mixer"].pop(key, None)
    with pytest.raises(ConfigError):
        hb.RidotarConfig.from_dict(bare).model_spec()
    shapes = {n: p.shape for n, p in table.items()}
    assert hb.RidotarConfig.from_dict(bare).with_tensor_shapes(shapes) == c
    with pytest.raises(ConfigError):
        c.with_tensor_shapes({"l0.mix.dq": (25, 64)})
    d = str(tmp_path / "m")
    rt.write_model(d, rt.MIXED, 3, state_ranks=False)
    assert hb.load_config(d) == c

    def changed(i, path, value, drop=False):
        cfg = copy.deepcopy(rt.MIXED)
        at = cfg["layers"][i]
        for k in path[:-1]:
            at = at[k]
        if drop:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return cfg
    for bad in ({**rt.MIXED, "layers": []}, {**rt.MIXED, "width": 0}, {k: v for k, v in rt.MIXED.items() if k != "norm"},
                {**rt.MIXED, "norm": {"eps": 1e-5, "groups": 7}}, {**rt.MIXED, "token_side": {"dim": 0}}, changed(0, ("type",), "conv"),
                changed(3, ("mixer", "decay"), [0.5]), changed(3, ("mixer", "decay"), [0.5, 1.5, 0.1, 0.1]), changed(0, ("mixer", "rot", "dims"), 3),
                changed(0, ("mixer", "rot", "dims"), 10), changed(2, ("mixer", "kv_from"), 2), changed(2, ("mixer", "kv_from"), 1),
                changed(7, ("mixer", "kv_from"), 2), changed(7, ("mixer", "kv_from"), 4), changed(5, ("mixer", "rot", "base"), 51.0),
                changed(0, ("mlp", "router", "top"), 7), changed(0, ("mlp", "kind"), "dense"), changed(1, ("mixer", "dim"), None, drop=True),
                changed(0, ("mixer", "scale"), None, drop=True)):
        with pytest.raises(ConfigError):
            hb.RidotarConfig.from_dict(bad)


def test_plain_mechanisms_agree_with_their_definitions():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # the group-wise norm: unit mean square per run of neighbours, whatever the runs' sizes are; one group is the ordinary norm
    x, w = r(3, 12) * torch.tensor([1.0, 100.0, 0.01]).repeat_interleave(4), r(12)
    y = group_rms_norm(x, w, 0.0, 3) / w
    assert torch.allclose((y * y).reshape(3, 3, 4).mean(-1), torch.ones(3, 3, dtype=torch.float64))
    assert torch.allclose(group_rms_norm(x, w, 0.3, 1), rms_norm(x, w, 0.3))
    # the norm sits behind the sum, the gate in front of it
    b = r(3, 12)
    assert torch.allclose(gated_sum_norm(x, b, torch.full((3, 12), 40.0, dtype=torch.float64), 2.0, w, 0.1, 4), group_rms_norm(2 * x + b, w, 0.1, 4))
    assert torch.allclose(gated_sum_norm(x, b, torch.full((3, 12), -60.0, dtype=torch.float64), 2.0, w, 0.1, 4), group_rms_norm(2 * x, w, 0.1, 4))
    # the memories as explicit sums
    q, k, v, lam = r(6, 2, 3), r(6, 2, 3), r(6, 2, 4), [0.8, 1.0]
    out = fixed_decay_memory(q, k, v, lam)
    for h in range(2):
        assert torch.allclose(out[5, h], sum(lam[h] ** (5 - s) * (q[5, h] @ k[s, h]) * v[s, h] for s in range(6)))
    f = torch.rand(6, 2, 3, generator=g, dtype=torch.float64)
    out = forget_gate_memory(q, v, f)
    assert torch.allclose(out[5, 1], sum((q[5, 1] * (1 - f[s, 1]) * f[s + 1:, 1].prod(0)).sum() * v[s, 1] for s in range(6)))
    # a memory that forgets nothing is written nothing; one that forgets all holds the last value alone
    assert forget_gate_memory(q, v, torch.ones_like(f)).abs().max() == 0
    assert torch.allclose(forget_gate_memory(q, v, torch.zeros_like(f))[4, 0], q[4, 0].sum() * v[4, 0])
    # interleaved pairs; a score depends on the distance only
    t = r(1, 1, 6)
    got = rotate_pairs(t, torch.tensor([5]), 4, 100.0)[0, 0]
    for i, a in enumerate((5.0, 0.5)):
        assert torch.allclose(got[2 * i], t[0, 0, 2 * i] * math.cos(a) - t[0, 0, 2 * i + 1] * math.sin(a))
        assert torch.allclose(got[2 * i + 1], t[0, 0, 2 * i + 1] * math.cos(a) + t[0, 0, 2 * i] * math.sin(a))
    assert torch.equal(got[4:], t[0, 0, 4:])
    # causal softmax, and the latent attention's folded form: [Wuk^T q | q_r] against [c | k_r], values from the mixed latents
    T, H, d, dr, dv, rank = 6, 2, 3, 2, 4, 5
    q, c, kr, uk, uv = r(T, H, d + dr), r(T, rank), r(T, dr), r(H, d, rank), r(H, dv, rank)
    keys = torch.cat([torch.einsum("hdr,tr->thd", uk, c), kr[:, None].expand(T, H, dr)], -1)
    want = causal_softmax(q, keys, torch.einsum("hvr,tr->thv", uv, c), 0.4)
    s = torch.softmax(torch.stack([q[3, 1] @ keys[j, 1] for j in range(4)]) * 0.4, 0)
    assert torch.allclose(want[3, 1], sum(s[j] * (uv[1] @ c[j]) for j in range(4)))
    qf = torch.cat([torch.einsum("thd,hdr->thr", q[..., :d], uk), q[..., d:]], -1)
    mixed = causal_softmax(qf, torch.cat([c, kr], -1)[:, None].expand(T, H, rank + dr), c[:, None].expand(T, H, rank), 0.4)
    assert torch.allclose(torch.einsum("thr,hvr->thv", mixed, uv), want)
    # the router's scores are not divided by anything, and they multiply what an expert reads
    h, wr = r(1, 5), r(4, 5)
    chosen, scores = route(h, wr, 2)
    z = wr @ h[0]
    assert set(chosen[0].tolist()) == set(torch.topk(z, 2).indices.tolist()) and torch.allclose(scores[0], torch.sigmoid(z[chosen[0]]))
    w = {"router": wr, **{f"e{e}.{n}": r(*s) for e in range(4) for n, s in (("gate", (3, 5)), ("up", (3, 5)), ("down", (5, 3)))}}
    want = 0
    for e in chosen[0].tolist():
        hin = torch.sigmoid(z[e]) * h[0]
        want = want + w[f"e{e}.down"] @ (silu(w[f"e{e}.gate"] @ hin) * (w[f"e{e}.up"] @ hin))
    assert torch.allclose(moe_ff(h, w, {"router": {"experts": 4, "top": 2}})[0], want)
    # the side input: its norm makes its size independent of the table's
    e, wg, wp = r(3, 4), r(4, 12), r(12, 4)
    a, b = (token_side(x, x, e * f, wg, wp, torch.ones(12, dtype=torch.float64), 0.0) for f in (1.0, 7.0))
    assert torch.allclose(a, b) and torch.allclose(((a - x) ** 2).mean(-1), torch.ones(3, dtype=torch.float64))
    assert abs(gelu_tanh(torch.tensor(1.0)).item() - 0.841192) < 1e-5


# --------------------------------------------------------------------------- kernels alone
@pytest.mark.gpu
def test_group_norm_alone_and_behind_a_gated_sum():
    require_gpu()
    c = _context(torch.float32)
    ops, g = c.ops, torch.Generator().manual_seed(1)
    for width, groups in ((1, 1), (2, 2), (12, 3), (40, 5), (72, 9), (256, 16), (257, 1), (1000, 8), (2048, 8), (2500, 4), (4096, 1), (6000, 6), (9000, 2), (640, 160)):
        x, y = torch.randn(19, width, generator=g).cuda(), (torch.randn(38, width, generator=g) * 3).cuda()
        # runs of very different sizes: a norm over the wrong values shows
        x *= (10.0 ** (torch.arange(groups) % 5 - 2).float()).repeat_interleave(width // groups).cuda()
        w, bias = torch.randn(width, generator=g).cuda(), torch.randn(width, generator=g).cuda()
        big = torch.randn(19, width + 12, generator=g).cuda()
        for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 1e-2)):
            out = torch.empty(19, width, dtype=dtype, device=DEV)
            ops.group_rmsnorm(x, w, 1e-5, groups, out)
            want = group_rms_norm(x.double(), w.double(), 1e-5, groups)
            assert ((out.double() - want).abs() / want.abs().clamp(min=1.0)).max() < tol, (width, groups, dtype)
            rows = torch.tensor([18, 0, 5], dtype=torch.int32, device=DEV)
            some = torch.empty(3, width, dtype=dtype, device=DEV)
            ops.group_rmsnorm(x, w, 1e-5, groups, some, rows)
            assert torch.equal(some, out[rows.long()])
        for at in (8, 3):                               # the gate's logits as columns of a wider matrix, aligned and not
            gate = big[:, at: at + width]
            for n_sum in (1, 2):
                yy = y[: 19 * n_sum]
                total = yy.double().reshape(19, n_sum, width).sum(1)
                for gl, gb in ((gate, bias), (gate, None), (None, None)):
                    logits = torch.full((19, width), 60.0, dtype=torch.float64, device=DEV) if gl is None else gl.double() + (0 if gb is None else gb.double())
                    want = gated_sum_norm(x.double(), total, logits, 1.7, w.double(), 1e-4, groups)
                    x1, copy = x.clone(), torch.empty(19, width, dtype=torch.bfloat16, device=DEV)
                    ops.gated_sum_norm(x1, 1.7, yy, w, 1e-4, groups, gate=gl, gate_bias=gb, n_sum=n_sum, copy=copy)
                    assert ((x1.double() - want).abs() / want.abs().clamp(min=1.0)).max() < 3e-5, (width, groups, at, n_sum)
                    assert torch.equal(copy, x1.to(torch.bfloat16))
                    x2 = x.clone()
                    ops.gated_sum_norm(x2, 1.7, yy, w, 1e-4, groups, gate=gl, gate_bias=gb, n_sum=n_sum)
                    assert torch.equal(x1, x2)
        # the stream plus an ordinary norm, with a copy of the new rows
        x1, copy = x.clone(), torch.empty(19, width, dtype=torch.bfloat16, device=DEV)
        ops.rmsnorm_add(y[:19], w, 1e-5, 0.0, x1, copy=copy)
        want = x.double() + rms_norm(y[:19].double(), w.double(), 1e-5)
        assert ((x1.double() - want).abs() / want.abs().clamp(min=1.0)).max() < 3e-5 and torch.equal(copy, x1.to(torch.bfloat16))
    ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_side_part(dtype):
    require_gpu()
    from hilbert_pruned_8b_b200.config.spec import PartSpec
    from hilbert_pruned_8b_b200.parts import TOKEN_SIDES
    from hilbert_pruned_8b_b200.parts.token_side import SIDE_TABLE
    g = torch.Generator().manual_seed(2)
    vocab, rnd = 50, _rnd(dtype)

    class Step:
        pass
    for width, dim, T in ((64, 12, 9), (40, 1, 3), (256, 40, 70), (128, 200, 17), (72, 64, 1)):
        c = _context(dtype)
        layers = 3
        table = torch.randn(vocab, dim * layers, generator=g).to(torch.bfloat16)
        for layer in range(layers):
            part = TOKEN_SIDES.build(PartSpec("gelu_side", {"size": width, "dim": dim, "offset": layer * dim, "eps": 1e-5}), c)
            w = {"gate": torch.randn(dim, width, generator=g) * 2 / width ** 0.5, "proj": torch.randn(width, dim, generator=g) / dim ** 0.5,
                 "norm": torch.randn(width, generator=g) * 0.3 + 1}
            w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
            part.bind({k: (v.to(dtype) if v.dim() == 2 else v).to(DEV) for k, v in w.items()})
            step = Step()
            step.num_tokens, step.tokens, step.shared = T, torch.randint(0, vocab, (T,), generator=g).to(torch.int32).to(DEV), {SIDE_TABLE: table.to(dtype).to(DEV)}
            x = torch.randn(T, width, generator=g)
            h = x.to(dtype).cuda()
            e = table.double()[step.tokens.cpu().long()][:, layer * dim: (layer + 1) * dim]
            want = token_side(x.double(), rnd(x.double()), e, w["gate"].double(), w["proj"].double(), w["norm"].double(), 1e-5, rnd)
            x1, copy = x.cuda(), torch.empty(T, width, dtype=torch.bfloat16, device=DEV)
            part.forward(x1 if dtype == torch.float32 else h, x1, step, copy=copy if dtype == torch.bfloat16 else None)
            assert (x1.cpu().double() - want).abs().max() < (2e-4 if dtype == torch.float32 else 4e-2) * max(1.0, want.abs().max().item()), (width, dim, T, layer)
            assert dtype == torch.float32 or torch.equal(copy, x1.to(torch.bfloat16))
        c.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sigmoid_router_and_experts_with_weighted_inputs(dtype):
    require_gpu()
    from hilbert_pruned_8b_b200.config.spec import PartSpec
    from hilbert_pruned_8b_b200.parts import FEED_FORWARDS
    g, rnd = torch.Generator().manual_seed(3), _rnd(dtype)

    class Step:
        pass
    for n, (width, E, top, ff, T) in enumerate(((24, 3, 2, 10, 1), (64, 6, 2, 32, 5), (64, 5, 1, 24, 333), (40, 1, 1, 8, 70), (128, 40, 6, 64, 90), (56, 4, 4, 40, 33))):
        for tc in (True, False):
            c = _context(dtype)
            c.ops.use_tensor_cores = tc
            part = FEED_FORWARDS.build(PartSpec("moe", {"hidden_size": width, "num_experts": E, "top": top, "expert_size": ff, "router": "sigmoid",
                                                        "unit": "silu_glu", "weigh": "input"}), c)
            # scores far below one for most: an expert whose result (not its input) were weighted would differ
            w = {p.name: (torch.randn(tuple(p.shape), generator=g) * (1.5 if p.name == "router" else 2.0) / p.shape[1] ** 0.5).to(torch.bfloat16).float()
                 for p in part.params()}
            part.bind({k: v.to(dtype).to(DEV) for k, v in w.items()})
            h = (torch.randn(T, width, generator=g) * 1.5).to(torch.bfloat16)
            cfg = {"router": {"experts": E, "top": top}}
            want = moe_ff(h.double(), {k: v.double() for k, v in w.items()}, cfg, rnd)
            step = Step()
            step.num_tokens = T
            out = torch.full((T, width), 2.0, device=DEV)
            part.forward(h.to(dtype).cuda(), out, step, accumulate=True)
            tol = (1e-5 if dtype == torch.float32 else 2e-2) * max(1.0, want.abs().max().item())
            assert (out.cpu().double() - 2.0 - want).abs().max() < tol, (n, tc)
            assert part.sums_entries
            rows, k = part.forward_entries(h.to(dtype).cuda(), step)
            assert k == top and (rows.cpu().double().reshape(T, top, width).sum(1) - want).abs().max() < tol, (n, tc)
            part.forward(h.to(dtype).cuda(), out, step, accumulate=False)
            assert (out.cpu().double() - want).abs().max() < tol
            c.ops.check_errors()


# --------------------------------------------------------------------------- mixers alone
def _mixer_spec(layer, width):
    import hilbert_pruned_8b_b200 as hb
    return hb.RidotarConfig.from_dict(rt.config(width, 16, [rt.with_mlp(layer, None)], groups=1)).model_spec().layers[0].parts["mixer"]


def _mixer_weights(spec, seed):
    from hilbert_pruned_8b_b200.engine.model import describe_context
    from hilbert_pruned_8b_b200.parts import MIXERS
    g = torch.Generator().manual_seed(seed)
    return {p.name: rt.draw(p.name, tuple(p.shape), g).to(torch.bfloat16).float() for p in MIXERS.build(spec, describe_context()).params()}


def _close(got, want, dtype, what):
    for i, (a, b) in enumerate(zip(got, want)):
        err = (a - b).abs().max(1).values / b.abs().max().clamp(min=1.0)
        assert err.max() < (1e-4 if dtype == torch.float32 else 3e-2), f"{what}: sequence {i} position {int(err.argmax())}: {float(err.max()):.3e}"


def _inputs(width, seed, lengths=(70, 3, 131)):
    g = torch.Generator().manual_seed(seed)
    return [torch.randn(t, width, generator=g).to(torch.bfloat16).float() for t in lengths]


def _double(w):
    return {k: v.double() for k, v in w.items()}


FORGET = [(3, 8, 12), (1, 1, 3), (2, 4, 4), (2, 128, 64), (3, 40, 96), (1, 256, 20), (5, 20, 7), (4, 64, 200)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_forget_gate_memory_in_portions_against_the_recurrence(dtype):
    require_gpu()
    width, rnd = 48, _rnd(dtype)
    for n, (heads, d, dv) in enumerate(FORGET):
        layer = rt.hgrn2(heads, d, dv)
        spec = _mixer_spec(layer, width)
        w = _mixer_weights(spec, 20 + n)
        hs = _inputs(width, 30 + n)
        want = [hgrn2_mixer(h.double(), _double(w), layer["mixer"], 1e-5, rnd) for h in hs]
        c = _context(dtype)
        for sizes in ((200,), (1, 2, 3, 1, 64, 5, 200), (33, 1, 1, 1, 1, 1, 200)):
            run = _MixerRun(c, spec, w)
            _close(run.feed(hs, sizes), want, dtype, f"forget_gate_memory {(heads, d, dv)} portions {sizes}")
            _close(run.feed(hs, (7, 2, 200)), want, dtype, "slots used again")
        # long portions cut into chunks that run side by side: the same sums
        c.ops.HEAD_SCAN_CHUNK_FROM = 8
        c.ops.sm_count = 10 ** 6
        _close(_MixerRun(c, spec, w).feed(hs, (100, 200)), want, dtype, "chunks side by side")
    # gates next to one and next to the lower bound, bounds of zero and one: a memory that keeps everything and is written
    # nothing, one that forgets all at once, and a very slow one that must keep its distance to one
    layer = rt.hgrn2(2, 8, 8)
    spec = _mixer_spec(layer, width)
    for bias, low in ((40.0, 0.5), (-40.0, 0.0), (-40.0, 0.996), (9.0, 0.0), (0.0, 1.0)):
        w = _mixer_weights(spec, 9)
        w["f.b"], w["lower"] = torch.full_like(w["f.b"], bias), torch.full_like(w["lower"], low)
        hs = _inputs(width, 1, (290,))
        want = [hgrn2_mixer(hs[0].double(), _double({k: (v.to(torch.bfloat16).float() if k == "lower" else v) for k, v in w.items()}), layer["mixer"], 1e-5, rnd)]
        w["lower"] = w["lower"].to(torch.bfloat16).float()
        _close(_MixerRun(_context(dtype), spec, w).feed(hs, (40, 1, 1, 300)), want, dtype, f"gate bias {bias}, lower bound {low}")
        c = _context(dtype)
        c.ops.HEAD_SCAN_CHUNK_FROM = 8
        c.ops.sm_count = 10 ** 6
        _close(_MixerRun(c, spec, w).feed(hs, (300,)), want, dtype, f"chunks side by side, gate bias {bias}, lower bound {low}")


MEMORY = [(4, 12, 8, (0.5, 0.9, 0.97, 0.998)), (1, 1, 1, (1.0,)), (3, 5, 7, (0.0, 1.0, 0.75)), (2, 64, 32, (0.4, 0.9995)), (2, 128, 40, (0.99, 0.2)),
          (1, 256, 16, (0.9,))]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_fixed_decay_memory_in_portions_against_the_recurrence(dtype):
    require_gpu()
    width, rnd = 40, _rnd(dtype)
    for n, (heads, d, dv, decay) in enumerate(MEMORY):
        layer = rt.lightning(heads, d, dv, decay)
        spec = _mixer_spec(layer, width)
        w = _mixer_weights(spec, 50 + n)
        hs = _inputs(width, 60 + n)
        want = [lightning_mixer(h.double(), _double(w), layer["mixer"], 1e-5, rnd) for h in hs]
        c = _context(dtype)
        for sizes in ((200,), (1, 2, 3, 1, 64, 5, 200), (31, 1, 1, 32, 1, 1, 200)):
            run = _MixerRun(c, spec, w)
            _close(run.feed(hs, sizes), want, dtype, f"fixed decay {(heads, d, dv)} portions {sizes}")
            _close(run.feed(hs, (7, 2, 200)), want, dtype, "slots used again")


class _PairRun(_MixerRun):
    """A latent mixer that keeps its latents and one that reads them: feeds both, returns both results side by side."""

    def __init__(self, c, spec, weights, reader_spec, reader_weights):
        from hilbert_pruned_8b_b200.parts import MIXERS
        super().__init__(c, spec, weights)
        source, reader = self.mixer, MIXERS.build(reader_spec, c)
        reader.bind({k: (v.to(c.dtype) if v.dim() == 2 else v).to(DEV) for k, v in reader_weights.items()})
        self.readers = [reader]

        class Both:
            def forward(_, hin, out, step, cache, state, append, accumulate):
                half = out.shape[1] // 2
                a, b = torch.full((out.shape[0], half), 3.0, device=DEV), torch.full((out.shape[0], half), 5.0, device=DEV)
                source.forward(hin[:, :half].contiguous(), a, step, cache, state, True, accumulate=False)
                reader.forward(hin[:, half:].contiguous(), b, step, cache, state, False, accumulate=False)
                out[:, :half], out[:, half:] = a, b
        self.source, self.mixer = source, Both()


def _eye(rows, width, at):
    m = torch.zeros(rows, width)
    m[torch.arange(rows), at + torch.arange(rows)] = 1.0
    return m


# (heads, dim, rot_dim, vdim, kv_rank): the general kernel, the one-block-per-token kernel, the tensor-core prompt kernel on
# written-out keys of 64 to 192 numbers (bfloat16), sixteen heads, odd sizes
LATENTS = [(4, 16, 8, 12, 40), (1, 8, 2, 5, 9), (3, 3, 4, 3, 8), (16, 32, 32, 64, 64), (4, 96, 32, 96, 64), (2, 128, 64, 128, 192), (6, 40, 24, 20, 56)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention_with_far_probes_and_a_reader(dtype):
    require_gpu()
    import hilbert_pruned_8b_b200 as hb
    rnd = _rnd(dtype)
    for n, (H, d, dr, dv, rank) in enumerate(LATENTS):
        # the latent is cut out of the input, and so is the queries' latent (of the latent's size: a query that is a key's
        # direction), so that a probe can be written into the input; the second half of the width feeds the reader
        half = 2 * rank + dr
        layer = rt.latent(H, d, dr, dv, rank, rank, base=30.0, scale=6.0 / (d + dr) ** 0.5)
        other = rt.latent(H + 1, max(1, d - 2), dr, dv + 1, rank + 3, rank, base=30.0, kv_from=0, scale=1.5 / (d + dr) ** 0.5)
        specs = [ls.parts["mixer"] for ls in hb.RidotarConfig.from_dict(rt.config(half, 16, [rt.with_mlp(layer, None), rt.with_mlp(other, None)], groups=1)).model_spec().layers]
        g = torch.Generator().manual_seed(70 + n)
        w, w2 = _mixer_weights(specs[0], 80 + n), _mixer_weights(specs[1], 90 + n)
        w["dq"], w["dq.norm"] = _eye(rank, half, 0), torch.ones(rank)
        w["dkv"], w["dkv.norm"] = _eye(rank + dr, half, rank), torch.ones(rank)
        uk = (torch.randn(H, d, rank, generator=g) / rank ** 0.5).to(torch.bfloat16).float()
        w["uk"] = uk.reshape(H * d, rank)
        w["uq"] = torch.cat([uk, torch.randn(H, dr, rank, generator=g) * 0.3 / rank ** 0.5], dim=1).reshape(H * (d + dr), rank).to(torch.bfloat16).float()
        lengths = (200, 77, 1)
        hs = [torch.randn(t, 2 * half, generator=g) for t in lengths]
        for p, s in ((5, 0), (63, 1), (64, 3), (65, 63), (127, 64), (128, 127), (130, 2), (150, 66), (199, 4)):
            direction = torch.randn(rank, generator=g)
            hs[0][p, :rank] = direction                  # the query at p looks for the latent at s
            hs[0][s, rank: 2 * rank] = direction
        hs = [h.to(torch.bfloat16).float() for h in hs]
        want = []
        for h in hs:
            a, cached = latent_mixer(h[:, :half].double(), _double(w), layer["mixer"], 1e-5, torch.arange(h.shape[0]), None, rnd)
            b, _ = latent_mixer(h[:, half:].double(), _double(w2), other["mixer"], 1e-5, torch.arange(h.shape[0]), cached, rnd)
            want.append(torch.cat([a, b], 1))
        c = _context(dtype)
        for write_out in ((True, False) if dtype == torch.bfloat16 else (True,)):
            for sizes in ((300,), (60, 3, 1, 1, 1, 1, 1, 1, 1, 58, 1, 1, 1, 1, 1, 1, 1, 300), (2, 126, 1, 1, 300)):
                run = _PairRun(c, specs[0], w, specs[1], w2)
                run.source.write_out = run.readers[0].write_out = write_out
                _close(run.feed(hs, sizes), want, dtype, f"latent attention {(H, d, dr, dv, rank)} portions {sizes} written out {write_out}")
                _close(run.feed(hs, (150, 1, 1, 300)), want, dtype, "pages used again")
        if dtype == torch.float32 and d >= 12:
            # the probes do stand out: without the probed key, 195 tokens back, the result is another
            blind = hs[0].clone()
            blind[4, rank: 2 * rank] = 0
            a, _ = latent_mixer(blind[:, :half].double(), _double(w), layer["mixer"], 1e-5, torch.arange(200))
            assert (a[199] - want[0][199, :half]).abs().max() > 0.05 * want[0].abs().max()
    with pytest.raises(ValueError):
        run.readers[0].forward(None, None, None, None, None, True)           # a reader has nothing to append


# --------------------------------------------------------------------------- the engine
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompts_and_token_by_token(models, name, dtype):
    require_gpu()
    folder, cfg, plain = models[name]
    requests = _requests(cfg, [150, 64, 1, 2, 65], 100)
    eng = _engine(folder, dtype, 64 * 12)
    steps, _ = tt.trace_whole(requests)
    _check(eng, steps, plain, requests, dtype, f"{name} whole")
    steps, _ = tt.trace_tail(requests, tail=75)
    _check(eng, steps, plain, requests, dtype, f"{name} last 75 tokens one by one")
    assert all(g.pool.num_free == g.pool.size for g in eng.cache.groups)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_prompts_in_portions(models, name, dtype):
    require_gpu()
    folder, cfg, plain = models[name]
    requests = _requests(cfg, [170, 71], 200)
    eng = _engine(folder, dtype, 64 * 12)
    for sizes in ((2, 3, 1, 64, 1, 1, 5, 300), (63, 1, 1, 2, 300), (128, 1, 300)):
        steps = []
        for rid, toks in requests.items():
            at = 0
            for n in sizes:
                part = toks[at: at + n]
                if not part:
                    break
                steps.append({"step": len(steps), "entries": [{"id": rid, "tokens": part, "want": list(range(len(part)))}],
                              "end": [rid] if at + n >= len(toks) else []})
                at += n
        _check(eng, steps, plain, requests, dtype, f"{name} portions {sizes}")
    # steps cut by the engine itself
    small = _engine(folder, dtype, 64 * 12, max_step_tokens=48)
    steps, _ = tt.trace_whole(requests)
    _check(small, steps, plain, requests, dtype, f"{name} steps of 48 tokens")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", NAMES)
def test_unequal_batches_with_slots_and_pages_used_again(models, name, dtype):
    require_gpu()
    folder, cfg, plain = models[name]
    lengths = [(140, 100), (30, 3), (67, 64), (90, 1), (129, 128), (12, 12)]
    requests = _requests(cfg, [n for n, _ in lengths], 300)
    ids = list(requests)
    batches = [{ids[i]: (requests[ids[i]], lengths[i][1]) for i in (0, 1, 2)}, {ids[i]: (requests[ids[i]], lengths[i][1]) for i in (3, 4, 5)},
               {ids[i]: (requests[ids[i]], lengths[i][1]) for i in (1, 4)}]
    steps, peak = tt.trace_batches(batches)
    eng = _engine(folder, dtype, peak + 64, max_sequences=3)
    _check(eng, steps, plain, requests, dtype, f"{name} batches")
    assert all(g.pool.num_free == g.pool.size for g in eng.cache.groups)
    assert dtype == "bfloat16" or eng.graph_replays > 0


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding_and_fused_steps_against_separate_ones(models, name):
    require_gpu()
    folder, cfg, plain = models[name]
    requests = _requests(cfg, [420], 400)
    eng = _engine(folder, "float32", 64 * 8)
    steps, _ = tt.trace_tail(requests, tail=400)
    _check(eng, steps, plain, requests, "float32", f"{name} 400 decoded tokens")
    assert eng.graph_replays > 300
    # the experts' results summed by the mixture itself, and every gate a product of its own
    import hilbert_pruned_8b_b200 as hb
    from hilbert_pruned_8b_b200.config.spec import LayerSpec
    from hilbert_pruned_8b_b200.engine.step import Engine
    from hilbert_pruned_8b_b200.weights.loader import load_tensors
    import dataclasses
    spec = hb.load_config(folder).model_spec()
    spec = dataclasses.replace(spec, layers=[LayerSpec(l.prefix, l.parts, l.part_prefixes, l.block, {**l.block_params, "host_gate": False}) for l in spec.layers])
    plainer = Engine(spec, "float32", 64 * 8)
    plainer.model.bind(load_tensors(folder, plainer.model.weight_table(""), plainer.dtype, plainer.device), "")
    plainer._make_cache()
    for b, hosted in zip(plainer.model.blocks, eng.model.blocks):
        b.fuse_entries = False
        assert hosted.mixer_gate.hosted and not b.mixer_gate.hosted
    steps, _ = tt.trace_whole(requests)
    _check(plainer, steps, plain, requests, "float32", f"{name} separate steps")


@pytest.mark.gpu
def test_rewinding_a_sequence_with_memories_and_shared_latents(models):
    require_gpu()
    from hilbert_pruned_8b_b200.engine.batch import StepEntry
    folder, cfg, plain = models["mixed"]
    eng = _engine(folder, "float32", 64 * 8)
    a, b, c = tt.random_tokens(70, cfg["vocab"], 1), tt.random_tokens(9, cfg["vocab"], 2), tt.random_tokens(66, cfg["vocab"], 3)
    seq = eng.open_sequence()
    eng.step_chunked([StepEntry(seq, a, [])])
    snap = eng.snapshot(seq)
    eng.step_chunked([StepEntry(seq, c, [])])
    eng.restore(seq, snap)
    got = eng.step_chunked([StepEntry(seq, b, list(range(9)))]).cpu().double()
    want = plain["exact"].logits(a + b)[70:]
    assert (got - want).abs().max() < 1e-3 * max(1.0, want.abs().max().item())
    eng.close_sequence(seq)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_and_the_replay_program(models, dtype, tmp_path):
    require_gpu()
    import hilbert_pruned_8b_b200 as hb
    folder, cfg, plain = models["mixed"]
    prompts = [tt.random_tokens(n, cfg["vocab"], 500 + n) for n in (40, 3, 21, 1, 66)]
    llm = hb.load(folder, dtype=dtype, max_tokens=64 * 8, max_batch=3)        # two batches: slots are used again
    res = llm.generate(prompts, max_new_tokens=24, stop_token_ids=[])
    for prompt, r in zip(prompts, res):
        assert len(r.tokens) == 24
        if dtype == "float32":
            # every generated token is the plain model's choice given the tokens before it (two nearly tied logits aside)
            lg = plain["exact"].logits(prompt + r.tokens)
            for i, t in enumerate(r.tokens):
                row = lg[len(prompt) + i - 1]
                assert row[t] >= row.max() - 1e-3 * max(1.0, row.abs().max().item()), f"prompt of {len(prompt)} tokens, token {i}"
    assert llm.generator.stats.batches == 2
    assert all(g.pool.num_free == g.pool.size for g in llm.engine.cache.groups)
    requests = _requests(cfg, [70, 9], 600)
    steps, peak = tt.trace_batches([{rid: (toks, len(toks) - 5) for rid, toks in requests.items()}])
    got = tt.run_program(folder, dtype, steps, peak, str(tmp_path / "out"), cfg["vocab"])
    # the program drives the engine: the same logits, its decode steps from captured graphs
    want = tt.run_in_process(_engine(folder, dtype, peak), steps)
    assert sorted(got) == sorted(want) and all(torch.equal(got[k], want[k]) for k in want)
    _check(_engine(folder, dtype, peak), steps, plain, requests, dtype, "replayed steps")
