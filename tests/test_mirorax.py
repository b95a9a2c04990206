"""The Mirorax decoder against the plain implementation (tests/plain_mirorax.py): every mechanism alone (the sum behind two sublayers
with its factors, vectors and norm; the clamped gated unit; the biased router with silu experts and a shared expert; the
attention without positions and with a gate per element; the attention over latents with a window and a sink), then the
engine: whole prompts, token-by-token decoding, prompts in portions down to two tokens, unequal batches with slots and pages
used again, long decoding, greedy generation through the library's entry point and the replay program."""
import copy
import math

import pytest
import torch

import mirorax_tools as mt
import trace_tools as tt
from conftest import require_gpu
from plain_mirorax import (PlainMirorax, attention_mixer, clamped_unit, dense_ff, latent_mixer, layer_runs, moe_ff, parallel_sum, rms_norm,
                           rotate_pairs, route, silu, softmax_attention, to_bf16, visible)
from test_ridotar import _Choices
from test_tonovik import _MixerRun, _compare, _context, _reference, _requests

DTYPES = ["float32", "bfloat16"]
NAMES = list(mt.CONFIGS)
DEV = "cuda:0"


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (folder, config, {"exact" | dtype: plain model})"""
    out = {}
    for i, (name, cfg) in enumerate(mt.CONFIGS.items()):
        d = str(tmp_path_factory.mktemp("mirorax_" + name))
        tensors = mt.write_model(d, cfg, 40 + i)
        out[name] = (d, cfg, {"exact": PlainMirorax(cfg, tensors), "float32": PlainMirorax(cfg, tensors, dtype=torch.float32),
                              "bfloat16": PlainMirorax(cfg, tensors, round_to=torch.bfloat16)})
    return out


def _engine(folder, dtype, max_tokens, **kw):
    from hilbert_pruned_8b_b200.engine.step import Engine
    return Engine.from_folder(folder, dtype, max_tokens=max_tokens, **kw)


CLOSE_CALL = 0.3        # a choice may differ from the exact model's by so much of a logit (rounding moves logits by hundredths)


def _check(eng, steps, plain, requests, dtype, what):
    """Runs the steps and compares every wanted position with the plain models, which in bfloat16 take the experts that the
    library chose (nearly tied logits may go either way once the router's input is rounded)."""
    if dtype == "float32":
        _compare(tt.run_in_process(eng, steps), _reference(plain, requests, dtype), dtype, what)
        return
    choices = _Choices(eng)
    got = tt.run_in_process(eng, steps)

    class Followed:
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


def _double(w):
    return {k: v.double() for k, v in w.items()}


# --------------------------------------------------------------------------- without a GPU
def test_config_round_trip_weight_table_and_plan():
    import hilbert_pruned_8b_b200 as hb
    from hilbert_pruned_8b_b200.config import ConfigError, config_class_for
    from hilbert_pruned_8b_b200.engine.model import DecoderModel, describe_context, weight_table
    for cfg in mt.CONFIGS.values():
        assert config_class_for(cfg) is hb.MiroraxConfig
        c = hb.MiroraxConfig.from_dict(cfg)
        assert hb.MiroraxConfig.from_dict(c.to_dict()) == c
        table = weight_table(c.model_spec(), "")
        W, loop = cfg["width"], cfg.get("loop")
        assert ("loop.step" in table) == (loop is not None) and (loop is None or table["loop.step"].shape == (loop["times"], W))
        assert table["head"].shape == table["embed"].shape == (cfg["vocab"], W) and "final.norm" in table
        for i, layer in enumerate(cfg["layers"]):
            m, mlp, has = layer["mixer"], layer["mlp"], lambda n: f"l{i}.{n}" in table
            assert has("norm1") and has("ls1") and not has("norm2") and has("ls2") == (mlp is not None)
            plain = layer["type"] == "attention"
            assert all(has("mix." + n) == plain for n in ("k", "v", "g", "q.b", "k.b", "v.b", "o.b")) and not has("mix.g.b")
            assert all(has("mix." + n) != plain for n in ("dkv", "dkv.norm", "uk", "uv", "sink"))
            if plain:
                assert table[f"l{i}.mix.g"].shape == (m["heads"] * m["vdim"], W) and table[f"l{i}.mix.v.b"].shape == (m["kv_heads"] * m["vdim"],)
            assert has("mlp.gate") == (mlp is not None and mlp["kind"] == "dense")
            routed = mlp is not None and mlp["kind"] == "moe"
            assert has("mlp.router") == has("mlp.router.b") == routed and has("mlp.shared.down") == (routed and "shared" in mlp)
        # the order of the runs, and who adds a pass's vector
        plan = c.model_spec().plan
        assert [(e.layer, e.adds) for e in plan] == [(i, t if opens else None) for i, t, opens in layer_runs(len(cfg["layers"]), loop)]
        assert all(e.cache_of is None for e in plan)
    # every run of a layer keeps keys and values of its own; runs with one need share a group
    model = DecoderModel(hb.MiroraxConfig.from_dict(mt.MIXED).model_spec(), describe_context())
    needs = model.cache_needs()
    assert sorted(needs) == list(range(12)) and [needs[i].window for i in range(12)] == [None, 30, None, 70, 30, None, 70, 30, None, 70, None, 30]
    assert needs[1].head_dim == 48 and needs[1].value_dim == 40 and needs[0].num_kv_heads == 2 and needs[0].value_dim == 12

    def changed(i, path, value, drop=False):
        cfg = copy.deepcopy(mt.MIXED)
        at = cfg["layers"][i]
        for k in path[:-1]:
            at = at[k]
        if drop:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        return cfg
    for bad in ({**mt.MIXED, "layers": []}, {**mt.MIXED, "width": 0}, {k: v for k, v in mt.MIXED.items() if k != "norm"},
                {**mt.MIXED, "loop": {"start": 2, "stop": 2, "times": 1}}, {**mt.MIXED, "loop": {"start": 0, "stop": 7, "times": 1}},
                {**mt.MIXED, "loop": {"start": 0, "stop": 2, "times": 0}}, {**mt.MIXED, "loop": {"start": 0, "stop": 2}},
                changed(0, ("type",), "conv"), changed(0, ("mixer", "kv_heads"), 3), changed(0, ("mixer", "scale"), None, drop=True),
                changed(1, ("mixer", "mask"), None, drop=True), changed(1, ("mixer", "mask", "size"), 0), changed(1, ("mixer", "rot", "dims"), 3),
                changed(1, ("mixer", "rot", "dims"), 10), changed(1, ("mixer", "kv_rank"), None, drop=True), changed(1, ("mlp", "limit"), None, drop=True),
                changed(0, ("mlp", "router", "top"), 7), changed(0, ("mlp", "kind"), "sparse"), changed(0, ("mlp", "shared", "ff"), 0)):
        with pytest.raises(ConfigError):
            hb.MiroraxConfig.from_dict(bad)


def test_a_plan_that_adds_a_vector_the_model_does_not_have_is_refused():
    import dataclasses
    import hilbert_pruned_8b_b200 as hb
    from hilbert_pruned_8b_b200.config.spec import PlanEntry
    spec = hb.MiroraxConfig.from_dict(mt.MIXED).model_spec()
    for bad in (dataclasses.replace(spec, plan=[PlanEntry(0, adds=3)]), dataclasses.replace(spec, stream_vectors=None)):
        with pytest.raises(ValueError):
            bad.validate()


def test_plain_mechanisms_agree_with_their_definitions():
    g = torch.Generator().manual_seed(0)
    r = lambda *s: torch.randn(*s, generator=g, dtype=torch.float64)
    # windows: the token itself and the ones just in front of it
    m = visible(6, 3)
    assert m[5].tolist() == [False, False, False, True, True, True] and m[0].tolist() == [True] + [False] * 5
    assert torch.equal(visible(6, 1), torch.eye(6, dtype=torch.bool)) and torch.equal(visible(6), torch.tril(torch.ones(6, 6, dtype=torch.bool)))
    # a sink takes a share of the weights and brings no value; grouped heads read their own key/value head
    q, k, v, sink = r(6, 4, 3), r(6, 2, 3), r(6, 2, 5), r(4)
    out = softmax_attention(q, k, v, 0.7, visible(6, 3), sink)
    e = torch.stack([torch.exp(0.7 * q[5, 3] @ k[j, 1]) for j in (3, 4, 5)])
    want = sum(e[i] * v[j, 1] for i, j in enumerate((3, 4, 5))) / (e.sum() + torch.exp(sink[3]))
    assert torch.allclose(out[5, 3], want)
    assert torch.allclose(softmax_attention(q, k, v, 0.7, visible(6, 3), torch.full((4,), -1e9)), softmax_attention(q, k, v, 0.7, visible(6, 3)))
    # interleaved pairs; a score depends on the distance only
    t = r(1, 1, 6)
    got = rotate_pairs(t, torch.tensor([5]), 4, 100.0)[0, 0]
    for i, a in enumerate((5.0, 0.5)):
        assert torch.allclose(got[2 * i], t[0, 0, 2 * i] * math.cos(a) - t[0, 0, 2 * i + 1] * math.sin(a))
        assert torch.allclose(got[2 * i + 1], t[0, 0, 2 * i + 1] * math.cos(a) + t[0, 0, 2 * i] * math.sin(a))
    assert torch.equal(got[4:], t[0, 0, 4:])
    # the clamped unit: a gate is cut off above only, the other factor at both ends
    one = lambda x: torch.tensor([x], dtype=torch.float64)
    assert torch.allclose(clamped_unit(one(9.0), one(-9.0), 2.0), 2.0 * torch.sigmoid(one(3.404)) * (1.0 - 2.0))
    assert torch.allclose(clamped_unit(one(-9.0), one(0.5), 2.0), -9.0 * torch.sigmoid(one(-1.702 * 9)) * 1.5)
    # the router's bias counts for the choice and the weights, which are a softmax over the chosen alone
    h, wr, b = r(1, 5), r(4, 5), torch.tensor([0.0, 50.0, 0.0, 49.5], dtype=torch.float64)
    chosen, weights = route(h, wr, b, 2)
    z = wr @ h[0] + b
    assert set(chosen[0].tolist()) == {1, 3} and torch.allclose(weights.sum(), torch.tensor(1.0, dtype=torch.float64))
    assert torch.allclose(weights[0, 0] / weights[0, 1], torch.exp(z[chosen[0, 0]] - z[chosen[0, 1]]))
    w = {"router": wr, "router.b": b, **{f"{e}.{n}": r(*s) for e in ("e0", "e1", "e2", "e3", "shared") for n, s in (("gate", (3, 5)), ("up", (3, 5)), ("down", (5, 3)))}}
    unit = lambda e: w[e + ".down"] @ (silu(w[e + ".gate"] @ h[0]) * (w[e + ".up"] @ h[0]))
    want = unit("shared") + sum(weights[0, i] * unit(f"e{int(c)}") for i, c in enumerate(chosen[0]))
    assert torch.allclose(moe_ff(h, w, {"router": {"experts": 4, "top": 2}, "shared": {"ff": 3}})[0], want)
    # the order of the runs
    assert layer_runs(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, None, False)]
    assert layer_runs(2, None) == [(0, None, False), (1, None, False)]


# --------------------------------------------------------------------------- kernels and parts alone
@pytest.mark.gpu
def test_parallel_sum_with_every_term_present_and_absent():
    require_gpu()
    c = _context(torch.float32)
    ops, g = c.ops, torch.Generator().manual_seed(1)
    T = 17
    r = lambda *s: torch.randn(*s, generator=g).cuda()
    for width in (1, 3, 40, 64, 257, 1000, 2048, 2500, 4096, 6000, 9000):
        for n_sum, with_z, with_y, with_v, with_w in ((0, True, True, False, False), (0, False, True, True, False), (3, True, True, True, True),
                                                      (2, False, True, False, True), (4, True, False, False, False), (0, False, False, True, False)):
            x, y, z, rows = r(T, width), r(T, width) * 3, r(T, width), r(T * max(n_sum, 1), width) * 2
            a, b, v, nw, w = r(width), r(width), r(width) * 2, r(width), torch.rand(T, max(n_sum, 1), generator=g).cuda()
            second = n_sum > 0 or with_z
            fed = torch.zeros(T, width, dtype=torch.float64, device=DEV)
            if with_z:
                fed += z.double()
            if n_sum:
                weights = w.double() if with_w else torch.ones_like(w).double()
                fed += (rows.double().reshape(T, n_sum, width) * weights[:, :, None]).sum(1)
            want = parallel_sum(x.double(), y.double() if with_y else torch.zeros_like(y).double(), a.double(), fed if second else None, b.double())
            if with_v:
                want = want + v.double()
            kw = dict(y=y if with_y else None, a=a if with_y else None, z=z if with_z else None, entries=rows if n_sum else None, n_sum=n_sum,
                      entry_weights=w if n_sum and with_w else None, b=b if second else None, vector=v if with_v else None)
            bound = lambda got, ref: ((got.double() - ref).abs() / ref.abs().clamp(min=1.0)).max()
            x1 = x.clone()
            ops.parallel_sum(x1, **kw)
            assert bound(x1, want) < 3e-5, (width, n_sum)
            for dtype, tol in ((torch.float32, 5e-5), (torch.bfloat16, 1e-2)):
                x2, h = x.clone(), torch.empty(T, width, dtype=dtype, device=DEV)
                ops.parallel_sum(x2, then=(nw, 1e-4, 0.0), then_out=h, **kw)
                assert torch.equal(x1, x2) and bound(h, rms_norm(want, nw.double(), 1e-4)) < tol, (width, n_sum, dtype)
    ops.check_errors()


class _Step:
    pass


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_clamped_gated_unit(dtype):
    require_gpu()
    from hilbert_pruned_8b_b200.config.spec import PartSpec
    from hilbert_pruned_8b_b200.parts import FEED_FORWARDS
    g, rnd = torch.Generator().manual_seed(2), _rnd(dtype)
    for width, ff, limit, T in ((40, 1, 0.5, 3), (64, 72, 0.9, 5), (128, 130, 3.0, 70), (256, 512, 0.0, 300), (72, 24, 1e6, 1)):
        c = _context(dtype)
        part = FEED_FORWARDS.build(PartSpec("clamped_glu", {"hidden_size": width, "intermediate_size": ff, "limit": limit}), c)
        w = {p.name: (torch.randn(tuple(p.shape), generator=g) * 1.5 / p.shape[1] ** 0.5).to(torch.bfloat16).float() for p in part.params()}
        part.bind({k: v.to(dtype).to(DEV) for k, v in w.items()})
        h = torch.randn(T, width, generator=g).to(torch.bfloat16)
        want = dense_ff(h.double(), _double(w), {"limit": limit}, rnd)
        step = _Step()
        step.num_tokens = T
        out = torch.full((T, width), 2.0, device=DEV)
        part.forward(h.to(dtype).cuda(), out, step, accumulate=True)
        tol = (1e-5 if dtype == torch.float32 else 2e-2) * max(1.0, want.abs().max().item())
        assert (out.cpu().double() - 2.0 - want).abs().max() < tol, (width, ff, limit)
        part.forward(h.to(dtype).cuda(), out, step, accumulate=False)
        assert (out.cpu().double() - want).abs().max() < tol
        c.ops.check_errors()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_biased_router_with_silu_experts_and_a_shared_expert(dtype):
    require_gpu()
    from hilbert_pruned_8b_b200.config.spec import PartSpec
    from hilbert_pruned_8b_b200.parts import FEED_FORWARDS
    g, rnd = torch.Generator().manual_seed(3), _rnd(dtype)
    for n, (width, E, top, ff, shared, T) in enumerate(((24, 3, 2, 10, 7, 1), (64, 6, 2, 32, 64, 5), (64, 5, 1, 24, 0, 333), (40, 1, 1, 8, 8, 70),
                                                        (128, 40, 6, 64, 192, 90), (56, 4, 4, 40, 20, 33), (264, 4, 2, 200, 64, 700),
                                                        (72, 8, 2, 40, 24, 31), (64, 16, 4, 72, 64, 31))):       # (small tiles, and experts with more rows than one holds)
        for tc in ("tcgen05", "mma.sync", None):          # the products' three kernels (where the step has rows enough and bfloat16 for them)
            c = _context(dtype, cap=1024)
            c.ops.use_tensor_cores, c.ops.use_tcgen05_experts = tc is not None, tc == "tcgen05"
            c.ops.call_log = []
            part = FEED_FORWARDS.build(PartSpec("moe", {"hidden_size": width, "num_experts": E, "top": top, "expert_size": ff, "shared_size": shared,
                                                        "router": "top_logits", "router_bias": True, "unit": "silu_glu"}), c)
            w = {p.name: (torch.randn(tuple(p.shape), generator=g) * (2.0 if len(p.shape) == 1 else 2.0 / p.shape[-1] ** 0.5)).to(torch.bfloat16).float()
                 for p in part.params()}
            part.bind({k: (v.to(dtype) if v.dim() == 2 else v).to(DEV) for k, v in w.items()})
            h = (torch.randn(T, width, generator=g) * 1.5).to(torch.bfloat16)
            if T == 31:
                w["router.b"][:2] += 12.0                  # every token's choice: 31 rows for an expert
                part.bind({k: (v.to(dtype) if v.dim() == 2 else v).to(DEV) for k, v in w.items()})
            cfg = {"router": {"experts": E, "top": top}, "shared": {"ff": shared} if shared else None}
            want = moe_ff(h.double(), _double(w), cfg, rnd)
            if top < E and T > 1:                          # the bias does decide
                assert (moe_ff(h.double(), {**_double(w), "router.b": torch.zeros(E).double()}, cfg, rnd) - want).abs().max() > 0.05
            step = _Step()
            step.num_tokens = T
            tol = (1e-5 if dtype == torch.float32 else 2e-2) * max(1.0, want.abs().max().item())
            out = torch.full((T, width), 2.0, device=DEV)
            part.forward(h.to(dtype).cuda(), out, step, accumulate=True)
            assert (out.cpu().double() - 2.0 - want).abs().max() < tol, (n, tc)
            part.forward(h.to(dtype).cuda(), out, step, accumulate=False)
            assert (out.cpu().double() - want).abs().max() < tol, (n, tc)
            rows, k, weights, base = part.forward_weighted(h.to(dtype).cuda(), step)
            assert k == top and part.weighs_entries and (base is None) == (shared == 0)
            total = (rows.cpu().double().reshape(T, top, width) * weights.cpu().double()[:, :, None]).sum(1)
            assert (total + (0 if base is None else base.cpu().double()) - want).abs().max() < tol, (n, tc)
            assert ("hb_moe_tc" in c.ops.call_log) == (tc == "tcgen05" and dtype == torch.bfloat16 and width % 8 == 0 and ff % 8 == 0)
            c.ops.check_errors()


# --------------------------------------------------------------------------- mixers alone
def _mixer_spec(layer, width):
    import hilbert_pruned_8b_b200 as hb
    return hb.MiroraxConfig.from_dict(mt.config(width, 16, [mt.with_mlp(layer, None)])).model_spec().layers[0].parts["mixer"]


def _close(got, want, dtype, what):
    for i, (a, b) in enumerate(zip(got, want)):
        err = (a - b).abs().max(1).values / b.abs().max().clamp(min=1.0)
        assert err.max() < (1e-4 if dtype == torch.float32 else 3e-2), f"{what}: sequence {i} position {int(err.argmax())}: {float(err.max()):.3e}"


def _eye(rows, width, at):
    m = torch.zeros(rows, width)
    m[torch.arange(rows), at + torch.arange(rows)] = 1.0
    return m


PORTIONS = ((300,), (60, 3, 1, 1, 1, 1, 1, 1, 1, 58, 1, 1, 1, 1, 1, 1, 1, 300), (2, 126, 1, 1, 300))
# the kernels of a step, one after the other taken away, so that each of them meets every case
KERNELS = ("use_tcgen05_sink_attention", "use_group_attention", "use_mma_attention", "use_flash_sink_attention")

# (heads, kv heads, dim, vdim): one head, odd sizes (the general kernel), groups of one, some and more query heads than one tile of rows
# holds, sizes the tcgen05 prompt kernel pads and does not pad, sizes of keys and values that differ both ways, sizes it does not take
ATTENTIONS = [(1, 1, 8, 8), (3, 1, 5, 7), (4, 2, 16, 24), (2, 2, 64, 64), (6, 3, 40, 32), (20, 1, 24, 48), (33, 1, 16, 8), (4, 1, 128, 104), (2, 1, 136, 64),
              (2, 2, 192, 128), (2, 1, 200, 16), (1, 1, 24, 136), (16, 4, 64, 64)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_attention_without_positions_and_with_a_gate_per_element(dtype):
    require_gpu()
    rnd = _rnd(dtype)
    for n, (H, G, d, dv) in enumerate(ATTENTIONS):
        width, g = H * d + G * d, torch.Generator().manual_seed(20 + n)
        layer = mt.attention(H, G, d, dv, scale=1.0 / d ** 0.5)
        spec = _mixer_spec(layer, width)
        # q and k are cut out of the input, so that a probe can be written into it: a query and a key far back in one direction
        # give a score that stands out among hundreds
        w = {"q": _eye(H * d, width, 0), "k": _eye(G * d, width, H * d), "v": torch.randn(G * dv, width, generator=g) / width ** 0.5,
             "g": torch.randn(H * dv, width, generator=g) * 2 / width ** 0.5, "o": torch.randn(width, H * dv, generator=g) / (H * dv) ** 0.5,
             "q.b": torch.randn(H * d, generator=g) * 0.2, "k.b": torch.randn(G * d, generator=g) * 0.2, "v.b": torch.randn(G * dv, generator=g),
             "o.b": torch.randn(width, generator=g)}
        w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
        hs = [torch.randn(t, width, generator=g) for t in (200, 77, 1)]
        for i, (p, s) in enumerate(((5, 0), (63, 1), (64, 0), (65, 63), (127, 64), (128, 127), (130, 2), (150, 66), (199, 4))):
            head = i % H
            direction = torch.randn(d, generator=g)
            direction *= (14.0 * d ** 0.5) ** 0.5 / direction.norm()      # a score of 14 where the others' spread is about one
            hs[0][p, head * d: (head + 1) * d] = direction
            at = H * d + head // (H // G) * d
            hs[0][s, at: at + d] = direction
        hs = [h.to(torch.bfloat16).float() for h in hs]
        want = [attention_mixer(h.double(), _double(w), layer["mixer"], rnd) for h in hs]
        c = _context(dtype)
        what = f"attention {(H, G, d, dv)}"
        for sizes in PORTIONS:
            run = _MixerRun(c, spec, w)
            _close(run.feed(hs, sizes), want, dtype, f"{what} portions {sizes}")
            _close(run.feed(hs, (150, 1, 1, 300)), want, dtype, f"{what}, pages used again")
        for flag in KERNELS:
            setattr(c.ops, flag, False)
            _close(_MixerRun(c, spec, w).feed(hs, (150, 1, 1, 300)), want, dtype, f"{what} without {flag}")
        run = _MixerRun(c, spec, w)
        run.mixer.use_heads_kernel = False
        _close(run.feed(hs, (150, 1, 1, 300)), want, dtype, f"{what}, the general kernel")
        if dtype == torch.float32 and d >= 16:
            # the probes do stand out: without the probed key, 195 tokens back, the result is another
            blind = hs[0].clone()
            blind[4, H * d:] = 0
            assert (attention_mixer(blind.double(), _double(w), layer["mixer"])[199] - want[0][199]).abs().max() > 0.01 * want[0].abs().max()


# (heads, dim, rot_dim, rotated dims, vdim, kv_rank, window)
LATENTS = [(4, 16, 8, 8, 12, 40, 30), (1, 8, 2, 2, 5, 9, 1), (3, 3, 4, 2, 3, 8, 64), (2, 8, 0, 0, 8, 16, 2), (16, 32, 32, 32, 64, 64, 65), (4, 96, 32, 32, 96, 64, 127),
           (20, 24, 8, 8, 72, 64, 128), (2, 128, 64, 64, 128, 192, 63), (33, 8, 8, 4, 8, 32, 100), (6, 40, 24, 24, 20, 56, 1000), (2, 136, 64, 32, 128, 256, 70),
           (4, 128, 64, 64, 128, 512, 130)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_attention_with_probes_at_the_window_s_edge_and_a_sink(dtype):
    require_gpu()
    rnd = _rnd(dtype)
    for n, (H, d, dr, rotated, dv, rank, window) in enumerate(LATENTS):
        # the latent is cut out of the input, and the queries come from another part of it through the keys' own matrix: a query
        # that holds a latent's direction looks for that latent
        width, g = 2 * rank + dr, torch.Generator().manual_seed(70 + n)
        layer = mt.latent(H, d, dr, dv, rank, window, base=30.0, scale=6.0 / (d + dr) ** 0.5, rotated=rotated)
        spec = _mixer_spec(layer, width)
        uk = (torch.randn(H, d, rank, generator=g) / rank ** 0.5).to(torch.bfloat16).float()
        q = torch.zeros(H, d + dr, width)
        q[:, :d, :rank] = uk
        q[:, d:, :rank] = torch.randn(H, dr, rank, generator=g) * 0.3 / rank ** 0.5
        w = {"q": q.reshape(H * (d + dr), width), "dkv": _eye(rank + dr, width, rank), "dkv.norm": torch.ones(rank), "uk": uk.reshape(H * d, rank),
             "uv": torch.randn(H * dv, rank, generator=g) / rank ** 0.5, "sink": torch.randn(H, generator=g) * 2 + 1,
             "o": torch.randn(width, H * dv, generator=g) / (H * dv) ** 0.5}
        w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
        hs = [torch.randn(t, width, generator=g) for t in (200, 77, 1)]
        # keys just inside and just outside the window, next to one another, at page borders and at the sequence's start
        probes = []
        for p in (5, 62, 63, 64, 65, 127, 128, 130, 150, 191, 192, 199):
            probes += [(p, s) for s in (p - window + 1, p - window, p - 1, 0) if 0 <= s < p]
        taken = set()
        for p, s in probes[n % 4::2]:
            if p in taken or s in taken:
                continue
            taken |= {p, s}
            direction = torch.randn(rank, generator=g)
            hs[0][p, :rank] = direction
            hs[0][s, rank: 2 * rank] = direction
        hs = [h.to(torch.bfloat16).float() for h in hs]
        cfg = layer["mixer"]
        want = [latent_mixer(h.double(), _double(w), cfg, 1e-5, torch.arange(h.shape[0]), rnd) for h in hs]
        c = _context(dtype)
        what = f"latent attention {(H, d, dr, dv, rank, window)}"
        for sizes in PORTIONS:
            for write_out in ((True, False) if dtype == torch.bfloat16 else (True,)):
                run = _MixerRun(c, spec, w)
                run.mixer.write_out = write_out
                _close(run.feed(hs, sizes), want, dtype, f"{what} portions {sizes} written out {write_out}")
                _close(run.feed(hs, (150, 1, 1, 300)), want, dtype, f"{what}, pages used again")
        for flag in KERNELS:
            setattr(c.ops, flag, False)
            _close(_MixerRun(c, spec, w).feed(hs, (150, 1, 1, 300)), want, dtype, f"{what} without {flag}")
        if dtype == torch.float32 and d >= 12:
            # a window one token longer or shorter and a sink left out are seen
            other = lambda **kw: latent_mixer(hs[0].double(), _double({**w, **kw.pop("w", {})}), {**cfg, **kw}, 1e-5, torch.arange(200))
            scale = want[0].abs().max()
            assert (other(w={"sink": torch.full((H,), -50.0)}) - want[0]).abs().max() > 0.05 * scale
            if window < 150:
                for size in (window - 1, window + 1):
                    assert (other(mask={"size": size}) - want[0]).abs().max() > 0.02 * scale, (what, size)


@pytest.mark.gpu
def test_a_sink_that_takes_nearly_everything_and_one_that_takes_nothing():
    require_gpu()
    layer = mt.latent(4, 64, 32, 64, 64, 70)
    spec, width, g = _mixer_spec(layer, 96), 96, torch.Generator().manual_seed(5)
    from hilbert_pruned_8b_b200.engine.model import describe_context
    from hilbert_pruned_8b_b200.parts import MIXERS
    w = {p.name: mt.draw(p.name, tuple(p.shape), g).to(torch.bfloat16).float() for p in MIXERS.build(spec, describe_context()).params()}
    w["sink"] = torch.tensor([60.0, -60.0, 8.0, 0.0])
    w["o"] = w["o"] * 4
    hs = [torch.randn(150, width, generator=g).to(torch.bfloat16).float()]
    for dtype in (torch.float32, torch.bfloat16):
        want = [latent_mixer(hs[0].double(), _double(w), layer["mixer"], 1e-5, torch.arange(150), _rnd(dtype))]
        for sizes in ((200,), (100, 1, 1, 1, 200), (10, 5, 200)):
            _close(_MixerRun(_context(dtype), spec, w).feed(hs, sizes), want, dtype, f"sinks, portions {sizes}")


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
    # pages behind a window go back while a sequence is still decoded
    seq = eng.open_sequence()
    from hilbert_pruned_8b_b200.engine.batch import StepEntry
    eng.step_chunked([StepEntry(seq, requests["r0"][:300], [])])
    eng.step_chunked([StepEntry(seq, [1], [])])
    for gi, group in enumerate(eng.cache.groups):
        held, reach = sum(p is not None for p in seq.pages[gi]), group.need.window
        assert held == 5 if reach is None else held <= (reach + 63) // 64 + 1, (held, reach)
    eng.close_sequence(seq)
    # every norm, every pass's vector and every expert's sum a kernel of its own
    plainer = _engine(folder, "float32", 64 * 8)
    for b in plainer.model.blocks:
        assert b.adds_vector
        b.fuse_norms = b.fuse_entries = False
        assert not b.adds_vector
    steps, _ = tt.trace_tail(requests, tail=4)
    _check(plainer, steps, plain, requests, "float32", f"{name} separate steps")
    # and the decoded tokens of a bfloat16 engine through captured graphs are those of its eager steps
    fast, eager = _engine(folder, "bfloat16", 64 * 8), _engine(folder, "bfloat16", 64 * 8)
    eager.use_graphs = False
    steps, _ = tt.trace_tail(requests, tail=60)
    a, b = tt.run_in_process(fast, steps), tt.run_in_process(eager, steps)
    assert fast.graph_replays > 40 and eager.graph_replays == 0
    # (the key ranges of an attention differ, so two nearly tied experts may be chosen either way at a few tokens)
    apart = sorted(((a[k] - b[k]).abs().max() / b[k].abs().max()).item() for k in b)
    assert apart[len(apart) // 2] <= 0.01 and apart[(9 * len(apart)) // 10] <= 0.05


@pytest.mark.gpu
def test_rewinding_a_sequence_inside_a_window(models):
    require_gpu()
    from hilbert_pruned_8b_b200.engine.batch import StepEntry
    folder, cfg, plain = models["mixed"]
    eng = _engine(folder, "float32", 64 * 8)
    a, b, c = tt.random_tokens(70, cfg["vocab"], 1), tt.random_tokens(9, cfg["vocab"], 2), tt.random_tokens(6, cfg["vocab"], 3)
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
