"""Mezadra on the CPU: the configuration reader and the model specification, what its layers ask of the cache manager, and the plain
implementation (tests/plain_mezadra.py) against cases small enough to be written out by hand."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_mezadra as plain
from mezadra_cases import MEZADRA, drawn, load_plain, near_uniform, write_model

F = torch.float64


def _model(cfg, **env):
    from stride_b200.config import resolve_architecture
    from stride_b200.parts import BuildEnv, DecoderModel
    arch = resolve_architecture(cfg)
    return DecoderModel(arch.model_spec(arch.parse_config(cfg)),
                        BuildEnv(device=torch.device("cpu"), compute_dtype=torch.float32, max_tokens=8, max_positions=64, **env))


def test_configurations_parse_and_plan_their_tensors():
    from stride_b200.config import ConfigError, resolve_architecture
    from stride_b200.weights.random_init import model_plan
    for cfg in [c for c, _, _ in MEZADRA.values()] + [drawn(s) for s in range(20)]:
        arch = resolve_architecture(cfg)
        assert arch.name == "Mezadra"
        spec = arch.model_spec(arch.parse_config(cfg))
        assert len(spec.schedule) == len(spec.layers) == len(cfg["layers"])
        plan, W = model_plan(cfg), cfg["width"]
        assert plan["head"].shape == plan["embed"].shape == (cfg["vocab"], W) and plan["final.norm"].shape == (W,)
        mixing = []
        for i, l in enumerate(cfg["layers"]):
            p, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
            assert plan[p + "norm1"].shape == (W,) and (p + "norm2" in plan) == (mlp is not None)
            assert plan[p + "mix.q"].shape == (m["heads"] * m["dim"], W) and plan[p + "mix.o"].shape == (W, m["heads"] * m["vdim"])
            if l["type"] == "lightning":
                assert plan[p + "mix.k"].shape == (m["heads"] * m["dim"], W) and plan[p + "mix.norm"].shape == (m["heads"] * m["vdim"],)
                assert plan[p + "mix.g"].shape == plan[p + "mix.v"].shape == (m["heads"] * m["vdim"], W)
            else:
                taps = m.get("conv", 0)
                assert all((f"{p}mix.{r}.conv" in plan) == (taps > 0) for r in "qkv") and plan[p + "mix.sink"].shape == (m["heads"],)
                if taps:
                    assert plan[p + "mix.v.conv"].shape == (m["kv_heads"] * m["vdim"], taps)
                assert (p + "mix.vmix" in plan) == bool(m.get("v_mix"))
                if m.get("v_mix"):
                    assert plan[p + "mix.vmix"].shape == ()
                    mixing.append(spec.layers[i].mixer.params["value_mix"])
            if mlp and mlp["kind"] == "moe":
                assert plan[p + "mlp.router"].shape == (mlp["router"]["experts"], W)
                assert (p + "mlp.shared.sg" in plan) == (p + "mlp.shared.down" in plan) == ("shared" in mlp)
                assert f"{p}mlp.e{mlp['router']['experts'] - 1}.up" in plan and f"{p}mlp.e{mlp['router']['experts']}.up" not in plan
        assert mixing == ["keep", "mix", "mix", "mix", "mix", "mix"][:len(mixing)]
    base = MEZADRA["M"][0]

    def refused(edit, match):
        bad = copy.deepcopy(base)
        edit(bad)
        with pytest.raises(ConfigError, match=match):
            resolve_architecture(bad).parse_config(bad)

    refused(lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads")
    refused(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=11), "rot.dims")
    refused(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=24), "rot.dims")
    refused(lambda c: c["layers"][3]["mixer"].update(vdim=11), "v_mix")
    refused(lambda c: c["layers"][1]["mixer"]["decay"].pop(), "decay")
    refused(lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "router")
    refused(lambda c: c["layers"][1]["mlp"].pop("limit"), "limit")
    refused(lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse")
    refused(lambda c: c["layers"][1].update(type="retention"), "retention")
    refused(lambda c: c["layers"][2]["mixer"].pop("scale"), "scale")
    refused(lambda c: c.pop("width"), "width")


def test_what_the_layers_ask_of_the_cache_manager():
    """Pages and, behind a convolution of more than one tap, a record of the last taps - 1 inputs, in 32-bit."""
    from stride_b200.cache.manager import CacheManager
    needs = _model(MEZADRA["M"][0]).cache_needs()
    pages, record = needs[0]
    assert (pages.kind, pages.kv_heads, pages.head_dim, pages.window) == ("pages", 2, 27, 0)
    assert record.kind == "state" and record.state_shape == (2 * (4 * 22 + 2 * (22 + 27)),) and record.state_dtype == torch.float32
    assert needs[1].kind == "state" and needs[1].state_shape == (3, 20, 37)
    plain_needs = _model(MEZADRA["O"][0]).cache_needs()
    assert plain_needs[0].kind == plain_needs[1].kind == "pages"        # no convolution, and one of a single tap
    pool = CacheManager(needs, device="cpu", max_slots=2, max_context=64, page_size=16, num_pages=4)
    cache = pool.layer_cache(0)
    assert cache.parts[0].pages.shape[1:] == (2, 2, 16, 27) and cache.parts[1].state.shape == (3, record.state_shape[0])


def test_a_plan_made_for_one_step_is_the_native_plan():
    """How a step's entries are cut for the tensor-core attention: the context's own cut and the native program's agree."""
    import numpy as np
    from stride_b200.kernels.native import StepProgram
    from stride_b200.parts import Workspace
    from stride_b200.parts.context import step_context
    R = 512
    ws = Workspace("cpu", R)
    program = StepProgram(ws, R, 4 * R + 64, 512)
    entries = [(0, 200, 37), (1, 1, 300), (2, 2, 0), (3, 31, 5), (4, 4, 1000)]
    staging = np.zeros(13 * R + 64, dtype=np.int32)
    i32 = lambda v: np.ascontiguousarray(v, dtype=np.int32).ctypes.data_as(__import__("ctypes").POINTER(__import__("ctypes").c_int32))
    for group, rows in ((4, 128), (1, 64), (16, 128), (3, 64)):
        k = program.plan(group, rows, 1, -1)
        count, first = np.array([e[1] for e in entries], dtype=np.int32), np.array([e[2] for e in entries], dtype=np.int32)
        program.prepare(len(entries), i32(count), i32(first), int(count.sum()), 0, 0, i32(staging), torch.from_numpy(staging))
        q = program.step.plan[k]
        work, tiles, items, chunks = step_context(entries, ws, torch.bfloat16, rows=R).tile_plan(group, rows)
        assert (q.tiles, q.items, q.chunks, q.fused) == (tiles, items, chunks, 0) and not q.list


# ---------------------------------------------------------------------------------------------- the plain implementation by hand
def test_convolution_and_rotation_by_hand():
    u = torch.tensor([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]], dtype=F)
    taps = torch.tensor([[4.0, 5.0, 1.0], [0.0, 0.0, 2.0]], dtype=F)
    assert plain.short_conv(u, taps).tolist() == [[1.0, 20.0], [2.0 + 5.0, 40.0], [3.0 + 10.0 + 4.0, 60.0]]
    assert torch.equal(plain.short_conv(u, torch.ones(2, 1, dtype=F)), u)
    x = torch.tensor([[[1.0, 5.0, 2.0, 7.0, 9.0]]], dtype=F)                   # one token, one head of five; four are turned: (1, 2) and (5, 7)
    y = plain.rotated(x, 100.0, 4, first=3)[0, 0]
    c, s = math.cos(3.0), math.sin(3.0)
    c1, s1 = math.cos(0.3), math.sin(0.3)                                      # 100^(-2/4) = 1/10
    assert torch.allclose(y, torch.tensor([c - 2 * s, 5 * c1 - 7 * s1, 2 * c + s, 7 * c1 + 5 * s1, 9.0], dtype=F))


def test_softmax_norm_cap_by_hand():
    w = plain.sink_softmax(torch.log(torch.tensor([[1.0, 7.0], [2.0, 3.0]], dtype=F)), torch.tensor(math.log(5.0), dtype=F))
    assert torch.allclose(w, torch.tensor([[1 / 6, 0.0], [2 / 10, 3 / 10]], dtype=F))
    assert torch.allclose(plain.unit_rms(torch.tensor([[3.0, 4.0]], dtype=F), 12.5), torch.tensor([[3.0 / 5, 4.0 / 5]], dtype=F))
    x = torch.tensor([2.0, -100.0], dtype=F)
    assert torch.allclose(plain.capped(x, 4.0), torch.tensor([4 * math.tanh(0.5), -4.0], dtype=F)) and plain.capped(x, 0) is x


def test_attention_by_hand():
    """One head of two elements, the second always 0: q and k become (+-sqrt 2, 0), scores +-2 scale; values mixed with given ones."""
    t = {"p.q": torch.tensor([[1.0], [0.0]]), "p.k": torch.tensor([[3.0], [0.0]]), "p.v": torch.tensor([[5.0]]), "p.o": torch.tensor([[10.0]]),
         "p.sink": torch.tensor([0.0]), "p.vmix": torch.tensor(0.25)}
    h = torch.tensor([[1.0], [-1.0]], dtype=F)
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "vdim": 1, "scale": 0.5, "softcap": 2.0}
    y, own = plain.attention(h, t, "p.", m, 0.0, first_values=torch.tensor([[9.0], [1.0]], dtype=F))
    assert own.tolist() == [[5.0], [-5.0]]
    v = [0.75 * 5 + 0.25 * 9, 0.75 * -5 + 0.25 * 1]
    e = math.exp(2 * math.tanh(0.5))                                            # score +1 capped at 2
    want = [10 * v[0] * e / (e + 1), 10 * (v[0] / e + v[1] * e) / (1 / e + e + 1)]
    assert torch.allclose(y.flatten(), torch.tensor(want, dtype=F))
    y, _ = plain.attention(h, t, "p.", m, 0.0)
    assert torch.allclose(y.flatten()[0], torch.tensor(10 * 5 * e / (e + 1), dtype=F))


def test_recurrence_by_hand():
    q, k, v = (torch.tensor(x, dtype=F) for x in ([[[1.0, 0.0]], [[1.0, 2.0]]], [[[2.0, 3.0]], [[1.0, 0.0]]], [[[10.0]], [[1.0]]]))
    o = plain.linear_recurrence(q, k, v, torch.tensor([0.5], dtype=F))
    assert o.flatten().tolist() == [20.0, (0.5 * 20 + 1) + 2 * (0.5 * 30)]


def test_feed_forwards_by_hand():
    one = torch.ones(1, 1)
    t = {"p.gate": one * 3.0, "p.up": one * -5.0, "p.down": one * 2.0}
    y = plain.clamped_gated(torch.tensor([[1.0], [-0.1]], dtype=F), t, "p.", 1.5)
    sig = lambda z: 1 / (1 + math.exp(-z))
    assert torch.allclose(y.flatten(), torch.tensor([2 * 1.5 * sig(1.702 * 1.5) * (-1.5 + 1), 2 * -0.3 * sig(1.702 * -0.3) * (0.5 + 1)], dtype=F))
    y = plain.clamped_gated(torch.tensor([[-10.0]], dtype=F), t, "p.", 1.5)      # the gate has no lower limit, `up` has both
    assert torch.allclose(y.flatten(), torch.tensor([2 * -30.0 * sig(1.702 * -30.0) * 2.5], dtype=F))
    t = {"p.router": torch.tensor([[1.0], [-1.0], [2.0]])}
    for e, s in enumerate((1.0, 3.0, 7.0)):
        t.update({f"p.e{e}.gate": one, f"p.e{e}.up": one, f"p.e{e}.down": one * s})
    t.update({"p.shared.gate": one, "p.shared.up": one, "p.shared.down": one * 100, "p.shared.sg": one * 0.5})
    h = torch.tensor([[1.0], [-2.0]], dtype=F)
    chosen = plain.route(h, t, "p.", 2)
    assert [[e for e, _ in row] for row in chosen] == [[2, 0], [1, 0]] and math.isclose(chosen[1][0][1], sig(2.0))
    y = plain.experts(h, t, "p.", {"router": {"experts": 3, "top": 2}, "shared": {"ff": 1}})
    f = lambda x: x * sig(x) * x                                                # an expert of size 1 with unit matrices
    want = [7 * f(sig(2.0)) + f(sig(1.0)) + 100 * f(1.0) * sig(0.5),
            3 * f(-2 * sig(2.0)) + f(-2 * sig(-2.0)) + 100 * f(-2.0) * sig(-1.0)]
    assert torch.allclose(y.flatten(), torch.tensor(want, dtype=F))


def test_every_part_of_the_design_moves_the_plain_logits(tmp_path):
    """Faults planted in the plain implementation's inputs: each moves the logits far beyond what the engine is held to, so the tests
    on the GPU would notice the same fault there."""
    from conftest import logit_tolerance, random_tokens
    folder = write_model(tmp_path / "u", "M", config=near_uniform(MEZADRA["M"][0]))
    cfg, w = load_plain(folder)
    toks = random_tokens(cfg["vocab"], 60, 5)
    want = plain.run(cfg, w, toks).float()
    tol = logit_tolerance("float32", want)

    def moved(edit_cfg=None, edit_w=None, tokens=toks, of=slice(45, None), config=None, weights=None, ref=None):
        c, t = copy.deepcopy(config or cfg), dict(weights or w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(t)
        got = plain.run(c, t, tokens).float()
        return float((got - (want if ref is None else ref)).abs().max(dim=1).values[of].min())

    def scaled(name, factor):
        return lambda t: t.update({name: (t[name].float() * factor).to(t[name].dtype)})

    for i in (0, 2, 3, 5):                                                       # the attention layers
        p = f"l{i}.mix."
        assert moved(edit_w=lambda t: t.update({p + "sink": torch.full_like(t[p + "sink"], -60.0)})) > 10 * tol
        for r in "qkv":
            assert moved(edit_w=lambda t: t.update({f"{p}{r}.conv": t[f"{p}{r}.conv"].flip(1)})) > 4 * tol, (i, r)
    for i in (3, 5):
        assert moved(edit_w=lambda t: t.update({f"l{i}.mix.vmix": torch.zeros((), dtype=torch.bfloat16)})) > 10 * tol
        assert moved(lambda c: c["layers"][i]["mixer"].update(v_mix=False)) > 10 * tol
    assert moved(edit_w=lambda t: t.update({"l2.mix.vmix": t["l2.mix.vmix"] * 0})) == 0      # the first one only keeps
    assert moved(lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.9, 0.975])) > 10 * tol
    assert moved(edit_w=scaled("l1.mix.g", 0.0)) > 10 * tol
    assert moved(lambda c: c["layers"][1]["mlp"].update(limit=0.8)) > 10 * tol
    assert moved(edit_w=lambda t: t.update({"l0.mlp.router": t["l0.mlp.router"].roll(1, 0)})) > 10 * tol
    assert moved(edit_w=scaled("l0.mlp.shared.sg", 0.0)) > 10 * tol
    assert moved(edit_w=scaled("l0.norm1", 1.1)) > 10 * tol
    assert moved(lambda c: c["embedding"].update(scale=2.6)) > 10 * tol
    assert moved(lambda c: c["norm"].update(eps=3e-2)) > 10 * tol
    other = list(toks)
    other[0] = (other[0] + 1) % cfg["vocab"]                                     # attention close to uniform: the first key is never forgotten
    assert moved(tokens=other) > 10 * tol
    sharp = MEZADRA["M"][0]                                                      # what only shows where scores differ: the cap and the angles
    ref = plain.run(sharp, w, toks).float()
    tol = logit_tolerance("float32", ref)
    for i in (0, 2, 5):
        assert moved(lambda c: c["layers"][i]["mixer"].update(softcap=0.0), config=sharp, ref=ref) > 5 * tol
    for i in (0, 2, 3):
        assert moved(lambda c: c["layers"][i]["mixer"]["rot"].update(base=600.0), config=sharp, ref=ref) > 5 * tol
