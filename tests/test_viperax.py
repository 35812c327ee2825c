"""Viperax on the CPU: the configuration reader and the model specification, the windows of caches that several layers read, random
tables, and the plain implementation (tests/plain_viperax.py) against cases small enough to be written out by hand."""
from __future__ import annotations

import copy
import math

import pytest
import torch

import plain_viperax as plain
from viperax_cases import VIPERAX, drawn, load_plain, near_uniform, write_model

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
    for cfg in [c for c, _, _ in VIPERAX.values()] + [drawn(s) for s in range(20)]:
        arch = resolve_architecture(cfg)
        assert arch.name == "Viperax"
        spec = arch.model_spec(arch.parse_config(cfg))
        assert len(spec.schedule) == len(spec.layers) == len(cfg["layers"])
        assert [e.cache_of for e in spec.schedule] == [l["mixer"].get("kv_from") for l in cfg["layers"]]
        plan, W, S = model_plan(cfg), cfg["width"], cfg["streams"]
        assert plan["head"].shape == plan["embed"].shape == (cfg["vocab"], W) and plan["final.norm"].shape == (W,)
        for i, l in enumerate(cfg["layers"]):
            p, m, mlp = f"l{i}.", l["mixer"], l["mlp"]
            own = m.get("kv_from") is None
            assert (p + "mix.dkv" in plan) == (p + "mix.dkv.norm" in plan) == own
            assert plan[p + "mix.uk"].shape == (m["heads"] * m["dim"], m["kv_rank"]) and plan[p + "mix.sink"].shape == (m["heads"],)
            assert plan[p + "mix.g"].shape == (m["heads"] * m["vdim"], W) and plan[p + "hc1.mix"].shape == (S, S)
            assert (p + "norm2" in plan) == (p + "hc2.out" in plan) == (mlp is not None)
            if mlp and mlp["kind"] == "moe":
                assert plan[p + "mlp.table"].shape == (cfg["vocab"], mlp["router"]["top"]) and plan[p + "mlp.table"].integer
                assert (p + "mlp.shared.down" in plan) == ("shared" in mlp)
                assert f"{p}mlp.e{mlp['router']['experts'] - 1}.up" in plan and f"{p}mlp.e{mlp['router']['experts']}.up" not in plan
    base = VIPERAX["X"][0]

    def refused(edit, match):
        bad = copy.deepcopy(base)
        edit(bad)
        with pytest.raises(ConfigError, match=match):
            resolve_architecture(bad).parse_config(bad)

    refused(lambda c: c["layers"][1]["mixer"].update(kv_from=1), "kv_from")
    refused(lambda c: c["layers"][3]["mixer"].update(kv_from=1), "kv_from")          # layer 1 stores no latents itself
    refused(lambda c: c["layers"][1]["mixer"].update(kv_rank=45), "kv_from")
    refused(lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "router")
    refused(lambda c: c["layers"][0]["mlp"].update(kind="sparse"), "sparse")
    refused(lambda c: c["layers"][2].update(type="attention"), "attention")
    refused(lambda c: c.pop("streams"), "streams")
    refused(lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank")


def test_a_cache_that_others_read_keeps_their_longest_window():
    """The pages of a layer stay while any of its readers still sees a token of them."""
    from stride_b200.cache.manager import CacheManager
    x = _model(VIPERAX["X"][0]).cache_needs()
    assert x[0].window == 29 and x[1] == ("shared", 0) and x[2].window == 40 and x[3] == ("shared", 0)
    y = _model(VIPERAX["Y"][0]).cache_needs()
    assert y[0].window == 0 and y[1].window == 0                   # one of the two sees everything
    z = _model(VIPERAX["Z"][0]).cache_needs()
    assert z[0].window == 64
    pool = CacheManager(x, device="cpu", max_slots=1, max_context=96, page_size=8, num_pages=12)
    slot = pool.acquire_slot()
    pool.ensure(slot, 64)
    pool.trim(slot)
    held = {g.window: set(g.held[slot]) for g in pool.groups}
    assert held[29] == {4, 5, 6, 7}                                # positions 64 - 28 = 36 and on: pages 4 to 7
    assert held[40] == {3, 4, 5, 6, 7}


def test_random_tables_name_different_experts_of_their_range():
    from stride_b200.weights.random_init import random_tensors
    for cfg, seed, _ in VIPERAX.values():
        t = random_tensors(cfg, seed)
        for i, l in enumerate(cfg["layers"]):
            if l["mlp"] and l["mlp"]["kind"] == "moe":
                table, r = t[f"l{i}.mlp.table"], l["mlp"]["router"]
                assert table.dtype == torch.int32 and int(table.min()) >= 0 and int(table.max()) < r["experts"]
                assert all(len(set(row)) == r["top"] for row in table.tolist())
                assert len(set(table.flatten().tolist())) == r["experts"]
            mix = t[f"l{i}.hc1.mix"].float()
            assert (mix - torch.eye(cfg["streams"])).abs().mean() < 0.5


def test_table_experts_refuse_a_table_that_names_what_is_not_there():
    from stride_b200.parts import BuildEnv, PartSpec, part_class
    t = {"table": "t", "gate": ("g",), "up": ("u",), "down": ("d",)}
    part = part_class("feed_forward", "table_experts")(PartSpec("table_experts", {"hidden_size": 4, "vocab_size": 3, "intermediate_size": 2, "experts": 1,
                                                                                  "top": 1}, t),
                                                       BuildEnv(torch.device("cpu"), torch.float32, 4, 8))
    tensors = {"t": torch.tensor([[0], [1], [0]], dtype=torch.int32), "g": torch.zeros(2, 4), "u": torch.zeros(2, 4), "d": torch.zeros(4, 2)}
    with pytest.raises(ValueError, match="names experts"):
        part.bind(tensors)


# ---------------------------------------------------------------------------------------------- the plain implementation by hand
def test_streams_by_hand():
    X = torch.tensor([[[1.0, 2.0]], [[10.0, 20.0]]], dtype=F)
    assert plain.read_streams(X, torch.tensor([3.0, 0.5], dtype=F)).tolist() == [[8.0, 16.0]]
    mix = torch.tensor([[1.0, 2.0], [0.0, 0.5]], dtype=F)            # from 0 to 1 twice, from 1 to 0 not at all
    new = plain.write_streams(X, mix, torch.tensor([1.0, -1.0], dtype=F), torch.tensor([[100.0, 0.0]], dtype=F))
    assert new.tolist() == [[[101.0, 2.0]], [[2.0 + 5.0 - 100.0, 4.0 + 10.0]]]


def test_norms_sink_and_window_by_hand():
    x = torch.tensor([[1.0, 3.0]], dtype=F)
    g = torch.tensor([2.0, 4.0], dtype=F)
    assert torch.allclose(plain.layer_norm(x, g, 3.0), torch.tensor([[-2.0 / 2.0, 4.0 / 2.0]], dtype=F))       # variance 1, plus 3
    assert torch.allclose(plain.rms_norm(x, g, 4.0), torch.tensor([[2.0 / 3.0, 12.0 / 3.0]], dtype=F))          # mean square 5, plus 4
    seen = plain.visible(4, 2)
    assert seen.tolist() == [[True, False, False, False], [True, True, False, False], [False, True, True, False], [False, False, True, True]]
    assert plain.visible(3, 0).tolist() == [[True, False, False], [True, True, False], [True, True, True]]
    w = plain.sink_softmax(torch.log(torch.tensor([[1.0, 7.0], [2.0, 3.0]], dtype=F)), plain.visible(2, 0), torch.tensor(math.log(5.0), dtype=F))
    assert torch.allclose(w, torch.tensor([[1 / 6, 0.0], [2 / 10, 3 / 10]], dtype=F))


def test_latent_attention_by_hand():
    """One head of one-element queries, keys and values, latents of one element whose norm leaves +-gain: the scores are +-1."""
    t = {"p.q": torch.tensor([[1.0]]), "p.g": torch.tensor([[0.0]]), "p.uk": torch.tensor([[2.0]]), "p.uv": torch.tensor([[3.0]]),
         "p.o": torch.tensor([[10.0]]), "p.sink": torch.tensor([0.0]), "p.dkv": torch.tensor([[5.0]]), "p.dkv.norm": torch.tensor([1.0])}
    h = torch.tensor([[1.0], [-1.0]], dtype=F)
    c = plain.latents(h, t, "p.", 0.0)
    assert c.tolist() == [[1.0], [-1.0]]
    y = plain.latent_attention(h, c, t, "p.", {"heads": 1, "dim": 1, "vdim": 1, "scale": 0.5})
    e = math.e                                                   # scores: (0, 0) +1; (1, 0) -1, (1, 1) +1; gate sigmoid(0) = 1/2
    want = [10 * 0.5 * 3 * e / (e + 1), 10 * 0.5 * (3 / e - 3 * e) / (1 / e + e + 1)]
    assert torch.allclose(y.flatten(), torch.tensor(want, dtype=F))
    y1 = plain.latent_attention(h, c, t, "p.", {"heads": 1, "dim": 1, "vdim": 1, "scale": 0.5, "mask": {"size": 1}})
    assert torch.allclose(y1.flatten(), torch.tensor([want[0], -10 * 0.5 * 3 * e / (e + 1)], dtype=F))


def test_experts_and_head_by_hand():
    ones = torch.ones(1, 1)
    t = {"p.table": torch.tensor([[0, 1], [1, 0]], dtype=torch.int32)}
    for e, s in ((0, 1.0), (1, 3.0)):
        t[f"p.e{e}.gate"], t[f"p.e{e}.up"], t[f"p.e{e}.down"] = ones * 0 + 100.0, ones, ones * s          # silu(100) = 100
    t["p.shared.gate"], t["p.shared.up"], t["p.shared.down"] = ones * 100.0, ones, ones * 0.01
    mlp = {"router": {"experts": 2, "top": 2}, "shared": {"ff": 1}}
    y = plain.table_experts(torch.tensor([[1.0], [1.0]], dtype=F), [0, 1], t, "p.", mlp)
    assert torch.allclose(y, torch.full((2, 1), 100 * (1 + 3) / 2 + 1.0, dtype=F))
    t["p.table"] = torch.tensor([[0], [1]], dtype=torch.int32)
    y = plain.table_experts(torch.tensor([[1.0], [1.0]], dtype=F), [1, 0], t, "p.", {"router": {"experts": 2, "top": 1}})
    assert torch.allclose(y, torch.tensor([[300.0], [100.0]], dtype=F))
    x = torch.tensor([[4.0]], dtype=F)
    w = {"head": torch.tensor([[1.0], [-2.0]])}
    assert torch.allclose(plain.head(x, {"logit_scale": 0.5, "logit_softcap": 2.0}, w), torch.tensor([[2 * math.tanh(1.0), 2 * math.tanh(-2.0)]], dtype=F))
    assert plain.head(x, {}, w).tolist() == [[4.0, -8.0]]


def test_every_part_of_the_design_moves_the_plain_logits(tmp_path):
    """Faults planted in the plain implementation's inputs: each moves the logits far beyond what the engine is held to, so the tests
    on the GPU would notice the same fault there."""
    from conftest import logit_tolerance, random_tokens
    folder = write_model(tmp_path / "u", "X", transform=near_uniform)
    cfg, w = load_plain(folder)
    toks = random_tokens(cfg["vocab"], 60, 5)
    want = plain.run(cfg, w, toks).float()
    tol = logit_tolerance("float32", want)

    def moved(edit_cfg=None, edit_w=None, of=slice(45, None)):
        c, t = copy.deepcopy(cfg), dict(w)
        if edit_cfg:
            edit_cfg(c)
        if edit_w:
            edit_w(t)
        return float((plain.run(c, t, toks).float() - want).abs().max(dim=1).values[of].min())

    for layer in (0, 1, 2, 3):
        for delta in (1, -1):
            assert moved(lambda c: c["layers"][layer]["mixer"]["mask"].update(size=c["layers"][layer]["mixer"]["mask"]["size"] + delta)) > 5 * tol
        assert moved(edit_w=lambda t: t.update({f"l{layer}.mix.sink": torch.full_like(t[f"l{layer}.mix.sink"], -60.0)})) > 10 * tol
        assert moved(edit_w=lambda t: t.update({f"l{layer}.mix.g": t[f"l{layer}.mix.g"] * 0})) > 10 * tol
        assert moved(edit_w=lambda t: t.update({f"l{layer}.hc1.mix": t[f"l{layer}.hc1.mix"].T.contiguous()})) > 10 * tol
    assert moved(edit_w=lambda t: t.update({"l0.mlp.table": t["l0.mlp.table"].roll(1, 0)})) > 10 * tol
    assert moved(edit_w=lambda t: t.update({"l3.mlp.shared.down": t["l3.mlp.shared.down"] * 0})) > 10 * tol
    assert moved(lambda c: c.update(logit_softcap=9.5)) > 10 * tol
    assert moved(lambda c: c["norm"].update(eps=3e-2)) > 10 * tol
