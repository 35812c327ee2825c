"""Viperax through the engine against the plain implementation (tests/plain_viperax.py): every mechanism alone (streams, latent attention
with window, sink, gate and another layer's latents, experts by table, capped logits), then whole models of tiny configurations whole,
decoded token by token, in portions down to two tokens and in mixed batches with pages and slots used again, in 32-bit and in bfloat16;
window edges, sinks and far keys made to show; long decoding; batches against each request alone; greedy generation through the entry
point, its scheduler and the command line."""
from __future__ import annotations

import copy

import pytest
import torch

import plain_viperax as plain
from conftest import TraceRun, logit_tolerance, random_tokens
from test_replay_gpu import _Bits, _portions
from viperax_cases import VIPERAX, drawn, load_plain, near_uniform, write_model

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F = torch.float64
BF = torch.bfloat16
ROWS = 256


@pytest.fixture(scope="module")
def viperax_dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("viperax")
    out = {name: write_model(root / name, name) for name in VIPERAX}
    out["XU"] = write_model(root / "XU", "X", transform=near_uniform)
    return out


def _env(dtype, rows=ROWS):
    from stride_b200.parts import BuildEnv
    return BuildEnv(device=torch.device(DEV), compute_dtype=dtype, max_tokens=rows, max_positions=1024)


def _step(entries, dtype, tokens=None, rows=ROWS, workspace=None):
    """The context of a step of (slot, tokens, first position) entries."""
    from stride_b200.parts import Workspace
    from stride_b200.parts.context import step_context
    return step_context(entries, workspace or Workspace(DEV, rows), dtype, tokens)


# ---------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("S,W,out_dtype", [(1, 96, torch.float32), (2, 50, BF), (3, 260, BF), (4, 64, torch.float32), (5, 52, BF), (9, 33, torch.float32),
                                           (3, 2048, BF), (16, 128, BF)])
def test_streams_step(S, W, out_dtype):
    """Streams read, changed and normed in one pass: from the embedding output alone, with one and two sources (buffers, partial sums,
    constants), layer norm and RMS norm, biases; and the streams' sum on chosen rows at the end."""
    from stride_b200.kernels.native import ImmediateProgram
    g = torch.Generator().manual_seed(S * 100 + W)
    n, eps = 11, 1e-3
    rnd = lambda *shape: torch.randn(*shape, generator=g)
    e, X, a, b, pa, pb = rnd(n, W), rnd(S, n, W), rnd(n, W), rnd(n, W), rnd(3, n, W), rnd(9, n, W)
    mix, out, inp, gain, bias = rnd(S, S), rnd(S), rnd(S), rnd(W), rnd(W)
    dev = lambda t: t.to(DEV).contiguous()
    held = dev(X.transpose(0, 1))                                       # [n, S, W]
    ctx = _step([(0, n, 0)], BF)
    rows = [7, 0, 7, 10]
    R = (ctx.positions.data_ptr() - ctx.token_ids.data_ptr()) // 4
    wanted = torch.as_strided(ctx.token_ids, (len(rows),), (1,), ctx.token_ids.storage_offset() + 3 * R)
    wanted.copy_(torch.tensor(rows, dtype=torch.int32))
    tol = 2e-5 if out_dtype == torch.float32 else 2e-2

    def check(got, u, centred, biased):
        want = plain.layer_norm(u, gain.double(), eps) if centred else plain.rms_norm(u, gain.double(), eps)
        want = want + (bias.double() if biased else 0)
        assert (got.cpu().double() - want).abs().max() <= tol * max(1.0, float(want.abs().max()))

    sources = [("buffer", [dev(a), None, 1, 0, None, None, 1, 0], [1.0, 1.0], a.double()),
               ("sums", [None, dev(pa), 3, 512, None, None, 1, 0], [0.5, 1.0], 0.5 * pa.double().sum(0)),
               ("both", [dev(a), dev(pa), 3, 512, dev(b), dev(pb), 9, 1 << 30], [0.25, 2.0],
                0.25 * (a.double() + pa.double().sum(0)) + 2.0 * (b.double() + pb.double().sum(0)))]
    gd, bd, ind, md, od, ed = (dev(t) for t in (gain, bias, inp, mix, out, e))
    with ImmediateProgram(ctx, None) as program:
        for centred in (True, False):
            normed = torch.empty(n, W, dtype=out_dtype, device=DEV)
            # nothing stored yet: every stream is the embedding output
            program.add("streams", "sb_op_streams_step", [ed, W, 0, None, None, None, 1, 0, None, None, 1, 0, None, None, ind, gd, bd if centred else None,
                                                          int(centred), normed, out_dtype, S, W, 0], [1.0, 1.0, eps])
            check(normed, plain.read_streams(torch.stack([e.double()] * S), inp.double()), centred, centred)
            for what, args, constants, y in sources:
                for first in (True, False):
                    x = dev(torch.zeros(n, S, W)) if first else held.clone()
                    src = [ed, W, 0] if first else [x, S * W, W]
                    normed = torch.empty(n, W, dtype=out_dtype, device=DEV)
                    program.add("streams", "sb_op_streams_step", [*src, x, *args, md, od, ind, gd, None, int(centred), normed, out_dtype, S, W, 0],
                                [*constants, eps])
                    old = torch.stack([e.double()] * S) if first else X.double()
                    new = plain.write_streams(old, mix.double(), out.double(), y)
                    assert (x.cpu().double().transpose(0, 1) - new).abs().max() <= 1e-5 * float(new.abs().max()), what
                    check(normed, plain.read_streams(new, inp.double()), centred, False)
                    if not first:                                       # the end of a model: the sum of the streams on the wanted rows
                        program.step.wanted = len(rows)
                        x = held.clone()
                        last = torch.empty(len(rows), W, dtype=out_dtype, device=DEV)
                        program.add("streams", "sb_op_streams_step", [x, S * W, W, None, *args, md, od, None, gd, None, int(centred), last, out_dtype, S, W, 1],
                                    [*constants, eps])
                        check(last, new.sum(0)[rows], centred, False)
                        assert torch.equal(x, held)


def _moe_case(W, vocab, E, top, ff, shared, g, scale=0.3):
    t = {"p.table": torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(vocab)]).to(torch.int32)}
    for name, F_ in [*((f"p.e{e}.", ff) for e in range(E)), *([("p.shared.", shared)] if shared else [])]:
        for r, shape in (("gate", (F_, W)), ("up", (F_, W)), ("down", (W, F_))):
            t[name + r] = (torch.randn(*shape, generator=g) * scale).to(BF)
    params = {"hidden_size": W, "vocab_size": vocab, "intermediate_size": ff, "experts": E, "top": top, "shared": shared}
    names = {r: tuple(f"p.e{e}.{r}" for e in range(E)) for r in ("gate", "up", "down")}
    return t, params, {"table": "p.table", **names, **({f"shared_{r}": f"p.shared.{r}" for r in ("gate", "up", "down")} if shared else {})}


@pytest.mark.parametrize("W,E,top,ff,shared,n,dtype", [
    (24, 5, 2, 40, 0, 23, torch.float32), (72, 3, 3, 33, 17, 9, torch.float32), (64, 1, 1, 24, 40, 50, torch.float32),
    (64, 4, 1, 72, 40, 200, BF), (136, 6, 3, 48, 0, 256, BF), (64, 40, 2, 24, 64, 37, BF), (256, 3, 2, 200, 128, 256, BF), (100, 4, 2, 36, 12, 40, BF),
    (64, 300, 8, 16, 0, 130, BF), (64, 7, 7, 16, 0, 1, BF)])
def test_experts_by_table(W, E, top, ff, shared, n, dtype):
    """The part alone, adding to a stream (blocks without several streams fold it), against the plain experts; one expert much more
    popular than the others, a token still being chosen read from its slot, experts that nobody chose, a token alone in the same bits."""
    from stride_b200.parts import PartSpec, ResidualStream, Workspace, part_class
    g = torch.Generator().manual_seed(W + E)
    vocab = 61
    t, params, names = _moe_case(W, vocab, E, top, ff, shared, g)
    toks = torch.randint(0, vocab, (n,), generator=g)
    toks[: n // 2] = 3                                                  # half of the rows choose the same experts
    part = part_class("feed_forward", "table_experts")(PartSpec("table_experts", params, names), _env(dtype))
    part.bind({k: v.to(DEV) for k, v in t.items()})
    assert part.tensor_core == (dtype == BF and W % 8 == 0 and ff % 8 == 0)
    ws = Workspace(DEV, ROWS)
    h = torch.randn(n, W, generator=g).to(BF)
    mlp = {"router": {"experts": E, "top": top}, **({"shared": {"ff": shared}} if shared else {})}
    base = torch.randn(n, W, generator=g)

    def run(rows):
        fed = toks[rows].tolist()
        ctx = _step([(1, len(rows), 0)], dtype, fed, workspace=ws)
        if len(rows) == n:
            ctx.token_ids[n - 1] = -1
        ctx.sampled = torch.tensor([0, int(toks[n - 1]), 0], dtype=torch.int32, device=DEV)
        stream = ResidualStream(base[rows].to(DEV))
        part.forward(ctx, h[rows].to(DEV, dtype), stream)
        stream.fold()
        return stream.h.cpu()

    got = run(list(range(n)))
    want = plain.table_experts(h.double(), toks.tolist(), t, "p.", mlp, None if dtype == torch.float32 else BF)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    assert (got.double() - base.double() - want).abs().max() <= tol * float(want.abs().max())
    for i in sorted({0, n // 2, n - 1}):
        assert torch.equal(run([i])[0], got[i]), f"row {i} alone differs from the row in company"
    assert torch.equal(run(list(range(n))), got)


def _latent_case(H, D, V, R, W, g, own=True, scale=0.4):
    t = {"p.q": torch.randn(H * D, W, generator=g), "p.g": torch.randn(H * V, W, generator=g), "p.uk": torch.randn(H * D, R, generator=g),
         "p.uv": torch.randn(H * V, R, generator=g), "p.o": torch.randn(W, H * V, generator=g), "p.sink": torch.randn(H, generator=g) + 1.0}
    if own:
        t.update({"p.dkv": torch.randn(R, W, generator=g), "p.dkv.norm": 1.0 + 0.3 * torch.randn(R, generator=g)})
    for k in t:
        t[k] = (t[k] * (W ** -0.5 if k in ("p.q", "p.g", "p.dkv") else R ** -0.5 if k in ("p.uk", "p.uv") else (H * V) ** -0.5 if k == "p.o" else 1.0)).to(BF)
    return t


def _latent_part(H, D, V, R, W, window, scale, eps, dtype, t, own=True):
    from stride_b200.parts import PartSpec, part_class
    names = {r: "p." + r for r in ("q", "uk", "uv", "sink", "g", "o")}
    if own:
        names.update(dkv="p.dkv", dkv_norm="p.dkv.norm")
    part = part_class("mixer", "latent_attention")(
        PartSpec("latent_attention", {"hidden_size": W, "num_heads": H, "key_dim": D, "value_dim": V, "q_rank": 0, "kv_rank": R, "scale": scale,
                                      "norm_eps": eps, "window": window, "sink": True, "gate": True, "own_latent": own}, names), _env(dtype))
    assert set(part.tensor_plan()) == set(t)
    part.bind({k: v.to(DEV) for k, v in t.items()})
    return part


@pytest.mark.parametrize("H,D,V,R,W,window,window2,page,dtype", [
    (3, 22, 27, 44, 60, 9, 30, 8, torch.float32), (4, 32, 32, 64, 96, 50, 0, 16, torch.float32), (1, 8, 5, 16, 40, 1, 7, 8, torch.float32),
    (4, 32, 48, 64, 128, 37, 64, 16, BF), (16, 16, 32, 96, 128, 64, 1, 64, BF), (8, 24, 40, 512, 96, 100, 33, 32, BF), (5, 20, 12, 40, 72, 21, 40, 8, BF)])
def test_latent_attention_alone(H, D, V, R, W, window, window2, page, dtype):
    """Two mixers over one cache: the first stores the latents, the second reads them with other heads and another window. Two requests
    of unequal length fed in portions beside single tokens, in pages handed out in a shuffled order and full of large numbers."""
    from stride_b200.cache.manager import LayerCache
    from stride_b200.parts import ResidualStream, Workspace
    g = torch.Generator().manual_seed(H * 1000 + R)
    eps, scale = 1e-4, 0.8
    H2 = 2 * H if H < 16 else 2
    lengths = [130, 61]
    t1, t2 = _latent_case(H, D, V, R, W, g), _latent_case(H2, D, V, R, W, g, own=False)
    p1, p2 = _latent_part(H, D, V, R, W, window, scale, eps, dtype, t1), _latent_part(H2, D, V, R, W, window2, scale, eps, dtype, t2, own=False)
    per = -(-max(lengths) // page)
    need = p1.cache_need()
    assert (need.kv_heads, need.head_dim, need.planes, need.window) == (1, R, 1, window) and p2.cache_need().window == window2
    perm = torch.randperm(2 * per + 3, generator=g)[:2 * per].view(2, per).to(torch.int32).to(DEV).contiguous()
    pages = torch.full((2 * per + 3, 1, 1, page, R), 1e4, dtype=dtype, device=DEV)
    c1 = LayerCache(pages=pages, block_table=perm, page_size=page)
    c2 = LayerCache(pages=pages, block_table=perm, page_size=page, writes=False)
    h = [torch.randn(n, W, generator=g).to(BF) for n in lengths]
    h2 = [torch.randn(n, W, generator=g).to(BF) for n in lengths]
    ws = Workspace(DEV, ROWS)
    schedule = [[(0, 70), (1, 2)], [(1, 30)], [(0, 1), (1, 1)], [(0, 2), (1, 28)]] + [[(0, 1)]] * 3 + [[(0, 54)]]
    fed, got = [0, 0], [[[], []], [[], []]]
    for step in schedule:
        entries = [(r, n, fed[r]) for r, n in step]
        for k, (part, cache, hs) in enumerate(((p1, c1, h), (p2, c2, h2))):
            ctx = _step(entries, dtype, workspace=ws)
            x = torch.cat([hs[r][fed[r]:fed[r] + n] for r, n in step]).to(DEV, dtype)
            stream = ResidualStream(torch.zeros(ctx.n, W, device=DEV))
            part.forward(ctx, x, stream, cache)
            stream.fold()
            out, at = stream.h.cpu().double(), 0
            for r, n in step:
                got[k][r].append(out[at:at + n])
                at += n
        for r, n in step:
            fed[r] += n
    assert fed == lengths
    rnd = None if dtype == torch.float32 else BF
    for r in range(2):
        c = plain.latents(h[r].double(), t1, "p.", eps, rnd)
        for k, (t, hs, heads, win) in enumerate(((t1, h, H, window), (t2, h2, H2, window2))):
            m = {"heads": heads, "dim": D, "vdim": V, "scale": scale, **({"mask": {"size": win}} if win else {})}
            want = plain.latent_attention(hs[r].double(), c, t, "p.", m, rnd)
            diff = (torch.cat(got[k][r]) - want).abs().max()
            assert diff <= (2e-5 if rnd is None else 2e-2) * float(want.abs().max()), f"mixer {k}, request {r}: {diff}"


@pytest.mark.parametrize("dtype", [torch.float32, BF])
def test_one_key_that_stands_out_is_seen_up_to_the_edge_of_the_window(dtype):
    """One position's latent answers every query with a score far above the others: while it lies inside the window the result is its
    value, one position later it is not."""
    from stride_b200.cache.manager import LayerCache
    from stride_b200.parts import ResidualStream, Workspace
    g = torch.Generator().manual_seed(9)
    H, D, V, R, W, window, page, n, loud = 4, 32, 32, 64, 64, 70, 16, 160, 37
    t = _latent_case(H, D, V, R, W, g)
    h = torch.randn(n, W, generator=g)
    h[:, :8] = h[:, :8].abs() + 1.0                                     # every query has a positive share along the first directions ..
    t["p.q"] = torch.zeros(H * D, W, dtype=BF)
    t["p.q"][:, :8] = 0.3
    t["p.uk"] = torch.zeros(H * D, R, dtype=BF)
    t["p.uk"][:, 5] = 1.0                                               # .. and scores element 5 of the latent,
    t["p.dkv"][5] = 0.0
    t["p.dkv"][5, 20] = 1.0
    h[:, 20] = 0.0
    h[loud, 20] = 40.0                                                  # which one token alone has
    h = h.to(BF)
    part = _latent_part(H, D, V, R, W, window, 0.5, 1e-5, dtype, t)
    per = n // page
    cache = LayerCache(pages=torch.full((per, 1, 1, page, R), 1e4, dtype=dtype, device=DEV), page_size=page,
                       block_table=torch.randperm(per, generator=g).view(1, per).to(torch.int32).to(DEV))
    rows, ws, at = [], Workspace(DEV, ROWS), 0
    for k in (50, 2, 53, 1, 1, 1, 1, 51):
        ctx = _step([(0, k, at)], dtype, workspace=ws)
        stream = ResidualStream(torch.zeros(k, W, device=DEV))
        part.forward(ctx, h[at:at + k].to(DEV, dtype), stream, cache)
        stream.fold()
        rows.append(stream.h.cpu().double())
        at += k
    assert at == n
    got, rnd = torch.cat(rows), None if dtype == torch.float32 else BF
    c = plain.latents(h.double(), t, "p.", 1e-5, rnd)
    m = {"heads": H, "dim": D, "vdim": V, "scale": 0.5, "mask": {"size": window}}
    want = plain.latent_attention(h.double(), c, t, "p.", m, rnd)
    assert (got - want).abs().max() <= (2e-5 if rnd is None else 2e-2) * float(want.abs().max())
    for delta in (1, -1):                                               # the edge shows, at its own place and nowhere else
        other = plain.latent_attention(h.double(), c, t, "p.", {**m, "mask": {"size": window + delta}}, rnd)
        moved = (other - want).abs().max(dim=1).values
        edge = loud + window + (0 if delta > 0 else -1)
        assert float(moved[edge]) > 0.2 * float(want.abs().max()) and (got[edge] - want[edge]).abs().max() < 0.1 * float(moved[edge])


def test_layer_norm_without_bias_capped_logits_and_fresh_branches():
    from stride_b200.kernels import ops
    from stride_b200.kernels.linear import Linear
    from stride_b200.kernels.native import ImmediateProgram
    from stride_b200.parts.branch import emit_on_branch
    g = torch.Generator().manual_seed(2)
    h, w = torch.randn(7, 90, generator=g), torch.randn(90, generator=g)
    out = torch.empty(7, 90, device=DEV)
    ops.layernorm(h.to(DEV), w.to(DEV), None, 1e-3, out)
    want = plain.layer_norm(h.double(), w.double(), 1e-3)
    assert (out.cpu().double() - want).abs().max() <= 1e-5 * float(want.abs().max())
    for shape in ((3, 77), (2, 4096)):
        for scale, cap in ((0.5, 15.0), (1.0, 0.0), (2.0, 3.0)):
            x = 8 * torch.randn(*shape, generator=g)
            d = x.to(DEV)
            ops.cap_logits(d, scale, cap)
            want = cap * torch.tanh(x.double() * scale / cap) if cap else x.double() * scale
            assert (d.cpu().double() - want).abs().max() <= 1e-5 * float(want.abs().max())
    # a branch whose contents mean nothing: the first projection stores, a second one adds, an operation that wants the buffer finds zeros
    for dtype, K in ((torch.float32, 24), (BF, 20)):
        ctx = _step([(0, 5, 0)], dtype)
        lin = Linear((torch.randn(16, K, generator=g)).to(BF).to(DEV), dtype)
        x = torch.randn(5, K, generator=g).to(BF).to(DEV, dtype)
        branch = torch.full((5, 16), float("nan"), device=DEV)
        want = x.double() @ lin.weight.double().T
        with ImmediateProgram(ctx, None) as program:
            source = emit_on_branch(program, branch, lambda: (lin.emit_add(program, x), lin.emit_add(program, x)), fresh=True)
            assert source[0] is branch and source[1] is None
            assert (branch.double() - 2 * want).abs().max() <= 1e-5 * float(want.abs().max())
            branch.fill_(float("nan"))
            emit_on_branch(program, branch, lambda: program.h, fresh=True)
            assert float(branch.abs().max()) == 0.0


# ---------------------------------------------------------------------------------------------- whole models
def _engine(model_dir, dtype, page, pages, rows=ROWS, slots=4, **kw):
    from stride_b200.engine.engine import Engine, EngineOptions
    return Engine(model_dir, EngineOptions(dtype=dtype, max_rows=rows, max_full_rows=rows, max_slots=slots, kv_pages=pages,
                                           page_size=page, max_context=pages * page, device=DEV, **kw))


def _noise(cfg, w, tokens):
    """The largest |plain with bfloat16 rounding - plain exact| over the sequence's logits."""
    return float((plain.run(cfg, w, tokens, BF) - plain.run(cfg, w, tokens)).abs().max())


def test_every_layer_against_the_plain_streams(viperax_dirs):
    """The sum of the streams after every layer, in 32-bit, for a prompt in one step."""
    from stride_b200.engine.engine import StepEntry
    for name in VIPERAX:
        cfg, w = load_plain(viperax_dirs[name])
        toks = random_tokens(cfg["vocab"], 37, 12)
        want = []
        plain.run(cfg, w, toks, after_layer=lambda i, x: want.append(x))
        eng = _engine(viperax_dirs[name], "float32", VIPERAX[name][2], 8, native_step=False)
        slot = eng.cache.acquire_slot()
        eng.cache.ensure(slot, len(toks))
        seen = []
        for block in eng.model.blocks:
            def run(ctx, stream, cache, inner=block.forward):
                inner(ctx, stream, cache)
                s = stream.streams
                old = s.x[:len(toks)].cpu().double().transpose(0, 1) if s.held else torch.stack([stream.h[:len(toks)].cpu().double()] * s.count)
                sources, mix, out = s.update
                y = torch.zeros(len(toks), s.width, dtype=F)
                for buffer, pending, c in sources:
                    if buffer is not None:
                        y += c * buffer[:len(toks)].cpu().double()
                    if pending is not None:
                        flat, P = pending[:2]
                        y += c * flat.reshape(-1)[:P * y.numel()].view(P, *y.shape).sum(0).cpu().double()
                seen.append(plain.write_streams(old, mix.cpu().double(), out.cpu().double(), y).sum(0))
            block.forward = run
        eng.step([StepEntry(slot, 0, toks, list(range(len(toks))))])
        assert len(seen) == len(want) == len(cfg["layers"])
        for k, (a, b) in enumerate(zip(seen, want)):
            assert (a - b).abs().max() <= 2e-4 * max(1.0, float(b.abs().max())), f"{name}: the streams after layer {k} differ"


LENGTHS = {"X": [70, 130, 45, 33, 2], "Y": [300, 65, 140, 129, 40], "Z": [48, 90, 17, 64, 5], "S": [66, 40, 90, 34, 3]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(VIPERAX))
def test_replay_modes(name, dtype, viperax_dirs, tmp_path):
    """Through bin/trace_run: whole; all but the last 32 tokens, then token by token; portions down to two tokens; mixed batches in a
    pool so small that pages are used again, four slots for five requests. Against the plain implementation (bfloat16: rounding at the
    same places; the largest deviation within the largest rounding noise of the same sequence), and all four in the same bits."""
    cfg, _, page = VIPERAX[name]
    vocab = cfg["vocab"]
    reqs = [random_tokens(vocab, n, 300 + i) for i, n in enumerate(LENGTHS[name])]
    pcfg, w = load_plain(viperax_dirs[name])
    bf = dtype == "bfloat16"
    want = [plain.run(pcfg, w, r, BF if bf else None).float() for r in reqs]
    tols = [_noise(pcfg, w, r) if bf else logit_tolerance(dtype, want[i]) for i, r in enumerate(reqs)]
    per = lambda n: -(-n // page) * page
    longest = sorted((per(len(r)) for r in reqs), reverse=True)
    pool = max(longest[0] + longest[1] + page, 4 * page)
    tr = TraceRun(viperax_dirs[name], dtype, tmp_path, pool, page, extra=("--kv-shuffle", "5"))
    bits = _Bits()

    def compare(got, i, a, b, what):
        diff = (got - want[i][a:b]).abs()
        assert diff.max() <= tols[i], f"{name} {dtype} {what}: max |diff| {diff.max():.3e} > {tols[i]:.3e} at {a + int(diff.max(dim=1).values.argmax())}"
        bits.check(i, a, got, f"{name} {what}")

    try:
        for i, r in enumerate(reqs):
            s = tr.run([(f"w{i}", r, range(len(r)))], end=[f"w{i}"])
            compare(tr.logits(s, vocab), i, 0, len(r), f"whole request {i}")
        for i, r in enumerate(reqs):
            cut = max(1, len(r) - 32)
            s = tr.run([(f"d{i}", r[:cut], [cut - 1])], end=[f"d{i}"] if cut == len(r) else [])
            compare(tr.logits(s, vocab), i, cut - 1, cut, f"request {i} prefill end")
            for p in range(cut, len(r)):
                s = tr.run([(f"d{i}", r[p:p + 1], [0])], end=[f"d{i}"] if p == len(r) - 1 else [])
                compare(tr.logits(s, vocab), i, p, p + 1, f"request {i} decode at {p}")
        for i, r in enumerate(reqs):
            cuts = _portions(len(r), [7, 2, 19, 3, 2, 31, 5])
            for j, (a, b) in enumerate(cuts):
                s = tr.run([(f"p{i}", r[a:b], range(b - a))], end=[f"p{i}"] if j == len(cuts) - 1 else [])
                compare(tr.logits(s, vocab), i, a, b, f"request {i} portion {a}:{b}")
        fed, turn = [0] * len(reqs), [0] * len(reqs)
        sizes = [[9, 1, 1, 4, 1], [2, 13, 1, 1, 1, 6], [5, 1, 1, 1], [17, 1, 2, 1, 1], [3, 1, 8, 1]]
        live, waiting, steps = [], list(range(len(reqs))), 0
        while live or waiting:
            while waiting and len(live) < 4 and sum(per(len(reqs[i])) for i in live) + per(len(reqs[waiting[0]])) <= pool:
                live.append(waiting.pop(0))
            entries, ends, spans = [], [], []
            for k, i in enumerate(list(live)):
                if (steps + k) % 5 == 4 and len(live) > 1:
                    continue                                            # this request sits the step out and goes on later
                n = min(sizes[i][turn[i] % len(sizes[i])], len(reqs[i]) - fed[i])
                turn[i] += 1
                a, b = fed[i], fed[i] + n
                entries.append((f"m{i}", reqs[i][a:b], range(n) if steps % 3 else []))      # (steps whose logits nobody wants in between)
                spans.append((i, a, b))
                fed[i] = b
                if b == len(reqs[i]):
                    ends.append(f"m{i}")
                    live.remove(i)
            s = tr.run(entries, end=ends)
            if steps % 3:
                got, at = tr.logits(s, vocab), 0
                for i, a, b in spans:
                    compare(got[at:at + b - a], i, a, b, f"mixed step {steps} request {i} {a}:{b}")
                    at += b - a
            steps += 1
    finally:
        tr.close()


def test_window_edges_show_and_agree(viperax_dirs):
    """With attention close to uniform every visible key carries weight (that a window one token off shows is checked on the plain
    implementation): the engine agrees at every position, in a prompt whose windows straddle pages and decoding token by token with pages
    given back behind the longest window of a cache's readers."""
    from stride_b200.engine.engine import StepEntry
    cfg, w = load_plain(viperax_dirs["XU"])
    toks = random_tokens(cfg["vocab"], 100, 77)
    want = plain.run(cfg, w, toks).float()
    eng = _engine(viperax_dirs["XU"], "float32", 16, 7, slots=1)
    slot = eng.cache.acquire_slot()
    eng.cache.ensure(slot, 50)
    got = [eng.step([StepEntry(slot, 0, toks[:50], list(range(50)))]).cpu().clone()]
    for t in range(50, 100):
        eng.cache.ensure(slot, t + 1)
        got.append(eng.step([StepEntry(slot, t, [toks[t]], [0])]).cpu().clone())
        eng.cache.trim(slot)
    assert (torch.cat(got) - want).abs().max() <= logit_tolerance("float32", want)
    held = {g.window: sorted(g.held[slot]) for g in eng.cache.groups}
    assert held[29][0] == (100 - 28) // 16 and held[40][0] == (100 - 39) // 16
    eng.cache.check()


def test_the_first_tokens_of_a_sequence(viperax_dirs):
    """Positions 0, 1, 2, .. one by one in a slot that another request used: a sink beside a single key, windows with fewer keys than
    their size."""
    from stride_b200.engine.engine import StepEntry
    for name in sorted(VIPERAX):
        cfg, w = load_plain(viperax_dirs[name])
        eng = _engine(viperax_dirs[name], "float32", VIPERAX[name][2], 16)
        for seed in (3, 4):
            toks = random_tokens(cfg["vocab"], 12, seed)
            want = plain.run(cfg, w, toks).float()
            slot = eng.cache.acquire_slot()
            got = []
            for t in range(12):
                eng.cache.ensure(slot, t + 1)
                got.append(eng.step([StepEntry(slot, t, [toks[t]], [0])]).cpu().clone())
            assert (torch.cat(got) - want).abs().max() <= logit_tolerance("float32", want)
            eng.cache.release_slot(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_slot_reuse(dtype, viperax_dirs):
    """A short prompt, then 400 tokens one by one (every window passes over decoded tokens, pages behind them are given back and taken
    again: the pool is far smaller than the sequence), against the plain implementation; then the same slot again for another request."""
    from stride_b200.engine.engine import StepEntry
    cfg, w = load_plain(viperax_dirs["XU"])
    eng = _engine(viperax_dirs["XU"], dtype, 16, 26, slots=1)
    for seed in (1, 2):
        toks = random_tokens(cfg["vocab"], 410, seed)
        bf = dtype == "bfloat16"
        want = plain.run(cfg, w, toks, BF if bf else None).float()
        slot = eng.cache.acquire_slot()
        eng.cache.ensure(slot, 10)
        got = [eng.step([StepEntry(slot, 0, toks[:10], list(range(10)))]).cpu().clone()]
        for t in range(10, 410):
            eng.cache.ensure(slot, t + 1)
            got.append(eng.step([StepEntry(slot, t, [toks[t]], [0])]).cpu().clone())
            eng.cache.trim(slot)
        assert (torch.cat(got) - want).abs().max() <= (_noise(cfg, w, toks) if bf else logit_tolerance("float32", want))
        eng.cache.release_slot(slot)
        eng.cache.check()


def test_a_far_token_shows_through_the_unbounded_layers(viperax_dirs, tmp_path):
    """Two layers of Y see every earlier token. One early token's latent is made loud: another token in its place moves the plain
    logits 300 tokens later far beyond the tolerance, and the engine, fed in portions that cut pages and then token by token, agrees."""
    from stride_b200.engine.engine import StepEntry

    def loud(tensors):
        near_uniform(tensors)
        for n in tensors:
            if n.endswith("mix.sink"):
                tensors[n] = tensors[n] - 2.0
            if n.endswith("mix.o"):
                tensors[n] = (tensors[n].float() * 3.0).to(BF)
        e = tensors["embed"].float()
        e[7] *= 8.0
        tensors["embed"] = e.to(tensors["embed"].dtype)

    folder = write_model(tmp_path / "far", "Y", transform=loud)
    cfg, w = load_plain(folder)
    toks = [t if t != 7 else 8 for t in random_tokens(cfg["vocab"], 330, 21)]
    toks[13] = 7
    want = plain.run(cfg, w, toks).float()
    tol = logit_tolerance("float32", want)
    other = list(toks)
    other[13] = 8
    assert (plain.run(cfg, w, other).float()[-20:] - want[-20:]).abs().max(dim=1).values.min() > 10 * tol
    eng = _engine(folder, "float32", 32, 14)
    slot = eng.cache.acquire_slot()
    got, at = [], 0
    for n in (45, 2, 150, 83, 3, 17):
        eng.cache.ensure(slot, at + n)
        got.append(eng.step([StepEntry(slot, at, toks[at:at + n], list(range(n)))]).cpu().clone())
        eng.cache.trim(slot)
        at += n
    for t in range(at, len(toks)):
        eng.cache.ensure(slot, t + 1)
        got.append(eng.step([StepEntry(slot, t, [toks[t]], [0])]).cpu().clone())
        eng.cache.trim(slot)
    assert (torch.cat(got) - want).abs().max() <= tol


@pytest.mark.parametrize("native", [True, False])
def test_batches_of_unequal_requests_against_each_alone(viperax_dirs, native):
    """Four requests of unequal length in one step, then single tokens of some beside portions of others: every logit has the bits of
    the request run alone; the native step program and the part-by-part driver agree."""
    from stride_b200.engine.engine import StepEntry
    for name in ("Y", "X", "S"):
        cfg, _, page = VIPERAX[name]
        reqs = [random_tokens(cfg["vocab"], n, 40 + n) for n in (150, 3, 64, 31)]
        for dtype in ("float32", "bfloat16"):
            eng = _engine(viperax_dirs[name], dtype, page, 48, native_step=native)
            assert (eng._program is not None) == native
            alone = []
            for r in reqs:
                slot = eng.cache.acquire_slot()
                eng.cache.ensure(slot, len(r))
                alone.append(eng.step([StepEntry(slot, 0, r, list(range(len(r))))]).cpu().clone())
                eng.cache.release_slot(slot)
            slots = [eng.cache.acquire_slot() for _ in reqs]
            fed, got = [0] * 4, [[] for _ in reqs]
            plan = [[100, 2, 30, 1], [1, 1, 20, 30], [49, 0, 1, 0], [1, 1, 13, 0]]      # tokens of each request per step; then one by one
            step = 0
            while any(fed[i] < len(reqs[i]) for i in range(4)):
                entries, who = [], []
                for i, r in enumerate(reqs):
                    n = plan[step][i] if step < len(plan) else 1
                    n = min(n, len(r) - fed[i])
                    if n > 0:
                        eng.cache.ensure(slots[i], fed[i] + n)
                        entries.append(StepEntry(slots[i], fed[i], r[fed[i]:fed[i] + n], list(range(n))))
                        who.append((i, n))
                        fed[i] += n
                out, at = eng.step(entries).cpu(), 0
                for i, n in who:
                    got[i].append(out[at:at + n].clone())
                    at += n
                step += 1
            for i in range(4):
                assert torch.equal(torch.cat(got[i]), alone[i]), f"{name} {dtype}: request {i} in company differs from the request alone"


def test_steps_of_many_tokens_give_the_bits_of_small_ones(tmp_path):
    """More tokens than the projections leave partial sums for, experts' rows in tiles of every size: the bits of portions of a few."""
    from stride_b200.engine.engine import StepEntry
    folder = write_model(tmp_path / "m", "Y")
    toks = random_tokens(VIPERAX["Y"][0]["vocab"], 900, 5)
    for dtype in ("bfloat16", "float32"):
        out = []
        for sizes in ([900], [300, 40, 17, 1, 130, 412], [64] * 14 + [4]):
            eng = _engine(folder, dtype, 64, 16, rows=1024)
            slot = eng.cache.acquire_slot()
            at, got = 0, []
            for n in sizes:
                eng.cache.ensure(slot, at + n)
                got.append(eng.step([StepEntry(slot, at, toks[at:at + n], list(range(n)))]).cpu().clone())
                at += n
            eng.check_kernels()
            out.append(torch.cat(got))
        assert torch.equal(out[0], out[1]) and torch.equal(out[0], out[2]), dtype


def test_greedy_generation_through_the_entry_point(viperax_dirs):
    """LLM.generate with its scheduler (three requests on two slots, prompts cut into portions, decode steps replayed from CUDA
    graphs, the experts' table read for tokens that are still being chosen): the tokens of greedy decoding with the plain implementation."""
    from stride_b200 import LLM
    cfg, w = load_plain(viperax_dirs["X"])
    prompts = [random_tokens(cfg["vocab"], n, 500 + n) for n in (5, 41, 23)]
    llm = LLM(viperax_dirs["X"], dtype="float32", concurrency=2, max_rows=32, prefill_chunk=8, kv_pages=12, page_size=16,
              max_slots=2, max_context=128, device=DEV)
    outs = llm.generate(prompts, max_new_tokens=12)
    sure = 0
    for p, o in zip(prompts, outs):
        seq = list(p)
        for tok in o.tokens:
            ref = plain.run(cfg, w, seq)[-1]
            top = torch.topk(ref, 2).values
            if float(top[0] - top[1]) > 1e-3:       # (a near tie may go either way)
                assert tok == int(ref.argmax())
                sure += 1
            seq.append(tok)
        assert len(o.tokens) == 12 and o.finish_reason == "length"
    assert sure > 18
    bf = LLM(viperax_dirs["Y"], dtype="bfloat16", concurrency=4, max_rows=64, prefill_chunk=16, kv_pages=16, page_size=32,
             max_slots=4, max_context=256, device=DEV)
    outs = bf.generate([random_tokens(VIPERAX["Y"][0]["vocab"], n, n) for n in (70, 9, 33, 120, 64)], max_new_tokens=8)
    assert all(len(o.tokens) == 8 for o in outs)


def test_command_line_generates_what_the_entry_point_generates(viperax_dirs, tmp_path):
    """bin/stride_cli on a Viperax folder (greedy, float32 and bfloat16): the tokens of LLM.generate."""
    import json
    import subprocess
    import sys
    from conftest import ROOT
    from stride_b200 import LLM
    cfg = VIPERAX["Z"][0]
    prompts = [random_tokens(cfg["vocab"], n, 900 + n) for n in (3, 50, 21)]
    (tmp_path / "in.jsonl").write_text("".join(json.dumps({"id": i, "tokens": p}) + "\n" for i, p in enumerate(prompts)))
    for path, dtype in (("exact", "float32"), ("tc", "bfloat16")):
        out = tmp_path / f"out_{path}.jsonl"
        subprocess.run([sys.executable, str(ROOT / "bin" / "stride_cli"), "--model", str(viperax_dirs["Z"]), "--input", str(tmp_path / "in.jsonl"),
                        "--output", str(out), "--max-new", "6", "--concurrency", "2", "--max-rows", "32", "--prefill-chunk", "16",
                        "--kv-blocks", "24", "--page-size", "8", "--max-slots", "4", "--max-context", "128", "--path", path], check=True, timeout=600)
        got = [json.loads(l) for l in out.read_text().splitlines()]
        llm = LLM(viperax_dirs["Z"], dtype=dtype, concurrency=2, max_rows=32, prefill_chunk=16, kv_pages=24, page_size=8, max_slots=4,
                  max_context=128, device=DEV)
        want = llm.generate(prompts, max_new_tokens=6)
        assert [g["tokens"] for g in got] == [w.tokens for w in want] and all(g["finish"] == "length" for g in got)


@pytest.mark.parametrize("seed", range(31, 41))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Whole, and in portions down to one token with pages trimmed on the way, in 32-bit against the plain implementation and in bfloat16 in
    equal bits between the two ways of feeding."""
    from stride_b200.engine.engine import StepEntry
    cfg = drawn(seed)
    folder = write_model(tmp_path / "m", f"R{seed}", config=cfg, seed=seed)
    pcfg, w = load_plain(folder)
    toks = random_tokens(cfg["vocab"], 75, seed)
    want = plain.run(pcfg, w, toks).float()
    for dtype in ("float32", "bfloat16"):
        got = []
        for cuts in ([75], [9, 1, 2, 30, 1, 1, 17, 5, 1, 1, 7]):
            eng = _engine(folder, dtype, 16, 12)
            slot = eng.cache.acquire_slot()
            rows, at = [], 0
            for n in cuts:
                eng.cache.ensure(slot, at + n)
                rows.append(eng.step([StepEntry(slot, at, toks[at:at + n], list(range(n)))]).cpu().clone())
                eng.cache.trim(slot)
                at += n
            got.append(torch.cat(rows))
        assert torch.equal(got[0], got[1]), f"seed {seed} {dtype}: in portions it differs from the whole"
        if dtype == "float32":
            assert (got[0] - want).abs().max() <= logit_tolerance("float32", want), f"seed {seed}: {cfg}"
        else:
            assert (got[0] - plain.run(pcfg, w, toks, BF).float()).abs().max() <= 2.0 * _noise(pcfg, w, toks)
