"""Mezadra through the engine against the plain implementation (tests/plain_mezadra.py): every mechanism alone (convolution, rotation, unit
heads and mixed values in front of the attention; capped scores and sinks in every attention kernel; clamped gates; experts behind a sigmoid
router; norms on results with their second output), then whole models of tiny configurations whole, decoded token by token, in portions
down to two tokens and in mixed batches with pages and slots used again, in 32-bit and in bfloat16; far keys made to show; long decoding;
batches against each request alone; greedy generation through the entry point, its scheduler and the command line."""
from __future__ import annotations

import pytest
import torch

import plain_mezadra as plain
from conftest import TraceRun, logit_tolerance, random_tokens
from mezadra_cases import MEZADRA, drawn, load_plain, near_uniform, write_model
from test_replay_gpu import _Bits, _portions

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F = torch.float64
BF = torch.bfloat16
ROWS = 256


@pytest.fixture(scope="module")
def mezadra_dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("mezadra")
    out = {name: write_model(root / name, name) for name in MEZADRA}
    for name in ("M", "N"):
        out[name + "U"] = write_model(root / (name + "U"), name, config=near_uniform(MEZADRA[name][0]))
    return out


def _env(dtype, rows=ROWS):
    from stride_b200.parts import BuildEnv
    return BuildEnv(device=torch.device(DEV), compute_dtype=dtype, max_tokens=rows, max_positions=4096)


def _step(entries, dtype, tokens=None, rows=ROWS, workspace=None):
    """The context of a step of (slot, tokens, first position) entries."""
    from stride_b200.parts import Workspace
    from stride_b200.parts.context import step_context
    return step_context(entries, workspace or Workspace(DEV, rows), dtype, tokens)


# ---------------------------------------------------------------------------------------------- mechanisms alone
@pytest.mark.parametrize("taps,H,G,D,V,rot,unit,dtype,page", [
    (4, 4, 2, 32, 24, 16, 1, torch.float32, 16), (3, 3, 3, 21, 18, 10, 1, torch.float32, 8), (1, 2, 1, 40, 40, 0, 1, torch.float32, 8),
    (0, 4, 1, 16, 48, 16, 0, torch.float32, 24), (16, 2, 2, 12, 70, 4, 1, torch.float32, 16), (4, 8, 2, 128, 128, 128, 1, BF, 64),
    (2, 6, 2, 64, 64, 32, 1, BF, 32), (5, 5, 5, 9, 7, 2, 0, BF, 8)])
def test_what_stands_in_front_of_the_attention(taps, H, G, D, V, rot, unit, dtype, page):
    """Three requests fed in portions of 1 to 70 tokens beside single ones: q, the cached k and v, the kept and the mixed values, against the
    plain functions; records of slots that another request left are not read at a sequence's start; the record holds the last inputs."""
    from stride_b200.kernels.native import ImmediateProgram
    from stride_b200.parts import Workspace
    g = torch.Generator().manual_seed(taps * 100 + D)
    C, lengths, eps, lam, base = H * D + G * (D + V), [100, 41, 7], 1e-3, 0.3, 700.0
    halo = max(taps - 1, 0)
    conv = torch.randn(C, taps, generator=g) if taps else None
    u = [torch.randn(n, C, generator=g) for n in lengths]
    first = [torch.randn(n, G * V, generator=g) for n in lengths]
    half = rot // 2
    a = torch.arange(256, dtype=F).view(-1, 1) * base ** (-2.0 * torch.arange(half, dtype=F) / max(rot, 1))
    table = torch.stack([a.cos(), a.sin()], -1).float().to(DEV).contiguous() if rot else None
    slots, per = [2, 0, 3], -(-128 // page)
    blocks = torch.randperm(4 * per + 1, generator=g)[:4 * per].view(4, per).to(torch.int32).to(DEV).contiguous()
    record = torch.full((4, max(halo * C, 1)), 1e4, device=DEV)
    taps_dev = conv.T.contiguous().to(DEV) if taps else None
    pages = {m: torch.zeros(4 * per + 1, 2, G, page, max(D, V), dtype=dtype, device=DEV) for m in ("own", "keep", "mix")}
    ws = Workspace(DEV, ROWS)
    got = {m: [[] for _ in lengths] for m in ("q", "keep")}
    fed = [0, 0, 0]
    for step in ([(0, 1), (1, 2)], [(2, 3), (0, 70)], [(1, 1), (0, 1), (2, 1)], [(0, 2), (1, 30)], [(0, 18), (2, 1)], [(1, 8), (2, 2)], [(0, 8)]):
        ctx = _step([(slots[r], n, fed[r]) for r, n in step], dtype, workspace=ws)
        rows = torch.cat([u[r][fed[r]:fed[r] + n] for r, n in step]).to(DEV)
        kept_in = torch.cat([first[r][fed[r]:fed[r] + n] for r, n in step]).to(DEV)
        # the projection's output as three partial sums, of which the kernel sees the total
        parts = torch.stack([rows * 0.5, rows * 0.25, rows * 0.25]).contiguous()
        before = record.clone()
        for m, mode in (("own", 0), ("keep", 1), ("mix", 2)):
            record.copy_(before)
            q = torch.zeros(ctx.n, H * D, dtype=dtype, device=DEV)
            kept = torch.full((ctx.n, G * V), 7.0, device=DEV) if m == "keep" else kept_in
            p = pages[m]
            with ImmediateProgram(ctx, None) as program:
                program.add("short_conv", "sb_op_conv_qkv", [parts, C, 3, 512, taps_dev, taps, record if halo else None, halo * C, table, rot, unit, kept, mode,
                                                             q, dtype, p, blocks, per, page, p.stride(0), p.stride(1), p.stride(2), H, G, D, V, max(D, V)],
                            [eps, lam])
            if m == "keep":
                at = 0
                for r, n in step:
                    got["q"][r].append(q[at:at + n].cpu().double())
                    got["keep"][r].append(kept[at:at + n].cpu().double())
                    at += n
        for r, n in step:
            fed[r] += n
            if halo:
                tail = torch.cat([torch.zeros(halo, C), u[r][:fed[r]]])[-halo:]
                assert (record[slots[r]].view(halo, C).cpu() - tail).abs().max() <= 1e-5
    assert fed == lengths
    tol = 2e-5 if dtype == torch.float32 else 1.2e-2
    for r, n in enumerate(lengths):
        y = plain.short_conv(u[r].double(), conv.double()) if taps else u[r].double()
        q, k, v = y[:, :H * D].view(n, H, D), y[:, H * D:(H + G) * D].view(n, G, D), y[:, (H + G) * D:]
        if rot:
            q, k = plain.rotated(q, base, rot), plain.rotated(k, base, rot)
        if unit:
            q, k = plain.unit_rms(q, eps), plain.unit_rms(k, eps)
        close = lambda have, want, what: (have - want).abs().max() <= tol * max(1.0, float(want.abs().max())) or pytest.fail(f"{what} of request {r}")
        close(torch.cat(got["q"][r]), q.reshape(n, H * D), "queries")
        close(torch.cat(got["keep"][r]), v, "kept values")
        where = blocks[slots[r]].cpu()
        for m, want_v in (("own", v), ("keep", v), ("mix", (1 - lam) * v + lam * first[r].double())):
            cached = pages[m].cpu().double()[where.long()]                           # [per, 2, G, page, row]
            flat = cached.permute(1, 0, 3, 2, 4).reshape(2, per * page, G, max(D, V))
            close(flat[0, :n, :, :D], k, "cached keys")
            close(flat[1, :n, :, :V].reshape(n, G * V), want_v, f"cached values ({m})")


def _attention_case(H, G, D, V, W, taps, g, mixes=True):
    t = {"p.q": torch.randn(H * D, W, generator=g), "p.k": torch.randn(G * D, W, generator=g), "p.v": torch.randn(G * V, W, generator=g),
         "p.o": torch.randn(W, H * V, generator=g) * (H * V) ** -0.5, "p.sink": torch.randn(H, generator=g) + 1.0}
    for r in "qkv":
        t["p." + r] *= W ** -0.5
        if taps:
            t[f"p.{r}.conv"] = torch.randn(t["p." + r].shape[0], taps, generator=g) * 0.5 + 0.3
    if mixes:
        t["p.vmix"] = torch.tensor(0.4)
    return {k: v.to(BF) for k, v in t.items()}


def _attention_part(H, G, D, V, W, m, eps, dtype, t, value_mix):
    from stride_b200.parts import PartSpec, part_class
    rot = m.get("rot")
    names = {r: "p." + r for r in ("q", "k", "v", "o", "sink")}
    if m.get("conv"):
        names.update({f"{r}_conv": f"p.{r}.conv" for r in "qkv"})
    if value_mix:
        names["lambda"] = "p.vmix"
    position = PartSpec("rope", {"head_dim": D, "rotary_dim": rot["dims"], "theta": rot["base"], "exact_angles": True}) if rot else None
    part = part_class("mixer", "conv_attention")(
        PartSpec("conv_attention", {"hidden_size": W, "num_heads": H, "num_kv_heads": G, "key_dim": D, "value_dim": V, "scale": m["scale"], "norm_eps": eps,
                                    "taps": m.get("conv", 0), "qk_unit": True, "position": position, "cap": m.get("softcap", 0.0), "sink": True,
                                    "value_mix": value_mix}, names), _env(dtype))
    assert set(part.tensor_plan()) == set(t)
    part.bind({k: v.to(DEV) for k, v in t.items()})
    return part


def _cache(part, slots, per, page, dtype, g):
    """The mixer's cache: pages handed out in a shuffled order and full of large numbers, records full of them too."""
    from stride_b200.cache.manager import LayerCache
    need = part.cache_need()
    pages_need, record = need if isinstance(need, list) else (need, None)
    blocks = torch.randperm(slots * per + 3, generator=g)[:slots * per].view(slots, per).to(torch.int32).to(DEV).contiguous()
    pages = torch.full((slots * per + 3, 2, pages_need.kv_heads, page, pages_need.head_dim), 1e4, dtype=dtype, device=DEV)
    paged = LayerCache(pages=pages, block_table=blocks, page_size=page)
    if record is None:
        return paged
    return LayerCache(parts=[paged, LayerCache(state=torch.full((slots, *record.state_shape), 1e4, device=DEV))])


@pytest.mark.parametrize("H,G,D,V,W,taps,rot,cap,scale,page,dtype", [
    (4, 2, 22, 27, 60, 3, (10, 50.0), 1.5, 0.5, 8, torch.float32), (3, 3, 64, 64, 96, 4, (32, 1000.0), 4.0, 0.3, 16, torch.float32),
    (2, 1, 16, 40, 40, 0, None, 0.0, 0.4, 8, torch.float32),
    (8, 2, 64, 64, 128, 4, (32, 1000.0), 3.0, 0.15, 64, BF), (4, 4, 128, 128, 128, 3, (128, 500.0), 2.0, 0.1, 16, BF), (16, 1, 64, 64, 64, 2, None, 0.0, 0.1, 8, BF),
    (6, 2, 64, 64, 72, 4, (8, 30.0), 5.0, 0.2, 24, BF), (6, 2, 64, 64, 72, 4, (24, 30.0), 5.0, 0.2, 64, BF),
    (12, 1, 128, 128, 64, 3, (16, 30.0), 4.0, 0.1, 32, BF), (12, 4, 64, 32, 64, 5, (12, 30.0), 3.0, 0.2, 32, BF), (4, 2, 48, 80, 96, 4, (48, 1000.0), 3.0, 0.2, 16, BF), (5, 5, 20, 12, 72, 2, (4, 9.0), 2.0, 0.5, 8, BF)])
def test_attention_alone(H, G, D, V, W, taps, rot, cap, scale, page, dtype):
    """Two mixers, the second of which mixes its values with the first one's: two requests of unequal length fed in portions beside single
    tokens (long enough that a row's keys are folded over several chunks), in every attention kernel the shapes choose."""
    from stride_b200.parts import ResidualStream, Workspace
    g = torch.Generator().manual_seed(H * 1000 + D + V)
    eps, lengths = 1e-4, [620, 61]
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale, "softcap": cap, **({"conv": taps} if taps else {}),
         **({"rot": {"dims": rot[0], "base": rot[1]}} if rot else {})}
    ts = [_attention_case(H, G, D, V, W, taps, g) for _ in range(2)]
    parts = [_attention_part(H, G, D, V, W, m, eps, dtype, t, mode) for t, mode in zip(ts, ("keep", "mix"))]
    assert parts[0]._fixed_heads() == (dtype == BF and D == V and D in (64, 128))
    per = -(-max(lengths) // page)
    caches = [_cache(p, 2, per, page, dtype, g) for p in parts]
    h = [torch.randn(n, W, generator=g).to(BF) for n in lengths]
    ws = Workspace(DEV, ROWS)
    schedule = [[(0, 70), (1, 2)], [(1, 30)], [(0, 1), (1, 1)], [(0, 2), (1, 28)]] + [[(0, 1)]] * 3 + [[(0, 200)], [(0, 3)], [(0, 200)], [(0, 131)]] + [[(0, 1)]] * 10
    fed, got = [0, 0], [[[], []], [[], []]]
    for step in schedule:
        entries = [(r, n, fed[r]) for r, n in step]
        x = torch.cat([h[r][fed[r]:fed[r] + n] for r, n in step]).to(DEV, dtype)
        for k, (part, cache) in enumerate(zip(parts, caches)):      # (the kept values of a step lie in the workspace)
            ctx = _step(entries, dtype, workspace=ws)
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
        y0, own = plain.attention(h[r].double(), ts[0], "p.", m, eps, None, rnd)
        y1, _ = plain.attention(h[r].double(), ts[1], "p.", m, eps, own, rnd)
        for k, want in enumerate((y0, y1)):
            diff = (torch.cat(got[k][r]) - want).abs().max()
            assert diff <= (3e-5 if rnd is None else 2e-2) * float(want.abs().max()), f"mixer {k}, request {r}: {diff}"


@pytest.mark.parametrize("D,page", [(64, 64), (128, 64), (64, 24)])
def test_a_long_context_with_cap_and_sinks(D, page):
    """One decoded token and a short portion over thousands of keys: chunk records folded by a kernel of their own, by the last CTA, in
    clusters; the sinks raised so that a row that forgets its own is far off."""
    from stride_b200.kernels.native import ImmediateProgram
    from stride_b200.parts.attention import emit_tensor_core_attention
    g = torch.Generator().manual_seed(D)
    H, G, cap, scale = 4, 2, 3.0, 0.25
    lengths = [9000, 700, 300, 5]
    per = -(-9000 // page)
    pages = torch.randn(4 * per, 2, G, page, D, generator=g).to(BF).to(DEV)
    blocks = torch.randperm(4 * per, generator=g).view(4, per).to(torch.int32).to(DEV).contiguous()
    sinks = torch.tensor([6.0, 9.0, -3.0, 8.0])
    for entries in ([(0, 1, 8999)], [(0, 1, 8999), (1, 1, 699), (2, 1, 299), (3, 1, 4)], [(1, 1, 699), (3, 1, 4)], [(0, 4, 8996), (1, 40, 660)]):
        n = sum(e[1] for e in entries)
        ctx = _step(entries, BF)
        q = torch.randn(n, H * D, generator=g).to(BF)
        out = torch.zeros(n, H * D, dtype=BF, device=DEV)
        tc5 = page in (16, 32, 64)
        with ImmediateProgram(ctx, None) as program:
            plan = program.plan(H // G, 128 if tc5 else 64, 1, -1)
            emit_tensor_core_attention(program, q.to(DEV), out, pages, blocks, H, G, D, 0, scale, plan, tc5, cap=cap, sinks=sinks.to(DEV))
        torch.cuda.synchronize()
        got, at = out.cpu().double().view(n, H, D), 0
        for slot, count, first in entries:
            seen = pages[blocks[slot].long()].permute(1, 2, 0, 3, 4).reshape(2, G, per * page, D).cpu().double()
            for j in range(count):
                for a in range(H):
                    s = plain.capped(scale * (seen[0, a // 2, :first + j + 1] @ q[at].double().view(H, D)[a]), cap)
                    e = torch.exp(s)
                    want = (e @ seen[1, a // 2, :first + j + 1]) / (e.sum() + torch.exp(sinks[a].double()))
                    assert (got[at, a] - want).abs().max() <= 1e-2 * float(want.abs().max()) + 1e-4, (entries, slot, j, a)
                at += 1


@pytest.mark.parametrize("dtype,D", [(torch.float32, 32), (BF, 64), (BF, 32)])
def test_one_key_that_stands_out_is_never_out_of_sight(dtype, D):
    """One early position's key answers every query with a score near the cap while the others lie far below: it is seen from every later
    position, in portions and decoded, and the result without it or without the cap would be another."""
    from stride_b200.parts import ResidualStream, Workspace
    g = torch.Generator().manual_seed(9)
    H, G, V, W, page, n, loud = 4, 2, D, 64, 16, 330, 21
    m = {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": 16.0 / D, "softcap": 5.0}
    t = _attention_case(H, G, D, V, W, 0, g, mixes=False)
    t["p.q"], t["p.k"] = torch.zeros(H * D, W, dtype=BF), torch.zeros(G * D, W, dtype=BF)
    for a in range(H):                                                  # every query points along its first element ..
        t["p.q"][a * D, 0] = 1.0
    for a in range(G):                                                  # .. and a key does so by what its token has in element 1
        t["p.k"][a * D, 1], t["p.k"][a * D + 1, 2] = 1.0, 1.0
    h = torch.randn(n, W, generator=g)
    h[:, 0], h[:, 1], h[:, 2] = 1.0, 0.0, 1.0
    h[loud, 1], h[loud, 2] = 1.0, 0.0
    h = h.to(BF)
    part = _attention_part(H, G, D, V, W, m, 1e-6, dtype, t, None)
    cache = _cache(part, 1, -(-n // page), page, dtype, g)
    rows, ws, at = [], Workspace(DEV, ROWS), 0
    for k in (50, 2, 153, 1, 1, 1, 1, 31, 90):
        ctx = _step([(0, k, at)], dtype, workspace=ws)
        stream = ResidualStream(torch.zeros(k, W, device=DEV))
        part.forward(ctx, h[at:at + k].to(DEV, dtype), stream, cache)
        stream.fold()
        rows.append(stream.h.cpu().double())
        at += k
    assert at == n
    got, rnd = torch.cat(rows), None if dtype == torch.float32 else BF
    want, _ = plain.attention(h.double(), t, "p.", m, 1e-6, None, rnd)
    assert (got - want).abs().max() <= (3e-5 if rnd is None else 2e-2) * float(want.abs().max())
    without = h.clone()
    without[loud, 1], without[loud, 2] = 0.0, 1.0
    for other in (plain.attention(without.double(), t, "p.", m, 1e-6, None, rnd)[0], plain.attention(h.double(), t, "p.", {**m, "softcap": 0.0}, 1e-6, None, rnd)[0]):
        assert float((other - want)[loud + 1:].abs().max(dim=1).values.min()) > 0.04 * float(want.abs().max())


@pytest.mark.parametrize("n,W,ff,dtype", [(5, 40, 24, torch.float32), (64, 100, 37, BF), (16, 64, 40, BF), (200, 128, 200, BF), (700, 256, 512, BF),
                                          (700, 64, 1024, BF), (300, 512, 4096, BF)])
def test_clamped_gate(n, W, ff, dtype):
    """The gated feed-forward with clamps in every form of the product, with activations on both sides of both clamps; few rows in the bits of
    many."""
    from stride_b200.parts import PartSpec, ResidualStream, Workspace, part_class
    g = torch.Generator().manual_seed(n + ff)
    limit = 0.75
    t = {"p.gate": torch.randn(ff, W, generator=g) * 1.5 * W ** -0.5, "p.up": torch.randn(ff, W, generator=g) * 1.5 * W ** -0.5,
         "p.down": torch.randn(W, ff, generator=g) * ff ** -0.5}
    t = {k: v.to(BF) for k, v in t.items()}
    part = part_class("feed_forward", "gated")(PartSpec("gated", {"hidden_size": W, "intermediate_size": ff, "activation": "clamped", "limit": limit,
                                                                  "slope": 1.702}, {r: "p." + r for r in ("gate", "up", "down")}), _env(dtype, 1024))
    part.bind({k: v.to(DEV) for k, v in t.items()})
    h = torch.randn(n, W, generator=g).to(BF)
    ws = Workspace(DEV, 1024)

    def run(rows):
        ctx = _step([(0, len(rows), 0)], dtype, rows=1024, workspace=ws)
        stream = ResidualStream(torch.zeros(len(rows), W, device=DEV))
        part.forward(ctx, h[rows].to(DEV, dtype), stream)
        stream.fold()
        return stream.h.cpu()

    got = run(list(range(n)))
    want = plain.clamped_gated(h.double(), t, "p.", limit, None if dtype == torch.float32 else BF)
    assert (got.double() - want).abs().max() <= (2e-5 if dtype == torch.float32 else 1.5e-2) * float(want.abs().max())
    for wrong in (limit * 1.05, 1e9):
        assert (plain.clamped_gated(h.double(), t, "p.", wrong) - want).abs().max() > 0.02 * float(want.abs().max())
    assert torch.equal(run([0, n - 1]), got[[0, n - 1]])


def _moe_case(W, E, top, ff, shared, g, scale=0.3):
    t = {"p.router": (torch.randn(E, W, generator=g) * W ** -0.5).to(BF)}
    for name, F_ in [*((f"p.e{e}.", ff) for e in range(E)), *([("p.shared.", shared)] if shared else [])]:
        for r, shape in (("gate", (F_, W)), ("up", (F_, W)), ("down", (W, F_))):
            t[name + r] = (torch.randn(*shape, generator=g) * scale).to(BF)
    names = {r: tuple(f"p.e{e}.{r}" for e in range(E)) for r in ("gate", "up", "down")}
    if shared:
        t["p.shared.sg"] = (torch.randn(1, W, generator=g) * 0.3).to(BF)
        names.update({f"shared_{r}": f"p.shared.{r}" for r in ("gate", "up", "down", "sg")})
    params = {"hidden_size": W, "intermediate_size": ff, "experts": E, "top": top, "shared": shared, "shared_gate": bool(shared)}
    return t, params, {"router": "p.router", **names}


@pytest.mark.parametrize("W,E,top,ff,shared,n,dtype", [
    (24, 5, 2, 40, 0, 23, torch.float32), (72, 3, 3, 33, 17, 9, torch.float32), (64, 1, 1, 24, 40, 50, torch.float32),
    (64, 4, 1, 72, 40, 200, BF), (136, 6, 3, 48, 0, 256, BF), (64, 40, 2, 24, 64, 37, BF), (256, 3, 2, 200, 128, 256, BF), (100, 4, 2, 36, 12, 40, BF),
    (64, 300, 8, 16, 24, 130, BF), (64, 7, 7, 16, 0, 1, BF), (64, 33, 2, 16, 8, 5, BF)])
def test_experts_behind_a_sigmoid_router(W, E, top, ff, shared, n, dtype):
    """The part alone, adding to a stream (blocks that do not fold its sources themselves), against the plain experts; half of the rows alike,
    experts that nobody chose, a token alone in the same bits."""
    from stride_b200.parts import PartSpec, ResidualStream, Workspace, part_class
    g = torch.Generator().manual_seed(W + E)
    t, params, names = _moe_case(W, E, top, ff, shared, g)
    part = part_class("feed_forward", "sigmoid_experts")(PartSpec("sigmoid_experts", params, names), _env(dtype))
    assert set(part.tensor_plan()) == set(t)
    part.bind({k: v.to(DEV) for k, v in t.items()})
    assert part.tensor_core == (dtype == BF and W % 8 == 0 and ff % 8 == 0)
    ws = Workspace(DEV, ROWS)
    h = torch.randn(n, W, generator=g)
    h[: n // 2] = h[0]
    h = h.to(BF)
    mlp = {"router": {"experts": E, "top": top}, **({"shared": {"ff": shared}} if shared else {})}
    base = torch.randn(n, W, generator=g)

    def run(rows):
        ctx = _step([(1, len(rows), 0)], dtype, workspace=ws)
        stream = ResidualStream(base[rows].to(DEV))
        part.forward(ctx, h[rows].to(DEV, dtype), stream)
        stream.fold()
        return stream.h.cpu()

    got = run(list(range(n)))
    want = plain.experts(h.double(), t, "p.", mlp, None if dtype == torch.float32 else BF)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    # (rows whose last chosen and first refused expert are closer than 32-bit sums tell apart may go either way: none here)
    z = torch.topk(h.double() @ t["p.router"].double().T, min(top + 1, E)).values
    assert E == top or float((z[:, top - 1] - z[:, top]).min()) > 1e-5
    assert (got.double() - base.double() - want).abs().max() <= tol * float(want.abs().max())
    for i in sorted({0, n // 2, n - 1}):
        assert torch.equal(run([i])[0], got[i]), f"row {i} alone differs from the row in company"


@pytest.mark.parametrize("W", [92, 64, 2048, 33])
def test_norms_on_results_with_row_factors_and_a_second_output(W):
    """dst += gain y / rms(y) with y = ca a + cb row_factor b from buffers and partial sums; the new rows once more as bfloat16."""
    from stride_b200.kernels.native import ImmediateProgram
    from stride_b200.parts.branch import ALWAYS, emit_fold
    g = torch.Generator().manual_seed(W)
    n, eps = 9, 1e-3
    dev = lambda t: t.to(DEV).contiguous()
    dst, a, pa, pb, rf, gain = (torch.randn(*s, generator=g) for s in ((n, W), (n, W), (3, n, W), (9, n, W), (n,), (W,)))
    for norm in (eps, None):
        ctx = _step([(0, n, 0)], BF)
        copy = torch.zeros(n, W, dtype=BF, device=DEV)
        h = dev(dst)
        with ImmediateProgram(ctx, None) as program:
            program.h = h
            sources = [(dev(a), (dev(pa), 3, W, ALWAYS), 0.5), (None, (dev(pb), 9, W, ALWAYS), dev(rf))]
            emit_fold(program, sources, dev(gain), W, norm_eps=norm, copy=copy if norm else None)
        y = 0.5 * (a.double() + pa.double().sum(0)) + rf.double()[:, None] * pb.double().sum(0)
        want = dst.double() + gain.double() * (plain.unit_rms(y, eps) if norm else y)
        assert (h.cpu().double() - want).abs().max() <= 2e-5 * float(want.abs().max())
        if norm:
            assert torch.equal(copy, h.to(BF))


# ---------------------------------------------------------------------------------------------- whole models
def _engine(model_dir, dtype, page, pages, rows=ROWS, slots=4, **kw):
    from stride_b200.engine.engine import Engine, EngineOptions
    return Engine(model_dir, EngineOptions(dtype=dtype, max_rows=rows, max_full_rows=rows, max_slots=slots, kv_pages=pages,
                                           page_size=page, max_context=pages * page, device=DEV, **kw))


def _noise(cfg, w, tokens):
    """The largest |plain with bfloat16 rounding - plain exact| over the sequence's logits."""
    return float((plain.run(cfg, w, tokens, BF) - plain.run(cfg, w, tokens)).abs().max())


def _steady(cfg, w, tokens, margin=2e-2):
    """False if some token's last chosen and first refused expert are so close that bfloat16 rounding may tell them apart the other way."""
    near = [False]
    inner = plain.route

    def watch(h, tensors, p, top):
        z = h @ plain.w(tensors, p + "router").T
        if z.shape[1] > top:
            v = torch.topk(z, top + 1).values
            near[0] = near[0] or float((v[:, top - 1] - v[:, top]).min()) < margin
        return inner(h, tensors, p, top)

    plain.route = watch
    try:
        plain.run(cfg, w, tokens)
    finally:
        plain.route = inner
    return not near[0]


def test_every_layer_against_the_plain_residual(mezadra_dirs):
    """The residual after every layer, in 32-bit, for a prompt in one step."""
    from stride_b200.engine.engine import StepEntry
    for name in MEZADRA:
        cfg, w = load_plain(mezadra_dirs[name])
        toks = random_tokens(cfg["vocab"], 37, 12)
        want = []
        plain.run(cfg, w, toks, after_layer=lambda i, x: want.append(x))
        eng = _engine(mezadra_dirs[name], "float32", MEZADRA[name][2], 8, native_step=False)
        slot = eng.cache.acquire_slot()
        eng.cache.ensure(slot, len(toks))
        seen = []
        for block in eng.model.blocks:
            def run(ctx, stream, cache, inner=block.forward):
                inner(ctx, stream, cache)
                assert stream.pending is None
                seen.append(stream.h[:len(toks)].cpu().double())
            block.forward = run
        eng.step([StepEntry(slot, 0, toks, list(range(len(toks))))])
        assert len(seen) == len(want) == len(cfg["layers"])
        for k, (a, b) in enumerate(zip(seen, want)):
            assert (a - b).abs().max() <= 2e-4 * max(1.0, float(b.abs().max())), f"{name}: the residual after layer {k} differs"


LENGTHS = {"M": [70, 130, 45, 33, 2], "N": [300, 65, 140, 129, 40], "O": [48, 90, 17, 64, 5], "Q": [66, 40, 90, 34, 3]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(MEZADRA))
def test_replay_modes(name, dtype, mezadra_dirs, tmp_path):
    """Through bin/trace_run: whole; all but the last 32 tokens, then token by token; portions down to two tokens; mixed batches in a
    pool so small that pages are used again, four slots for five requests. Against the plain implementation (bfloat16: rounding at the
    same places; the largest deviation within the largest rounding noise of the same sequence, for requests whose experts rounding cannot
    change), and all four in the same bits."""
    cfg, _, page = MEZADRA[name]
    vocab = cfg["vocab"]
    pcfg, w = load_plain(mezadra_dirs[name])
    reqs = [random_tokens(vocab, n, 300 + i) for i, n in enumerate(LENGTHS[name])]
    bf = dtype == "bfloat16"
    want = [plain.run(pcfg, w, r, BF if bf else None).float() for r in reqs]
    tols = [_noise(pcfg, w, r) if bf else logit_tolerance(dtype, want[i]) for i, r in enumerate(reqs)]
    per = lambda n: -(-n // page) * page
    longest = sorted((per(len(r)) for r in reqs), reverse=True)
    pool = max(longest[0] + longest[1] + page, 4 * page)
    tr = TraceRun(mezadra_dirs[name], dtype, tmp_path, pool, page, extra=("--kv-shuffle", "5"))
    bits, seen = _Bits(), [[] for _ in reqs]

    def compare(got, i, a, b, what):
        bits.check(i, a, got, f"{name} {what}")
        diff = (got - want[i][a:b]).abs().max(dim=1).values
        if not bf:
            assert diff.max() <= tols[i], f"{name} {dtype} {what}: max |diff| {diff.max():.3e} > {tols[i]:.3e} at {a + int(diff.argmax())}"
        seen[i].append(diff)

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
    if bf:
        for i, r in enumerate(reqs):
            d = torch.cat(seen[i])
            if _steady(pcfg, w, r):
                assert d.max() <= tols[i], f"{name} request {i}: max |diff| {d.max():.3e} > {tols[i]:.3e}"
            else:       # an expert that rounding may change moves single tokens (and what they are seen by) as far as that expert reaches
                assert d.median() <= tols[i], f"{name} request {i}: median |diff| {d.median():.3e} > {tols[i]:.3e}"


def test_every_key_counts_and_agrees(mezadra_dirs):
    """With attention close to uniform every key carries weight (that another first token shows at every later position is checked on the
    plain implementation): the engine agrees in a prompt whose portions straddle pages and decoding token by token."""
    from stride_b200.engine.engine import StepEntry
    for name, page in (("MU", 16), ("NU", 32)):
        cfg, w = load_plain(mezadra_dirs[name])
        toks = random_tokens(cfg["vocab"], 150, 77)
        want = plain.run(cfg, w, toks).float()
        eng = _engine(mezadra_dirs[name], "float32", page, 10, slots=1)
        slot = eng.cache.acquire_slot()
        got, at = [], 0
        for n in (50, 2, 31, 17):
            eng.cache.ensure(slot, at + n)
            got.append(eng.step([StepEntry(slot, at, toks[at:at + n], list(range(n)))]).cpu().clone())
            at += n
        for t in range(at, 150):
            eng.cache.ensure(slot, t + 1)
            got.append(eng.step([StepEntry(slot, t, [toks[t]], [0])]).cpu().clone())
        assert (torch.cat(got) - want).abs().max() <= logit_tolerance("float32", want)
        eng.cache.check()


def test_the_first_tokens_of_a_sequence(mezadra_dirs):
    """Positions 0, 1, 2, .. one by one, and as portions of two, in a slot that another request used: a sink beside a single key, taps that
    reach in front of the sequence, a record and a state that another request left."""
    from stride_b200.engine.engine import StepEntry
    for name in sorted(MEZADRA):
        cfg, w = load_plain(mezadra_dirs[name])
        eng = _engine(mezadra_dirs[name], "float32", MEZADRA[name][2], 16, slots=1)
        for seed, size in ((3, 1), (4, 1), (5, 2), (6, 3)):
            toks = random_tokens(cfg["vocab"], 12, seed)
            want = plain.run(cfg, w, toks).float()
            slot = eng.cache.acquire_slot()
            got = []
            for t in range(0, 12, size):
                eng.cache.ensure(slot, t + size)
                got.append(eng.step([StepEntry(slot, t, toks[t:t + size], list(range(size)))]).cpu().clone())
            assert (torch.cat(got) - want).abs().max() <= logit_tolerance("float32", want), (name, seed)
            eng.cache.release_slot(slot)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_slot_reuse(dtype, mezadra_dirs):
    """A short prompt, then 400 tokens one by one, against the plain implementation; then the same slot and pages for another request."""
    from stride_b200.engine.engine import StepEntry
    cfg, w = load_plain(mezadra_dirs["NU"])
    eng = _engine(mezadra_dirs["NU"], dtype, 32, 13, slots=1)
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
        diff = (torch.cat(got) - want).abs().max(dim=1).values
        if bf:
            assert diff.median() <= 0.5 * _noise(cfg, w, toks)
        else:
            assert diff.max() <= logit_tolerance("float32", want)
        eng.cache.release_slot(slot)
        eng.cache.check()


def test_a_far_token_shows(tmp_path):
    """Another token near the start moves the plain logits 300 tokens later far beyond the tolerance; the engine, fed in portions that cut
    pages and then token by token, agrees."""
    from stride_b200.engine.engine import StepEntry

    def loud(tensors):
        for n in tensors:
            if n.endswith("mix.sink"):
                tensors[n] = tensors[n] - 3.0
        e = tensors["embed"].float()
        e[7] *= 8.0
        tensors["embed"] = e.to(tensors["embed"].dtype)

    folder = write_model(tmp_path / "far", "N", transform=loud, config=near_uniform(MEZADRA["N"][0]))
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
        at += n
    for t in range(at, len(toks)):
        eng.cache.ensure(slot, t + 1)
        got.append(eng.step([StepEntry(slot, t, [toks[t]], [0])]).cpu().clone())
    assert (torch.cat(got) - want).abs().max() <= tol


@pytest.mark.parametrize("native", [True, False])
def test_batches_of_unequal_requests_against_each_alone(mezadra_dirs, native):
    """Four requests of unequal length in one step, then single tokens of some beside portions of others: every logit has the bits of
    the request run alone; the native step program and the part-by-part driver agree."""
    from stride_b200.engine.engine import StepEntry
    for name in ("N", "M", "Q"):
        cfg, _, page = MEZADRA[name]
        reqs = [random_tokens(cfg["vocab"], n, 40 + n) for n in (150, 3, 64, 31)]
        for dtype in ("float32", "bfloat16"):
            eng = _engine(mezadra_dirs[name], dtype, page, 48, native_step=native)
            assert (eng._program is not None) == native
            other = _engine(mezadra_dirs[name], dtype, page, 48)             # alone: always the native program
            alone = []
            for r in reqs:
                slot = other.cache.acquire_slot()
                other.cache.ensure(slot, len(r))
                alone.append(other.step([StepEntry(slot, 0, r, list(range(len(r))))]).cpu().clone())
                other.cache.release_slot(slot)
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
    folder = write_model(tmp_path / "m", "N")
    toks = random_tokens(MEZADRA["N"][0]["vocab"], 900, 5)
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


def test_greedy_generation_through_the_entry_point(mezadra_dirs):
    """LLM.generate with its scheduler (three requests on two slots, prompts cut into portions, decode steps replayed from CUDA
    graphs): the tokens of greedy decoding with the plain implementation."""
    from stride_b200 import LLM
    cfg, w = load_plain(mezadra_dirs["M"])
    prompts = [random_tokens(cfg["vocab"], n, 500 + n) for n in (5, 41, 23)]
    llm = LLM(mezadra_dirs["M"], dtype="float32", concurrency=2, max_rows=32, prefill_chunk=8, kv_pages=12, page_size=16,
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
    bf = LLM(mezadra_dirs["N"], dtype="bfloat16", concurrency=4, max_rows=64, prefill_chunk=16, kv_pages=16, page_size=32,
             max_slots=4, max_context=256, device=DEV)
    outs = bf.generate([random_tokens(MEZADRA["N"][0]["vocab"], n, n) for n in (70, 9, 33, 120, 64)], max_new_tokens=8)
    assert all(len(o.tokens) == 8 for o in outs)


def test_a_preempted_request_generates_the_same_tokens(mezadra_dirs):
    """A pool too small for all requests at once: the youngest is taken off its slot and pages and recomputed from its first token, in a slot
    whose record and state another request left."""
    from stride_b200 import LLM
    cfg = MEZADRA["M"][0]
    prompts = [random_tokens(cfg["vocab"], n, 700 + n) for n in (30, 28, 33)]
    kw = dict(dtype="float32", concurrency=3, max_rows=64, prefill_chunk=16, page_size=16, max_slots=3, max_context=96, device=DEV)
    roomy = LLM(mezadra_dirs["M"], kv_pages=24, **kw).generate(prompts, max_new_tokens=24)
    tight = LLM(mezadra_dirs["M"], kv_pages=8, **kw).generate(prompts, max_new_tokens=24)
    assert [o.tokens for o in tight] == [o.tokens for o in roomy]


def test_command_line_generates_what_the_entry_point_generates(mezadra_dirs, tmp_path):
    """bin/stride_cli on a Mezadra folder (greedy, float32 and bfloat16): the tokens of LLM.generate."""
    import json
    import subprocess
    import sys
    from conftest import ROOT
    from stride_b200 import LLM
    cfg = MEZADRA["O"][0]
    prompts = [random_tokens(cfg["vocab"], n, 900 + n) for n in (3, 50, 21)]
    (tmp_path / "in.jsonl").write_text("".join(json.dumps({"id": i, "tokens": p}) + "\n" for i, p in enumerate(prompts)))
    for path, dtype in (("exact", "float32"), ("tc", "bfloat16")):
        out = tmp_path / f"out_{path}.jsonl"
        subprocess.run([sys.executable, str(ROOT / "bin" / "stride_cli"), "--model", str(mezadra_dirs["O"]), "--input", str(tmp_path / "in.jsonl"),
                        "--output", str(out), "--max-new", "6", "--concurrency", "2", "--max-rows", "32", "--prefill-chunk", "16",
                        "--kv-blocks", "24", "--page-size", "8", "--max-slots", "4", "--max-context", "128", "--path", path], check=True, timeout=600)
        got = [json.loads(l) for l in out.read_text().splitlines()]
        llm = LLM(mezadra_dirs["O"], dtype=dtype, concurrency=2, max_rows=32, prefill_chunk=16, kv_pages=24, page_size=8, max_slots=4,
                  max_context=128, device=DEV)
        want = llm.generate(prompts, max_new_tokens=6)
        assert [g["tokens"] for g in got] == [w.tokens for w in want] and all(g["finish"] == "length" for g in got)


@pytest.mark.parametrize("seed", range(41, 53))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Whole, and in portions down to one token, in 32-bit against the plain implementation and in bfloat16 in equal bits between the two ways
    of feeding."""
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
                at += n
            got.append(torch.cat(rows))
        assert torch.equal(got[0], got[1]), f"seed {seed} {dtype}: in portions it differs from the whole"
        if dtype == "float32":
            assert (got[0] - want).abs().max() <= logit_tolerance("float32", want), f"seed {seed}: {cfg}"
        else:
            diff = (got[0] - plain.run(pcfg, w, toks, BF).float()).abs().max(dim=1).values
            assert diff.median() <= _noise(pcfg, w, toks)
            assert not _steady(pcfg, w, toks) or diff.max() <= 2.0 * _noise(pcfg, w, toks)
