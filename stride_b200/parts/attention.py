"""Grouped-query attention over the paged cache.

One step of it, for all tokens of the batch at once: q, k, v = W x; rotate q and k
by the position encoding; append k and v to the request's pages; every token then
attends to the keys of its own request at positions first..pos (its own included),
first = 0 or pos - window + 1; the result goes through the output projection
into the residual. Order and formulas as in arhaamatiq/stride (Qkv: src/kernels.cu:204-284;
attention: src/kernel_common.h:90-309; scale = float(pow(double(D), -0.5)), src/engine.cpp:151;
output projection added to the residual: src/kernels.cu:294-325). The token's own key is in the
cache before attention runs, so a portion of a prompt needs no mask tensor.
"""
from __future__ import annotations

import math

import numpy as np
import torch

from ..kernels import ops
from ..kernels.linear import Linear
from ..kernels.native import NO_PHASE
from .base import CacheNeed, Mixer, part_class, register_part
from .spec import TensorPlan


def page_where(pages, table) -> list:
    return [pages, table, table.shape[1], pages.shape[3], pages.stride(0), pages.stride(1), pages.stride(2)]


def tensor_core_head(dtype, num_heads: int, num_kv_heads: int, head_dim: int) -> bool:
    """True if the tensor-core attention kernels with heads of fixed size take this shape."""
    return dtype == torch.bfloat16 and head_dim in (64, 128) and num_heads // num_kv_heads <= 16


def emit_tensor_core_attention(program, q, out, pages, table, H: int, G: int, D: int, window: int, scale: float, plan: int, tc5: bool,
                               projected=None, cap: float = 0.0, sinks=None) -> None:
    """Prompt portions on the tcgen05 kernel where the page size allows it (`tc5`; else, and decoded tokens and very short portions always,
    on the mma.sync kernels), each finding its share of the step in the step's tile plan. projected: (q | k | v partial sums, their width,
    K ranges, rotation table) where the decode kernel may rotate and append itself. cap: scores are capped softly; sinks: a term exp(sink)
    per head in the denominator."""
    ws, where = program.workspace, page_where(pages, table)
    if tc5:
        program.add("attention_tc5", "sb_op_attention_tc5", [q, out, pages, pages.shape[0], *where[1:], H, G, D, window, plan, sinks], [scale, cap],
                    chain=NO_PHASE)
    # the decode kernel's chunk records: as many as the step's decode entries and their longest context need
    need = ops.attention_tc_scratch
    scratch = program.growing_buffer("attn.scratch", torch.float32, (plan, G, D), lambda step: need(step.plan[plan].items, G, step.plan[plan].chunks, D))
    counters = ws.raw("attn.counters", (ws.max_tokens * G,), torch.int32)
    qkv, width, S, cos_sin = projected or (None, 0, 1, None)
    phase = None
    if projected is not None:
        phase = lambda chain: chain.attention(qkv, S, cos_sin, out, pages, table, scratch, counters, H, G, D, window, scale, plan)
    program.add("attention_tc", "sb_op_attention_tc",
                [q, out, *where, scratch, 0, counters, H, G, D, window, plan, int(tc5), qkv, width, S, program.few_tokens, cos_sin, sinks],
                [scale, cap], chain=phase)


@register_part("mixer", "attention")
class AttentionMixer(Mixer):
    """params: hidden_size, num_heads, num_kv_heads, head_dim, window (0 = all keys),
    position (a PartSpec of category "position", or None), scale (default head_dim ** -0.5),
    values_from_keys (True: there is no value projection; a token's values are its keys as projected, before rotation).
    tensors: q, k, v (unless values_from_keys), o."""
    graph_safe = True


    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.num_heads = int(p["num_heads"])
        self.num_kv_heads = int(p["num_kv_heads"])
        self.head_dim = int(p["head_dim"])
        self.window = int(p.get("window", 0) or 0)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"attention: {self.num_heads} heads do not divide into {self.num_kv_heads} key/value heads")
        scale = p.get("scale")
        self.scale = float(np.float32(math.pow(float(self.head_dim), -0.5))) if scale is None else float(scale)
        pos = p.get("position")
        self.position = part_class("position", pos.kind)(pos, env) if pos is not None else None
        self.values_from_keys = bool(p.get("values_from_keys", False))
        self.qkv = self.o = None

    @property
    def qkv_width(self):
        return (self.num_heads + (1 if self.values_from_keys else 2) * self.num_kv_heads) * self.head_dim

    def tensor_plan(self):
        t, D = self.spec.tensors, self.head_dim
        plan = {t["q"]: TensorPlan((self.num_heads * D, self.hidden)),
                t["k"]: TensorPlan((self.num_kv_heads * D, self.hidden)),
                t["o"]: TensorPlan((self.hidden, self.num_heads * D))}
        if not self.values_from_keys:
            plan[t["v"]] = TensorPlan((self.num_kv_heads * D, self.hidden))
        if self.position is not None:
            plan.update(self.position.tensor_plan())      # a position part may have tensors of its own (a learned table)
        return plan

    def bind(self, tensors):
        t = self.spec.tensors
        ws = [tensors[t[r]] for r in (("q", "k") if self.values_from_keys else ("q", "k", "v"))]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.to(torch.float32) for w in ws]
        self.qkv = Linear(torch.cat(ws, dim=0), self.env.compute_dtype)
        self.o = Linear(tensors[t["o"]], self.env.compute_dtype)
        if self.position is None:
            # No rotation: a table of cos = 1, sin = 0 is never read because rotary_dim is 0.
            self._cos_sin, self._rotary = torch.zeros(1, device=self.env.device), 0
        else:
            self.position.bind(tensors)
            table, rotary = getattr(self.position, "cos_sin", None), getattr(self.position, "rotary_dim", None)
            if not isinstance(table, torch.Tensor) or rotary is None or table.dim() != 3 or table.shape[-1] != 2 \
                    or rotary % 2 or not 0 <= rotary <= self.head_dim or (rotary and table.shape[1] != rotary // 2):
                raise TypeError(f"the position part '{self.spec.params['position'].kind}' does not offer what the attention mixer's kernels "
                                f"read: cos_sin [positions, rotary_dim / 2, 2] float32 and an even rotary_dim <= head_dim {self.head_dim} "
                                f"(see parts.base.PositionEncoding); an encoding of another nature needs a mixer of its own")
            self._cos_sin, self._rotary = table, int(rotary)

    def weight_bytes(self):
        return self.qkv.weight_bytes() + self.o.weight_bytes()

    def cache_need(self):
        return CacheNeed("pages", kv_heads=self.num_kv_heads, head_dim=self.head_dim, window=self.window,
                         dtype=self.env.act_dtype)

    def kernel_libraries(self):
        if self.env.compute_dtype != torch.bfloat16:
            return {"gemm_f32", "elementwise", "attention_generic"}
        G = self.num_heads // self.num_kv_heads
        if self.head_dim in (64, 128) and G <= 16:
            return {"gemm_tc", "elementwise", "attention_tc", "attention_tc5"}
        return {"gemm_tc", "elementwise", "attention_generic"}

    def forward(self, ctx, x, stream, cache):
        n, ws, D = ctx.n, ctx.workspace, self.head_dim
        qkv = self.qkv.forward_partials(x, ws.raw("attn.qkv", (self.qkv.partial_elems(ws.max_tokens),), torch.float32))
        mixed = ws.get("attn.out", n, (self.num_heads * D,), ctx.act_dtype)
        G = self.num_heads // self.num_kv_heads
        tensor_core = tensor_core_head(ctx.act_dtype, self.num_heads, self.num_kv_heads, D)
        plan = None
        if tensor_core:
            tc5 = ops.attention_tc5_supported(self.num_heads, self.num_kv_heads, D, cache.page_size)
            plan = ctx.tile_plan(G, 128 if tc5 else 64)
        if (plan is not None and plan[1] == 0 and cache.writes and self._rotary == D and not self.values_from_keys
                and plan[2] * self.num_kv_heads * plan[3] <= ops.attention_decode_rope_limit()):
            # only decoded tokens and very short portions, few enough for all CTAs to run at once: rotation and append
            # happen inside the decode kernel (the same bits; with more CTAs than that the separate kernel is faster)
            work, _, n_items, chunks = plan
            scratch = ws.grow("attn.scratch", ops.attention_tc_scratch(n_items, self.num_kv_heads, chunks, D), torch.float32)
            counters = ws.raw("attn.counters", (ws.max_tokens * self.num_kv_heads,), torch.int32)
            ops.attention_decode_rope(qkv, self._cos_sin, mixed, cache.pages, cache.block_table, ctx.entry_meta, work, n_items,
                                      chunks, scratch, counters, self.num_heads, self.num_kv_heads, D, self.window, self.scale)
            self.o.forward_add(mixed, stream, ws.raw("attn.o_partials", (self.o.partial_elems(ws.max_tokens),), torch.float32))
            return
        q = ws.get("attn.q", n, (self.num_heads * D,), ctx.act_dtype)
        ops.rope_append(qkv, ctx.positions, ctx.slots, self._cos_sin, self._rotary, q, cache.pages, cache.block_table,
                        self.num_heads, self.num_kv_heads, D, write_kv=cache.writes, values_from_keys=self.values_from_keys)
        if tensor_core:
            # prompt portions: the tcgen05 kernel where the page size allows it (tiles of 128 rows), else mma.sync (64 rows);
            # decoded tokens and very short portions: the split-key decode kernel
            work, n_tiles, n_items, chunks = plan
            if tc5 and n_tiles:
                ops.attention_tc5(q, mixed, cache.pages, cache.block_table, ctx.entry_meta, work, n_tiles, self.num_heads,
                                  self.num_kv_heads, D, self.window, self.scale)
                work, n_tiles = work[2 * n_tiles:], 0
            if n_tiles or n_items:
                scratch = ws.grow("attn.scratch", ops.attention_tc_scratch(n_items, self.num_kv_heads, chunks, D), torch.float32)
                counters = ws.raw("attn.counters", (ws.max_tokens * self.num_kv_heads,), torch.int32)
                ops.attention_tc(q, mixed, cache.pages, cache.block_table, ctx.entry_meta, work, n_tiles, n_items, chunks,
                                 scratch, self.num_heads, self.num_kv_heads, D, self.window, self.scale, counters=counters)
        else:
            ops.attention_generic(q, mixed, cache.pages, cache.block_table, ctx.positions, ctx.slots,
                                  self.num_heads, self.num_kv_heads, D, self.window, self.scale)
        self.o.forward_add(mixed, stream, ws.raw("attn.o_partials", (self.o.partial_elems(ws.max_tokens),), torch.float32))

    def emit(self, program, x, cache):
        """`forward` as operations of the native step program: the projection, then rotation and append, the
        attention kernels that this shape takes (each finds its share of the step in the step's tile plan, or skips),
        the output projection."""
        ws, env, D = program.workspace, self.env, self.head_dim
        act, T = env.act_dtype, ws.max_tokens
        qkv = ws.raw("attn.qkv", (self.qkv.partial_elems(T),), torch.float32)
        S = self.qkv.emit_partials(program, x, qkv)
        mixed = ws.get("attn.out", T, (self.num_heads * D,), act)
        q = ws.get("attn.q", T, (self.num_heads * D,), act)
        G = self.num_heads // self.num_kv_heads
        tensor_core = tensor_core_head(act, self.num_heads, self.num_kv_heads, D)
        pages, table = cache.pages, cache.block_table
        where = page_where(pages, table)
        plan = -1
        if tensor_core:
            tc5 = ops.attention_tc5_supported(self.num_heads, self.num_kv_heads, D, cache.page_size)
            fused = cache.writes and self._rotary == D and not self.values_from_keys
            plan = program.plan(G, 128 if tc5 else 64, self.num_kv_heads, ops.attention_decode_rope_limit() if fused else -1)
        # (in a step of decoded tokens only, rotation and append can happen inside the attention kernel: the decode chain
        # counts on it, so it takes this mixer only with a fully rotated head and a cache of its own)
        program.add("elementwise", "sb_op_rope_append",
                    [qkv, self.qkv_width, S, program.few_tokens, self._cos_sin, self._rotary, q, q.dtype, pages, pages.dtype, table,
                     table.shape[1], pages.shape[3], pages.stride(0), pages.stride(1), pages.stride(2), self.num_heads,
                     self.num_kv_heads, D, int(cache.writes), plan, int(self.values_from_keys)],
                    chain=NO_PHASE if tensor_core and fused else None)
        if tensor_core:
            emit_tensor_core_attention(program, q, mixed, pages, table, self.num_heads, self.num_kv_heads, D, self.window, self.scale, plan, tc5,
                                       projected=(qkv, self.qkv_width, S, self._cos_sin))
        else:
            program.add("attention_generic", "sb_op_attention_generic",
                        [q, mixed, q.dtype, *where, self.num_heads, self.num_kv_heads, D, self.window], [self.scale])
        self.o.emit_add(program, mixed, ws.raw("attn.o_partials", (self.o.partial_elems(T),), torch.float32))
