"""Softmax attention over the paged cache whose q, k and v pass a short causal convolution over time (kernels: csrc/short_conv.cu in front;
csrc/attention_tc5.cu and attention_tc.cu for heads of 64 or 128 in the bfloat16 engine, csrc/masked_attention.cu otherwise).

q, k, v = W x, no biases; each channel of them convolved over the last `taps` tokens (the last tap the current token's, zeros before the
start). The first `rotary_dim` elements of every q and k head may be rotated by the position, and every head of them may then be divided by
its root mean square (no gain). score = scale q.k, softly capped, c tanh(score / c), where the design has a cap; i sees every j <= i (or
those within a window); the softmax's denominator may hold one more term exp(sink) per head.

Values may be mixed across layers: one mixer of a step keeps its values (`value_mix` "keep"), later ones (`value_mix` "mix") cache
(1 - lambda) v + lambda v_kept of the same token, lambda a stored number.

Per request the record [taps - 1, channels] float32 holds the convolution's last inputs, beside the pages of keys and values."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..kernels.linear import Linear
from ..kernels.native import ImmediateProgram
from .base import CacheNeed, Mixer, part_class, register_part
from .attention import emit_tensor_core_attention, tensor_core_head
from .masked_attention import _emit_attend, _page_where
from .spec import TensorPlan

MAX_TAPS = 16


@register_part("mixer", "conv_attention")
class ConvAttentionMixer(Mixer):
    """params: hidden_size, num_heads, num_kv_heads, key_dim, value_dim, scale, norm_eps, taps (0: no convolution), qk_unit (heads divided by
    their root mean square behind the rotation), position (a PartSpec of category "position" offering cos_sin, or None), cap (0: none),
    window (0: every earlier key), sink, value_mix (None, "keep" or "mix").
    tensors: q, k, v, o and, as the parameters say, q_conv, k_conv, v_conv [channels, taps], sink [heads], lambda (one number; it belongs to
    every mixer with `value_mix`, also to the one that keeps)."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.H, self.G, self.D, self.V = int(p["num_heads"]), int(p["num_kv_heads"]), int(p["key_dim"]), int(p["value_dim"])
        self.scale, self.eps, self.cap = float(p["scale"]), float(p.get("norm_eps", 1e-6)), float(p.get("cap") or 0.0)
        self.taps, self.unit, self.window = int(p.get("taps", 0) or 0), bool(p.get("qk_unit")), int(p.get("window", 0) or 0)
        self.has_sink, self.value_mix = bool(p.get("sink")), p.get("value_mix")
        if self.H % self.G:
            raise ValueError(f"attention with a short convolution: {self.H} heads do not divide into {self.G} key/value heads")
        if not 0 <= self.taps <= MAX_TAPS:
            raise ValueError(f"attention with a short convolution: {self.taps} taps (at most {MAX_TAPS})")
        if max(self.D, self.V) > 640:
            raise ValueError(f"attention with a short convolution: key size {self.D} / value size {self.V} exceed 640, the most the kernel holds")
        if self.value_mix not in (None, "keep", "mix"):
            raise ValueError(f"attention with a short convolution: value_mix {self.value_mix!r}")
        pos = p.get("position")
        self.position = part_class("position", pos.kind)(pos, env) if pos is not None else None
        self.channels = self.H * self.D + self.G * (self.D + self.V)
        self.record = max(self.taps - 1, 0) * self.channels
        self.qkv = self.o = self.conv = self.sinks = self.cos_sin = None
        self.rot, self.lam = 0, 0.0

    def tensor_plan(self):
        t, H, G, D, V, W = self.spec.tensors, self.H, self.G, self.D, self.V, self.hidden
        plan = {t["q"]: TensorPlan((H * D, W)), t["k"]: TensorPlan((G * D, W)), t["v"]: TensorPlan((G * V, W)), t["o"]: TensorPlan((W, H * V))}
        if self.taps:
            plan.update({t["q_conv"]: TensorPlan((H * D, self.taps)), t["k_conv"]: TensorPlan((G * D, self.taps)),
                         t["v_conv"]: TensorPlan((G * V, self.taps))})
        if self.has_sink:
            plan[t["sink"]] = TensorPlan((H,), zero_mean=True)
        if self.value_mix is not None:
            plan[t["lambda"]] = TensorPlan(())
        if self.position is not None:
            plan.update(self.position.tensor_plan())
        return plan

    def bind(self, tensors):
        t, f32 = self.spec.tensors, torch.float32
        ws = [tensors[t[r]] for r in ("q", "k", "v")]
        if len({w.dtype for w in ws}) > 1:
            ws = [w.to(f32) for w in ws]
        self.qkv = Linear(torch.cat(ws, dim=0), self.env.compute_dtype)
        self.o = Linear(tensors[t["o"]], self.env.compute_dtype)
        if self.taps:
            self.conv = torch.cat([tensors[t[r]].to(f32) for r in ("q_conv", "k_conv", "v_conv")]).T.contiguous()       # [taps, channels]
        if self.has_sink:
            self.sinks = tensors[t["sink"]].to(f32).contiguous()
        if self.value_mix is not None:
            self.lam = float(tensors[t["lambda"]].to(f32))
        if self.position is not None:
            self.position.bind(tensors)
            table, rot = getattr(self.position, "cos_sin", None), getattr(self.position, "rotary_dim", None)
            if not isinstance(table, torch.Tensor) or not rot or rot % 2 or rot > self.D or tuple(table.shape[1:]) != (rot // 2, 2):
                raise TypeError(f"the position part '{self.spec.params['position'].kind}' does not offer cos_sin [positions, rotary_dim / 2, 2] "
                                f"for an even rotary_dim <= {self.D} (see parts.base.PositionEncoding)")
            self.cos_sin, self.rot = table, int(rot)

    def weight_bytes(self):
        return self.qkv.weight_bytes() + self.o.weight_bytes()

    def cache_need(self):
        pages = CacheNeed("pages", kv_heads=self.G, head_dim=max(self.D, self.V), window=self.window, dtype=self.env.act_dtype)
        if not self.record:
            return pages
        return [pages, CacheNeed("state", state_shape=(self.record,), state_dtype=torch.float32)]

    def kernel_libraries(self):
        attend = {"attention_tc", "attention_tc5"} if self._fixed_heads() else {"masked_attention"}
        return attend | {"short_conv", "gemm_tc" if self.env.compute_dtype == torch.bfloat16 else "gemm_f32"}

    def _fixed_heads(self) -> bool:
        return self.D == self.V and tensor_core_head(self.env.act_dtype, self.H, self.G, self.D)

    def _tiles(self, pages) -> bool:
        return self.env.act_dtype == torch.bfloat16 and ops.masked_attention_tiles_supported(self.H, self.G, self.D, self.V, pages.shape[4],
                                                                                             pages.stride(1))

    def forward(self, ctx, x, stream, cache):
        with ImmediateProgram(ctx, stream) as program:
            self.emit(program, x, cache)

    def emit(self, program, x, cache):
        ws, f32, act, H, G, D, V = program.workspace, torch.float32, self.env.act_dtype, self.H, self.G, self.D, self.V
        T = ws.max_tokens
        paged, state = (cache.parts[0], cache.parts[1].state) if self.record else (cache, None)
        pages, table = paged.pages, paged.block_table
        qkv = ws.raw("cattn.qkv", (self.qkv.partial_elems(T),), f32)
        S = self.qkv.emit_partials(program, x, qkv)
        q = ws.get("cattn.q", T, (H * D,), act)
        mixed = ws.get("cattn.out", T, (H * V,), act)
        kept = ws.get("cattn.kept_values", T, (G * V,), f32) if self.value_mix is not None else None
        program.add("short_conv", "sb_op_conv_qkv",
                    [qkv, self.channels, S, program.few_tokens, self.conv, self.taps, state, self.record, self.cos_sin, self.rot, int(self.unit), kept,
                     {None: 0, "keep": 1, "mix": 2}[self.value_mix], q, q.dtype, pages, table, *_page_where(pages, table), H, G, D, V, pages.shape[4]],
                    [self.eps, self.lam])
        if self._fixed_heads():
            tc5 = ops.attention_tc5_supported(H, G, D, pages.shape[3])
            plan = program.plan(H // G, 128 if tc5 else 64, 1, -1)
            emit_tensor_core_attention(program, q, mixed, pages, table, H, G, D, self.window, self.scale, plan, tc5, cap=self.cap, sinks=self.sinks)
        else:
            _emit_attend(program, q, mixed, paged, None, self.sinks, H, G, D, V, self.window, 0, self.scale, self._tiles(pages), cap=self.cap)
        self.o.emit_add(program, mixed, ws.raw("cattn.o_partials", (self.o.partial_elems(T),), f32))
