"""Several residual streams side by side (hyper-connections).

In place of one residual x there are S streams x_1 .. x_S, all equal to the embedding output at first. A sublayer reads a weighted sum of
them, u = sum_s in[s] x_s, y = sublayer(norm(u)), and then all streams change at once, x_t <- sum_s mix[s, t] x_s + out[t] y. Behind the last
layer the streams' sum is what the final norm sees. All of it in 32-bit.

"hyper_connection" (category "streams") holds one sublayer's three weights; the blocks "hyper" and "hyper_mixer" run a mixer and a
feed-forward, or a mixer alone, between them. The sublayers are the parts that other blocks use, each on a branch that nothing clears:
its last projection stores its result or leaves partial sums. What a sublayer left and how the streams take it in stays noted on the program
(`Streams.update`) until the next sublayer, or the end of the model, reads the streams: one kernel then does both and norms on the way
(csrc/streams.cu)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from ..kernels.native import ImmediateProgram
from .base import Block, Part, register_part
from .branch import emit_on_branch, pending_limit
from .spec import TensorPlan


@dataclass
class Streams:
    """Where the streams of a step stand while its operations are laid out."""
    count: int
    width: int
    x: torch.Tensor                      # [max_tokens, count, width] float32
    held: bool = False                   # False: nothing was stored yet, every stream is the embedding output
    update: Optional[tuple] = None       # (sources, mix, out): a sublayer's result that the streams have not taken in yet


def streams_of(program, count: int, width: int) -> Streams:
    if program.streams is None:
        ws = program.workspace
        program.streams = Streams(count, width, ws.get("streams.x", ws.max_tokens, (count, width), torch.float32))
    s = program.streams
    if (s.count, s.width) != (count, width):
        raise ValueError(f"{count} streams of {width} elements in a model that has {s.count} of {s.width}")
    return s


def emit_read(program, streams: Streams, weights, norm, out: torch.Tensor, last: bool = False) -> None:
    """out = norm(sum_s weights[s] x_s) once the pending update is taken in; `last`: on the rows whose logits are wanted, and the streams
    themselves are not stored any more."""
    centred, gain, bias, eps = norm.form()
    S, W, x = streams.count, streams.width, streams.x
    program.need_folded("streams side by side")
    source = [x, S * W, W] if streams.held else [program.h, W, 0]
    keep = streams.update is not None and not last
    args, constants = [], []
    sources, mix, share = streams.update or ([], None, None)
    for buffer, pending, c in [*sources, (None, None, 1.0), (None, None, 1.0)][:2]:
        flat, P = (pending or (None, 1))[:2]
        args += [buffer, flat, P, pending_limit(pending) or program.few_tokens]
        constants.append(c)
    program.add("streams", "sb_op_streams_step", [*source, x if keep else None, *args, mix, share, weights, gain, bias, int(centred), out, out.dtype,
                                                  S, W, int(last)], [*constants, eps])
    if keep:
        streams.held, streams.update = True, None


@register_part("streams", "hyper_connection")
class HyperConnection(Part):
    """params: hidden_size, streams. tensors: in [streams], out [streams], mix [streams, streams] (from, to)."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden, self.count = int(spec.params["hidden_size"]), int(spec.params["streams"])
        if not 1 <= self.count <= 16:
            raise ValueError(f"hyper-connections: {self.count} streams (1 to 16)")
        self.read = self.share = self.mix = None

    def tensor_plan(self):
        t, S = self.spec.tensors, self.count
        return {t["in"]: TensorPlan((S,)), t["out"]: TensorPlan((S,)), t["mix"]: TensorPlan((S, S), near_identity=True)}

    def bind(self, tensors):
        t = self.spec.tensors
        self.read, self.share, self.mix = (tensors[t[r]].to(torch.float32).contiguous() for r in ("in", "out", "mix"))

    def kernel_libraries(self):
        return {"streams"}

    def emit_sublayer(self, program, norm, part, run) -> None:
        """Read the streams through `norm`, run `part` (`run(emit, x)` calls its emit with whatever else it takes) on a branch, note the result."""
        ws, W, f32 = program.workspace, self.hidden, torch.float32
        streams = streams_of(program, self.count, W)
        x = ws.get("block.x", ws.max_tokens, (W,), self.env.act_dtype)
        emit_read(program, streams, self.read, norm, x)
        if hasattr(part, "emit_sources"):
            sources = run(part.emit_sources, x)
        else:
            branch = ws.get("streams.branch", ws.max_tokens, (W,), f32)
            sources = [(*emit_on_branch(program, branch, lambda: run(part.emit, x), fresh=True), 1.0)]
        if not 1 <= len(sources) <= 2:
            raise ValueError("streams take in one or two branches")
        streams.update = (sources, self.mix, self.share)


class _StreamsBlock(Block):
    graph_safe = True
    norms_itself = True          # the norms in front of sublayers, and the model's last one, run inside the streams' kernel

    def kernel_libraries(self):
        return set().union(*(self.parts[role].kernel_libraries() for role, category in self.ROLES.items() if category != "norm"))

    def forward(self, ctx, stream, cache):
        with ImmediateProgram(ctx, stream) as program:
            self.emit(program, cache)


@register_part("block", "hyper")
class HyperBlock(_StreamsBlock):
    ROLES = {"mixer_norm": "norm", "mixer": "mixer", "mixer_streams": "streams",
             "feed_forward_norm": "norm", "feed_forward": "feed_forward", "feed_forward_streams": "streams"}

    def emit(self, program, cache):
        self.mixer_streams.emit_sublayer(program, self.mixer_norm, self.mixer, lambda f, x: f(program, x, cache))
        self.feed_forward_streams.emit_sublayer(program, self.feed_forward_norm, self.feed_forward, lambda f, x: f(program, x))


@register_part("block", "hyper_mixer")
class HyperMixerBlock(_StreamsBlock):
    """The first half alone: a layer without a feed-forward."""
    ROLES = {"mixer_norm": "norm", "mixer": "mixer", "mixer_streams": "streams"}

    def emit(self, program, cache):
        self.mixer_streams.emit_sublayer(program, self.mixer_norm, self.mixer, lambda f, x: f(program, x, cache))
