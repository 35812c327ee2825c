"""Feed-forwards that are no plain gated product.

"polynorm": W_down act(W_up x) with act(z) = a N(z) + b N(z^2) + c N(z^3) + e, powers element by element, N(y) =
y / sqrt(mean(y^2) + eps) over a token's row, and a, b, c, e four stored numbers.

"routed": `experts` small feed-forwards W_down relu(W_up x)^2 of which every token uses `top`, plus `identity` experts
without weights whose output is their input. Router logits z = W_r x in true float32; scores s = softmax(z) over all
experts; the `top` experts with the largest s + correction are chosen; a chosen expert weighs s / (sum of the chosen
s + 1e-20) * scale. The experts' up matrices lie side by side as one matrix, so do the down matrices: the hidden
activations of experts that a token did not choose are exact zeros (times weight 0), so one product each way is the
weighted sum of the chosen experts; identity experts add their weight times x. Kernels between the products:
csrc/feed_forward.cu; the identity experts' share: csrc/branch.cu.

Two parameters make other routed designs of it. `weights_from` "logits": the stored vector is the router's bias, z = W_r x + b, the
`top` largest z are chosen and weigh by the softmax over the chosen z alone. `expert` "silu_gated": an expert is
W_down (silu(W_gate x) * (W_up x)); its gate and up matrices lie one above the other in the side-by-side product.

"table_experts": gated experts without a router, chosen by a stored table of token ids; the products run grouped, every expert on the rows
that chose it (csrc/grouped_gemm.cu). "sigmoid_experts": the same grouped products behind a router, whose chosen scores are sigmoids taken as
they are and multiply the experts' inputs."""
from __future__ import annotations

import torch

from ..kernels import ops
from ..kernels.linear import Linear
from ..kernels.native import ImmediateProgram
from .base import FeedForward, register_part
from .branch import ALWAYS, emit_fold, emit_on_branch
from .mlp import SwiGLU
from .spec import PartSpec, TensorPlan


@register_part("feed_forward", "polynorm")
class PolyNormFeedForward(FeedForward):
    """params: hidden_size, intermediate_size, eps. tensors: up, down, coefficients [4]."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden, self.intermediate = int(spec.params["hidden_size"]), int(spec.params["intermediate_size"])
        self.eps = float(spec.params["eps"])
        self.up = self.down = None
        self.coefficients = (0.0, 0.0, 0.0, 0.0)

    def tensor_plan(self):
        t = self.spec.tensors
        return {t["up"]: TensorPlan((self.intermediate, self.hidden)), t["down"]: TensorPlan((self.hidden, self.intermediate)),
                t["coefficients"]: TensorPlan((4,))}

    def bind(self, tensors):
        t = self.spec.tensors
        self.up = Linear(tensors[t["up"]], self.env.compute_dtype)
        self.down = Linear(tensors[t["down"]], self.env.compute_dtype)
        self.coefficients = tuple(float(v) for v in tensors[t["coefficients"]].to(torch.float32).cpu().tolist())

    def weight_bytes(self):
        return self.up.weight_bytes() + self.down.weight_bytes()

    def kernel_libraries(self):
        return {"feed_forward", "gemm_tc" if self.env.compute_dtype == torch.bfloat16 else "gemm_f32"}

    def forward(self, ctx, x, stream):
        n, ws = ctx.n, ctx.workspace
        up = self.up.forward_partials(x, ws.raw("polynorm.up", (self.up.partial_elems(ws.max_tokens),), torch.float32))
        z = ws.get("polynorm.z", n, (self.intermediate,), ctx.act_dtype)
        ops.polynorm(up, z, self.coefficients, self.eps)
        self.down.forward_add(z, stream, ws.raw("polynorm.down_partials", (self.down.partial_elems(ws.max_tokens),), torch.float32))

    def emit(self, program, x):
        ws = program.workspace
        T = ws.max_tokens
        up = ws.raw("polynorm.up", (self.up.partial_elems(T),), torch.float32)
        S = self.up.emit_partials(program, x, up)
        z = ws.get("polynorm.z", T, (self.intermediate,), self.env.act_dtype)
        eps_bits = int(torch.tensor(self.eps, dtype=torch.float32).view(torch.int32).item())
        program.add("feed_forward", "sb_op_polynorm", [up, S, program.few_tokens, z, z.dtype, self.intermediate, eps_bits], self.coefficients)
        self.down.emit_add(program, z, ws.raw("polynorm.down_partials", (self.down.partial_elems(T),), torch.float32))


@register_part("feed_forward", "routed")
class RoutedFeedForward(FeedForward):
    """params: hidden_size, intermediate_size (of one expert), experts, identity (experts without weights, listed last by the
    router), top, scale (1 by default), weights_from ("scores" by default, or "logits"), expert ("relu2" by default, or "silu_gated").
    tensors: router [experts + identity, hidden], correction [experts + identity], up and down (lists of names, one per expert), gate
    (the same, for gated experts)."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden, self.intermediate = int(p["hidden_size"]), int(p["intermediate_size"])
        self.experts, self.identity, self.top = int(p["experts"]), int(p.get("identity", 0)), int(p["top"])
        self.scale = float(p.get("scale", 1.0))
        self.biased = {"scores": False, "logits": True}[p.get("weights_from", "scores")]
        self.gated = {"relu2": False, "silu_gated": True}[p.get("expert", "relu2")]
        self.outputs = self.experts + self.identity
        if not 0 < self.top <= self.outputs or self.outputs > 256:
            raise ValueError(f"routed feed-forward: {self.top} of {self.outputs} experts (at most 256)")
        self.router = self.correction = self.up = self.down = None

    def tensor_plan(self):
        t = self.spec.tensors
        plan = {t["router"]: TensorPlan((self.outputs, self.hidden)), t["correction"]: TensorPlan((self.outputs,), zero_mean=True)}
        for name in (*t["up"], *(t["gate"] if self.gated else ())):
            plan[name] = TensorPlan((self.intermediate, self.hidden))
        for name in t["down"]:
            plan[name] = TensorPlan((self.hidden, self.intermediate))
        return plan

    def bind(self, tensors):
        t = self.spec.tensors

        def side_by_side(names, dim):
            ws = [tensors[n] for n in names]
            if len({w.dtype for w in ws}) > 1:
                ws = [w.to(torch.float32) for w in ws]
            return torch.cat(ws, dim=dim)

        self.router = tensors[t["router"]].contiguous()
        self.correction = tensors[t["correction"]].to(torch.float32).contiguous()
        if self.experts:
            rows = t["up"] if not self.gated else [name for pair in zip(t["gate"], t["up"]) for name in pair]
            self.up = Linear(side_by_side(rows, 0), self.env.compute_dtype)
            self.down = Linear(side_by_side(t["down"], 1), self.env.compute_dtype)

    def weight_bytes(self):
        own = self.router.numel() * self.router.element_size()
        return own + (self.up.weight_bytes() + self.down.weight_bytes() if self.experts else 0)

    def kernel_libraries(self):
        return {"feed_forward", "branch", "gemm_f32", "gemm_tc" if self.env.compute_dtype == torch.bfloat16 else "gemm_f32"}

    def forward(self, ctx, x, stream):
        n, ws, E, F = ctx.n, ctx.workspace, self.experts, self.intermediate
        logits = ws.get("routed.logits", n, (self.outputs,), torch.float32)
        ops.gemm_f32(x, self.router, logits)
        weights = ws.get("routed.weights", n, (self.outputs,), torch.float32)
        ops.moe_route(logits, self.correction, weights, self.top, self.scale, self.biased)
        if self.identity:
            stream.fold()
            ops.row_scaled_add(stream.h, x, weights, E, self.identity)
        if E:
            up = self.up.forward_partials(x, ws.raw("routed.up", (self.up.partial_elems(ws.max_tokens),), torch.float32))
            z = ws.get("routed.z", n, (E * F,), ctx.act_dtype)
            ops.moe_activate(up, weights, z, E, F, self.gated)
            self.down.forward_add(z, stream, ws.raw("routed.down_partials", (self.down.partial_elems(ws.max_tokens),), torch.float32))

    def emit(self, program, x):
        ws, E, F, X = program.workspace, self.experts, self.intermediate, self.outputs
        T, f32 = ws.max_tokens, torch.float32
        logits = ws.get("routed.logits", T, (X,), f32)
        program.add("gemm_f32", "sb_op_linear_f32", [x, x.dtype, x.stride(0), self.router, self.router.dtype, self.router.stride(0), logits, X, X,
                                                     self.hidden, 0, 0])
        weights = ws.get("routed.weights", T, (X,), f32)
        program.add("feed_forward", "sb_op_moe_route", [logits, X, self.correction, self.correction.dtype, weights, X, self.top, int(self.biased)],
                    [self.scale])
        if self.identity:
            program.need_folded("identity experts")
            program.add("branch", "sb_op_row_scaled_add", [program.h, x, x.dtype, weights, X, E, self.identity, self.hidden])
        if E:
            up = ws.raw("routed.up", (self.up.partial_elems(T),), f32)
            S = self.up.emit_partials(program, x, up)
            z = ws.get("routed.z", T, (E * F,), self.env.act_dtype)
            program.add("feed_forward", "sb_op_moe_activate", [up, S, program.few_tokens, weights, X, z, z.dtype, E, F, int(self.gated)])
            self.down.emit_add(program, z, ws.raw("routed.down_partials", (self.down.partial_elems(T),), f32))


class GroupedExpertsFeedForward(FeedForward):
    """Gated experts W_down (silu(W_gate x) * (W_up x)) of which every token uses `top`, and perhaps a shared one of the same form: the
    step's (token, choice) pairs are sorted by expert and every projection is one launch over the experts in use, each on its own rows
    (csrc/grouped_gemm.cu); the choices of a token come back as `top` partial sums, which whoever takes the result in adds in their order.
    Which experts a token uses is a subclass's business. params: hidden_size, intermediate_size (of one expert), experts, top, shared (the
    shared expert's intermediate size; 0: none). tensors: gate, up, down (lists of names, one per expert), shared_gate, shared_up, shared_down."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden, self.intermediate = int(p["hidden_size"]), int(p["intermediate_size"])
        self.experts, self.top, self.shared_size = int(p["experts"]), int(p["top"]), int(p.get("shared", 0) or 0)
        if not 0 < self.top <= self.experts or self.experts > 1024:
            raise ValueError(f"grouped experts: {self.top} of {self.experts} experts (at most 1024)")
        t = spec.tensors
        self.shared = SwiGLU(PartSpec("gated", {"hidden_size": self.hidden, "intermediate_size": self.shared_size},
                                      {"gate": t["shared_gate"], "up": t["shared_up"], "down": t["shared_down"]}), env) if self.shared_size else None
        self.gate_up = self.down = None
        self.tensor_core = False

    def tensor_plan(self):
        t, plan = self.spec.tensors, {}
        for name in (*t["gate"], *t["up"]):
            plan[name] = TensorPlan((self.intermediate, self.hidden))
        for name in t["down"]:
            plan[name] = TensorPlan((self.hidden, self.intermediate))
        if self.shared is not None:
            plan.update(self.shared.tensor_plan())
        return plan

    def bind(self, tensors):
        t = self.spec.tensors

        def one_below_the_other(names):
            ws = [tensors[n] for n in names]
            if len({w.dtype for w in ws}) > 1:
                ws = [w.to(torch.float32) for w in ws]
            return torch.cat(ws, dim=0).contiguous()

        self.gate_up = one_below_the_other([name for pair in zip(t["gate"], t["up"]) for name in pair])      # [E (F gate rows, F up rows), hidden]
        self.down = one_below_the_other(t["down"])                                                          # [E hidden, F]
        self.tensor_core = (self.env.compute_dtype == torch.bfloat16 and self.gate_up.dtype == self.down.dtype == torch.bfloat16
                            and self.hidden % 8 == 0 and self.intermediate % 8 == 0)
        if self.shared is not None:
            self.shared.bind(tensors)

    def weight_bytes(self):
        """Of a step of one token: its `top` experts and the shared one."""
        one = (self.gate_up.numel() * self.gate_up.element_size() + self.down.numel() * self.down.element_size()) // self.experts
        return self.top * one + (self.shared.weight_bytes() if self.shared is not None else 0)

    def kernel_libraries(self):
        return {"grouped_gemm", "branch"} | (self.shared.kernel_libraries() if self.shared is not None else set())

    def forward(self, ctx, x, stream):
        with ImmediateProgram(ctx, stream) as program:
            self.emit(program, x)

    def emit(self, program, x):
        program.need_folded("grouped experts")
        emit_fold(program, self.emit_sources(program, x), None, self.hidden, fresh=True)

    def _emit_grouped(self, program, x, choice, vocab: int, pair_weight, scale: float) -> list:
        """The chosen experts' and the shared expert's results as branches with constants. choice [vocab, top]: the experts of every token
        id; with vocab 0, [tokens of the step, top]. pair_weight [top, tokens]: a factor on every pair's input, or None."""
        ws, E, top, F, W, tc = program.workspace, self.experts, self.top, self.intermediate, self.hidden, int(self.tensor_core)
        T, i32, act = ws.max_tokens, torch.int32, self.env.act_dtype
        order = ws.raw("experts.order", (T * top,), i32)
        tiles = ws.raw("experts.tiles", (3 * T * top + 1,), i32)
        lib = "grouped_gemm"
        program.add(lib, "sb_op_expert_sort", [choice, vocab, top, E, getattr(program, "sampled", None), order, tiles, tc])
        if tc:
            xs = ws.raw("experts.x", (T * top, W), act)
            program.add(lib, "sb_op_expert_gather", [x, x.stride(0), x.element_size(), order, top, xs, W])
        else:
            xs = x
        z = ws.raw("experts.z", (T * top, F), act)
        program.add(lib, "sb_op_expert_linear", [xs, xs.stride(0), xs.dtype, self.gate_up, self.gate_up.dtype, z, z.dtype, 2 * F, W, E, top, 1,
                                                 order, tiles, tc, pair_weight])
        out = ws.raw("experts.out", (T * top * W,), torch.float32)
        program.add(lib, "sb_op_expert_linear", [z, F, z.dtype, self.down, self.down.dtype, out, out.dtype, W, F, E, top, 0, order, tiles, tc])
        sources = [(None, (out, top, W, ALWAYS), scale)]
        if self.shared is not None:
            branch = ws.get("experts.shared", T, (W,), torch.float32)
            sources.append((*emit_on_branch(program, branch, lambda: self.shared.emit(program, x), fresh=True), 1.0))
        return sources


@register_part("feed_forward", "sigmoid_experts")
class SigmoidExpertsFeedForward(GroupedExpertsFeedForward):
    """Grouped experts behind a router in 32-bit: z = W_r x, the `top` experts with the largest z are chosen, and the score of a chosen one,
    s = sigmoid(z) as it is, multiplies the expert's input: sum of expert(s x). The shared expert's result may be multiplied by a gate per
    token, sigmoid(W_sg x): one more row of the router's product.
    params further: shared_gate (False by default). tensors further: router [experts, hidden], shared_sg [1, hidden]."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.shared_gate = bool(spec.params.get("shared_gate")) and self.shared_size > 0
        self.router = None

    def tensor_plan(self):
        t, plan = self.spec.tensors, super().tensor_plan()
        plan[t["router"]] = TensorPlan((self.experts, self.hidden))
        if self.shared_gate:
            plan[t["shared_sg"]] = TensorPlan((1, self.hidden))
        return plan

    def bind(self, tensors):
        super().bind(tensors)
        t = self.spec.tensors
        rows = [tensors[t["router"]], *([tensors[t["shared_sg"]]] if self.shared_gate else [])]
        if len({w.dtype for w in rows}) > 1:
            rows = [w.to(torch.float32) for w in rows]
        self.router = torch.cat(rows, dim=0).contiguous()

    def weight_bytes(self):
        return super().weight_bytes() + self.router.numel() * self.router.element_size()

    def kernel_libraries(self):
        return super().kernel_libraries() | {"gemm_f32"}

    def emit_sources(self, program, x):
        """The result as branches with constants, left to the caller to add."""
        ws, E, top, f32 = program.workspace, self.experts, self.top, torch.float32
        T, X = ws.max_tokens, self.router.shape[0]
        logits = ws.get("experts.logits", T, (X,), f32)
        program.add("gemm_f32", "sb_op_linear_f32", [x, x.dtype, x.stride(0), self.router, self.router.dtype, self.router.stride(0), logits, X, X,
                                                     self.hidden, 0, 0])
        choice = ws.raw("experts.choice", (T * top,), torch.int32)
        weights = ws.raw("experts.weights", (T * top,), f32)
        gate = ws.raw("experts.shared_gate", (T,), f32) if self.shared_gate else None
        program.add("grouped_gemm", "sb_op_expert_choose", [logits, X, E, top, choice, weights, gate])
        sources = self._emit_grouped(program, x, choice, 0, weights, 1.0)
        if gate is not None:
            sources[1] = (*sources[1][:2], gate)
        return sources


@register_part("feed_forward", "table_experts")
class TableExpertsFeedForward(GroupedExpertsFeedForward):
    """Grouped experts without a router, chosen by the token alone: a stored table names `top` experts for every token id, each with weight
    1 / top. params further: vocab_size. tensors further: table [vocab, top]."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.vocab = int(spec.params["vocab_size"])
        self.table = None

    def tensor_plan(self):
        return {self.spec.tensors["table"]: TensorPlan((self.vocab, self.top), integer=True, below=self.experts), **super().tensor_plan()}

    def bind(self, tensors):
        t = self.spec.tensors
        self.table = tensors[t["table"]].contiguous()
        low, high = int(self.table.min()), int(self.table.max())
        if low < 0 or high >= self.experts:
            raise ValueError(f"experts by table: '{t['table']}' names experts {low} .. {high} of {self.experts}")
        super().bind(tensors)

    def emit_sources(self, program, x):
        """The result as branches with constants, left to the caller to add."""
        return self._emit_grouped(program, x, self.table, self.vocab, None, 1.0 / self.top)
