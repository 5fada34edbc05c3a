"""A routed feed-forward: a mixture of small experts, of which each token uses a few.

With h the input, R = experts + identity router outputs:

    z = Wr h (float32)          s = softmax(z) over all R outputs
    choice = s + correction     the ``top`` largest choice values are taken, looking only inside the ``keep`` of
                                ``count`` groups of neighbouring outputs whose best choice value is largest
    w_k = s_k / (sum of the chosen s + 1e-20)
    out = sum_k w_k E_k(h)      E_e(h) = Wdown_e relu(Wup_e h)^2 for an expert, h itself for an identity output

Parameters change six things: the scores may be each output's own logistic function instead of the softmax; the weights
the chosen scores as they are instead of over their sum, and all times a constant; a weight may multiply its expert's INPUT,
E(w h), instead of the output; a group's value may be the sum of its two largest choice values; an expert may be a gated
feed-forward, Wdown (silu(Wgate h) Wup h), or a clamped gated one, Wdown (g sigmoid(alpha g) (u + offset)) with g =
min(Wgate h, L) and u = clamp(Wup h, -L, L), gate and up rows interleaved in one matrix (the plain gate is the clamped one
with L infinite, alpha 1 and offset 0); and the feed-forward that every token uses may be multiplied by one gate per token,
sigmoid(wg h).  That gate's row lies below the router's in one matrix.

The correction steers the choice only; the weights use the plain scores.  Identity outputs are the last ``identity``
router outputs and have no tensors.  The sum over a token's choices is formed in float32 in the order of the choice
and added into the float32 stream.

Three ways through the experts.  A step of very few tokens lets each (token, choice) pair read its expert's rows
directly (``experts_direct``: two kernels).  A step of some tokens whose choices between them reach most experts
anyway (a decode batch, a short portion: at least twice as many pairs as experts, at most ``DENSE_MAX_TOKENS``
tokens) goes through ALL experts: one product of the tokens with every up matrix, ``experts_dense_weigh`` (the
chosen experts' activated rows times their weights, zeros elsewhere), one product with the down matrices side by
side along k that adds into the stream; every expert's weights cross the memory bus once, on the tensor cores, and
the work wasted on zeros is free while the step is bound by those bytes.  Neither reads anything from the host, so
both can be captured into a CUDA graph.  A step of many tokens groups the pairs by expert and runs one ordinary product per
expert and projection over that expert's block of rows (``experts_group`` -> products ->
``experts_combine_add``); the host reads the group sizes, which a step with prompt portions may do.

On the dense path a gated feed-forward that every token uses is one expert more: its rows lie below the experts' in the up
matrix and beside them in the down matrix, and the kernel between the products multiplies its values by the token's gate.

The down matrices are kept side by side, [hidden, experts, inner]: expert e's matrix is the strided view [:, e, :].
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

from .base import FEED_FORWARDS, FeedForward, ParamSpec, StepContext, build_part

DIRECT_MAX_TOKENS = 32      # steps of up to this many tokens (and every step of single tokens) avoid the grouped path
DENSE_MAX_TOKENS = 256      # beyond this many tokens the wasted products of the dense path would cost more than its bytes


@FEED_FORWARDS.register("routed_experts")
class RoutedExperts(FeedForward):
    """params: ``hidden_size``, ``intermediate_size`` (an expert's inner width), ``experts``, ``top``, optional
    ``identity`` (default 0), ``group_count`` / ``group_keep`` (default 1 / 1: no groups), ``correction`` (bool,
    default True: the checkpoint holds a correction of the choice), ``activation`` (``"relu_squared"`` or
    ``"clamped_glu"``, the latter with ``limit`` and optionally ``alpha``, default 1.702, and ``up_offset``, default 1, or
    ``"swiglu"``), ``group_value`` (``"best"`` or ``"two_best"``), ``weights_scale`` (default 1), ``shared_gate`` (bool, default
    False: one logistic gate per token on the shared feed-forward; parameter ``shared_gate.weight`` [1, hidden]), ``score`` (``"softmax"`` or ``"logistic"``), ``weights_over_sum`` (bool, default True), ``weigh`` (``"output"`` or
    ``"input"``; the latter without identity experts), ``router_bias`` (bool, default False: a bias added to the router's logits, so it
    steers the choice and the weights alike), ``shared`` (None, or the PartSpec of a feed-forward that every token
    uses and whose output is added; its parameters are this part's under ``shared.<local name>``).
    With no correction and no groups the weights are the softmax over the chosen logits alone: a chosen output's share
    of the softmax over all, divided by the chosen ones' sum, is the same number.
    weights: ``router.weight`` [experts + identity, hidden], ``router.bias`` and ``correction`` (float32 [experts +
    identity]), ``experts.<e>.up.weight`` [inner, hidden] (and ``experts.<e>.gate.weight`` of gated ones),
    ``experts.<e>.down.weight`` [hidden, inner]."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.hidden = int(p["hidden_size"])
        self.inner_size = int(p["intermediate_size"])
        self.experts = int(p["experts"])
        self.identity = int(p.get("identity", 0))
        self.top = int(p["top"])
        self.group_count = int(p.get("group_count", 1))
        self.group_keep = int(p.get("group_keep", 1))
        self.has_correction = bool(p.get("correction", True))
        self.has_router_bias = bool(p.get("router_bias", False))
        shared = p.get("shared")
        self.shared: Optional[FeedForward] = build_part(FEED_FORWARDS, shared, env) if shared is not None else None
        if self.shared is not None:
            self.graph_safe = bool(self.shared.graph_safe)
        self.shared_gate = bool(p.get("shared_gate", False))
        if self.shared_gate and self.shared is None:
            raise ValueError("routed_experts: a gate on the shared feed-forward needs one")
        group_value = str(p.get("group_value", "best"))
        if group_value not in ("best", "two_best"):
            raise ValueError(f"routed_experts: group_value {group_value!r} is 'best' or 'two_best'")
        self.group_pairs = group_value == "two_best"
        self.weights_scale = float(p.get("weights_scale", 1.0))
        self.shared_inner = 0                  # inner width of a shared feed-forward that runs as one expert more
        self.router_bias: Optional[torch.Tensor] = None
        self.outputs = self.experts + self.identity
        activation = str(p.get("activation", "relu_squared"))
        self.gate = None                       # (limit, alpha, offset) of clamped gated experts
        if activation == "clamped_glu":
            self.gate = (float(p["limit"]), float(p.get("alpha", 1.702)), float(p.get("up_offset", 1.0)))
            if not self.gate[0] > 0.0:
                raise ValueError("routed_experts: the limit must be positive")
        elif activation == "swiglu":
            self.gate = (math.inf, 1.0, 0.0)
        elif activation != "relu_squared":
            raise ValueError(f"routed_experts: unknown activation '{p.get('activation')}'")
        self.matrices = 2 if self.gate is None else 3
        self.logistic = str(p.get("score", "softmax")) == "logistic"
        self.over_sum = bool(p.get("weights_over_sum", True))
        self.weigh_input = str(p.get("weigh", "output")) == "input"
        if str(p.get("score", "softmax")) not in ("softmax", "logistic") or str(p.get("weigh", "output")) not in ("output", "input"):
            raise ValueError(f"routed_experts: score {p.get('score')!r} or weigh {p.get('weigh')!r} is not known")
        if self.weigh_input and (self.identity or self.gate is None):
            raise ValueError("routed_experts: weights on the input go with gated experts and without identity experts")
        if min(self.hidden, self.inner_size, self.top, self.group_count, self.group_keep) <= 0 or self.experts < 0 \
                or self.identity < 0 or self.outputs <= 0:
            raise ValueError("routed_experts: sizes must be positive")
        if self.outputs % self.group_count or self.group_keep > self.group_count:
            raise ValueError(f"routed_experts: {self.group_count} groups ({self.group_keep} kept) of {self.outputs} router outputs")
        if self.top > (self.outputs // self.group_count) * self.group_keep:
            raise ValueError(f"routed_experts: {self.top} choices do not fit the kept groups")
        if self.outputs > 1024:
            raise ValueError("routed_experts: the router kernel takes up to 1024 outputs")
        self.w_router: Optional[torch.Tensor] = None
        self.correction: Optional[torch.Tensor] = None
        self.w_up: Optional[torch.Tensor] = None         # [experts, inner, hidden]; gated: [experts, 2 inner, hidden]
        self.w_down: Optional[torch.Tensor] = None       # [hidden, experts, inner]
        self.up_rows: Optional[torch.Tensor] = None      # all up (and gate) rows, a joined shared feed-forward's last
        self.down_columns: Optional[torch.Tensor] = None # all down matrices side by side, likewise

    def param_specs(self) -> Dict[str, ParamSpec]:
        specs = {"router.weight": ParamSpec((self.outputs, self.hidden))}
        if self.has_correction:
            specs["correction"] = ParamSpec((self.outputs,), role="vector")
        if self.has_router_bias:
            specs["router.bias"] = ParamSpec((self.outputs,), role="vector")
        if self.shared_gate:
            specs["shared_gate.weight"] = ParamSpec((1, self.hidden))
        if self.shared is not None:
            specs.update({f"shared.{local}": param for local, param in self.shared.param_specs().items()})
        for e in range(self.experts):
            if self.gate is not None:
                specs[f"experts.{e}.gate.weight"] = ParamSpec((self.inner_size, self.hidden))
            specs[f"experts.{e}.up.weight"] = ParamSpec((self.inner_size, self.hidden))
            specs[f"experts.{e}.down.weight"] = ParamSpec((self.hidden, self.inner_size))
        return specs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_router = tensors["router.weight"].contiguous()
        if self.shared_gate:
            # the gate's row below the router's, and rows of zeros up to a multiple of four (rows of logits on 16 bytes)
            gate = tensors["shared_gate.weight"]
            spare = gate.new_zeros((-(self.outputs + 1) % 4, self.hidden))
            self.w_router = torch.cat([self.w_router, gate, spare], dim=0).contiguous()
        self.correction = tensors["correction"].contiguous() if self.has_correction else None
        self.router_bias = tensors["router.bias"].contiguous() if self.has_router_bias else None
        if self.router_bias is not None and self.shared_gate:
            self.router_bias = torch.cat([self.router_bias, self.router_bias.new_zeros(self.w_router.shape[0] - self.outputs)])
        if self.shared is not None:
            self.shared.load({name[len("shared."):]: t for name, t in tensors.items() if name.startswith("shared.")})
        if self.experts:
            if self.gate is None:
                self.w_up = torch.stack([tensors[f"experts.{e}.up.weight"] for e in range(self.experts)]).contiguous()
            else:
                self.w_up = torch.stack([torch.stack([tensors[f"experts.{e}.gate.weight"], tensors[f"experts.{e}.up.weight"]], dim=1)
                                         .reshape(2 * self.inner_size, self.hidden) for e in range(self.experts)]).contiguous()
            self.w_down = torch.stack([tensors[f"experts.{e}.down.weight"] for e in range(self.experts)], dim=1).contiguous()
            self.up_rows = self.w_up.view(-1, self.hidden)
            self.down_columns = self.w_down.view(self.hidden, -1)
            self.join_shared()
        else:
            self.w_up = torch.empty((0, self.inner_size, self.hidden), dtype=self.w_router.dtype, device=self.w_router.device)
            self.w_down = torch.empty((self.hidden, 0, self.inner_size), dtype=self.w_router.dtype, device=self.w_router.device)

    def join_shared(self) -> None:
        """A gated feed-forward that every token uses becomes the last block of the experts' matrices."""
        matrices = getattr(self.shared, "gated_matrices", None)
        if matrices is None or self.gate is None or self.gate[1:] != (1.0, 0.0) or self.weigh_input:
            return
        gate_up, down = matrices()
        routed = self.experts * self.inner_size
        self.shared_inner = down.shape[1]
        self.up_rows = torch.cat([self.up_rows, gate_up], dim=0).contiguous()
        self.down_columns = torch.cat([self.down_columns, down], dim=1).contiguous()
        self.w_up = self.up_rows[:2 * routed].view(self.experts, 2 * self.inner_size, self.hidden)
        self.w_down = self.down_columns[:, :routed].unflatten(1, (self.experts, self.inner_size))
        self.shared.adopt_matrices(self.up_rows[2 * routed:], self.down_columns[:, routed:])

    def param_bytes(self) -> int:
        """What one token's step reads: the router and the chosen experts (a large batch touches more of them)."""
        item = self.env.dtype.itemsize
        extra = self.shared.param_bytes() if self.shared is not None else 0
        return (self.outputs * self.hidden + min(self.top, self.experts) * self.matrices * self.inner_size * self.hidden) * item + 4 * self.outputs + extra

    def dense(self, tokens: int) -> bool:
        """Whether a step of this many tokens runs all experts (its choices reach most of them anyway)."""
        return bool(self.experts) and 2 * self.experts <= tokens * self.top and tokens <= DENSE_MAX_TOKENS

    def step_param_bytes(self, tokens: int) -> int:
        """What a step of ``tokens`` tokens reads: the router, and all experts on the dense path, else as many as
        uniform choices would reach on average."""
        item = self.env.dtype.itemsize
        reached = self.experts if self.dense(tokens) else self.experts * (1.0 - (1.0 - min(self.top / self.outputs, 1.0)) ** tokens)
        extra = self.shared.param_bytes() if self.shared is not None else 0
        return int((self.outputs * self.hidden + reached * self.matrices * self.inner_size * self.hidden) * item) + 4 * self.outputs + extra

    def flops(self, tokens: int, pairs: float) -> float:
        extra = self.shared.flops(tokens, pairs) if self.shared is not None else 0.0
        return 2.0 * tokens * (self.outputs * self.hidden + self.top * self.matrices * self.inner_size * self.hidden) + extra

    def route(self, h):
        """(ids int32 [T, top], weights float32 [T, top], the gate logits of the shared feed-forward [T] or None); the logits
        are a float32 product of the rows as given, which may lack their norm's factor."""
        logits = self.ops.linear(h, self.w_router, self.router_bias, self.ops.GEMM_STORE_F32)
        ids, weights = self.ops.router_topk(logits, self.correction, self.top, self.group_count, self.group_keep,
                                            logistic=self.logistic, over_sum=self.over_sum, group_pairs=self.group_pairs,
                                            factor=self.weights_scale, outputs=self.outputs)
        return ids, weights, logits[:, self.outputs] if self.shared_gate else None

    def takes_deferred_at(self, tokens: int) -> bool:
        # on the dense path two products read the rows, and nothing else does
        return self.gate is not None and self.dense(tokens) and (self.shared is None or self.shared_inner > 0)

    def last_product(self, h: torch.Tensor, ctx: StepContext):
        """On the dense path of gated experts everything ends in one product with all down matrices."""
        ops, tokens = self.ops, h.shape[0]
        if not self.takes_deferred_at(tokens):
            return None
        ids, weights, gate = self.route(h)
        z = ops.linear(h, self.up_rows, None, ops.GEMM_STORE)
        a = ops.experts_dense_gate(z, ids, weights, self.experts, self.gate, self.weigh_input, self.shared_inner, gate)
        return a, self.down_columns

    def forward_add(self, h: torch.Tensor, x: torch.Tensor, ctx: StepContext, next_norm=None):
        if self.shared_gate:
            self.ops.add_to_stream(x, self.forward_f32(h, ctx))
            return None
        h = self.add_routed(h, x, ctx)
        if self.shared is not None:
            # the feed-forward every token uses adds last, and with it whatever it can do for the next norm
            return self.shared.forward_add(h, x, ctx, next_norm=next_norm)
        return None

    def add_routed(self, h: torch.Tensor, x: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        """Adds the chosen experts' weighted outputs into ``x`` (with a gate on the shared feed-forward, whose output ``x``
        then holds: into gate * x); returns the rows as the experts read them."""
        ops = self.ops
        complete = getattr(h, "complete", None)
        h = h if complete is None else complete()
        ids, weights, x_gate = self.route(h)
        tokens = h.shape[0]
        few = ctx.max_q_len <= 1 or tokens <= DIRECT_MAX_TOKENS
        if self.dense(tokens) and self.gate is not None and x_gate is None:
            z = ops.linear(h, self.w_up.view(self.experts * 2 * self.inner_size, self.hidden), None, ops.GEMM_STORE)
            a = ops.experts_dense_gate(z, ids, weights, self.experts, self.gate, self.weigh_input)
            ops.linear(a, self.w_down.view(self.hidden, self.experts * self.inner_size), None, ops.GEMM_ADD_F32, out=x)
            return h
        if self.dense(tokens) and self.gate is None and x_gate is None:
            z = ops.linear(h, self.w_up.view(self.experts * self.inner_size, self.hidden), None, ops.GEMM_STORE)
            ops.experts_dense_weigh(z, ids, weights, h, x, self.experts)
            ops.linear(z, self.w_down.view(self.hidden, self.experts * self.inner_size), None, ops.GEMM_ADD_F32, out=x)
            return h
        if few or self.experts == 0:
            ops.experts_direct(h, self.w_up, self.w_down, ids, weights, x, gate=self.gate, weigh_input=self.weigh_input,
                               x_gate=x_gate)
            return h
        place, offsets, grouped = ops.experts_group(h, ids, self.experts, in_weights=weights if self.weigh_input else None)
        bounds: List[int] = offsets.tolist()             # the host learns the group sizes: not a captured step
        rows = bounds[-1]
        inner = torch.empty((max(rows, 1), self.inner_size), dtype=h.dtype, device=h.device)
        outputs = torch.empty((max(rows, 1), self.hidden), dtype=torch.float32, device=h.device)
        # the gate is the product's own epilogue, where it has it
        fused = {(1.702, 1.0): ops.GEMM_GLU_CLAMPED, (1.0, 0.0): ops.GEMM_SWIGLU}.get(self.gate[1:] if self.gate else None)
        if fused == ops.GEMM_SWIGLU and self.gate[0] != math.inf:
            fused = None
        for e in range(self.experts):
            lo, hi = bounds[e], bounds[e + 1]
            if hi > lo:
                if fused is not None:
                    ops.linear(grouped[lo:hi], self.w_up[e], None, fused, out=inner[lo:hi],
                               alpha=self.gate[0] if fused == ops.GEMM_GLU_CLAMPED else 1.0)
                elif self.gate is not None:
                    both = ops.linear(grouped[lo:hi], self.w_up[e], None, ops.GEMM_STORE_F32)
                    ops.gated_clamp_act(both, *self.gate, self.env.dtype, out=inner[lo:hi])
                else:
                    ops.linear(grouped[lo:hi], self.w_up[e], None, ops.GEMM_STORE, out=inner[lo:hi])
        if rows and self.gate is None:
            ops.activation(inner[:rows], ops.ACT_RELU_SQUARED)
        for e in range(self.experts):
            lo, hi = bounds[e], bounds[e + 1]
            if hi > lo:
                ops.linear(inner[lo:hi], self.w_down[:, e, :], None, ops.GEMM_STORE_F32, out=outputs[lo:hi])
        ops.experts_combine_add(outputs, place, None if self.weigh_input else weights, h, x, x_gate=x_gate)
        return h

    def forward_f32(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        last = self.last_product(h, ctx) if self.shared_inner else None
        if last is not None:
            return self.ops.linear(last[0], last[1], None, self.ops.GEMM_STORE_F32)
        if self.shared is not None:
            # the feed-forward every token uses writes the rows, the chosen experts add to them
            complete = getattr(h, "complete", None)
            h = h if complete is None else complete()
            out = self.shared.forward_f32(h, ctx)
            self.add_routed(h, out, ctx)
            return out
        out = torch.zeros((h.shape[0], self.hidden), dtype=torch.float32, device=h.device)
        self.forward_add(h, out, ctx)
        return out

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        return self.ops.to_run_dtype(self.forward_f32(h, ctx), self.env.dtype)
