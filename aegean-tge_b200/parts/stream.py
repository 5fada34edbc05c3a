"""Parts that act on the whole residual: steps before a layer, and a residual made of several streams.

Steps that change the whole stream before a layer runs (``LayerSpec.entry``):

``reinject``: x <- W [x; x0] + step[index], with x0 the embedding output of the same tokens, W [H, 2H] (the
columns of x first) and ``step`` one row per pass over a run of layers.  The product reads [x | x0] in the
products' number format and writes the float32 stream, the step's row added as the product's bias.

Several streams (hyper-connections): the residual is S rows per token, x [T, S, width], all the embedding output at the
start.  ``connected_rmsnorm`` is a sublayer's norm together with its connection (a [S], B [S, S], c [S]):

    u = sum_s a_s x_s      y = f(n(u))      x_t <- sum_s B[s, t] x_s + c_t y, all t at once from the old ones

Its ``forward`` gives n(u); its ``update`` and ``update_product`` write the streams back and, in the same kernel, give what
the next sublayer's norm reads.  Without a connection (``connected`` False) it is the norm of the streams' sum, which the
head reads.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from .base import NORMS, STREAM_STEPS, Norm, ParamSpec, StepContext, StreamStep


@STREAM_STEPS.register("reinject")
class Reinject(StreamStep):
    """params: ``hidden_size``, ``index`` (which row of ``step`` this visit adds), ``count`` (rows of ``step``).
    weights: ``weight`` [hidden, 2 hidden], ``step`` (float32 [count, hidden])."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        self.hidden = int(spec.params["hidden_size"])
        self.index = int(spec.params["index"])
        self.count = int(spec.params["count"])
        if self.hidden <= 0 or not 0 <= self.index < self.count:
            raise ValueError(f"reinject: row {self.index} of {self.count}, width {self.hidden}")
        self.weight: Optional[torch.Tensor] = None
        self.step: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.hidden, 2 * self.hidden)), "step": ParamSpec((self.count, self.hidden), role="vector")}

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.weight = tensors["weight"].contiguous()
        self.step = tensors["step"][self.index].contiguous()

    def param_bytes(self) -> int:
        return 2 * self.hidden * self.hidden * self.env.dtype.itemsize + 4 * self.hidden

    def flops(self, tokens: int, pairs: float) -> float:
        return 2.0 * tokens * 2 * self.hidden * self.hidden

    def forward(self, x: torch.Tensor, x0: torch.Tensor, ctx: StepContext) -> None:
        both = self.ops.concat_rows(x, x0, self.env.dtype)
        self.ops.linear(both, self.weight, self.step, self.ops.GEMM_STORE_F32, out=x)


@NORMS.register("connected_rmsnorm")
class ConnectedRMSNorm(Norm):
    """params: ``size`` (a stream's width), ``eps``, ``streams``, optional ``connected`` (default True; False: all streams are
    added up, and nothing is written back), ``unit_offset`` (the weight is stored around zero), ``optional`` (a checkpoint may
    lack the parameters; the norm then does not exist).  weights: ``weight`` and, connected, ``in`` [S], ``mix`` [S, S]
    (indexed [from, to]) and ``out`` [S], all float32.

    A step of up to ``ops.DEFER_MAX_TOKENS`` bfloat16 rows spreads every row over many blocks and hands the rows on without
    their norm's factor; a caller whose next part does not take such rows gets them completed."""
    graph_safe = True

    def __init__(self, spec, env):
        super().__init__(spec, env)
        p = spec.params
        self.size, self.eps, self.streams = int(p["size"]), float(p["eps"]), int(p["streams"])
        if self.size <= 0 or not self.eps > 0.0 or not 0 < self.streams <= 16:
            raise ValueError(f"connected_rmsnorm: size {self.size}, eps {self.eps}, {self.streams} streams (1 to 16)")
        self.connected = bool(p.get("connected", True))
        self.unit_offset = bool(p.get("unit_offset", False))
        self.optional = bool(p.get("optional", False))
        self.weight: Optional[torch.Tensor] = None
        self.into: Optional[torch.Tensor] = None
        self.mix: Optional[torch.Tensor] = None
        self.out: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        specs = {"weight": ParamSpec((self.size,), role="vector", optional=self.optional)}
        if self.connected:
            for name, shape in (("in", (self.streams,)), ("mix", (self.streams, self.streams)), ("out", (self.streams,))):
                specs[name] = ParamSpec(shape, role="vector", optional=self.optional)
        return specs

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        weight = tensors.get("weight") if self.optional else tensors["weight"]
        if weight is None:
            return
        self.weight = (weight.float() + 1.0 if self.unit_offset else weight).contiguous()
        if self.connected and not (self.optional and "mix" not in tensors):
            self.into, self.mix, self.out = (tensors[name].contiguous() for name in ("in", "mix", "out"))

    def reads(self):
        """What the kernels need to give this norm's rows: (combination or None, weight, eps)."""
        if self.weight is None:
            raise RuntimeError("connected_rmsnorm: the checkpoint holds no weight for this norm")
        return self.into, self.weight, self.eps

    def few(self, x: torch.Tensor) -> bool:
        return self.env.dtype == torch.bfloat16 and x.shape[0] <= self.ops.DEFER_MAX_TOKENS

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None, defer: bool = False):
        into, weight, eps = self.reads()
        if rows is None and self.few(x):
            h = self.ops.streams_defer(x, (into, weight, eps))
            return h if defer else h.complete()
        return self.ops.streams_norm(x, into, weight, eps, self.env.dtype, rows=rows)

    def update(self, x: torch.Tensor, y: torch.Tensor, following: Optional["ConnectedRMSNorm"], defer: bool = False):
        """Writes the sublayer's output y (float32 [T, width]) back into the streams; returns ``following``'s rows of the
        new streams (None without one)."""
        reads = following.reads() if following is not None else None
        if self.few(x):
            h = self.ops.streams_defer(x, reads, y, 1, self.mix, self.out)
            return h if defer or h is None else h.complete()
        return self.ops.streams_update(x, y, self.mix, self.out, reads, self.env.dtype)

    def update_product(self, x: torch.Tensor, rows: torch.Tensor, weight: torch.Tensor, following: Optional["ConnectedRMSNorm"],
                       defer: bool = False):
        """:meth:`update` with y = rows . weight^T; of few rows the product's partial sums go straight to the update."""
        partial = self.ops.linear_partials(rows, weight) if self.few(x) else None
        if partial is None:
            return self.update(x, self.ops.linear(rows, weight, None, self.ops.GEMM_STORE_F32), following, defer)
        reads = following.reads() if following is not None else None
        h = self.ops.streams_defer(x, reads, partial[0], partial[1], self.mix, self.out)
        return h if defer or h is None else h.complete()
