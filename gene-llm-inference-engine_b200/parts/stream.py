"""What replaces the residual stream ahead of a run of the schedule (the start of a pass over layers that run several times)."""
from __future__ import annotations

import torch

from ..ops import kernels
from ..ops.linear import Linear
from .registry import register_stream_input


@register_stream_input("embedding_mix")
class EmbeddingMix:
    """x <- W [x; x0] with x0 the embedding's output. W = [W_x, W_0]: W_0 x0 is the same for every pass of a step and is
    computed once, when the step begins; a pass starts its stream from it and adds W_x x, so that only half of W is read per
    pass. The kernel that ends the layer before may hand the stream over in the compute dtype and put W_0 x0 in its place in
    the same pass (``start``, ``taken``, ``ctx.carry``).

    Params: ``hidden_size``. Weights: ``weight`` [hidden, 2 hidden] (the columns of x first)."""

    graph_safe = True

    def __init__(self, params, weights, build):
        D = self.hidden_size = int(params["hidden_size"])
        w = weights["weight"]
        if tuple(w.shape) != (D, 2 * D):
            raise ValueError(f"embedding mix: the weight has shape {tuple(w.shape)}, expected ({D}, {2 * D})")
        self.w_x = Linear(w[:, :D].contiguous(), build.compute_dtype, build.device, tiles=build.weight_tiles)
        self.w_0 = Linear(w[:, D:].contiguous(), build.compute_dtype, build.device, tiles=build.weight_tiles)
        self.dtype = build.compute_dtype

    def start(self, ctx) -> torch.Tensor:
        """What a pass's stream starts from, W_0 x0 [T, hidden] 32-bit."""
        return ctx.scratch("stream_start", (ctx.n_tokens, self.hidden_size), torch.float32)

    def taken(self, ctx) -> torch.Tensor:
        """The stream as the product reads it, [T, hidden] in the compute dtype."""
        return ctx.scratch("stream_taken", (ctx.n_tokens, self.hidden_size), self.dtype)

    def begin(self, ctx, x: torch.Tensor) -> None:
        """``x``: the embedding's output, as the step's first run finds it."""
        start, taken, x0 = self.start(ctx), self.taken(ctx), x

        def launch():
            if self.dtype is torch.float32:
                self.w_0.forward(x0, start)
            else:
                kernels.scale_cast(x0, start, taken, 0.0)
                self.w_0.forward(taken, start)
        ctx.recorded(self, ("begin", ctx.n_tokens), launch)

    def forward(self, ctx, x: torch.Tensor) -> None:
        start, taken = self.start(ctx), self.taken(ctx)
        handed = ctx.carry.pop("stream_handed", None) == (x.data_ptr(), id(self))

        def launch():
            if not handed:
                kernels.take_stream(x, start, taken)
            self.w_x.forward(taken, x, accumulate=True)
        ctx.recorded(self, ("pass", ctx.n_tokens, handed), launch)


@register_stream_input("embedding_add")
class EmbeddingAdd:
    """x <- x + x0 with x0 the embedding's output, which is kept when a step begins. The kernel that ends the layer before may
    add it in its own pass (``kept``, ``ctx.carry``). Params: ``hidden_size``."""

    graph_safe = True

    def __init__(self, params, weights, build):
        self.hidden_size = int(params["hidden_size"])

    def kept(self, ctx) -> torch.Tensor:
        """x0 [T, hidden] 32-bit."""
        return ctx.scratch("stream_start", (ctx.n_tokens, self.hidden_size), torch.float32)

    def begin(self, ctx, x: torch.Tensor) -> None:
        x0 = self.kept(ctx)
        ctx.recorded(self, ("begin", ctx.n_tokens), lambda: kernels.scale_cast(x, x0, None, 1.0))

    def forward(self, ctx, x: torch.Tensor) -> None:
        if ctx.carry.pop("stream_handed", None) == (x.data_ptr(), id(self)):
            return                      # added by the kernel that ended the layer before
        x0 = self.kept(ctx)
        ctx.recorded(self, ("pass", ctx.n_tokens), lambda: kernels.add_stream(x, x0))
