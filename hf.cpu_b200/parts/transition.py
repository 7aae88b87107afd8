"""Steps on the stream between layers.

``join_embedding``: in front of pass t of a stretch of layers that runs several times,

    x <- W_in [x; x0] + step_t         x0: the embedding output,  W_in [E, 2 E] (x first),  step [passes, E]

W_in is kept as its two halves: ``c = W_0 x0`` is the same in every pass and is made once per step of the engine, so a pass
costs the product with x only.  That product's (partial) sums, c and the pass's vector meet in one pass over the stream
that also norms it for the layer behind; the block in front hands the stream over as that product's operand.  The sums
and the stream are float32; the product's operands have the run's type.  (The reference runs its layers once, in order,
src/model.c:574.)
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config.base import UnsupportedError
from ..weights.loader import TensorSpec
from .base import Transition, register_part
from .norm import RmsNorm, StreamCast


class JoinEmbedding(Transition):
    graph_safe = True
    OFFSET = "join_offset"              # scratch: W_0 x0 of the step's tokens, float32

    def __init__(self, hidden_size: int, passes: int, tensor: str, step_tensor: str, first: bool = False, **_):
        self.E, self.passes, self.tensor, self.step_tensor = int(hidden_size), int(passes), tensor, step_tensor
        # whether the first pass starts at the embedding itself (no layer in front): its operand is then x0's
        self.first = bool(first)
        if self.passes < 0:
            raise UnsupportedError("a stretch of layers runs a number of times that is not negative")
        self.w_x = self.w_0 = self.step = None
        self._cast = StreamCast()

    def tensor_specs(self):
        return [TensorSpec(self.tensor, (self.E, 2 * self.E)), TensorSpec(self.step_tensor, (self.passes, self.E))]

    def bind(self, tensors, run_dtype, device):
        w = tensors[self.tensor]
        self.w_x, self.w_0 = w[:, :self.E].contiguous(), w[:, self.E:].contiguous()
        self.step = tensors[self.step_tensor].to(torch.float32).contiguous()

    def weight_bytes(self):
        """Per pass (the embedding's half is read once a step: shared out over the passes)."""
        b = self.w_x.numel() * self.w_x.element_size()
        return b + b // max(self.passes, 1)

    def flops(self, rows):
        """Per pass, as for :meth:`weight_bytes`."""
        return 2.0 * rows * self.w_x.numel() * (1.0 + 1.0 / max(self.passes, 1))

    def operand_norm(self):
        return self._cast

    def begin(self, ctx, x):
        if self.passes < 1:
            return
        x0 = self._cast.forward(x, ctx.buf("join_x0", x.shape, ctx.run_dtype))
        with kernels.phase("join"):
            kernels.linear(x0, self.w_0, None, ctx.buf(self.OFFSET, x.shape, torch.float32), accumulate=False)

    def enter(self, ctx, x, number, ready, norm, out):
        if ready is None:
            ready = ctx.buf("join_x0", x.shape, ctx.run_dtype)
            if number > 0 or not self.first:
                ready = self._cast.forward(x, ctx.buf("join_operand", x.shape, ctx.run_dtype))
        nxt = (norm.weight, norm.eps) if isinstance(norm, RmsNorm) else None
        with kernels.phase("join"):
            kernels.linear_rms_tail(ready, self.w_x, ctx.buf("join_sums", x.shape, torch.float32), x, bias=self.step[number],
                                    base=ctx.buf(self.OFFSET, x.shape, torch.float32), nxt=nxt, out=out if nxt is not None else None)
        return nxt is not None


register_part("transition", "join_embedding", JoinEmbedding)
