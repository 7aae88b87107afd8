"""Dense gated feed-forward: ``h = act(x Wg^T) * (x Wu^T)``; ``out = h Wd^T`` added to the
residual; no biases (src/model.c:612-623, src/mathx.c:34: ``act`` = silu, the reference's only one;
``activation`` may also name relu or gelu_tanh).  ``bias_suffix`` adds a bias to each of the three products.
``activation`` "clamped" with ``clamp`` = {limit, alpha, offset}: with g and u the gate's and the up product's results, ``h =
min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u, -limit, limit) + offset)``.  Gate and up are one matrix product over the
concatenated rows, as the reference serves both with one pass over the activations
(src/model.c:612-615)."""
from __future__ import annotations

import torch

from .. import kernels
from ..config.base import UnsupportedError
from ..weights.loader import TensorSpec, fused_rows
from .base import FeedForward, register_part


class SwiGlu(FeedForward):
    graph_safe = True

    def __init__(self, hidden_size: int, intermediate_size: int, prefix: str, names=None, activation: str = "silu", clamp=None,
                 bias_suffix=None, **_):
        self.E, self.F = int(hidden_size), int(intermediate_size)
        if activation not in ("silu", "relu", "gelu_tanh", "clamped"):
            raise UnsupportedError(f"gated feed-forward: activation '{activation}' is not supported")
        if (activation == "clamped") != bool(clamp):
            raise UnsupportedError("gated feed-forward: the clamped activation and its constants come together")
        self.activation = activation
        self.clamp = (float(clamp["limit"]), float(clamp["alpha"]), float(clamp["offset"])) if clamp else None
        n = {"gate": "gate_proj.weight", "up": "up_proj.weight", "down": "down_proj.weight"}
        n.update(names or {})
        self.names = {k: f"{prefix}.{v}" for k, v in n.items()}
        self.bias_names = {k: v + bias_suffix for k, v in self.names.items()} if bias_suffix else {}
        self.w_gate_up = self.w_down = self.b_gate_up = self.b_down = None

    def tensor_specs(self):
        s = [TensorSpec(self.names["gate"], (self.F, self.E)), TensorSpec(self.names["up"], (self.F, self.E)),
             TensorSpec(self.names["down"], (self.E, self.F))]
        if self.bias_names:
            s += [TensorSpec(self.bias_names["gate"], (self.F,)), TensorSpec(self.bias_names["up"], (self.F,)),
                  TensorSpec(self.bias_names["down"], (self.E,))]
        return s

    def bind(self, tensors, run_dtype, device):
        # rows alternate gate_i, up_i, so that a product's epilogue finds both of a pair side by side
        self.w_gate_up = fused_rows(tensors, [self.names["gate"], self.names["up"]], device, interleave=True)
        self.w_down = tensors[self.names["down"]].contiguous()
        if self.bias_names:
            self.b_gate_up = torch.stack([tensors[self.bias_names["gate"]], tensors[self.bias_names["up"]]], 1).reshape(-1).contiguous()
            self.b_down = tensors[self.bias_names["down"]].contiguous()

    @property
    def operand_width(self):
        """Width of the down product's operand (what :meth:`operand` writes)."""
        return self.F

    def operand(self, ctx, xn, out):
        """The down product's operand into ``out`` [T, F], which may be a column slice of a wider array."""
        gu = ctx.buf("ffn_gate_up", (xn.shape[0], 2 * self.F), xn.dtype)
        with kernels.phase("gate_up"):
            kernels.linear_glu(xn, self.w_gate_up, gu, out, self.activation, bias=self.b_gate_up, clamp=self.clamp)

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_gate_up, self.w_down))

    def flops(self, rows):
        return 2.0 * rows * (self.w_gate_up.numel() + self.w_down.numel())

    def _hidden(self, ctx, xn):
        h = ctx.buf("ffn_h", (xn.shape[0], self.F), xn.dtype)
        self.operand(ctx, xn, h)
        return h

    def forward(self, ctx, xn, residual, accumulate=True):
        """``accumulate=False`` stores the output in ``residual`` (float32) instead of adding it."""
        h = self._hidden(ctx, xn)
        with kernels.phase("down"):
            kernels.linear(h, self.w_down, self.b_down, residual, accumulate=accumulate)

    def forward_into_norm(self, ctx, xn, y_buf, residual, post, next_norm, out):
        """residual += post(feed-forward output), the down product handed to the norm."""
        h = self._hidden(ctx, xn)
        with kernels.phase("down"):
            return post.add_product_into(h, self.w_down, self.b_down, y_buf, residual, next_norm, out)

    def forward_then_norm(self, ctx, xn, residual, norm, out):
        args = norm.fused_args()
        if args is None:
            self.forward(ctx, xn, residual)
            return False
        h = self._hidden(ctx, xn)
        with kernels.phase("down"):
            kernels.linear_residual_norm(h, self.w_down, self.b_down, residual, args[0], args[1], out, **(args[2] if len(args) > 2 else {}))
        return True


class Mlp(FeedForward):
    """The feed-forward without a gate: ``down(act(up x))``; ``activation`` as the product kernels name them (``relu2``
    is the square of relu).  The activation runs in the up product's epilogue, the down product ends in the sum with the
    stream and the following norm, as the gated form's does."""
    graph_safe = True

    def __init__(self, hidden_size: int, intermediate_size: int, prefix: str, activation: str = "relu2", names=None, **_):
        self.E, self.F = int(hidden_size), int(intermediate_size)
        if activation not in kernels.ACTIVATIONS or activation == "none":
            raise UnsupportedError(f"feed-forward: activation '{activation}' is not supported")
        self.activation = activation
        n = {"up": "up", "down": "down"}
        n.update(names or {})
        self.names = {k: f"{prefix}.{v}" for k, v in n.items()}
        self.w_up = self.w_down = None

    def tensor_specs(self):
        return [TensorSpec(self.names["up"], (self.F, self.E)), TensorSpec(self.names["down"], (self.E, self.F))]

    def bind(self, tensors, run_dtype, device):
        self.w_up = tensors[self.names["up"]].contiguous()
        self.w_down = tensors[self.names["down"]].contiguous()

    def weight_bytes(self):
        return sum(w.numel() * w.element_size() for w in (self.w_up, self.w_down))

    def flops(self, rows):
        return 2.0 * rows * (self.w_up.numel() + self.w_down.numel())

    def _hidden(self, ctx, xn):
        h = ctx.buf("ffn_h", (xn.shape[0], self.F), xn.dtype)
        with kernels.phase("gate_up"):
            kernels.linear_act(xn, self.w_up, h, self.activation)
        return h

    def forward(self, ctx, xn, residual, accumulate=True):
        h = self._hidden(ctx, xn)
        with kernels.phase("down"):
            kernels.linear(h, self.w_down, None, residual, accumulate=accumulate)

    def forward_into_norm(self, ctx, xn, y_buf, residual, post, next_norm, out):
        h = self._hidden(ctx, xn)
        with kernels.phase("down"):
            return post.add_product_into(h, self.w_down, None, y_buf, residual, next_norm, out)

    def forward_then_norm(self, ctx, xn, residual, norm, out):
        args = norm.fused_args()
        if args is None:
            self.forward(ctx, xn, residual)
            return False
        h = self._hidden(ctx, xn)
        with kernels.phase("down"):
            kernels.linear_residual_norm(h, self.w_down, None, residual, args[0], args[1], out, **(args[2] if len(args) > 2 else {}))
        return True


register_part("ffn", "mlp", Mlp)
register_part("ffn", "swiglu", SwiGlu)
register_part("ffn", "gated", SwiGlu)               # the same part under the name that does not fix the activation
