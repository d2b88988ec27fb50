"""Dense gated feed-forward.  Reference: src/models/turbo_generic.rs:105-110
— down(silu(gate x) * (up x)), no biases; :1980 — residual sum.  Gate and up
weights are concatenated at bind time so that one product yields both.
`activation` names the gate's function: "silu" (the default, SwiGLU) or
"gelu_tanh", 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).

Beside it the form without a gate, down(max(up x, 0)^2), whose first product applies
its activation in its own last step."""
from __future__ import annotations

import torch

from .. import kernels
from ..config import ConfigError
from .base import FeedForward, Runtime, StepContext, WeightSpec


class SwiGLU(FeedForward):
    takes_pending_norm = True           # x goes to kernels.linear only
    padded_rows_ok = True               # row by row
    can_store_result = True

    def __init__(self, spec):
        super().__init__(spec)
        self.activation = kernels.activation_code(self.params.get("activation", "silu"))
        self.hidden = int(self.params["hidden_size"])
        self.inter = int(self.params["intermediate_size"])
        self.names = dict(self.params.get("names", {"gate": "gate_proj", "up": "up_proj", "down": "down_proj"}))
        self.suffix = self.params.get("weight_suffix", ".weight")     # what follows a projection's name in a tensor's
        self.w_gate_up = self.w_down = None

    def _n(self, which):
        return f"{self.prefix}{self.names[which]}{self.suffix}"

    def weight_specs(self):
        return [WeightSpec(self._n("gate"), (self.inter, self.hidden), "matrix"),
                WeightSpec(self._n("up"), (self.inter, self.hidden), "matrix"),
                WeightSpec(self._n("down"), (self.hidden, self.inter), "matrix")]

    def bind(self, tensors, runtime: Runtime, shared=None):
        g, u = tensors[self._n("gate")], tensors[self._n("up")]
        if g.dtype != u.dtype:
            g, u = g.to(torch.float32), u.to(torch.float32)
        self.w_gate_up = torch.cat([g, u], dim=0).contiguous()
        self.w_down = tensors[self._n("down")].contiguous()

    def forward(self, x, ctx: StepContext, residual):
        act = kernels.linear(x, self.w_gate_up, swiglu=True, activation=self.activation,
                             out_dtype=ctx.runtime.act_dtype)
        kernels.mark("gate_up")
        kernels.linear(act, self.w_down, out=residual, accumulate=not ctx.store_result)
        kernels.mark("down")


class PlainFeedForward(FeedForward):
    """down(act(up x)) with act the square of relu, no biases."""
    padded_rows_ok = True               # row by row
    can_store_result = True

    def __init__(self, spec):
        super().__init__(spec)
        self.activation = kernels.activation_code(self.params.get("activation", "square_relu"))
        if self.activation != kernels.ACT_SQUARE_RELU:
            raise ConfigError("a feed-forward without a gate has the activation square_relu")
        self.hidden, self.inter = int(self.params["hidden_size"]), int(self.params["intermediate_size"])
        self.names = dict(self.params.get("names", {"up": "up", "down": "down"}))
        self.w_up = self.w_down = None

    def _n(self, which):
        return self.prefix + self.names[which]

    def weight_specs(self):
        return [WeightSpec(self._n("up"), (self.inter, self.hidden), "matrix"),
                WeightSpec(self._n("down"), (self.hidden, self.inter), "matrix")]

    def bind(self, tensors, runtime: Runtime, shared=None):
        self.w_up = tensors[self._n("up")].contiguous()
        self.w_down = tensors[self._n("down")].contiguous()

    def forward(self, x, ctx: StepContext, residual):
        act = kernels.linear(x, self.w_up, activation=self.activation, out_dtype=ctx.runtime.act_dtype)
        kernels.mark("up")
        kernels.linear(act, self.w_down, out=residual, accumulate=not ctx.store_result)
        kernels.mark("down")
