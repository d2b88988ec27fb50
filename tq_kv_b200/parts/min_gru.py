"""A mixer whose memory is one number per channel, with an update gate that does not look at it (minGRU):

    z = sigmoid(W_z x + b_z),   u = W_x x + b_x,   c = u + 1/2 for u >= 0, sigmoid(u) below
    S_t = (1 - z) S_{t-1} + z c                       entry by entry, `width` channels
    out = W_o (S_t * silu(W_g x)) * result_scale

S starts at zero, is float32 and lives in the cache's per-sequence state.  The three projections of x are one product
(float32 result); the recurrence and its result's gate are one kernel (csrc/gru_scan.cu), which also applies
`result_scale`, in float32.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache import StateRequest
from .base import Mixer, Runtime, StepContext, WeightSpec, float32_vector, stack_rows


class MinGRUMixer(Mixer):
    graph_capturable = True             # slots and lengths are read on the device
    can_store_result = True

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden, self.width = int(p["hidden_size"]), int(p["width"])
        self.result_scale = float(p.get("result_scale", 1.0))
        self.names = dict(p["names"])
        self.stride = -(-self.width // 8) * 8           # columns of a projection in the product's result
        self.w_in = self.bias = self.w_o = None

    def _n(self, which: str) -> str:
        return self.prefix + self.names[which]

    def weight_specs(self):
        n, h = self.width, self.hidden
        return [WeightSpec(self._n("update"), (n, h), "matrix"), WeightSpec(self._n("update_bias"), (n,), "bias"),
                WeightSpec(self._n("candidate"), (n, h), "matrix"), WeightSpec(self._n("candidate_bias"), (n,), "bias"),
                WeightSpec(self._n("gate"), (n, h), "matrix"), WeightSpec(self._n("out"), (h, n), "matrix")]

    def bind(self, tensors, runtime: Runtime, shared=None):
        rows, biases = [], []
        for w, b in (("update", "update_bias"), ("candidate", "candidate_bias"), ("gate", None)):
            padded, bias = stack_rows([tensors[self._n(w)]], [None if b is None else float32_vector(tensors[self._n(b)])])
            rows.append(padded)
            biases.append(bias)
        self.w_in, self.bias = stack_rows(rows, biases)
        self.w_o = tensors[self._n("out")].contiguous()

    def state_request(self):
        return StateRequest((self.width,), torch.float32)

    def input_rows(self):
        return self.w_in, self.bias

    def forward(self, x, ctx: StepContext, residual):
        proj = kernels.linear(x, self.w_in, bias=self.bias, out_dtype=torch.float32)
        kernels.mark("qkv")
        self.run(proj, ctx, residual, accumulate=not ctx.store_result)

    def run(self, proj, ctx: StepContext, residual, accumulate: bool) -> None:
        """The mixer on its projected rows (float32 [T, input rows], may be a column slice of wider rows)."""
        b, n, s = ctx.batch, self.width, self.stride
        y = torch.empty((proj.shape[0], n), dtype=ctx.runtime.act_dtype, device=proj.device)
        kernels.gru_scan(proj[:, :n], proj[:, s:s + n], proj[:, 2 * s:2 * s + n], ctx.state, b.cu_seqlens, b.slots, y,
                         n_seqs=b.n_seqs, scale=self.result_scale, single_tokens=b.single_tokens)
        kernels.mark("gru")
        kernels.linear(y, self.w_o, out=residual, accumulate=accumulate)
        kernels.mark("o")
