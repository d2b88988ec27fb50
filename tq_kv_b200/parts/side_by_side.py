"""Several mixers side by side on the same input.  Each branch's result is
RMS-normed over the model width with a weight of its own; the block's
residual stream gets `scale` times their sum (0.5 for the mean of two).  Where no
branch has such a norm (`out_norm` None), the results are simply added: each
branch's last product adds into the stream (a branch scales its own result, its
part's `result_scale`), and branches that run from projected rows (`input_rows`,
`run`) share ONE product of the input.

A branch is any registered mixer; what it asks of the cache is passed on: at
most one branch may ask for keys and values and at most one for per-sequence
state (a schedule entry owns one cache group and one state tensor).
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config import ConfigError
from .base import Mixer, Runtime, StepContext, WeightSpec, float32_vector, stack_rows
from .registry import make_part


class SideBySideMixer(Mixer):
    takes_pending_norm = True           # (run once here: the branches share its result)
    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.width = int(p["width"])
        self.eps = float(p.get("eps", 0.0))
        self.scale = float(p.get("scale", 1.0))
        self.branches = [make_part(b["part"]) for b in p["branches"]]
        self.norm_names = [b.get("out_norm") for b in p["branches"]]
        self.plain_sum = all(n is None for n in self.norm_names)
        if not self.plain_sum and any(n is None for n in self.norm_names):
            raise ConfigError("a side-by-side mixer norms every branch's result or none")
        if self.plain_sum and self.scale != 1.0:
            raise ConfigError("a side-by-side mixer without norms leaves the scales to its branches")
        self.one_product = self.plain_sum and all(hasattr(b, "input_rows") for b in self.branches)
        self.can_store_result = self.plain_sum and all(b.can_store_result for b in self.branches)
        self.accepts_rider = self.one_product
        self.w_in = self.bias = None
        self.columns: list = []
        if not 1 <= len(self.branches) <= 4:
            raise ConfigError("a side-by-side mixer has one to four branches")
        if sum(b.cache_request() is not None for b in self.branches) > 1 \
                or sum(b.state_request() is not None for b in self.branches) > 1:
            raise ConfigError("a side-by-side mixer can hold one branch with keys and values and one with state")
        self.norm_w: list = []

    @property
    def graph_capturable(self):
        return all(getattr(b, "graph_capturable", True) for b in self.branches)

    @property
    def padded_rows_ok(self):
        return all(getattr(b, "padded_rows_ok", False) for b in self.branches)

    def weight_specs(self):
        specs = [ws for b in self.branches for ws in b.weight_specs()]
        return specs + [WeightSpec(n, (self.width,), "norm_scale") for n in self.norm_names if n is not None]

    def ignored_weights(self):
        return [n for b in self.branches for n in b.ignored_weights()]

    def bind(self, tensors, runtime: Runtime, shared=None):
        for b in self.branches:
            b.bind(tensors, runtime, shared)
        self.norm_w = [float32_vector(tensors[n]) for n in self.norm_names if n is not None]
        if not self.one_product:
            return
        rows = [b.input_rows() for b in self.branches] + ([self.rider.rider_rows()] if self.rider is not None else [])
        self.w_in, self.bias = stack_rows([w for w, _ in rows], [bias for _, bias in rows])
        self.columns, at = [], 0
        for w, _ in rows:
            self.columns.append((at, at + w.shape[0]))
            at += w.shape[0]
        for b in self.branches:
            b.w_in = None                           # its rows live in the one product's weight now

    def cache_request(self):
        for b in self.branches:
            r = b.cache_request()
            if r is not None:
                return r
        return None

    def state_request(self):
        for b in self.branches:
            r = b.state_request()
            if r is not None:
                return r
        return None

    def check_step(self, start_pos, step_lens, owns_cache):
        for b in self.branches:
            b.check_step(start_pos, step_lens, owns_cache)

    def forward(self, x, ctx: StepContext, residual):
        if isinstance(x, kernels.PendingNorm):
            x = x.materialize()
        if self.one_product:
            proj = kernels.linear(x, self.w_in, bias=self.bias, out_dtype=torch.float32)
            kernels.mark("qkv")
            for i, b in enumerate(self.branches):
                lo, hi = self.columns[i]
                b.run(proj[:, lo:hi], ctx, residual, accumulate=i > 0 or not ctx.store_result)
            if self.rider is not None:
                lo, hi = self.columns[-1]
                ctx.rider_out = proj[:, lo:hi]
            return
        if self.plain_sum:
            stored, ctx.store_result = ctx.store_result, False
            if stored:
                residual.zero_()
            for b in self.branches:
                b.forward(x, ctx, residual)
            return
        outs = []
        for b in self.branches:
            y = torch.zeros_like(residual)          # a branch adds its result into what it is given
            b.forward(x, ctx, y)
            outs.append(y)
        kernels.add_normed(residual, list(zip(outs, self.norm_w)), self.eps, self.scale)
        kernels.mark("norms")
