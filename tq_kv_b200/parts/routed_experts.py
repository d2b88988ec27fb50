"""A feed-forward of `experts` small layers of which each token uses `top`.

Expert e is  W_down[e] (silu(W_gate[e] x) * (W_up[e] x)),  or with `gated` False
W_down[e] max(W_up[e] x, 0)^2;  no biases.  Which experts a
token uses is `routing`:
  "table"   there is no router: a table [vocab, top] of expert indices (the
            entries of a row differ) names them by the token's id; each has the
            weight 1 / top.
  "router"  scores s = sigmoid(W_router x), computed in float32; the `top` experts
            with the largest scores are chosen (the lowest index first among equals);
            their weights are  router_scale * s / (sum of the chosen s + weight_sum_floor).
  "softmax_router"  logits z = W_router x (+ the bias `router_bias` names), in float32; the
            `top` largest are chosen; their weights are the softmax over the chosen logits.
  "group_router"  scores s = softmax(W_router x) over all experts, in float32; the choice
            goes by s + correction (a learned number per expert): the experts lie in
            `groups` equal groups of neighbours, a group counts as its largest choice
            score, and of the `keep_groups` best groups' experts the `top` best are
            chosen; their weights are their s as they are.
The result is the weighted sum of the chosen experts' results.  With `shared_size` > 0
a shared expert of that inner width (same form, tensors under `names["shared"]`) runs
for every token and is added; with `shared_gate` times sigmoid(w x), one number per token (the
row `names["shared_gate"]` rides in the router's product, and the experts' last kernel
adds the gated result).

The experts' weights are stacked at bind time ([E, 2F, W] gate rows then up rows,
and [E, W, F]).  Few rows (decoding) and the float32 path run every (token, expert)
pair as a row-times-matrix product of its own (csrc/routed_experts.cu); bfloat16
steps with many rows, or with at least two pairs per expert, are sorted by expert
and run as tiles of one matrix product per projection
(`kernels.routed_experts_tiles`): each expert's matrices are then read once.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..config import ConfigError
from .base import FeedForward, Runtime, StepContext, WeightSpec, float32_vector, stack_rows


class TableExperts(FeedForward):
    padded_rows_ok = True               # row by row
    can_store_result = True
    TILE_MIN_ROWS = 65                  # from this many rows on, bfloat16 steps run the sorted tiles
    # ... and from this many (token, expert) pairs per expert on: the row form reads an expert's matrices once per
    # pair, the tiles once per expert, so decode batches whose tokens share experts run the tiles too (measured at
    # 8 experts of 4,096 x 5,504, 2 per token: 8 rows 1.14 -> 1.09 ms a step, 64 rows 5.79 -> 1.33; 4 rows 0.83 -> 0.97)
    TILE_MIN_PAIRS_PER_EXPERT = 2

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.inter = int(p["intermediate_size"])
        self.n_experts = int(p["experts"])
        self.top = int(p["top"])
        self.routing = p.get("routing", "table")
        if self.routing not in ("table", "router", "softmax_router", "group_router"):
            raise ConfigError(f"routed experts: unknown routing '{self.routing}' (known: table, router, softmax_router, "
                              f"group_router)")
        self.gated = bool(p.get("gated", True))
        self.groups, self.keep_groups = int(p.get("groups", 1)), int(p.get("keep_groups", 1))
        if self.routing == "group_router":
            if self.groups < 1 or self.n_experts % self.groups or not 1 <= self.keep_groups <= self.groups:
                raise ConfigError(f"routed experts: {self.n_experts} experts in {self.groups} equal groups, {self.keep_groups} kept")
            if self.top > self.keep_groups * (self.n_experts // self.groups):
                raise ConfigError(f"routed experts: a token cannot use {self.top} experts of {self.keep_groups} groups of "
                                  f"{self.n_experts // self.groups}")
        self.has_router_bias = self.routing == "softmax_router" and bool(p.get("router_bias", False))
        self.accepts_rider = self.routing == "group_router"      # (rows beside the router's)
        self.vocab = int(p["vocab_size"]) if self.routing == "table" else 0
        self.router_scale = float(p.get("router_scale", 1.0))
        self.weight_sum_floor = float(p.get("weight_sum_floor", 0.0))
        self.shared_size = int(p.get("shared_size") or 0)
        self.shared_gate = bool(p.get("shared_gate", False))
        if self.shared_gate and (not self.shared_size or self.routing != "softmax_router"):
            raise ConfigError("routed experts: a gate on the shared expert needs one, beside a softmax_router")
        if not 1 <= self.top <= self.n_experts:
            raise ConfigError(f"routed experts: a token cannot use {self.top} of {self.n_experts} experts")
        self.names = dict(p.get("names", {"expert": "e{}.", "gate": "gate", "up": "up", "down": "down", "table": "table"}))
        self.names.setdefault("router", "router")
        self.names.setdefault("shared", "shared.")
        self.names.setdefault("correction", "correction")
        self.names.setdefault("router_bias", "router.b")
        self.names.setdefault("shared_gate", "shared.sg")
        self.w_gate_up = self.w_down = self.table = self.w_router = self.w_shared_gate_up = self.w_shared_down = None
        self.correction = self.router_bias = None
        self.projections = ("gate", "up") if self.gated else ("up",)      # the rows of an expert's first product

    def _e(self, e: int, which: str) -> str:
        return f"{self.prefix}{self.names['expert'].format(e)}{self.names[which]}"

    def weight_specs(self):
        specs = []
        for e in range(self.n_experts):
            specs += [WeightSpec(self._e(e, w), (self.inter, self.hidden), "matrix") for w in self.projections]
            specs.append(WeightSpec(self._e(e, "down"), (self.hidden, self.inter), "matrix"))
        if self.routing == "table":
            specs.append(WeightSpec(self.prefix + self.names["table"], (self.vocab, self.top),
                                    f"choice_table:{self.n_experts}"))
        else:
            specs.append(WeightSpec(self.prefix + self.names["router"], (self.n_experts, self.hidden), "matrix"))
        if self.routing == "group_router":
            specs.append(WeightSpec(self.prefix + self.names["correction"], (self.n_experts,), "bias"))
        if self.has_router_bias:
            specs.append(WeightSpec(self.prefix + self.names["router_bias"], (self.n_experts,), "bias"))
        if self.shared_gate:
            specs.append(WeightSpec(self.prefix + self.names["shared_gate"], (1, self.hidden), "matrix"))
        if self.shared_size:
            sp = self.prefix + self.names["shared"]
            specs += [WeightSpec(sp + self.names[w], (self.shared_size, self.hidden), "matrix") for w in self.projections]
            specs.append(WeightSpec(sp + self.names["down"], (self.hidden, self.shared_size), "matrix"))
        return specs

    def bind(self, tensors, runtime: Runtime, shared=None):
        n = len(self.projections)
        mats = [tensors[self._e(e, w)] for e in range(self.n_experts) for w in (*self.projections, "down")]
        if len({m.dtype for m in mats}) != 1:
            mats = [m.to(torch.float32) for m in mats]
        gu = [torch.cat(mats[(n + 1) * e:(n + 1) * e + n], dim=0) for e in range(self.n_experts)]
        self.w_gate_up = torch.stack(gu).contiguous()                        # [E, 2F, W] (without a gate [E, F, W])
        self.w_down = torch.stack([mats[(n + 1) * e + n] for e in range(self.n_experts)]).contiguous()   # [E, W, F]
        if self.shared_size:
            sp = self.prefix + self.names["shared"]
            rows = [tensors[sp + self.names[w]] for w in self.projections]
            if len({r.dtype for r in rows}) != 1:
                rows = [r.to(torch.float32) for r in rows]
            self.w_shared_gate_up = torch.cat(rows, dim=0).contiguous()
            self.w_shared_down = tensors[sp + self.names["down"]].contiguous()
        if self.routing == "router":
            self.w_router = tensors[self.prefix + self.names["router"]].contiguous()
            return
        if self.routing == "softmax_router":         # the router's rows, then the shared expert's gate
            rows = [(tensors[self.prefix + self.names["router"]],
                     float32_vector(tensors[self.prefix + self.names["router_bias"]]) if self.has_router_bias else None)]
            if self.shared_gate:
                rows.append((tensors[self.prefix + self.names["shared_gate"]], None))
            self.w_router, self.router_bias = stack_rows([w for w, _ in rows], [b for _, b in rows])
            return
        if self.routing == "group_router":           # the rider's rows first: their columns then start aligned
            rows = ([self.rider.rider_rows()] if self.rider is not None else []) \
                + [(tensors[self.prefix + self.names["router"]], None)]
            self.w_router, self.router_bias = stack_rows([w for w, _ in rows], [b for _, b in rows])
            self.router_col = rows[0][0].shape[0] if self.rider is not None else 0
            self.correction = float32_vector(tensors[self.prefix + self.names["correction"]])
            return
        table = tensors[self.prefix + self.names["table"]]
        if table.dtype != torch.int32:
            raise ConfigError(f"routed experts: the table {self.prefix + self.names['table']} must hold integers")
        lo, hi = int(table.min()), int(table.max())
        if lo < 0 or hi >= self.n_experts:
            raise ConfigError(f"routed experts: the table names experts {lo} .. {hi}; there are {self.n_experts}")
        self.table = table.contiguous()

    def forward(self, x, ctx: StepContext, residual):
        weights = None
        if self.routing == "table":
            choice = kernels.table_choice(ctx.batch.tokens, self.table, self.n_experts)
        elif self.routing == "group_router":
            proj = kernels.linear(x, self.w_router, bias=self.router_bias, out_dtype=torch.float32)
            kernels.mark("router")
            if self.rider is not None:
                ctx.rider_out = proj[:, :self.router_col]
            choice, weights = kernels.group_router_choice(proj[:, self.router_col:self.router_col + self.n_experts],
                                                          self.top, self.correction, self.groups, self.keep_groups)
        elif self.routing == "softmax_router":
            proj = kernels.linear(x, self.w_router, bias=self.router_bias, out_dtype=torch.float32)
            kernels.mark("router")
            choice, weights = kernels.router_choice(proj[:, :self.n_experts], self.top, softmax=True)
        else:
            logits = kernels.linear(x, self.w_router, out_dtype=torch.float32)
            choice, weights = kernels.router_choice(logits, self.top, self.router_scale, self.weight_sum_floor)
        T = x.shape[0]
        shared = {}
        if self.shared_gate:                # its result goes beside the experts', gated by their last kernel
            shared = {"shared": self._shared_result(x, ctx), "shared_gate": proj[:, self.n_experts:self.n_experts + 1]}
        if ((T >= self.TILE_MIN_ROWS or T * self.top >= self.TILE_MIN_PAIRS_PER_EXPERT * self.n_experts)
                and x.dtype == torch.bfloat16 and kernels.routed_tiles_ok(x, self.w_gate_up, self.w_down, self.gated)):
            kernels.routed_experts_tiles(x, self.w_gate_up, self.w_down, choice, residual,
                                         accumulate=not ctx.store_result, weights=weights, gated=self.gated, **shared)
        else:
            kernels.routed_experts_rows(x, self.w_gate_up, self.w_down, choice, residual,
                                        accumulate=not ctx.store_result, weights=weights, gated=self.gated, **shared)
        kernels.mark("experts")
        if self.shared_size and not self.shared_gate:
            self._shared_result(x, ctx, residual)

    def _shared_result(self, x, ctx, residual=None):
        """The shared expert's result, added into `residual` or (none given) in float32 rows of its own."""
        act = kernels.linear(x, self.w_shared_gate_up, swiglu=self.gated, out_dtype=ctx.runtime.act_dtype,
                             activation=kernels.ACT_SILU if self.gated else kernels.ACT_SQUARE_RELU)
        if residual is None:
            out = kernels.linear(act, self.w_shared_down, out_dtype=torch.float32)
        else:
            out = kernels.linear(act, self.w_shared_down, out=residual, accumulate=True)
        kernels.mark("shared_expert")
        return out
