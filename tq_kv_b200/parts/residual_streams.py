"""A residual stream kept as several parallel streams (hyper-connections), and the layer arrangement that
works on them.

Instead of one x there are S copies x_1 .. x_S, all equal to the embedding at the start.  Sublayer q of a layer
(1: the mixer, 2: the feed-forward) has three small tensors, `<layer>hc<q>.in` [S], `.out` [S] and `.mix`
[S, S] (indexed [from, to]):

    u = sum_s in[s] x_s;   y = sublayer(norm(u));   x_r <- sum_s mix[s, r] x_s + out[r] y   (all r at once).

At the end the model reads the sum of the streams.  The streams are float32 and every sum is float32.  Options of a
layer: a factor on what every sublayer writes (`residual_mult`, folded into out), and on a sublayer's result a vector
and a gate, y <- y * scale * sigmoid(R h + b) with h = norm(u), what the sublayer read (part `SublayerResult`); they
are applied where y enters the streams.

`ResidualStreams` holds the streams [S, T, W] and what the last sublayer still has to write.  The write is put off
until the next reader comes, so that one kernel per sublayer boundary does the write, the next read and the
norm on it (csrc/stream_mix.cu): a layer of two sublayers costs two launches, as many as the two norms of a
plain pre-norm layer.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import kernels
from ..config import ConfigError, LayerSpec
from .base import Part, Runtime, StepContext, WeightSpec, float32_vector
from .registry import make_part


class ResidualStreams:
    def __init__(self, x: torch.Tensor, n_streams: int):
        self.xs = kernels.streams_fill(x, n_streams)
        self.n_streams = n_streams
        self._pending: dict = {}                      # y, mix, write (y_scale, y_gate) of the sublayer that ran last
        self._ones: Optional[torch.Tensor] = None

    def write_later(self, y: torch.Tensor, mix: torch.Tensor, write: torch.Tensor, y_scale: Optional[torch.Tensor] = None,
                    y_gate: Optional[torch.Tensor] = None) -> None:
        self.flush()
        self._pending = {"y": y, "mix": mix, "write": write, "y_scale": y_scale, "y_gate": y_gate}

    def read(self, coefs: torch.Tensor, norm: Optional[dict], out_dtype, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """sum_s coefs[s] x_s (after the write that is still due), normed if a norm is given (its `stream_args()`);
        `rows`: of these tokens only — the streams are then left without the due write (it is applied on the way to
        the result only), so nothing may read them afterwards."""
        due, self._pending = self._pending, {}
        return kernels.streams_step(self.xs, read=coefs, out_dtype=out_dtype, rows=rows, **due, **(norm or {}))

    def read_sum(self, norm: Optional[dict], out_dtype, rows=None) -> torch.Tensor:
        if self._ones is None:
            self._ones = torch.ones(self.n_streams, dtype=torch.float32, device=self.xs.device)
        return self.read(self._ones, norm, out_dtype, rows)

    def flush(self) -> None:
        if self._pending:
            due, self._pending = self._pending, {}
            kernels.streams_step(self.xs, **due)

    def total(self) -> torch.Tensor:
        """The sum of the streams, float32 [T, W] (for whoever wants to look at the residual stream)."""
        return self.read_sum(None, torch.float32)


class StreamConnection(Part):
    """The three tensors of one sublayer's connection to the streams."""
    padded_rows_ok = True

    def __init__(self, spec):
        super().__init__(spec)
        self.n_streams = int(self.params["streams"])
        if not 1 <= self.n_streams <= kernels.streams.MAX_STREAMS:
            raise ConfigError(f"a residual of {self.n_streams} streams (1 to {kernels.streams.MAX_STREAMS})")
        self.mult = float(self.params.get("residual_mult", 1.0))
        self.names = dict(self.params.get("names", {"read": "in", "write": "out", "mix": "mix"}))
        self.read = self.write = self.mix = None

    def weight_specs(self):
        S = self.n_streams
        return [WeightSpec(self.prefix + self.names["read"], (S,), "stream_read"),
                WeightSpec(self.prefix + self.names["write"], (S,), "stream_write"),
                WeightSpec(self.prefix + self.names["mix"], (S, S), "stream_mix")]

    def bind(self, tensors, runtime: Runtime, shared=None):
        self.read = float32_vector(tensors[self.prefix + self.names["read"]])
        self.write = float32_vector(tensors[self.prefix + self.names["write"]])
        if self.mult != 1.0:
            self.write = self.write * self.mult
        self.mix = tensors[self.prefix + self.names["mix"]].to(torch.float32).contiguous()


class SublayerResult(Part):
    """What becomes of a sublayer's result before it enters the residual: times a vector (tensor `names["scale"]`, [W])
    and / or times sigmoid(R h + b) (`names["gate"]` [W, W], `names["gate_bias"]` [W]), h being what the sublayer
    read.  The gate's rows ride in the sublayer's first product where that part takes riders; else the product runs
    here."""
    padded_rows_ok = True

    def __init__(self, spec):
        super().__init__(spec)
        self.width = int(self.params["width"])
        self.names = dict(self.params["names"])
        self.scale = self.w_gate = self.gate_bias = None

    def _n(self, which):
        return self.prefix + self.names[which]

    def weight_specs(self):
        W, specs = self.width, []
        if "scale" in self.names:
            specs.append(WeightSpec(self._n("scale"), (W,), "norm_scale"))
        if "gate" in self.names:
            specs += [WeightSpec(self._n("gate"), (W, W), "matrix"), WeightSpec(self._n("gate_bias"), (W,), "bias")]
        return specs

    def bind(self, tensors, runtime: Runtime, shared=None):
        if "scale" in self.names:
            self.scale = float32_vector(tensors[self._n("scale")])
        if "gate" in self.names:
            self.w_gate = tensors[self._n("gate")].contiguous()
            self.gate_bias = float32_vector(tensors[self._n("gate_bias")])

    @property
    def has_rows(self) -> bool:
        return "gate" in self.names

    def rider_rows(self):
        """The gate's rows and their bias for the sublayer's own product, which keeps them from here on."""
        w, self.w_gate = self.w_gate, None
        return w, self.gate_bias

    def gate_logits(self, x) -> Optional[torch.Tensor]:
        if self.w_gate is None:
            return None
        return kernels.linear(x, self.w_gate, bias=self.gate_bias, out_dtype=torch.float32)


class StreamsBlock:
    """Pre-norm layer on parallel residual streams (kind `residual_streams`): the mixer's sublayer, then — unless
    the layer has none — the feed-forward's, each with a connection of its own (parts `mixer_streams`,
    `feed_forward_streams`) and, if the layer names them, what becomes of its result (`mixer_result`,
    `feed_forward_result`).  The norms must be ones that the streams' kernel applies (`stream_args`)."""
    padded_rows_ok = True               # as far as its parts are

    def __init__(self, spec: LayerSpec):
        self.spec = spec
        self.mixer_norm = make_part(spec.part("mixer_norm"))
        self.mixer = make_part(spec.part("mixer"))
        self.mixer_streams = make_part(spec.part("mixer_streams"))
        self.feed_forward = self.feed_forward_norm = self.feed_forward_streams = None
        if spec.feed_forward is not None:
            self.feed_forward_norm = make_part(spec.part("feed_forward_norm"))
            self.feed_forward = make_part(spec.part("feed_forward"))
            self.feed_forward_streams = make_part(spec.part("feed_forward_streams"))
        for n in (self.mixer_norm, self.feed_forward_norm):
            if n is not None and getattr(n, "stream_args", None) is None:
                raise ConfigError("a layer on residual streams takes norms that the streams' kernel applies")
        named = spec.parts()
        self.mixer_result = make_part(named["mixer_result"]) if "mixer_result" in named else None
        self.feed_forward_result = make_part(named["feed_forward_result"]) if "feed_forward_result" in named else None
        for part, result in ((self.mixer, self.mixer_result), (self.feed_forward, self.feed_forward_result)):
            if part is not None and result is not None and result.has_rows and part.accepts_rider:
                part.rider = result

    def parts(self):
        # (a result part comes before the part that may carry its rows: it is bound first)
        return [p for p in (self.mixer_norm, self.mixer_result, self.mixer, self.mixer_streams, self.feed_forward_norm,
                            self.feed_forward_result, self.feed_forward, self.feed_forward_streams) if p is not None]

    def forward(self, h: ResidualStreams, ctx: StepContext) -> None:
        if not isinstance(h, ResidualStreams):
            raise kernels.KernelError("a layer of kind 'residual_streams' runs in a model that keeps streams")
        self._sublayer(h, ctx, self.mixer_norm, self.mixer, self.mixer_streams, self.mixer_result)
        if self.feed_forward is not None:
            self._sublayer(h, ctx, self.feed_forward_norm, self.feed_forward, self.feed_forward_streams,
                           self.feed_forward_result)

    @staticmethod
    def _sublayer(h: ResidualStreams, ctx: StepContext, norm, part, conn, result) -> None:
        x = h.read(conn.read, norm.stream_args(), ctx.runtime.act_dtype)
        kernels.mark("norms")
        store = bool(getattr(part, "can_store_result", False))
        y = (torch.empty if store else torch.zeros)(h.xs.shape[1:], dtype=torch.float32, device=h.xs.device)
        ctx.store_result = store
        try:
            part.forward(x, ctx, y)
        finally:
            ctx.store_result = False
        if result is None:
            h.write_later(y, conn.mix, conn.write)
            return
        gate, ctx.rider_out = ctx.rider_out, None
        if gate is None:
            if part.rider is not None:
                raise kernels.KernelError("a part that carries the residual gate's rows left no result of them")
            gate = result.gate_logits(x)
            kernels.mark("residual_gate")
        h.write_later(y, conn.mix, conn.write, result.scale, gate)
