"""A mixer with a matrix of memory per head, updated by the delta rule with a decay per head and key channel:

    q, k = unit(silu(conv(W_q h))), unit(silu(conv(W_k h)))     key_heads x key_dim; q also times query_scale
    v = silu(conv(W_v h))                                       heads x value_dim
    beta = sigmoid(W_b h)                                       per head
    g = exp(-exp(A_log) * softplus(W_a2 (W_a1 h) + dt_bias))    heads x key_dim
    S' = diag(g) S_{t-1};   u = beta (v - S'^T k);   S_t = S' + k u^T;   o_t = S_t^T q      (the read sees the write)
    out = W_o (rms_norm_per_head(o) * w * sigmoid(W_g2 (W_g1 h)))       w has value_dim entries, shared by the heads

conv is a short causal convolution over time per channel (no bias); unit(x) = x / sqrt(sum(x^2) + unit_eps) per head;
head h reads the q and k of key head h // (heads / key_heads).  S starts at zero, is float32 and lives, with the
convolutions' last taps - 1 inputs, in the cache's per-sequence state (csrc/short_conv.cu, csrc/low_rank.cu,
csrc/channel_scan.cu; one token at a time csrc/linear_scan.cu).  Everything that reads h is one product with a float32 result, which may carry a rider's rows.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache import StateRequest
from ..config import ConfigError
from ..kernels.scan import MAX_CONV_TAPS, MAX_KEY_WIDTH
from .base import Mixer, Runtime, StepContext, WeightSpec, float32_vector, stack_rows
from .state_space import CONV_VECTOR


class ChannelDeltaMixer(Mixer):
    graph_capturable = True             # slots and lengths are read on the device
    can_store_result = True
    accepts_rider = True

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.key_heads = int(p["heads"]), int(p["key_heads"])
        self.key_dim, self.value_dim, self.taps = int(p["key_dim"]), int(p["value_dim"]), int(p["taps"])
        self.decay_rank, self.gate_rank = p.get("decay_rank"), p.get("gate_rank")        # None: the checkpoint says
        self.eps, self.unit_eps = float(p["eps"]), float(p.get("unit_eps", 1e-6))
        self.query_scale = float(p.get("query_scale", 1.0))
        self.names = dict(p["names"])
        if self.heads % self.key_heads:
            raise ConfigError(f"{self.heads} heads cannot share {self.key_heads} key heads")
        if self.key_dim > MAX_KEY_WIDTH or not 1 <= self.taps <= MAX_CONV_TAPS:
            raise kernels.KernelError(f"channel delta rule: key width {self.key_dim} or {self.taps} taps exceed the kernels' limits")
        self.qk, self.vw = self.key_heads * self.key_dim, self.heads * self.value_dim
        self.conv_channels = 2 * self.qk + self.vw
        self.state_floats = self.heads * self.key_dim * self.value_dim
        self.w_in = self.bias = self.conv_w = self.w_decay = self.w_gate = self.dt_bias = self.a_log = None
        self.norm_w = self.w_o = None

    def _n(self, which: str) -> str:
        return self.prefix + self.names[which]

    def weight_specs(self):
        h, H = self.hidden, self.heads
        ra, rg = (-1 if r is None else int(r) for r in (self.decay_rank, self.gate_rank))
        return [WeightSpec(self._n("q"), (self.qk, h), "matrix"), WeightSpec(self._n("k"), (self.qk, h), "matrix"),
                WeightSpec(self._n("v"), (self.vw, h), "matrix"),
                WeightSpec(self._n("q_conv"), (self.qk, self.taps), "conv"),
                WeightSpec(self._n("k_conv"), (self.qk, self.taps), "conv"),
                WeightSpec(self._n("v_conv"), (self.vw, self.taps), "conv"),
                WeightSpec(self._n("beta"), (H, h), "matrix"), WeightSpec(self._n("a_log"), (H,), "bias"),
                WeightSpec(self._n("decay_in"), (ra, h), "matrix"),
                WeightSpec(self._n("decay_out"), (H * self.key_dim, ra), "matrix"),
                WeightSpec(self._n("dt_bias"), (H * self.key_dim,), "bias"),
                WeightSpec(self._n("gate_in"), (rg, h), "matrix"), WeightSpec(self._n("gate_out"), (self.vw, rg), "matrix"),
                WeightSpec(self._n("norm"), (self.value_dim,), "norm_scale"),
                WeightSpec(self._n("out"), (h, self.vw), "matrix")]

    def bind(self, tensors, runtime: Runtime, shared=None):
        # one product for everything that reads h: q | k | v | (rider) | decay's inner | gate's inner | write logits
        parts = [(tensors[self._n(x)], None) for x in ("q", "k", "v")]
        if self.rider is not None:
            parts.append(self.rider.rider_rows())
        a1, g1 = tensors[self._n("decay_in")], tensors[self._n("gate_in")]
        parts += [(a1, None), (g1, None), (tensors[self._n("beta")], None)]
        self.w_in, self.bias = stack_rows([w for w, _ in parts], [b for _, b in parts])
        self.off_rider = self.conv_channels
        self.rider_width = parts[3][0].shape[0] if self.rider is not None else 0
        self.decay_rank, self.gate_rank = int(a1.shape[0]), int(g1.shape[0])
        self.off_a = self.off_rider + self.rider_width
        self.off_g = self.off_a + self.decay_rank
        self.off_b = self.off_g + self.gate_rank
        w_a, w_g = tensors[self._n("decay_out")], tensors[self._n("gate_out")]
        for w, n, r in ((w_a, "decay_out", self.decay_rank), (w_g, "gate_out", self.gate_rank)):
            if w.shape[1] != r:
                raise kernels.KernelError(f"channel delta rule: {self._n(n)} has shape {tuple(w.shape)}, its inner width is {r}")
        if w_a.dtype != w_g.dtype:
            w_a, w_g = w_a.to(torch.float32), w_g.to(torch.float32)
        self.w_decay, self.w_gate = w_a.contiguous(), w_g.contiguous()
        self.conv_w = torch.cat([float32_vector(tensors[self._n(x)]) for x in ("q_conv", "k_conv", "v_conv")],
                                dim=0).contiguous()
        self.dt_bias = float32_vector(tensors[self._n("dt_bias")])
        self.a_log = float32_vector(tensors[self._n("a_log")])
        self.norm_w = float32_vector(tensors[self._n("norm")]).repeat(self.heads).contiguous()
        self.w_o = tensors[self._n("out")].contiguous()

    def state_request(self):
        return StateRequest((self.state_floats + (self.taps - 1) * self.conv_channels,), torch.float32)

    def forward(self, x, ctx: StepContext, residual):
        b, dev = ctx.batch, residual.device
        qk, vw, C, H = self.qk, self.vw, self.conv_channels, self.heads
        proj = kernels.linear(x, self.w_in, bias=self.bias, out_dtype=torch.float32)
        kernels.mark("qkv")
        if self.rider is not None:
            ctx.rider_out = proj[:, self.off_rider:self.off_a]
        T = proj.shape[0]
        single = b.single_tokens
        cv = torch.empty((T, C), dtype=torch.float32, device=dev)
        scal = torch.empty((T, H, 4), dtype=torch.float32, device=dev)
        kernels.short_conv(proj[:, :C], self.conv_w, None, cv, ctx.state[:, self.state_floats:],
                           tok_seq=b.tok_seq, cu_seqlens=b.cu_seqlens, slots=b.slots, n_seqs=b.n_seqs,
                           regions=[(0, qk, self.key_dim, True, self.query_scale), (qk, qk, self.key_dim, True, 1.0),
                                    (2 * qk, vw, min(vw, CONV_VECTOR), False, 1.0)],
                           silu=True, single_tokens=single, unit_eps=self.unit_eps,
                           beta_raw=proj[:, self.off_b:self.off_b + H], scalars=scal)
        kernels.mark("conv")
        decay, gate, done = kernels.low_rank_gates(proj[:, self.off_a:self.off_g], self.w_decay, self.dt_bias, self.a_log,
                                                   proj[:, self.off_g:self.off_b], self.w_gate,
                                                   leave_logits=not single)
        kernels.mark("decay")
        o = torch.empty((T, vw), dtype=torch.float32, device=dev)
        kernels.channel_delta_scan(cv[:, :qk], cv[:, qk:2 * qk], cv[:, 2 * qk:], decay, scal,
                                   ctx.state[:, :self.state_floats], b.cu_seqlens, b.slots, o, n_seqs=b.n_seqs, heads=H,
                                   qk_heads=self.key_heads, key_dim=self.key_dim, value_dim=self.value_dim,
                                   single_tokens=single, dt_bias=None if done else self.dt_bias,
                                   a_log=None if done else self.a_log)
        kernels.mark("scan")
        y = torch.empty((T, vw), dtype=ctx.runtime.act_dtype, device=dev)
        kernels.group_rmsnorm(o, self.norm_w, self.eps, y, groups=H, gate=gate)
        kernels.mark("head_norm")
        kernels.linear(y, self.w_o, out=residual, accumulate=not ctx.store_result)
        kernels.mark("o")
