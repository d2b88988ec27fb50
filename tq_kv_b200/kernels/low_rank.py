"""Python entry points of the two-step projections: decays per key channel and a result's gate (csrc/low_rank.cu)."""
from __future__ import annotations

from typing import Optional

import torch

from ._lib import KernelError, check, core, dtype_code, need_contiguous, ptr, stream
from .gemm import linear

# From this inner width and this many tokens on, bfloat16 products run on the tensor cores (whole K tiles of 64).
TC_MIN_RANK = 64
TC_MIN_TOKENS = 65


def round_columns(x: torch.Tensor) -> torch.Tensor:
    """bfloat16 copy [T, n] of float32 rows that may be a column slice."""
    T, n = x.shape
    if x.dtype != torch.float32 or x.stride(1) != 1:
        raise KernelError("round_columns: float32 rows")
    out = torch.empty((T, n), dtype=torch.bfloat16, device=x.device)
    check(core().tq_round_columns(ptr(x), x.stride(0), ptr(out), n, T, stream()), "round_columns")
    return out


def low_rank_gates(low_decay: torch.Tensor, w_decay: torch.Tensor, dt_bias: torch.Tensor, a_log: torch.Tensor,
                   low_gate: torch.Tensor, w_gate: torch.Tensor, *, use_tc: Optional[bool] = None, leave_logits: bool = False):
    """The second halves of two two-step projections whose first halves are columns of one float32 buffer:
    decay[t, i] = exp(-exp(a_log[i // d]) * softplus(w_decay[i] . low_decay[t] + dt_bias[i])), d = len(dt_bias) //
    len(a_log), and gate[t, i] = w_gate[i] . low_gate[t]; both float32 [T, n].  The weights share one dtype.  Returns
    (decay, gate, done): with `leave_logits` the decays may be left as w_decay . low_decay, for a reader that makes them
    itself; `done` then is False."""
    T = low_decay.shape[0]
    na, ra = w_decay.shape
    np_, rp = w_gate.shape
    H = a_log.shape[0]
    for name, low, r in (("low_decay", low_decay, ra), ("low_gate", low_gate, rp)):
        if low.dtype != torch.float32 or tuple(low.shape) != (T, r) or low.stride(1) != 1 or low.stride(0) != low_decay.stride(0):
            raise KernelError(f"low_rank_gates: {name} must be float32 [T, {r}], a column slice of one buffer")
    if w_decay.dtype != w_gate.dtype or dt_bias.dtype != torch.float32 or tuple(dt_bias.shape) != (na,) \
            or a_log.dtype != torch.float32 or H < 1 or na % H:
        raise KernelError("low_rank_gates: weights of one dtype, dt_bias float32 [n], a_log float32 [heads]")
    need_contiguous(w_decay=w_decay, w_gate=w_gate, dt_bias=dt_bias, a_log=a_log)
    d = na // H
    if use_tc is None:
        use_tc = (w_decay.dtype == torch.bfloat16 and T >= TC_MIN_TOKENS and min(ra, rp) >= TC_MIN_RANK
                  and ra % 8 == 0 and rp % 8 == 0)
    if use_tc:
        decay = linear(round_columns(low_decay), w_decay, out_dtype=torch.float32)
        gate = linear(round_columns(low_gate), w_gate, out_dtype=torch.float32)
        if not leave_logits:
            check(core().tq_channel_decay(ptr(decay), ptr(dt_bias), ptr(a_log), d, na, T, stream()), "channel_decay")
        return decay, gate, not leave_logits
    decay = torch.empty((T, na), dtype=torch.float32, device=low_decay.device)
    gate = torch.empty((T, np_), dtype=torch.float32, device=low_decay.device)
    check(core().tq_low_rank_rows(ptr(low_decay), ra, ptr(w_decay), na, ptr(dt_bias), ptr(a_log), d, ptr(decay),
                                  ptr(low_gate), rp, ptr(w_gate), np_, ptr(gate), low_decay.stride(0), dtype_code(w_decay),
                                  T, stream()), "low_rank_rows")
    return decay, gate, True
