"""Python entry point of the per-channel gated recurrence (csrc/gru_scan.cu)."""
from __future__ import annotations

import torch

from ._lib import KernelError, check, core, dtype_code, need_contiguous, ptr, stream


def gru_scan(z: torch.Tensor, u: torch.Tensor, gate: torch.Tensor, state: torch.Tensor, cu_seqlens: torch.Tensor,
             slots: torch.Tensor, out: torch.Tensor, *, n_seqs: int, scale: float = 1.0, single_tokens: bool = False):
    """Per channel S_t = (1 - s(z_t)) S_{t-1} + s(z_t) c(u_t), s the sigmoid, c(u) = u + 1/2 for u >= 0 and s(u) below;
    out_t = scale * S_t * gate_t * s(gate_t).  z, u, gate: float32 [T, W] column slices of one buffer; out [T, W]
    float32 or bfloat16; state float32 [slots, W] (may be a column slice of the per-sequence state) is read before each
    sequence's first token of the step and written after its last."""
    T, W = z.shape
    for t in (z, u, gate):
        if t.dtype != torch.float32 or tuple(t.shape) != (T, W) or t.stride(1) != 1 or t.stride(0) != z.stride(0):
            raise KernelError("gru_scan: z, u and gate must be float32 [T, W], column slices of one buffer")
    if tuple(out.shape) != (T, W):
        raise KernelError("gru_scan: out must be [T, W]")
    if state.dtype != torch.float32 or state.dim() != 2 or state.shape[1] != W or state.stride(1) != 1:
        raise KernelError("gru_scan: state must be float32 [slots, W]")
    if single_tokens and T != n_seqs:
        raise KernelError("gru_scan: single_tokens needs one token per sequence")
    need_contiguous(out=out, cu_seqlens=cu_seqlens, slots=slots)
    check(core().tq_gru_scan(ptr(z), ptr(u), ptr(gate), z.stride(0), ptr(state), state.stride(0), ptr(cu_seqlens),
                             ptr(slots), int(n_seqs), T, int(single_tokens), W, float(scale), ptr(out), dtype_code(out),
                             stream()), "gru_scan")
    return out
