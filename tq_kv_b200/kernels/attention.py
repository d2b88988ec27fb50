"""Python entry point of the attention kernel (csrc/attention.cu)."""
from __future__ import annotations

import math
from typing import Optional

import torch

from ._lib import KernelError, check, core, dtype_code, need_contiguous, ptr, stream, tc_status_word

MAX_HEAD_DIM = 512    # of the general kernel; the Qwen2 configuration keeps its own limit of 256
NOT_SUPPORTED = 801     # cudaErrorNotSupported: a specialised kernel declines the shape
TENSOR_CORE_WIDTHS = (32, 64, 96, 128)      # head widths (keys and values alike) of the bfloat16 tensor-core kernels
USE_TC_ATTENTION = True  # prompts: the tcgen05 kernel (csrc/flash_prefill_tc.cu) before the mma.sync one


def check_head_geometry(n_heads: int, n_kv_heads: int, head_dim: int) -> None:
    """Raises for head sizes the attention kernels do not take."""
    if head_dim % 16 or not 16 <= head_dim <= MAX_HEAD_DIM:
        raise KernelError(f"attention: head_dim {head_dim} must be a multiple of 16 between 16 and {MAX_HEAD_DIM}")
    if n_kv_heads <= 0 or n_heads % n_kv_heads:
        raise KernelError(f"attention: {n_heads} heads cannot be shared among {n_kv_heads} key/value heads")
    if n_kv_heads > 65535:
        raise KernelError(f"attention: more than 65535 key/value heads ({n_kv_heads})")


def head_groups(n_heads: int, n_kv_heads: int) -> int:
    """Blocks per token of the decode kernel: it serves up to 16 query heads of a key/value head at once."""
    return n_kv_heads * -(-(n_heads // n_kv_heads) // 16)


def plan_splits(n_tokens: int, n_kv_heads: int, max_keys: int, sm_count: int) -> int:
    """Number of splits of the key range for a step: one while the grid fills
    the GPU or the key ranges are short, else as many as fill the GPU in one
    wave, with at least 128 keys per split of the longest range.  (Each
    token cuts its own range into that many equal parts.)"""
    blocks = n_tokens * n_kv_heads
    resident = 2 * sm_count                    # blocks of the decode kernel that run at once
    if blocks >= resident or max_keys <= 256:
        return 1
    # fill the GPU once: a grid a little over a whole number of waves wastes most of its last wave
    return max(1, min(resident // blocks, -(-max_keys // 128), 64))


def split_scratch_floats(n_tokens: int, n_heads: int, head_dim: int, n_splits: int) -> int:
    return n_tokens * n_heads * n_splits * (head_dim + 2) if n_splits > 1 else 0


def attention(q: torch.Tensor, out: torch.Tensor, *, n_heads: int, n_kv_heads: int, head_dim: int,
              tok_pos: torch.Tensor, tok_seq: torch.Tensor, cu_seqlens: torch.Tensor, start_pos: torch.Tensor,
              window: Optional[int], scale: Optional[float] = None,
              k_packed: Optional[torch.Tensor] = None, v_packed: Optional[torch.Tensor] = None,
              k_pages: Optional[torch.Tensor] = None, v_pages: Optional[torch.Tensor] = None,
              block_table: Optional[torch.Tensor] = None, table_width: int = 0, ring_pages: int = 0,
              page_tokens: int = 64, n_splits: int = 1,
              scratch: Optional[torch.Tensor] = None, use_flash: bool = True):
    """out[t, h] = softmax(q[t, h] · K / sqrt(head_dim)) · V over the keys
    max(0, pos-window+1) .. pos of the token's sequence.  q/out [T, nh*hd].
    Keys and values come from the step's packed rows (k_packed/v_packed
    [T, nkv*hd]; every sequence must then start at position 0 or carry its
    whole history in the step) or from the paged cache."""
    check_head_geometry(n_heads, n_kv_heads, head_dim)
    T = q.shape[0]
    if q.shape[1] != n_heads * head_dim or out.shape != q.shape or out.dtype != q.dtype:
        raise KernelError("attention: q and out must be [T, n_heads*head_dim] of one dtype")
    packed = k_packed is not None
    if packed:
        if v_packed is None or k_packed.dtype != q.dtype or k_packed.shape != (T, n_kv_heads * head_dim):
            raise KernelError("attention: packed keys/values must be [T, n_kv_heads*head_dim] of q's dtype")
    else:
        if k_pages is None or v_pages is None or block_table is None or k_pages.dtype != q.dtype:
            raise KernelError("attention: no key/value source of q's dtype was given")
        if tuple(k_pages.shape[1:]) != (n_kv_heads, page_tokens, head_dim):
            raise KernelError(f"attention: cache pages have shape {tuple(k_pages.shape)}")
    part_acc = part_ml = None
    if n_splits > 1:
        need = split_scratch_floats(T, n_heads, head_dim, n_splits)
        if scratch is None or scratch.dtype != torch.float32 or scratch.numel() < need:
            raise KernelError(f"attention: {n_splits} splits need {need} float32 of scratch")
        n_acc = T * n_heads * n_splits * head_dim
        part_acc, part_ml = scratch[:n_acc], scratch[n_acc:need]
    need_contiguous(q=q, out=out, k_packed=k_packed, v_packed=v_packed, k_pages=k_pages, v_pages=v_pages,
                    block_table=block_table)
    if scale is None:
        scale = 1.0 / math.sqrt(head_dim)
    n_seqs = cu_seqlens.shape[0] - 1
    if q.dtype == torch.bfloat16 and use_flash and USE_TC_ATTENTION and T > n_seqs:
        # prompts on the tcgen05 tensor cores (128-query tiles, S and P·V in tensor memory)
        st = core().tq_flash_prefill_tc(
            ptr(q), ptr(k_packed), ptr(v_packed), ptr(k_pages), ptr(v_pages),
            0 if k_pages is None else k_pages.shape[0], ptr(block_table), table_width, ring_pages, page_tokens,
            ptr(cu_seqlens), ptr(start_pos), n_seqs, T, int(window or 0), float(scale), ptr(out), n_heads,
            n_kv_heads, head_dim, ptr(tc_status_word(q.device)), stream())
        if st != NOT_SUPPORTED:
            check(st, "flash_prefill_tc")
            return out
    if q.dtype == torch.bfloat16 and use_flash and T > n_seqs:
        # prompts (some sequence brings several tokens): the tensor-core kernel with 64-query tiles
        st = core().tq_flash_prefill(
            ptr(q), ptr(k_packed), ptr(v_packed), ptr(k_pages), ptr(v_pages), ptr(block_table), table_width,
            ring_pages, page_tokens, ptr(cu_seqlens), ptr(start_pos), n_seqs, T, int(window or 0), float(scale),
            ptr(out), n_heads, n_kv_heads, head_dim, stream())
        if st != NOT_SUPPORTED:
            check(st, "flash_prefill")
            return out
    if not packed and q.dtype == torch.bfloat16 and use_flash:
        # the bandwidth-built kernel for the cache; it declines shapes outside its reach
        st = core().tq_flash_decode(
            ptr(q), ptr(k_pages), ptr(v_pages), ptr(block_table), table_width, ring_pages, page_tokens,
            ptr(tok_pos), ptr(tok_seq), int(window or 0), float(scale), ptr(out), ptr(part_acc), ptr(part_ml), T,
            n_heads, n_kv_heads, head_dim, n_splits, stream())
        if st != NOT_SUPPORTED:
            check(st, "flash_decode")
            if n_splits > 1:
                check(core().tq_attention_merge(ptr(part_acc), ptr(part_ml), ptr(out), dtype_code(out), T, n_heads,
                                                head_dim, n_splits, 0, stream()), "attention_merge")
            return out
    check(core().tq_attention(
        ptr(q), dtype_code(q), ptr(k_packed), ptr(v_packed), ptr(k_pages), ptr(v_pages), ptr(block_table),
        table_width, ring_pages, page_tokens, ptr(tok_pos), ptr(tok_seq), ptr(cu_seqlens), ptr(start_pos),
        int(window or 0), float(scale), ptr(out), ptr(part_acc), ptr(part_ml), T, n_heads, n_kv_heads, head_dim,
        n_splits, stream()), "attention", 2 if n_splits > 1 else 1)
    return out


def check_row_widths(n_heads: int, n_kv_heads: int, key_dim: int, value_dim: int) -> None:
    """Raises for head sizes the general attention kernel with options does not take."""
    for name, d in (("key", key_dim), ("value", value_dim)):
        if d % 8 or not 8 <= d <= MAX_HEAD_DIM:
            raise KernelError(f"attention: the {name} rows' width {d} must be a multiple of 8 between 8 and {MAX_HEAD_DIM}")
    if n_kv_heads <= 0 or n_heads % n_kv_heads or n_kv_heads > 65535:
        raise KernelError(f"attention: {n_heads} heads cannot be shared among {n_kv_heads} key/value heads")


def attention_ext(q: torch.Tensor, out: torch.Tensor, *, n_heads: int, n_kv_heads: int, key_dim: int,
                  value_dim: int, tok_pos: torch.Tensor, tok_seq: torch.Tensor, cu_seqlens: torch.Tensor,
                  start_pos: torch.Tensor, scale: float, window: Optional[int] = None, keep_first: int = 0,
                  softcap: Optional[float] = None, slopes: Optional[torch.Tensor] = None,
                  k_packed: Optional[torch.Tensor] = None, v_packed: Optional[torch.Tensor] = None,
                  k_pages: Optional[torch.Tensor] = None, v_pages: Optional[torch.Tensor] = None,
                  block_table: Optional[torch.Tensor] = None, table_width: int = 0, ring_pages: int = 0,
                  page_tokens: int = 64, n_splits: int = 1, scratch: Optional[torch.Tensor] = None,
                  gate: Optional[torch.Tensor] = None, use_fast: bool = True, sink=False,
                  chunk: Optional[int] = None, unmerged: bool = False):
    """Softmax attention with options: for the query at position i of head h and the key at position j <= i,

        s = q . k * scale;   s <- softcap * tanh(s / softcap)  (if a cap is given);
        s <- s - slopes[h] * (i - j)                            (if slopes are given);

    j is visible if i - j < window or j < keep_first (no window: every j <= i); with `chunk` (and no window) if
    i // chunk == j // chunk.  `sink`: a float32 tensor [n_heads] — the softmax's denominator counts one more key of
    score sink[h] that has no value, p_j = exp(s_j) / (exp(sink[h]) + sum exp(s)) — or True (a score of 0) or False.
    Value rows may have another width than the keys.  q [T, nh*key_dim], out [T, nh*value_dim]; keys and values as in `attention`.
    `gate` (float32 [T, nh*value_dim], or [T, nh] with one number per head, possibly a column slice of wider rows): out
    *= sigmoid(gate), in the
    attention kernel's last step where it can, else by a kernel of its own.
    `unmerged` (then `out` is None; no gate, no sink): the float32 results are returned for a kernel that goes on with
    them, (rows [T, nh, value_dim], None, 1) or, per split of the keys, (sums [T, nh, n, value_dim], their maxima and
    sums of weights [T, nh, n, 2], n), as `difference_of_maps` takes them.

    bfloat16 with keys and values of one width runs on the tensor cores: prompts on the tcgen05 kernel (heads of
    64 and 128) or the mma.sync one (32, 64, 96, 128), single tokens on the bandwidth-built cache kernel; all
    else, and float32, on the general kernel."""
    check_row_widths(n_heads, n_kv_heads, key_dim, value_dim)
    T = q.shape[0]
    if unmerged and (out is not None or gate is not None or sink is not False):
        raise KernelError("attention: unmerged results take no out, gate or sink")
    if q.shape[1] != n_heads * key_dim or (not unmerged and (tuple(out.shape) != (T, n_heads * value_dim)
                                                             or out.dtype != q.dtype)):
        raise KernelError("attention: q must be [T, n_heads*key_dim] and out [T, n_heads*value_dim] of one dtype")
    packed = k_packed is not None
    if packed:
        if (v_packed is None or k_packed.dtype != q.dtype or tuple(k_packed.shape) != (T, n_kv_heads * key_dim)
                or tuple(v_packed.shape) != (T, n_kv_heads * value_dim)):
            raise KernelError("attention: packed keys [T, n_kv_heads*key_dim] and values [T, n_kv_heads*value_dim] of q's dtype")
    else:
        if k_pages is None or v_pages is None or block_table is None or k_pages.dtype != q.dtype:
            raise KernelError("attention: no key/value source of q's dtype was given")
        if (tuple(k_pages.shape[1:]) != (n_kv_heads, page_tokens, key_dim)
                or tuple(v_pages.shape[1:]) != (n_kv_heads, page_tokens, value_dim)):
            raise KernelError(f"attention: cache pages have shapes {tuple(k_pages.shape)} / {tuple(v_pages.shape)}")
    if slopes is not None and (slopes.dtype != torch.float32 or tuple(slopes.shape) != (n_heads,)):
        raise KernelError("attention: slopes must be float32 [n_heads]")
    if keep_first and ring_pages:
        raise KernelError("attention: kept first tokens need a cache that keeps all keys")
    if chunk and window:
        raise KernelError("attention: a window or chunks, not both")
    if sink is True:
        sink = torch.zeros(n_heads, dtype=torch.float32, device=q.device)
    elif sink is False:
        sink = None
    if sink is not None and (sink.dtype != torch.float32 or tuple(sink.shape) != (n_heads,)):
        raise KernelError("attention: sink must be float32 [n_heads]")
    part_acc = part_ml = None
    if n_splits > 1 or unmerged:
        need = T * n_heads * n_splits * (value_dim + 2)
        if unmerged and scratch is None:
            scratch = torch.empty(need, dtype=torch.float32, device=q.device)
        if scratch is None or scratch.dtype != torch.float32 or scratch.numel() < need:
            raise KernelError(f"attention: {n_splits} splits need {need} float32 of scratch")
        n_acc = T * n_heads * n_splits * value_dim
        part_acc, part_ml = scratch[:n_acc], scratch[n_acc:need]
    need_contiguous(q=q, out=out, k_packed=k_packed, v_packed=v_packed, k_pages=k_pages, v_pages=v_pages,
                    block_table=block_table, slopes=slopes, sink=sink)
    if gate is not None and (gate.dtype != torch.float32 or tuple(gate.shape) not in (tuple(out.shape), (T, n_heads))
                             or (gate.stride(1) != 1 and gate.shape[1] > 1)):
        raise KernelError("attention: the gate must be float32 of the result's shape, or one number per head")
    head_gate = int(gate is not None and tuple(gate.shape) != tuple(out.shape))
    keep = int(keep_first) if window else 0
    n_seqs = cu_seqlens.shape[0] - 1
    fast = use_fast and q.dtype == torch.bfloat16 and key_dim == value_dim
    if fast and T > n_seqs:                                  # prompts (some sequence brings several tokens)
        gate_ok = gate is not None and (head_gate or (gate.stride(0) % 4 == 0 and gate.data_ptr() % 16 == 0))
        g_ptr, g_ld = (ptr(gate), gate.stride(0)) if gate_ok else (None, 0)
        st = NOT_SUPPORTED
        if USE_TC_ATTENTION:
            st = core().tq_flash_prefill_tc_ext(
                ptr(q), ptr(k_packed), ptr(v_packed), ptr(k_pages), ptr(v_pages),
                0 if k_pages is None else k_pages.shape[0], ptr(block_table), table_width, ring_pages, page_tokens,
                ptr(cu_seqlens), ptr(start_pos), n_seqs, T, int(window or 0), float(scale), float(softcap or 0.0),
                ptr(slopes), keep, ptr(sink), int(chunk or 0), g_ptr, g_ld, head_gate, ptr(part_acc if unmerged else out),
                int(unmerged), n_heads, n_kv_heads, key_dim, ptr(tc_status_word(q.device)), stream())
            if st != NOT_SUPPORTED:
                check(st, "flash_prefill_tc_ext")
        if st == NOT_SUPPORTED:
            st = core().tq_flash_prefill_ext(
                ptr(q), ptr(k_packed), ptr(v_packed), ptr(k_pages), ptr(v_pages), ptr(block_table), table_width,
                ring_pages, page_tokens, ptr(cu_seqlens), ptr(start_pos), n_seqs, T, int(window or 0), float(scale),
                float(softcap or 0.0), ptr(slopes), keep, ptr(sink), int(chunk or 0), g_ptr, g_ld, head_gate,
                ptr(part_acc if unmerged else out), int(unmerged), n_heads, n_kv_heads, key_dim, stream())
            if st != NOT_SUPPORTED:
                check(st, "flash_prefill_ext")
        if st != NOT_SUPPORTED:
            if unmerged:
                return part_acc, None, 1
            if gate is not None and not gate_ok:
                from .elementwise import sigmoid_gate
                sigmoid_gate(out, gate)
            return out
    if fast and not packed:
        st = core().tq_flash_decode_ext(
            ptr(q), ptr(k_pages), ptr(v_pages), ptr(block_table), table_width, ring_pages, page_tokens, ptr(tok_pos),
            ptr(tok_seq), int(window or 0), float(scale), float(softcap or 0.0), ptr(slopes), keep, ptr(sink),
            int(chunk or 0),
            ptr(out), ptr(part_acc), ptr(part_ml), T, n_heads, n_kv_heads, key_dim, n_splits, stream())
        if st != NOT_SUPPORTED:
            check(st, "flash_decode_ext")
            if unmerged:
                return part_acc, part_ml, n_splits
            if n_splits > 1:
                check(core().tq_attention_merge(ptr(part_acc), ptr(part_ml), ptr(out), dtype_code(out), T, n_heads,
                                                value_dim, n_splits, ptr(sink), stream()), "attention_merge")
            if gate is not None:
                from .elementwise import sigmoid_gate
                sigmoid_gate(out, gate)
            return out
    check(core().tq_attention_ext(
        ptr(q), dtype_code(q), ptr(k_packed), ptr(v_packed), ptr(k_pages), ptr(v_pages), ptr(block_table),
        table_width, ring_pages, page_tokens, ptr(tok_pos), ptr(tok_seq), ptr(cu_seqlens), ptr(start_pos),
        int(window or 0), float(scale), ptr(out), ptr(part_acc), ptr(part_ml), T, n_heads, n_kv_heads, key_dim,
        value_dim, float(softcap or 0.0), ptr(slopes), keep, ptr(sink), int(chunk or 0), n_splits, stream()),
        "attention_ext", 2 if n_splits > 1 and not unmerged else 1)
    if unmerged:
        return part_acc, part_ml, n_splits
    if gate is not None:
        from .elementwise import sigmoid_gate
        sigmoid_gate(out, gate)
    return out
