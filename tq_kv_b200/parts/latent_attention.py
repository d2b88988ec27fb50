"""Softmax attention whose keys and values come from a small latent per token.

With H heads, per head `dim` unrotated and `rot_dim` rotated query/key entries
and values of `value_dim`, and a latent of `kv_rank`:

    c_q = rms_norm(W_dq x) * w_q            q[h] = (W_uq c_q)[h] = [q_flat[h] (dim), q_rot[h] (rot_dim)]
    [c' , k_r'] = W_dkv x                   c = rms_norm(c') * w_kv,  k_r = rotate(k_r')   (shared by the heads)
    key[h] = [U_k[h] c, k_r]                value[h] = U_v[h] c
    score = (q_flat[h] . U_k[h] c + rotate(q_rot[h]) . k_r) * scale,   softmax over the keys j <= i
    out = W_o ((heads side by side) * sigmoid(W_g x))            (the gate is optional)

`output_gate` True gates entry by entry; "heads" gates every head with one number (W_g has a row per head).  `sink`:
the softmax's denominator counts one more key without a value whose score is a learned number per head (tensor `sink`).
rot_dim 0: there is no rotated part (and no position).

With `shared_kv` the layer has no W_dkv: it reads the cache of the schedule entry it is given (the normed latents and
rotated key parts of an earlier layer) with its own U_k, U_v, queries, window, sink and gate.  `cache_window` is the
window the cache keeps (default: `window`; wider where other layers with wider windows read this layer's cache; None:
all rows); `shares_packed` leaves a prompt's packed rows in the step's shared dict for those layers.

Without a query latent (`q_rank` absent) the queries are projected directly, q = W_q x.  With `window` the query at
position i reads the keys j with 0 <= i - j < window, and the cache is a ring of the window's rows.

Only c and k_r are cached: one row of kv_rank + rot_dim values per token (one key/value "head" whose value rows
are not used).  The attention itself runs in the latent's space: the query is carried there,
q~[h] = [U_k[h]^T q_flat[h], rotate(q_rot[h])], the attention kernels see one shared key/value head whose value
is the cached row itself, and the weighted mean of latents is expanded afterwards, U_v[h] mean(c)
(csrc/latent_attention.cu).  That is how everything that reads the pages runs (decoding, portions of prompts, a
prompt beside decoding rows).  Prompts from position 0 bring all their keys along: there the keys and values of all
heads are expanded once, by two matrix products, and the ordinary attention kernels run with this mixer's heads
(fewer operations per score, and the tensor-core prompt kernels take the heads' widths).  Rows are padded with
zeros to the next width of the tensor-core kernels, or (over 128 values) to a multiple of 16.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..cache import PAGE_TOKENS, KVRequest, ring_pages_for
from ..config import ConfigError
from ..kernels.attention import MAX_HEAD_DIM
from .base import Mixer, Runtime, StepContext, WeightSpec, float32_vector, stack_rows
from .registry import make_part

MAX_ROW = MAX_HEAD_DIM          # widest cached row (latent + rotated part) the attention kernels take


class LatentAttention(Mixer):
    padded_rows_ok = True               # causal, and rows past a sequence's new length are not cached
    can_store_result = True

    def __init__(self, spec):
        super().__init__(spec)
        p = self.params
        self.hidden = int(p["hidden_size"])
        self.heads, self.dim, self.rot_dim = int(p["heads"]), int(p["dim"]), int(p["rot_dim"])
        self.value_dim = int(p["value_dim"])
        self.q_rank, self.kv_rank = int(p.get("q_rank") or 0), int(p["kv_rank"])      # q_rank 0: q = W_q x directly
        self.window = int(p["window"]) if p.get("window") else None
        self.window_chunk = 1
        self.cache_window = self.window
        if "cache_window" in p:
            self.cache_window = int(p["cache_window"]) if p.get("cache_window") else None
        if self.cache_window is not None and (self.window is None or self.cache_window < self.window):
            raise ConfigError(f"latent attention: a cache of {self.cache_window} rows is too small for a window of {self.window}")
        self.shared_kv, self.shares_packed = bool(p.get("shared_kv", False)), bool(p.get("shares_packed", False))
        if self.shared_kv and self.q_rank:
            raise ConfigError("latent attention: a layer that reads another's latents projects its queries directly")
        self.sink = bool(p.get("sink", False))
        self.scale = float(p["scale"])
        self.eps = float(p["eps"])
        self.output_gate = p.get("output_gate") or False
        if self.output_gate not in (False, True, "heads"):
            raise ConfigError(f"latent attention: output_gate {self.output_gate} (False, True or heads)")
        self.head_gate = self.output_gate == "heads"
        self.names = dict(p["names"])
        self.position = make_part(p["position"]) if p.get("position") is not None else None
        if self.position is None and self.rot_dim:
            raise ConfigError("latent attention: a rotated part needs a position")
        self.rotary_dim = self.position.rotary_dim if self.position is not None else 0
        self.gate_rows = 0 if not self.output_gate else self.heads * (1 if self.head_gate else self.value_dim)
        need = self.kv_rank + self.rot_dim
        self.row = next((w for w in kernels.TENSOR_CORE_WIDTHS if w >= need), -(-need // 16) * 16)
        if self.row > MAX_ROW:
            raise ConfigError(f"latent attention: a cached row of {self.kv_rank} + {self.rot_dim} values exceeds the "
                              f"attention kernels' {MAX_ROW}")
        if self.rotary_dim > self.rot_dim:
            raise ConfigError("latent attention: more rotated entries than the rotated part holds")
        self.w_in = self.w_uq = self.w_uk = self.w_uv = self.w_o = self.q_norm_w = self.kv_norm_w = self.sinks = None
        self.cos = self.sin = None

    def _n(self, which: str) -> str:
        return self.prefix + self.names[which]

    def weight_specs(self):
        h, H = self.hidden, self.heads
        if self.q_rank:
            specs = [WeightSpec(self._n("q_down"), (self.q_rank, h), "matrix"),
                     WeightSpec(self._n("q_norm"), (self.q_rank,), "norm_scale"),
                     WeightSpec(self._n("q_up"), (H * (self.dim + self.rot_dim), self.q_rank), "matrix")]
        else:
            specs = [WeightSpec(self._n("q"), (H * (self.dim + self.rot_dim), h), "matrix")]
        if not self.shared_kv:
            specs += [WeightSpec(self._n("kv_down"), (self.kv_rank + self.rot_dim, h), "matrix"),
                      WeightSpec(self._n("kv_norm"), (self.kv_rank,), "norm_scale")]
        specs += [WeightSpec(self._n("k_up"), (H * self.dim, self.kv_rank), "matrix"),
                  WeightSpec(self._n("v_up"), (H * self.value_dim, self.kv_rank), "matrix"),
                  WeightSpec(self._n("out"), (h, H * self.value_dim), "matrix")]
        if self.sink:
            specs.append(WeightSpec(self._n("sink"), (H,), "sink"))
        if self.output_gate:
            specs.append(WeightSpec(self._n("gate"), (self.gate_rows, h), "matrix"))
        return specs

    def bind(self, tensors, runtime: Runtime, shared=None):
        ws = [tensors[self._n("q_down" if self.q_rank else "q")]]
        if not self.shared_kv:
            ws.append(tensors[self._n("kv_down")])
        self.q_cols = self.q_rank or self.heads * (self.dim + self.rot_dim)      # columns of the first projection
        if self.output_gate:
            ws.append(tensors[self._n("gate")])
        self.gate_col = self.q_cols + (0 if self.shared_kv else self.kv_rank + self.rot_dim)
        self.w_in, _ = stack_rows(ws)                           # query latent | key/value latent, rotated part | gate
        self.w_uq = tensors[self._n("q_up")].contiguous() if self.q_rank else None
        self.window_chunk = runtime.window_chunk
        act = runtime.act_dtype                                 # the per-head products read these in the activations' dtype
        self.w_uk = tensors[self._n("k_up")].to(act).contiguous()
        self.w_uv = tensors[self._n("v_up")].to(act).contiguous()
        self.w_ukv = torch.cat([self.w_uk, self.w_uv], dim=0).contiguous()     # prompts expand keys and values at once
        # the heads' width where keys and values are expanded: in bfloat16 up to the next one of the tensor-core kernels
        need = max(self.dim + self.rot_dim, self.value_dim)
        self.head_width = -(-need // 16) * 16
        if act == torch.bfloat16:
            self.head_width = next((w for w in kernels.TENSOR_CORE_WIDTHS if w >= need), self.head_width)
        self.plain_heads = bool(self.q_rank) and not self.rot_dim and self.dim == self.value_dim == self.head_width
        self.w_o = tensors[self._n("out")].contiguous()
        self.q_norm_w = float32_vector(tensors[self._n("q_norm")]) if self.q_rank else None
        self.kv_norm_w = float32_vector(tensors[self._n("kv_norm")]) if not self.shared_kv else None
        self.sinks = float32_vector(tensors[self._n("sink")]) if self.sink else None
        if self.position is not None:
            self.position.bind(tensors, runtime, shared)
            self.position.prepare(runtime, shared)
            self.cos, self.sin = self.position.cos, self.position.sin
        else:
            self.cos = self.sin = torch.zeros((1, 1), dtype=torch.float32, device=runtime.device)     # never read

    def cache_request(self):
        return None if self.shared_kv else KVRequest(1, self.row, self.cache_window, 1)

    def check_step(self, start_pos, step_lens, owns_cache):
        if self.shared_kv and owns_cache:
            raise kernels.KernelError("a layer without a latent of its own must be given another entry's cache")
        if self.cache_window is None or self._use_packed(start_pos, step_lens, owns_cache):
            return
        ring_tokens = ring_pages_for(self.cache_window, self.window_chunk - 1) * PAGE_TOKENS
        longest = max(step_lens)
        if longest > ring_tokens - self.window + 1:
            raise kernels.KernelError(
                f"a layer with a window of {self.cache_window} keeps {ring_tokens} rows per sequence and cannot continue "
                f"a sequence by {longest} tokens in one step (at most {ring_tokens - self.window + 1}; the engine's "
                f"window_chunk option sets this)")

    def _use_packed(self, start_pos, step_lens, owns_cache) -> bool:
        return (owns_cache or self.shared_kv) and all(s == 0 for s in start_pos) and any(n > 1 for n in step_lens)

    def forward(self, x, ctx: StepContext, residual):
        b, kv, dev = ctx.batch, ctx.kv, residual.device
        act = ctx.runtime.act_dtype
        H, row = self.heads, self.row
        proj = kernels.linear(x, self.w_in, out_dtype=torch.float32)
        kernels.mark("qkv")
        T = proj.shape[0]
        owns = kv is not None and kv.writes and not self.shared_kv
        packed = self._use_packed(b.host_start, b.host_lens, owns)
        cq = torch.empty((T, self.q_rank), dtype=act, device=dev) if self.q_rank else None
        rows = None
        if packed and self.shared_kv:
            rows = ctx.step_shared[("packed_rows", ctx.cache_entry)]
        elif packed:
            rows = torch.empty((T, row), dtype=act, device=dev)
            if self.shares_packed and ctx.step_shared is not None:
                ctx.step_shared[("packed_rows", ctx.entry)] = rows
        rot = dict(cos=self.cos, sin=self.sin, rot_dims=self.rotary_dim, tok_pos=b.tok_pos,
                   paired=self.position is not None and self.position.paired)
        if not self.shared_kv:
            kernels.latent_rows(proj, cq, off_q=0, off_kv=self.q_cols, q_rank=self.q_rank, kv_rank=self.kv_rank,
                                rot_dim=self.rot_dim, row_width=row, q_weight=self.q_norm_w, kv_weight=self.kv_norm_w,
                                eps=self.eps, tok_seq=b.tok_seq, new_lens=b.new_lens, row_out=rows,
                                pages=kv.k_pages if owns else None, block_table=kv.block_table if owns else None,
                                table_width=kv.table_width if owns else 0,
                                page_tokens=kv.page_tokens if kv is not None else 64,
                                ring_pages=kv.ring_pages if owns else 0, out_dtype=act, **rot)
            kernels.mark("rotary")
        if self.q_rank:
            q = kernels.linear(cq, self.w_uq, out_dtype=act if packed and self.plain_heads else torch.float32)
            kernels.mark("qkv")
        else:
            q = proj[:, :self.q_cols]
        gate = proj[:, self.gate_col:self.gate_col + self.gate_rows] if self.output_gate else None
        common = dict(n_heads=H, tok_pos=b.tok_pos, tok_seq=b.tok_seq, cu_seqlens=b.cu_seqlens, start_pos=b.start_pos,
                      window=self.window, scale=self.scale)
        y = torch.empty((T, H * self.value_dim), dtype=act, device=dev)
        if packed:
            # A prompt from position 0 brings all its keys along: they are expanded once (two matrix products for
            # all heads) and the ordinary attention kernels run with this mixer's heads as they are.
            hw = self.head_width
            lat = rows[:, :self.kv_rank]
            if self.plain_heads:
                # nothing to turn and nothing to fill up: the products leave the heads as the attention takes them
                qh = q
                kh = kernels.linear(lat, self.w_uk, out_dtype=act)
                vh = kernels.linear(lat, self.w_uv, out_dtype=act)
                kernels.mark("qkv")
            else:
                kfv = kernels.linear(lat, self.w_ukv, out_dtype=torch.float32)
                kernels.mark("qkv")
                qh, kh, vh = (torch.empty((T, H * hw), dtype=act, device=dev) for _ in range(3))
                kernels.latent_heads(q, kfv, rows, qh, kh, vh, heads=H, dim=self.dim, rot_dim=self.rot_dim,
                                     value_dim=self.value_dim, kv_rank=self.kv_rank, **rot)
                kernels.mark("rotary")
            if hw == self.value_dim:             # the heads' results are as wide as they have to be: gated in place
                self._attend(qh, y, hw, k_packed=kh, v_packed=vh, n_kv_heads=H, gate=gate, **common)
                kernels.mark("attention")
            else:
                oh = torch.empty((T, H * hw), dtype=act, device=dev)
                self._attend(qh, oh, hw, k_packed=kh, v_packed=vh, n_kv_heads=H, **common)
                kernels.mark("attention")
                kernels.latent_expand(oh, None, y, heads=H, kv_rank=hw, row_width=hw, value_dim=self.value_dim, gate=gate,
                                      head_gate=self.head_gate)
                kernels.mark("rotary")
            kernels.linear(y, self.w_o, out=residual, accumulate=not ctx.store_result)
            kernels.mark("o")
            return
        qa = torch.empty((T, H * row), dtype=act, device=dev)
        kernels.latent_query(q, self.w_uk, qa, heads=H, dim=self.dim, rot_dim=self.rot_dim, kv_rank=self.kv_rank,
                             row_width=row, **rot)
        kernels.mark("rotary")
        lat = torch.empty_like(qa)
        max_keys = b.max_new_len if self.window is None else min(b.max_new_len, self.window)
        n_splits = kernels.plan_splits(T, kernels.head_groups(H, 1), max_keys, ctx.runtime.sm_count)
        scratch = None
        if n_splits > 1:
            scratch = torch.empty(kernels.split_scratch_floats(T, H, row, n_splits), dtype=torch.float32, device=dev)
        self._attend(qa, lat, row, n_kv_heads=1, k_pages=kv.k_pages, v_pages=kv.k_pages, block_table=kv.block_table,
                     table_width=kv.table_width, ring_pages=kv.ring_pages, page_tokens=kv.page_tokens,
                     n_splits=n_splits, scratch=scratch, **common)
        kernels.mark("attention")
        kernels.latent_expand(lat, self.w_uv, y, heads=H, kv_rank=self.kv_rank, row_width=row,
                              value_dim=self.value_dim, gate=gate, head_gate=self.head_gate)
        kernels.mark("rotary")
        kernels.linear(y, self.w_o, out=residual, accumulate=not ctx.store_result)
        kernels.mark("o")

    def _attend(self, q, out, width, gate=None, **kw):
        """The attention kernels over rows of `width` entries, with the sink and the gate if there are any."""
        if self.sinks is None and gate is None:
            kernels.attention(q, out, head_dim=width, **kw)
        else:
            kernels.attention_ext(q, out, key_dim=width, value_dim=width, gate=gate,
                                  sink=False if self.sinks is None else self.sinks, **kw)
