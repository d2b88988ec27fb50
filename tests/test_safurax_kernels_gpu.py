"""The kernels that the Safurax decoder brought, each alone against float64 computations at other sizes: the layer norm,
the encoding of two maps per head, the difference of two maps on every attention kernel (with single keys planted far
away, at page borders and in one map only), the sink over caches whose values are their keys, a gate per head, the
router's softmax over the chosen and the gated shared result (GPU)."""
import math

import pytest
import torch

import plain_safurax as ps

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _close(got, want, tol, what=""):
    got, want = got.detach().double().cpu(), want.double().cpu()
    assert got.shape == want.shape, (what, got.shape, want.shape)
    err = float((got - want).abs().max())
    scale = float(want.abs().max()) or 1.0
    assert err <= tol * scale, f"{what}: {err:.3e} of {scale:.3e}"


def _ints(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ---- the layer norm ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,W", [(1, 84), (7, 192), (130, 2048), (200, 512), (3, 5), (2, 4096), (150, 8196), (5, 9001)])
def test_layer_norm(T, W):
    """Rows with a large mean beside a small spread: a variance taken as a difference of squares would be lost."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(W)
    x = (torch.randn(T, W, generator=g) + 30.0 * torch.randn(T, 1, generator=g)).to(DEV)
    w = torch.randn(W, generator=g).to(DEV)
    want = ps.layer_norm(x.double().cpu(), w.double().cpu(), 1e-5)
    out = torch.empty((T, W), dtype=torch.float32, device=DEV)
    _close(kernels.rmsnorm(x, w, 1e-5, out, centered=True), want, 2e-5, "float32")
    half = torch.empty((T, W), dtype=torch.bfloat16, device=DEV)
    _close(kernels.rmsnorm(x, w, 1e-5, half, centered=True), want, 5e-3, "bfloat16")
    rows = _ints([T - 1, 0, T // 2])
    out = torch.empty((3, W), dtype=torch.float32, device=DEV)
    _close(kernels.rmsnorm(x, w, 1e-5, out, rows, centered=True), want[rows.cpu().long()], 2e-5, "picked rows")
    flat = torch.full((1, W), 3.0, device=DEV)                # no spread at all: eps alone keeps the division finite
    out = torch.empty((1, W), dtype=torch.float32, device=DEV)
    assert float(kernels.rmsnorm(flat, w, 1e-5, out, centered=True).abs().max()) < 1e-2


# ---- two maps per head ------------------------------------------------------------------------------------------
MAP_CASES = [(4, 2, 64, 128, 128, 128), (2, 1, 32, 64, 64, 64), (6, 2, 20, 12, 64, 64), (3, 3, 6, 5, 16, 8),
             (4, 1, 48, 72, 96, 96), (2, 2, 96, 40, 192, 40), (16, 1, 16, 32, 32, 32)]


def _encoded(H, G, d, e, kr, vr, T, dtype, rot, seed, paged=True):
    """Projected rows with norm weights, and what the encoding kernel makes of them (packed, and in shuffled pages)."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(seed)
    ld = H * 2 * d + G * 2 * d + G * e + 3
    proj = torch.randn(T, ld, generator=g)
    qw, kw = torch.randn(d, generator=g) * 0.3 + 1.0, torch.randn(d, generator=g) * 0.3 + 1.0
    rate = torch.pow(torch.tensor(1e4, dtype=torch.float64), -2.0 * torch.arange(max(rot // 2, 1), dtype=torch.float64) / max(rot, 2)) / 4.0
    ang = torch.arange(T, dtype=torch.float64).reshape(-1, 1) * rate
    n_pages = -(-T // 64)
    pages = torch.randperm(n_pages + 2, generator=g)[:n_pages].tolist()
    k_pages = torch.full((n_pages + 2, G, 64, kr), 7.0, dtype=dtype, device=DEV)    # what a page held before
    v_pages = torch.full((n_pages + 2, G, 64, vr), 7.0, dtype=dtype, device=DEV)
    q = torch.full((T, H * 2 * kr), float("nan"), dtype=dtype, device=DEV)
    k = torch.full((T, G * kr), float("nan"), dtype=dtype, device=DEV)
    v = torch.full((T, G * vr), float("nan"), dtype=dtype, device=DEV)
    kernels.head_encode(proj.to(DEV), (_ints(list(range(T))), _ints([0] * T), _ints([T])), q, q_col=0, k_col=H * 2 * d,
                        v_col=(H + G) * 2 * d, n_heads=H, n_kv_heads=G, key_dim=d, value_dim=e, maps=2, key_row=kr, value_row=vr,
                        cos=torch.cos(ang).float().to(DEV) if rot else None, sin=torch.sin(ang).float().to(DEV) if rot else None,
                        rotary_dim=rot, norm_eps=1e-5, q_weight=qw.to(DEV), k_weight=kw.to(DEV), k_out=k, v_out=v,
                        k_pages=k_pages, v_pages=v_pages, block_table=_ints([pages]), table_width=n_pages)
    P, pos = proj.double(), torch.arange(T)
    args = (rot, 1e4, 4.0)
    want_q = ps.rms_norm(P[:, :H * 2 * d].reshape(T, H * 2, d), qw.double(), 1e-5)
    want_k = ps.rms_norm(P[:, H * 2 * d:(H + G) * 2 * d].reshape(T, G * 2, d), kw.double(), 1e-5)
    if rot:
        want_q, want_k = ps.rotate(want_q, pos, *args), ps.rotate(want_k, pos, *args)
    want_v = P[:, (H + G) * 2 * d:(H + G) * 2 * d + G * e].reshape(T, G, e)
    return (q, k, v, k_pages, v_pages, pages), (want_q.reshape(T, H, 2, d), want_k.reshape(T, G, 2, d), want_v)


@pytest.mark.parametrize("H,G,d,e,kr,vr", MAP_CASES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_maps_rows_and_the_zeros_around_them(H, G, d, e, kr, vr, dtype):
    T, rot = 70, max(2, d // 2 // 2 * 2)
    (q, k, v, k_pages, v_pages, pages), (wq, wk, wv) = _encoded(H, G, d, e, kr, vr, T, dtype, rot, H * 10 + d)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    q, k, v = q.reshape(T, H, 2, kr), k.reshape(T, G, kr), v.reshape(T, G, vr)
    for m in (0, 1):
        _close(q[:, :, m, m * d:(m + 1) * d], wq[:, :, m], tol, f"query of map {m}")
        _close(k[:, :, m * d:(m + 1) * d], wk[:, :, m], tol, f"key of map {m}")
        rest = torch.cat([q[:, :, m, :m * d], q[:, :, m, (m + 1) * d:]], dim=-1)
        assert float(rest.abs().max() if rest.numel() else 0.0) == 0.0
    _close(v[:, :, :e], wv, tol, "values")
    assert not k[:, :, 2 * d:].any() and not v[:, :, e:].any()
    for t in range(T):
        assert torch.equal(k_pages[pages[t // 64], :, t % 64], k[t]) and torch.equal(v_pages[pages[t // 64], :, t % 64], v[t])


def _difference_reference(q, k, v, rows, scale, factor, eps, out_scale, gate=None):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, e]: the rows' heads [R, H, e]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    mask = ps.visible(T)
    out = torch.zeros((len(rows), H, v.shape[2]), dtype=torch.float64)
    for h in range(H):
        g = h // (H // G)
        a1, a2 = (ps.softmax_head(q[rows, h, m], k[:, g, m], v[:, g], scale, mask[rows]) for m in (0, 1))
        out[:, h] = ps.rms(a1 - factor * a2, eps) * out_scale
    return out if gate is None else out * torch.sigmoid(gate).unsqueeze(-1)


def _check_difference(rows_dev, refs, H, G, e, kr, vr, dtype, scale, what, tol=None):
    """The rows through the packed prompt kernels, a portion over pages, and single tokens with one to five splits."""
    from tq_kv_b200 import kernels
    q, k, v, k_pages, v_pages, pages = rows_dev
    T = q.shape[0]
    factor, eps, out_scale = -0.7, 1e-5, 0.65
    g = torch.Generator().manual_seed(T + e)
    gate = torch.randn(T, H + 3, generator=g)
    gates = gate.to(DEV)[:, 3:]                               # a column slice
    want = _difference_reference(*refs, list(range(T)), scale, factor, eps, out_scale, gate[:, 3:].double())
    tol = tol or (3e-5 if dtype == torch.float32 else 3e-2)
    common = dict(n_heads=2 * H, n_kv_heads=G, key_dim=kr, value_dim=vr, scale=scale, unmerged=True)
    diff = dict(heads=H, row=vr, value_dim=e, factor=factor, eps=eps, out_scale=out_scale)
    paged = dict(k_pages=k_pages, v_pages=v_pages, table_width=len(pages), page_tokens=64)

    def finish(parts, g_rows, n):
        acc, ml, n_splits = parts
        out = torch.full((n, H * e), float("nan"), dtype=dtype, device=DEV)
        return kernels.difference_of_maps(acc, out, ml=ml, n_splits=n_splits, gate=g_rows, **diff).reshape(n, H, e)

    for fast in (True, False):
        parts = kernels.attention_ext(q, None, k_packed=k, v_packed=v, tok_pos=_ints(list(range(T))), tok_seq=_ints([0] * T),
                                      cu_seqlens=_ints([0, T]), start_pos=_ints([0]), use_fast=fast, **common)
        _close(finish(parts, gates, T), want, tol, f"{what} packed fast={fast}")
        a = T // 3
        for n_splits in (1, 2):
            parts = kernels.attention_ext(q[a:].contiguous(), None, tok_pos=_ints(list(range(a, T))), tok_seq=_ints([0] * (T - a)),
                                          cu_seqlens=_ints([0, T - a]), start_pos=_ints([a]), block_table=_ints([pages]),
                                          n_splits=n_splits, use_fast=fast, **paged, **common)
            _close(finish(parts, gates[a:], T - a), want[a:], tol, f"{what} portion fast={fast}, {n_splits} splits")
        rows = [r for r in (0, 1, 63, 64, 65, 127, 128, 199, T - 1) if r < T]
        for n_splits in (1, 3, 5):                            # (some splits of the short rows are empty)
            parts = kernels.attention_ext(q[rows].contiguous(), None, tok_pos=_ints(rows), tok_seq=_ints(list(range(len(rows)))),
                                          cu_seqlens=_ints(list(range(len(rows) + 1))), start_pos=_ints(rows),
                                          block_table=_ints([pages] * len(rows)), n_splits=n_splits, use_fast=fast, **paged, **common)
            _close(finish(parts, gates[rows].contiguous(), len(rows)), want[rows], tol, f"{what} single tokens fast={fast}, {n_splits} splits")


@pytest.mark.parametrize("H,G,d,e,kr,vr", MAP_CASES)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_difference_of_two_maps_on_every_attention_kernel(H, G, d, e, kr, vr, dtype):
    T = 260
    dev, _ = _encoded(H, G, d, e, kr, vr, T, dtype, 0, H + d)
    q, k, v = dev[:3]
    # the reference reads what the kernels read (rounded rows), so that the bound is the attention's own error
    refs = (torch.stack([q.reshape(T, H, 2, kr)[:, :, m, m * d:(m + 1) * d] for m in (0, 1)], dim=2).double().cpu(),
            torch.stack([k.reshape(T, G, kr)[:, :, m * d:(m + 1) * d] for m in (0, 1)], dim=2).double().cpu(),
            v.reshape(T, G, vr)[:, :, :e].double().cpu())
    _check_difference(dev, refs, H, G, e, kr, vr, dtype, 1.0 / math.sqrt(d), f"{H}/{G} x {d}/{e}")


@pytest.mark.parametrize("H,G,d,e,kr,vr", [(2, 1, 64, 128, 128, 128), (4, 2, 32, 64, 64, 64), (2, 1, 20, 12, 64, 64)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("which", [0, 1])
def test_single_keys_far_away_and_at_page_borders_in_one_map(H, G, d, e, kr, vr, dtype, which):
    """One key of ONE map stands out against every query of that map: its value decides that map's share of the
    result at every later row, near and far; the other map does not see it."""
    T = 260
    for key_at in (0, 1, 63, 64, 127, 128, 190):
        (q, k, v, k_pages, v_pages, pages), _ = _encoded(H, G, d, e, kr, vr, T, dtype, 0, d)
        g = torch.Generator().manual_seed(key_at)
        u = torch.randn(d, generator=g)
        u = (u / u.norm()).to(DEV)
        q4, k3, v3 = q.reshape(T, H, 2, kr), k.reshape(T, G, kr), v.reshape(T, G, vr)
        q4[:, :, which, which * d:(which + 1) * d] = u.to(dtype)
        k3 *= 0.1
        k3[key_at, :, which * d:(which + 1) * d] = (u * 14.0).to(dtype)
        v3[:, :, :e] = (v3[:, :, :e].float() * 0.1).to(dtype)
        v3[key_at, :, :e] = torch.linspace(4.0, 6.0, e, device=DEV).to(dtype)
        for t in range(T):
            k_pages[pages[t // 64], :, t % 64], v_pages[pages[t // 64], :, t % 64] = k3[t], v3[t]
        refs = (torch.stack([q4[:, :, m, m * d:(m + 1) * d] for m in (0, 1)], dim=2).double().cpu(),
                torch.stack([k3[:, :, m * d:(m + 1) * d] for m in (0, 1)], dim=2).double().cpu(), v3[:, :, :e].double().cpu())
        shares = [ps.softmax_head(refs[0][:, 0, m], refs[1][:, 0, m], refs[2][:, 0], 1.0, ps.visible(T)) for m in (0, 1)]
        assert float(shares[which][key_at:].min()) > 3.0                     # every later row holds the key's value in this map
        assert float(shares[1 - which][key_at + 40:].abs().max()) < 1.5      # ... and not in the other
        _check_difference((q, k, v, k_pages, v_pages, pages), refs, H, G, e, kr, vr, dtype, 1.0, f"key at {key_at}",
                          tol=1e-4 if dtype == torch.float32 else 4e-2)


# ---- the sink where values are the keys ---------------------------------------------------------------------------
@pytest.mark.parametrize("H,row", [(6, 96), (20, 64), (3, 32), (16, 128), (4, 144)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [None, 70])
def test_a_learned_sink_over_a_cache_whose_values_are_its_keys(H, row, dtype, window):
    """One shared row per token serves as key and value of all heads; a ring for the window; one key stands out at the
    window's last place and one past it."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(H + row)
    T = 210
    k = (torch.randn(T, row, generator=g) * 0.3).to(dtype)
    q = (torch.randn(T, H, row, generator=g) * 0.5).to(dtype)
    sink = torch.randn(H, generator=g) * 2.0 + 2.0
    u = torch.randn(row, generator=g)
    u = u / u.norm()
    rows = [0, 1, 63, 64, 69, 70, 71, 128, 200, T - 1]
    for r in (200, 128):                                     # the key at distance 69 (inside 70), the one at 70 (outside)
        k[r - 69], k[r - 70] = (u * 6.0).to(dtype), (-u * 9.0).to(dtype)
        q[r] = (u * 2.0).to(dtype)
    mask = ps.visible(T, window)
    want = torch.stack([ps.softmax_head(q[:, h].double(), k.double(), k.double(), 1.0, mask, sink[h].double()) for h in range(H)], 1)
    ring = 3 if window else 0
    table = [4, 1, 3] if window else [4, 1, 3, 0]
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for fast in (True, False):
        for n_splits in (1, 3):
            for t in rows:                                   # the ring holds the last positions of each row's own past
                pages = torch.zeros((5, 1, 64, row), dtype=dtype, device=DEV)
                for p in range(max(0, t + 1 - (ring or 4) * 64), t + 1):
                    lp = p // 64 % ring if ring else p // 64
                    pages[table[lp], 0, p % 64] = k[p].to(DEV)
                out = torch.empty((1, H * row), dtype=dtype, device=DEV)
                scratch = torch.empty(H * n_splits * (row + 2), dtype=torch.float32, device=DEV) if n_splits > 1 else None
                kernels.attention_ext(q[t].reshape(1, -1).to(DEV), out, n_heads=H, n_kv_heads=1, key_dim=row, value_dim=row,
                                      tok_pos=_ints([t]), tok_seq=_ints([0]), cu_seqlens=_ints([0, 1]), start_pos=_ints([t]),
                                      scale=1.0, window=window, sink=sink.to(DEV), k_pages=pages, v_pages=pages,
                                      block_table=_ints([table]), table_width=len(table), ring_pages=ring, n_splits=n_splits,
                                      scratch=scratch, use_fast=fast)
                _close(out.reshape(H, row), want[t], tol, f"row {t}, fast={fast}, {n_splits} splits")


# ---- many prompts at once -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("sink", [False, True])
def test_prompt_attention_under_load(sink):
    """Many more tiles than fit the device, over and over, with the values cold and the keys warm in the cache: a block
    whose first value tile comes late has scores of two tiles ready before its first product with values, and must
    neither wait for good nor mix tiles up."""
    from tq_kv_b200 import kernels
    H, d, n_seqs, L = 8, 128, 8, 1024
    T = n_seqs * L
    g = torch.Generator(device=DEV).manual_seed(1)
    q, k, v = (torch.randn(T, H * d, generator=g, device=DEV).to(torch.bfloat16) for _ in range(3))
    flush = torch.empty(64 << 20, dtype=torch.float32, device=DEV)
    pos = _ints(list(range(L)) * n_seqs)
    seq = _ints([b for b in range(n_seqs) for _ in range(L)])
    args = dict(n_heads=H, n_kv_heads=H, tok_pos=pos, tok_seq=seq, cu_seqlens=_ints([b * L for b in range(n_seqs + 1)]),
                start_pos=_ints([0] * n_seqs), window=None, scale=d ** -0.5, k_packed=k, v_packed=v)
    sinks = torch.full((H,), 1.0, device=DEV)
    first = None
    for i in range(250):
        if i % 5 == 0:
            flush.fill_(float(i))
        q2, k2 = q.clone(), k.clone()                        # (warm; the values were last read a launch or a flush ago)
        out = torch.empty_like(q)
        a = {**args, "k_packed": k2}
        if sink:
            kernels.attention_ext(q2, out, key_dim=d, value_dim=d, sink=sinks, **a)
        else:
            kernels.attention(q2, out, head_dim=d, **a)
        first = out if first is None else first
        if i % 25 == 24:
            kernels.check_tc_status()
            assert torch.equal(out, first)
    T0 = 200                                                 # and right: the first rows of one sequence by hand
    rows = slice(3 * L, 3 * L + T0)
    for h in (0, 5):
        c = slice(h * d, (h + 1) * d)
        want = ps.softmax_head(q[rows, c].double().cpu(), k[rows, c].double().cpu(), v[rows, c].double().cpu(), d ** -0.5,
                               ps.visible(T0), torch.tensor(1.0, dtype=torch.float64) if sink else None)
        _close(first[rows, c], want, 2e-2, f"head {h}")


@pytest.mark.parametrize("H,d", [(4, 64), (2, 128), (3, 32), (2, 96)])
@pytest.mark.parametrize("window", [None, 70])
def test_a_gate_per_head_in_the_prompt_kernels(H, d, window):
    from tq_kv_b200 import kernels
    T = 150
    g = torch.Generator().manual_seed(d)
    q, k, v = (torch.randn(T, H * d, generator=g).to(torch.bfloat16) for _ in range(3))
    gate = torch.randn(T, H + 3, generator=g)[:, 2:H + 2]
    sink = torch.randn(H, generator=g)
    for fast in (True, False):
        out = torch.empty((T, H * d), dtype=torch.bfloat16, device=DEV)
        wide = torch.zeros((T, H + 3), device=DEV)
        wide[:, 2:H + 2] = gate.to(DEV)
        kernels.attention_ext(q.to(DEV), out, n_heads=H, n_kv_heads=H, key_dim=d, value_dim=d, tok_pos=_ints(list(range(T))),
                              tok_seq=_ints([0] * T), cu_seqlens=_ints([0, T]), start_pos=_ints([0]), scale=d ** -0.5,
                              window=window, sink=sink.to(DEV), gate=wide[:, 2:H + 2], k_packed=k.to(DEV), v_packed=v.to(DEV),
                              use_fast=fast)
        for h in range(H):
            c = slice(h * d, (h + 1) * d)
            want = ps.softmax_head(q[:, c].double(), k[:, c].double(), v[:, c].double(), d ** -0.5, ps.visible(T, window),
                                   sink[h].double()) * torch.sigmoid(gate[:, h:h + 1].double())
            _close(out[:, c], want, 2e-2, f"head {h}, fast={fast}")


@pytest.mark.parametrize("T,H,d,r,n,row", [(1, 3, 20, 4, 24, 32), (17, 2, 128, 0, 128, 128), (40, 5, 96, 32, 96, 128),
                                           (64, 1, 130, 2, 200, 208), (5, 4, 12, 6, 10, 32), (33, 2, 64, 64, 512, 576)])
def test_the_latent_s_per_head_products(T, H, d, r, n, row):
    """The query into the latent's space and the mean latent out of it, in bfloat16, at sizes around the tensor-core
    tiles (one whose rows are no whole 16-byte pieces: the general kernel)."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(T + n)
    e = d + 3
    q = torch.randn(T, H * (d + r), generator=g).to(DEV)
    uk = (torch.randn(H * d, n, generator=g) / d ** 0.5).to(torch.bfloat16).to(DEV)
    uv = (torch.randn(H * e, n, generator=g) / n ** 0.5).to(torch.bfloat16).to(DEV)
    pos = torch.arange(T) * 7 + 1
    rate = torch.pow(torch.tensor(1e4, dtype=torch.float64), -2.0 * torch.arange(max(r // 2, 1), dtype=torch.float64) / max(r, 2))
    ang = torch.arange(T * 7 + 2, dtype=torch.float64).reshape(-1, 1) * rate
    qa = torch.full((T, H * row), float("nan"), dtype=torch.bfloat16, device=DEV)
    kernels.latent_query(q, uk, qa, heads=H, dim=d, rot_dim=r, kv_rank=n, row_width=row, cos=torch.cos(ang).float().to(DEV),
                         sin=torch.sin(ang).float().to(DEV), rot_dims=r, paired=False, tok_pos=pos.int().to(DEV))
    Q = q.double().cpu().reshape(T, H, d + r)
    got = qa.reshape(T, H, row)
    _close(got[..., :n], torch.einsum("thd,hdn->thn", Q[..., :d], uk.double().cpu().reshape(H, d, n)), 1.5e-2, "query")
    if r:
        _close(got[..., n:n + r], ps.rotate(Q[..., d:], pos, r, 1e4), 1e-2, "rotated part")
    assert not got[..., n + r:].any()
    lat = torch.randn(T, H * row, generator=g).to(torch.bfloat16).to(DEV)
    gate = torch.randn(T, H * e, generator=g).to(DEV)
    y = torch.full((T, H * e), float("nan"), dtype=torch.bfloat16, device=DEV)
    kernels.latent_expand(lat, uv, y, heads=H, kv_rank=n, row_width=row, value_dim=e, gate=gate)
    want = torch.einsum("thn,hen->the", lat.double().cpu().reshape(T, H, row)[..., :n], uv.double().cpu().reshape(H, e, n))
    _close(y.reshape(T, H, e), want * torch.sigmoid(gate.double().cpu().reshape(T, H, e)), 1.5e-2, "expanded")


# ---- the latent's kernels without rotation and with a gate per head -------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_rows_and_queries_without_a_rotated_part(dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(3)
    T, H, d, n, nq, row = 5, 3, 12, 20, 10, 32
    proj = torch.randn(T, nq + n, generator=g).to(DEV)
    wq, wkv = torch.randn(nq, generator=g).to(DEV), torch.randn(n, generator=g).to(DEV)
    none = torch.zeros((1, 1), device=DEV)
    cq, rows = torch.empty((T, nq), dtype=dtype, device=DEV), torch.empty((T, row), dtype=dtype, device=DEV)
    pos = _ints([0, 5, 63, 64, 900])
    kernels.latent_rows(proj, cq, off_q=0, off_kv=nq, q_rank=nq, kv_rank=n, rot_dim=0, row_width=row, q_weight=wq,
                        kv_weight=wkv, eps=1e-5, cos=none, sin=none, rot_dims=0, paired=False, tok_pos=pos, tok_seq=_ints([0] * T),
                        new_lens=_ints([901]), row_out=rows)
    P, tol = proj.double().cpu(), 1e-5 if dtype == torch.float32 else 1e-2
    _close(cq, ps.rms_norm(P[:, :nq], wq.double().cpu(), 1e-5), tol, "query latent")
    _close(rows[:, :n], ps.rms_norm(P[:, nq:], wkv.double().cpu(), 1e-5), tol, "latent")
    assert not rows[:, n:].any()
    q, uk = torch.randn(T, H * d, generator=g).to(DEV), torch.randn(H * d, n, generator=g).to(dtype).to(DEV)
    qa = torch.empty((T, H * row), dtype=dtype, device=DEV)
    kernels.latent_query(q, uk, qa, heads=H, dim=d, rot_dim=0, kv_rank=n, row_width=row, cos=none, sin=none, rot_dims=0,
                         paired=False, tok_pos=pos)
    want = torch.einsum("thd,hdn->thn", q.double().cpu().reshape(T, H, d), uk.double().cpu().reshape(H, d, n))
    _close(qa.reshape(T, H, row)[..., :n], want, tol, "query in the latent's space")
    assert not qa.reshape(T, H, row)[..., n:].any()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,n,row,e", [(6, 20, 32, 12), (1, 64, 96, 5), (4, 128, 128, 128)])
def test_the_expansion_with_a_gate_per_head(H, n, row, e, dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(H + n)
    T = 4
    lat = torch.randn(T, H * row, generator=g).to(dtype).to(DEV)
    uv = torch.randn(H * e, n, generator=g).to(dtype).to(DEV)
    gate = (torch.randn(T, H + 2, generator=g) * 2.0).to(DEV)[:, 1:H + 1]
    y = torch.empty((T, H * e), dtype=dtype, device=DEV)
    kernels.latent_expand(lat, uv, y, heads=H, kv_rank=n, row_width=row, value_dim=e, gate=gate, head_gate=True)
    want = torch.einsum("thn,hen->the", lat.double().cpu().reshape(T, H, row)[..., :n], uv.double().cpu().reshape(H, e, n))
    want = want * torch.sigmoid(gate.double().cpu()).unsqueeze(-1)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    _close(y.reshape(T, H, e), want, tol, "expanded")
    if e <= row:
        kernels.latent_expand(lat, None, y, heads=H, kv_rank=row, row_width=row, value_dim=e, gate=gate, head_gate=True)
        want = lat.double().cpu().reshape(T, H, row)[..., :e] * torch.sigmoid(gate.double().cpu()).unsqueeze(-1)
        _close(y.reshape(T, H, e), want, tol, "narrowed")
    x = torch.randn(T, H * e, generator=g).to(dtype).to(DEV)
    want = x.double().cpu().reshape(T, H, e) * torch.sigmoid(gate.double().cpu()).unsqueeze(-1)
    _close(kernels.sigmoid_gate(x, gate).reshape(T, H, e), want, tol, "gated in place")


# ---- the experts ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top", [(16, 4), (5, 5), (1, 1), (40, 3), (8, 1)])
def test_the_softmax_over_the_chosen_logits(E, top):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(E)
    z = (torch.randn(50, E + 3, generator=g) * 3.0).to(DEV)[:, :E]      # a column slice
    for zz in (z, (z + 200.0).contiguous(), (z * 30.0).contiguous()):   # (exp of the larger ones overflows on its own)
        choice, weights = kernels.router_choice(zz, top, softmax=True)
        val, idx = torch.topk(zz.double().cpu(), top, dim=-1)
        assert torch.equal(choice.cpu().long(), idx)
        _close(weights, torch.softmax(val, dim=-1), 2e-6, "weights")
    c, w = kernels.router_choice(torch.zeros((2, E), device=DEV), top, softmax=True)      # equal logits: the lowest indices
    assert c.cpu().tolist() == [list(range(top))] * 2 and torch.allclose(w.cpu(), torch.full((2, top), 1.0 / top))


@pytest.mark.parametrize("T,W,F,E,top", [(5, 96, 40, 6, 2), (200, 128, 64, 8, 3), (70, 84, 36, 3, 3), (3, 64, 16, 1, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("accumulate", [True, False])
def test_the_gated_shared_result_in_rows_and_in_tiles(T, W, F, E, top, dtype, accumulate):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(T + W)
    x = torch.randn(T, W, generator=g).to(dtype)
    gu = (torch.randn(E, 2 * F, W, generator=g) / W ** 0.5).to(dtype)
    dn = (torch.randn(E, W, F, generator=g) / F ** 0.5).to(dtype)
    z = torch.randn(T, E + 1, generator=g).to(DEV)
    shared = torch.randn(T, W, generator=g).to(DEV)
    choice, weights = kernels.router_choice(z[:, :E], top, softmax=True)
    xd, gd, dd = x.double(), gu.double(), dn.double()
    want = shared.double().cpu() * torch.sigmoid(z[:, E:].double().cpu())
    for t in range(T):
        for j in range(top):
            e_ = int(choice[t, j])
            a = ps.silu(gd[e_, :F] @ xd[t]) * (gd[e_, F:] @ xd[t])
            want[t] += float(weights[t, j]) * (dd[e_] @ (a.to(torch.bfloat16).double() if dtype == torch.bfloat16 else a))
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    forms = [kernels.routed_experts_rows]
    if dtype == torch.bfloat16 and kernels.routed_tiles_ok(x.to(DEV), gu.to(DEV), dn.to(DEV)):
        forms.append(kernels.routed_experts_tiles)
    for form in forms:
        base = torch.randn(T, W, generator=g).to(DEV)
        y = base.clone()
        form(x.to(DEV), gu.to(DEV), dn.to(DEV), choice, y, accumulate=accumulate, weights=weights, shared=shared,
             shared_gate=z[:, E:])
        _close(y - base if accumulate else y, want, tol, form.__name__)
