"""The kernels that the Gokapel decoder brought, each alone against float64 computations at other sizes: the delta rule
with a decay per key channel, the write strengths beside the convolution, the two-step projections, the per-channel
recurrence, the streams' kernel with its norm, scale and gate, the norm per head with weights and rotation, chunks and
learned sinks in every attention kernel (with single keys planted at the chunks' edges), the choice with groups,
experts without a gate, products through the square of relu (GPU)."""
import math

import pytest
import torch

import plain_gokapel as pg

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _close(got, want, tol, what=""):
    got, want = got.detach().double().cpu(), want.double().cpu()
    assert got.shape == want.shape, f"{what}: {tuple(got.shape)} vs {tuple(want.shape)}"
    err = float((got - want).abs().max())
    scale = float(want.abs().max()) or 1.0
    assert err <= tol * scale, f"{what}: {err:.3e} of {scale:.3e}"


def _ints(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _cu(lens):
    return _ints([sum(lens[:i]) for i in range(len(lens) + 1)])


# ---- the delta rule with a decay per key channel -----------------------------------------------------------------
@pytest.mark.parametrize("H,G,d,e,lens", [(6, 2, 20, 12, (1, 37, 2, 70)), (2, 2, 64, 64, (130,)), (4, 1, 128, 128, (33, 1, 9)),
                                          (3, 3, 18, 30, (5, 5)), (1, 1, 200, 40, (40,)), (32, 16, 128, 128, (12, 3, 20)),
                                          (24, 8, 64, 256, (9, 17, 4, 2)), (4, 2, 33, 7, (19, 20)),
                                          (2, 1, 256, 20, (3, 6)), (16, 8, 128, 128, (70,)), (5, 5, 30, 100, (4, 8, 1, 63))])
def test_the_channel_delta_scan_against_the_recurrence(H, G, d, e, lens):
    """A ragged batch with shuffled slots and states that are not zero, then every sequence continued token by token
    with the one-token kernel; sizes that take every form of the scan."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(H * 100 + d)
    n, more = len(lens), 3
    slots = [5, 2, 7, 0][:n]
    extra = 5                                                  # the state lies in wider rows
    state = torch.randn(8, H * d * e + extra, generator=g) * 0.2
    dev_state = state.to(DEV)
    S = state[:, :H * d * e].double().reshape(8, H, d, e)

    def draw(T):
        x = torch.randn(T, 2 * G * d + H * e, generator=g)
        q, k = pg.unit(x[:, :G * d].reshape(T, G, d)) * d ** -0.5, pg.unit(x[:, G * d:2 * G * d].reshape(T, G, d))
        buf = torch.cat([q.reshape(T, -1), k.reshape(T, -1), x[:, 2 * G * d:]], dim=1)
        w = torch.exp(-torch.exp(torch.randn(T, H * d, generator=g) * 2.0 - 2.0))
        scal = torch.randn(T, H, 4, generator=g)               # (only entry 1 may be read)
        scal[..., 1] = torch.sigmoid(scal[..., 1])
        return buf.float(), w.float(), scal.float()

    def reference(buf, w, scal, t, slot):
        q = buf[t, :G * d].double().reshape(G, d).repeat_interleave(H // G, 0)
        k = buf[t, G * d:2 * G * d].double().reshape(G, d).repeat_interleave(H // G, 0)
        v = buf[t, 2 * G * d:].double().reshape(H, e)
        st = w[t].double().reshape(H, d, 1) * S[slot]
        u = scal[t, :, 1].double().reshape(H, 1) * (v - torch.einsum("hde,hd->he", st, k))
        S[slot] = st + k.unsqueeze(-1) * u.unsqueeze(1)
        return torch.einsum("hde,hd->he", S[slot], q).reshape(-1)

    def run(buf, w, scal, cu, n_seqs, single):
        T = buf.shape[0]
        b, wd = buf.to(DEV), w.to(DEV)
        out = torch.empty((T, H * e), dtype=torch.float32, device=DEV)
        kernels.channel_delta_scan(b[:, :G * d], b[:, G * d:2 * G * d], b[:, 2 * G * d:], wd, scal.to(DEV),
                                   dev_state[:, :H * d * e], cu, _ints(slots), out, n_seqs=n_seqs, heads=H, qk_heads=G,
                                   key_dim=d, value_dim=e, single_tokens=single)
        return out

    T = sum(lens)
    buf, w, scal = draw(T)
    want, at = [], 0
    for b, L in enumerate(lens):
        want += [reference(buf, w, scal, at + i, slots[b]) for i in range(L)]
        at += L
    _close(run(buf, w, scal, _cu(lens), n, False), torch.stack(want), 2e-5, "prompt")
    for _ in range(more):
        buf, w, scal = draw(n)
        want = torch.stack([reference(buf, w, scal, b, slots[b]) for b in range(n)])
        _close(run(buf, w, scal, _ints(list(range(n + 1))), n, True), want, 2e-5, "one token")
    _close(dev_state[:, :H * d * e].reshape(8, H, d, e), S, 2e-5, "state")
    assert torch.equal(dev_state[:, H * d * e:].cpu(), state[:, H * d * e:])


def test_decays_made_from_their_logits_and_channels_that_fade_at_once():
    """The scan that makes the decays itself gives what it gives for ready ones; decays of exactly zero and one, and of
    1e-30 in every token, leave everything finite."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(8)
    H, d, e, lens = 3, 40, 24, (23, 2, 41)
    T, n = sum(lens), len(lens)
    buf = torch.randn(T, 2 * H * d + H * e, generator=g)
    buf[:, :2 * H * d] = pg.unit(buf[:, :2 * H * d].reshape(T, 2 * H, d)).reshape(T, -1)
    z, bias, a_log = torch.randn(T, H * d, generator=g) * 3.0, torch.randn(H * d, generator=g), torch.randn(H, generator=g)
    bias[:4] = torch.tensor([200.0, -200.0, 69.0, 30.0])
    a_log[0] = 0.0
    w = torch.exp(-torch.exp(a_log).repeat_interleave(d) * torch.nn.functional.softplus(z + bias)).double().float()
    scal = torch.sigmoid(torch.randn(T, H, 4, generator=g))
    outs = []
    for kw, x in (({}, w), (dict(dt_bias=bias.to(DEV), a_log=a_log.to(DEV)), z)):
        state = torch.zeros(n, H * d * e, device=DEV)
        b = buf.to(DEV)
        out = torch.empty((T, H * e), device=DEV)
        kernels.channel_delta_scan(b[:, :H * d], b[:, H * d:2 * H * d], b[:, 2 * H * d:], x.to(DEV), scal.to(DEV), state, _cu(lens),
                                   _ints(list(range(n))), out, n_seqs=n, heads=H, qk_heads=H, key_dim=d, value_dim=e, **kw)
        assert torch.isfinite(out).all() and torch.isfinite(state).all()
        outs.append(out)
    _close(outs[1], outs[0], 1e-5, "decays made inside")
    want = pg.delta_scan(*(x.double() for x in (buf[:23, :H * d].reshape(23, H, d), buf[:23, H * d:2 * H * d].reshape(23, H, d),
                                                buf[:23, 2 * H * d:].reshape(23, H, e), w[:23].reshape(23, H, d), scal[:23, :, 1])))
    _close(outs[0][:23], want.reshape(23, -1), 2e-5, "first sequence")


def test_write_strengths_beside_the_convolution():
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(3)
    lens, C, H, K = (7, 1, 40), 36, 5, 4
    T = sum(lens)
    x = torch.randn(T, C + H, generator=g)
    taps = torch.randn(C, K, generator=g)
    want, at = [], 0
    for L in lens:
        want.append(pg.short_conv(x[at:at + L, :C].double(), taps.double()))
        at += L
    xd = x.to(DEV)
    out, scal = torch.empty((T, C), device=DEV), torch.full((T, H, 4), 9.0, device=DEV)
    seq = _ints(sum(([i] * L for i, L in enumerate(lens)), []))
    kernels.short_conv(xd[:, :C], taps.to(DEV), None, out, torch.zeros(4, (K - 1) * C, device=DEV), tok_seq=seq, cu_seqlens=_cu(lens),
                       slots=_ints([3, 0, 1]), n_seqs=3, regions=[(0, C, 12, False, 1.0)], silu=True, beta_raw=xd[:, C:], scalars=scal)
    _close(out, torch.cat(want), 2e-6, "convolution")
    _close(scal[..., 1], torch.sigmoid(x[:, C:].double()), 1e-6, "write strength")
    assert float((scal[..., 0] - 1.0).abs().max()) == 0.0


@pytest.mark.parametrize("T,ra,rg,H,d,n", [(1, 20, 28, 2, 56, 120), (9, 10, 14, 6, 20, 72), (70, 64, 72, 4, 64, 256),
                                           (300, 128, 64, 4, 128, 512), (64, 7, 300, 3, 11, 50)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_two_step_projections(T, ra, rg, H, d, n, dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(T + ra)
    low = torch.randn(T, 3 + ra + rg + 2, generator=g)
    wa, wg = (torch.randn(H * d, ra, generator=g) / ra ** 0.5).to(dtype), (torch.randn(n, rg, generator=g) / rg ** 0.5).to(dtype)
    bias, a_log = torch.randn(H * d, generator=g) * 2.0, torch.randn(H, generator=g)
    bias[:3] = torch.tensor([40.0, -40.0, 15.0])               # decays of nearly zero and of exactly one
    ld = low.to(DEV)
    args = (ld[:, 3:3 + ra], wa.to(DEV), bias.to(DEV), a_log.to(DEV), ld[:, 3 + ra:3 + ra + rg], wg.to(DEV))
    tc = dtype == torch.bfloat16 and T >= 65 and min(ra, rg) >= 64
    for use_tc in (None, False):
        decay, gate, done = kernels.low_rank_gates(*args, use_tc=use_tc)
        assert done
        on_tc = tc and use_tc is None
        la, lg = (t.to(torch.bfloat16).double() if on_tc else t.double() for t in (low[:, 3:3 + ra], low[:, 3 + ra:3 + ra + rg]))
        z = la @ wa.double().T + bias.double()
        want = torch.exp(-torch.exp(a_log.double()).repeat_interleave(d) * torch.nn.functional.softplus(z))
        _close(decay, want, 2e-5, f"decay tc={on_tc}")
        _close(gate, lg @ wg.double().T, 2e-5, f"gate tc={on_tc}")


# ---- the per-channel recurrence -----------------------------------------------------------------------------------
@pytest.mark.parametrize("W,lens", [(58, (1, 127, 3)), (256, (128,)), (17, (129, 8, 9)), (96, (300, 2)), (32, (257, 1, 1, 130))])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_gru_over_runs_of_tokens_and_one_by_one(W, lens, dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(W)
    n, T = len(lens), sum(lens)
    slots = [5, 2, 7, 0][:n]
    state = torch.randn(8, W + 3, generator=g)
    dev_state = state.to(DEV)
    S = state[:, :W].double().clone()

    def step(x, t, slot):
        z, u, gt = x[t, :W].double(), x[t, W:2 * W].double(), x[t, 2 * W:].double()
        z = torch.sigmoid(z)
        S[slot] = (1 - z) * S[slot] + z * torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
        return 0.7 * S[slot] * gt * torch.sigmoid(gt)

    def run(x, cu, single):
        xd = x.to(DEV)
        out = torch.empty((x.shape[0], W), dtype=dtype, device=DEV)
        kernels.gru_scan(xd[:, :W], xd[:, W:2 * W], xd[:, 2 * W:], dev_state[:, :W], cu, _ints(slots), out, n_seqs=n, scale=0.7,
                         single_tokens=single)
        return out

    tol = 5e-6 if dtype == torch.float32 else 5e-3
    x = torch.randn(T, 3 * W, generator=g) * 2.0
    x[:, :W] -= 2.0                                            # long memories beside short ones
    x[0, W] = 0.0                                              # u = 0 belongs to the upper branch
    want, at = [], 0
    for b, L in enumerate(lens):
        want += [step(x, at + i, slots[b]) for i in range(L)]
        at += L
    _close(run(x, _cu(lens), False), torch.stack(want), tol, "prompt")
    for _ in range(3):
        x = torch.randn(n, 3 * W, generator=g) * 2.0
        want = torch.stack([step(x, b, slots[b]) for b in range(n)])
        _close(run(x, _ints(list(range(n + 1))), True), want, tol, "one token")
    _close(dev_state[:, :W], S, 5e-6, "state")
    assert torch.equal(dev_state[:, W:].cpu(), state[:, W:])


# ---- the streams -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("S,T,W", [(1, 5, 96), (2, 70, 256), (3, 33, 84), (4, 7, 130), (6, 9, 64), (2, 3, 4096)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_a_write_that_is_scaled_and_gated_and_a_norm_without_statistics(S, T, W, dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(S * 1000 + W)
    xs, y = torch.randn(S, T, W, generator=g), torch.randn(T, W, generator=g)
    gates = torch.randn(T, W + 8, generator=g) * 3.0
    scale, nw, nb = torch.randn(W, generator=g), torch.randn(W, generator=g), torch.randn(W, generator=g)
    mix, write, read = torch.randn(S, S, generator=g), torch.randn(S, generator=g), torch.randn(S, generator=g)
    alpha = torch.tensor([0.8])
    rows = [0, T - 1, T // 2]
    tol = 2e-6 if dtype == torch.float32 else 5e-3
    for off in (0, 3, 4):                                      # the gate's columns may start anywhere in wider rows
        for with_scale in (True, False):
            gt = gates[:, off:off + W]
            yy = y.double() * torch.sigmoid(gt.double()) * (scale.double() if with_scale else 1.0)
            new = torch.einsum("st,saw->taw", mix.double(), xs.double()) + write.double().reshape(S, 1, 1) * yy
            u = torch.einsum("s,saw->aw", read.double(), new)
            want = torch.tanh(0.8 * u) * nw.double() + nb.double()
            gd = gates.to(DEV)[:, off:off + W]
            kw = dict(y=y.to(DEV), mix=mix.to(DEV), write=write.to(DEV), read=read.to(DEV), norm_weight=nw.to(DEV),
                      norm_bias=nb.to(DEV), alpha=alpha.to(DEV), out_dtype=dtype, y_gate=gd,
                      y_scale=scale.to(DEV) if with_scale else None)
            x = xs.to(DEV)
            sel = kernels.streams_step(x, rows=_ints(rows), **kw)
            assert torch.equal(x.cpu(), xs)                    # a selection of rows leaves the streams alone
            _close(sel, want[rows], tol, "rows")
            _close(kernels.streams_step(x, **kw), want, tol, "all rows")
            _close(x, new, 2e-6, "streams")


def test_the_norm_without_statistics_as_a_part():
    from tq_kv_b200.config import PartSpec
    from tq_kv_b200.parts import Runtime, make_part
    g = torch.Generator().manual_seed(1)
    n = make_part(PartSpec("dynamic_tanh_norm", {"width": 50, "weight_name": "n"}))
    t = {"n": torch.randn(50, generator=g), "n.b": torch.randn(50, generator=g), "n.alpha": torch.tensor(0.4)}
    assert {s.name: tuple(s.shape) for s in n.weight_specs()} == {"n": (50,), "n.b": (50,), "n.alpha": ()}
    n.bind({k: v.to(DEV) for k, v in t.items()}, Runtime(torch.device(DEV), torch.float32, 64))
    x = torch.randn(7, 50, generator=g)
    want = pg.dyt(x.double(), 0.4, t["n"].double(), t["n.b"].double())
    _close(n.forward(x.to(DEV), torch.float32), want, 2e-6)
    _close(n.forward(x.to(DEV), torch.bfloat16, rows=_ints([6, 2])), want[[6, 2]], 5e-3)


# ---- heads --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("H,G,d,e,rot", [(6, 2, 64, 64, 48), (4, 2, 24, 16, 24), (3, 1, 128, 8, 2), (2, 2, 96, 96, 48)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_heads_normed_with_shared_weights_then_turned_and_scaled_values(H, G, d, e, rot, dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(d)
    T, page = 70, 64
    proj = torch.randn(T, 5 + H * d + G * d + G * e, generator=g) * 3.0
    qw, kw = torch.randn(d, generator=g), torch.randn(d, generator=g)
    pos = torch.arange(T) + 30
    rate = 5e3 ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)
    ang = torch.arange(128, dtype=torch.float64).reshape(-1, 1) * rate
    x = proj[:, 5:].double()
    q = pg.rms(x[:, :H * d].reshape(T, H, d), 1e-5) * qw.double()
    k = pg.rms(x[:, H * d:(H + G) * d].reshape(T, G, d), 1e-5) * kw.double()
    q, k = pg.rotate(q, pos, rot, 5e3), pg.rotate(k, pos, rot, 5e3)
    v = x[:, (H + G) * d:].reshape(T, G, e) * 0.37
    qo, ko, vo = (torch.empty((T, n), dtype=dtype, device=DEV) for n in (H * d, G * d, G * e))
    k_pages, v_pages = torch.zeros((3, G, page, d), dtype=dtype, device=DEV), torch.zeros((3, G, page, e), dtype=dtype, device=DEV)
    pages = [2, 0]
    pd = proj.to(DEV)[:, 5:]
    kernels.head_encode(pd, (pos.int().to(DEV), _ints([0] * T), _ints([100])), qo, q_col=0, k_col=H * d, v_col=(H + G) * d, n_heads=H,
                        n_kv_heads=G, key_dim=d, value_dim=e, cos=torch.cos(ang).float().to(DEV), sin=torch.sin(ang).float().to(DEV),
                        rotary_dim=rot, norm_eps=1e-5, paired=True, q_weight=qw.to(DEV), k_weight=kw.to(DEV), v_scale=0.37, k_out=ko,
                        v_out=vo, k_pages=k_pages, v_pages=v_pages, block_table=_ints([pages]), table_width=2, page_tokens=page)
    tol = 3e-6 if dtype == torch.float32 else 5e-3
    _close(qo.reshape(T, H, d), q, tol, "q")
    _close(ko.reshape(T, G, d), k, tol, "k")
    _close(vo.reshape(T, G, e), v, tol, "v")
    for t in (0, 33, 34, 69):
        p = int(pos[t])
        assert torch.equal(k_pages[pages[p // page], :, p % page], ko[t].reshape(G, d))
        assert torch.equal(v_pages[pages[p // page], :, p % page], vo[t].reshape(G, e))


# ---- chunks and sinks, on every attention kernel --------------------------------------------------------------------
def _pages_of(k, v, pages, dtype):
    T, G, d = k.shape
    kp = torch.zeros((len(pages), G, 64, d), dtype=dtype, device=DEV)
    vp = torch.zeros((len(pages), G, 64, v.shape[2]), dtype=dtype, device=DEV)
    for p in range(T):
        kp[pages[p // 64], :, p % 64] = k[p].to(DEV)
        vp[pages[p // 64], :, p % 64] = v[p].to(DEV)
    return kp, vp


@pytest.mark.parametrize("H,G,d,e", [(4, 2, 64, 64), (2, 1, 128, 128), (6, 2, 32, 32), (4, 1, 40, 24), (8, 4, 96, 96)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunk", [None, 1, 33, 64, 90, 150])
def test_chunks_and_sinks_in_prompts_over_pages_and_in_splits(H, G, d, e, dtype, chunk):
    """The same rows through the packed prompt kernels, the paged prompt kernels, single tokens over the cache with
    one and with several splits (the merge step then adds the sink once), and the general kernel."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(d + H)
    T, scale = 300, 0.8 / math.sqrt(d)
    q, k, v = (torch.randn(T, h, w, generator=g).to(dtype) for h, w in ((H, d), (G, d), (G, e)))
    q[200] *= 6.0                                            # rows whose scores are large: the sink takes nearly nothing
    sinks = torch.tensor([(-3.0, 0.0, 2.5, 6.0)[h % 4] for h in range(H)])
    want = pg.softmax_heads(q.double(), k.double(), v.double(), scale, pg.visible(T, chunk), sinks.double())
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    qd, kd, vd = (t.reshape(T, -1).to(DEV) for t in (q, k, v))
    pos, seq, cu, start = _ints(list(range(T))), _ints([0] * T), _ints([0, T]), _ints([0])
    common = dict(n_heads=H, n_kv_heads=G, key_dim=d, value_dim=e, scale=scale, chunk=chunk, sink=sinks.to(DEV))
    for fast in (True, False):
        out = torch.empty((T, H * e), dtype=dtype, device=DEV)
        kernels.attention_ext(qd, out, k_packed=kd, v_packed=vd, tok_pos=pos, tok_seq=seq, cu_seqlens=cu, start_pos=start,
                              use_fast=fast, **common)
        _close(out.reshape(T, H, e), want, tol, f"packed fast={fast}")
    pages = [4, 0, 3, 1, 2]
    k_pages, v_pages = _pages_of(k, v, pages, dtype)
    paged = dict(k_pages=k_pages, v_pages=v_pages, block_table=_ints([pages]), table_width=5, page_tokens=64)
    for first in (100, 191, 192):                            # portions over the pages
        n = T - first
        out = torch.empty((n, H * e), dtype=dtype, device=DEV)
        kernels.attention_ext(qd[first:], out, tok_pos=pos[first:], tok_seq=seq[first:], cu_seqlens=_ints([0, n]),
                              start_pos=_ints([first]), **paged, **common)
        _close(out.reshape(n, H, e), want[first:], tol, f"a portion from {first} over pages")
    rows = [0, 1, 32, 33, 63, 64, 65, 89, 90, 149, 150, 191, 192, 200, 299]      # single tokens, each a sequence of its own
    for n_splits in (1, 3):
        for fast in (True, False):
            out = torch.empty((len(rows), H * e), dtype=dtype, device=DEV)
            scratch = torch.empty(kernels.split_scratch_floats(len(rows), H, e, n_splits), dtype=torch.float32, device=DEV) \
                if n_splits > 1 else None
            kernels.attention_ext(qd[rows].contiguous(), out, tok_pos=_ints(rows), tok_seq=_ints(list(range(len(rows)))),
                                  cu_seqlens=_ints(list(range(len(rows) + 1))), start_pos=_ints(rows),
                                  k_pages=k_pages, v_pages=v_pages, block_table=_ints([pages] * len(rows)), table_width=5,
                                  page_tokens=64, n_splits=n_splits, scratch=scratch, use_fast=fast, **common)
            _close(out.reshape(len(rows), H, e), want[rows], tol, f"single tokens, {n_splits} splits, fast={fast}")


@pytest.mark.parametrize("d", [32, 64, 128])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_single_keys_at_the_chunks_edges_and_page_borders(d, dtype):
    """One key is made to stand out by e^12 against the query; its value reaches every later row of its own chunk
    wholly and no row of another chunk, in prompts and for single tokens."""
    from tq_kv_b200 import kernels
    H = G = 2
    T, chunk = 420, 130
    g = torch.Generator().manual_seed(d)
    sinks = torch.tensor([0.0, 3.0])
    for key_at in (0, 63, 64, 129, 130, 191, 259, 260, 389):
        k, v = torch.randn(T, G, d, generator=g) * 0.1, torch.randn(T, G, d, generator=g) * 0.1
        qv = torch.randn(d, generator=g)
        qv = qv / qv.norm()
        k[key_at] = qv * 12.0
        v[key_at] = 5.0
        q = qv.expand(T, H, d).clone()
        q, k, v = q.to(dtype), k.to(dtype), v.to(dtype)
        want = pg.softmax_heads(q.double(), k.double(), v.double(), 1.0, pg.visible(T, chunk), sinks.double())
        last = key_at // chunk * chunk + chunk - 1             # the last row of the key's chunk
        assert float(want[min(last, T - 1)].min()) > 4.0 and (last + 1 >= T or float(want[last + 1].abs().max()) < 1.0)
        qd, kd, vd = (t.reshape(T, -1).to(DEV) for t in (q, k, v))
        common = dict(n_heads=H, n_kv_heads=G, key_dim=d, value_dim=d, scale=1.0, chunk=chunk, sink=sinks.to(DEV))
        out = torch.empty((T, H * d), dtype=dtype, device=DEV)
        kernels.attention_ext(qd, out, k_packed=kd, v_packed=vd, tok_pos=_ints(list(range(T))), tok_seq=_ints([0] * T),
                              cu_seqlens=_ints([0, T]), start_pos=_ints([0]), **common)
        tol = 2e-5 if dtype == torch.float32 else 2e-2
        _close(out.reshape(T, H, d), want, tol, f"prompt, key at {key_at}")
        pages = [6, 2, 5, 0, 3, 1, 4]
        k_pages, v_pages = _pages_of(k, v, pages, dtype)
        rows = [r for r in (key_at - 1, key_at, last - 1, last, last + 1, last + 2) if 0 <= r < T]
        for n_splits in (1, 2):
            out = torch.empty((len(rows), H * d), dtype=dtype, device=DEV)
            scratch = torch.empty(kernels.split_scratch_floats(len(rows), H, d, n_splits), dtype=torch.float32, device=DEV) \
                if n_splits > 1 else None
            kernels.attention_ext(qd[rows].contiguous(), out, tok_pos=_ints(rows), tok_seq=_ints(list(range(len(rows)))),
                                  cu_seqlens=_ints(list(range(len(rows) + 1))), start_pos=_ints(rows), k_pages=k_pages,
                                  v_pages=v_pages, block_table=_ints([pages] * len(rows)), table_width=7, page_tokens=64,
                                  n_splits=n_splits, scratch=scratch, **common)
            _close(out.reshape(len(rows), H, d), want[rows], tol, f"single tokens, key at {key_at}, {n_splits} splits")


def test_a_window_beside_chunks_is_refused():
    from tq_kv_b200 import kernels
    q = torch.zeros((1, 64), device=DEV)
    with pytest.raises(kernels.KernelError, match="window or chunks"):
        kernels.attention_ext(q, torch.empty_like(q), n_heads=1, n_kv_heads=1, key_dim=64, value_dim=64, scale=1.0, window=4, chunk=4,
                              k_packed=q, v_packed=q, tok_pos=_ints([0]), tok_seq=_ints([0]), cu_seqlens=_ints([0, 1]),
                              start_pos=_ints([0]))


# ---- the feed-forwards ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E,top,count,keep", [(10, 3, 2, 1), (16, 4, 4, 2), (6, 3, 3, 2), (5, 5, 1, 1), (1, 1, 1, 1), (40, 3, 40, 3),
                                              (64, 8, 8, 4), (12, 12, 3, 3), (256, 8, 8, 4)])
def test_the_choice_with_groups_and_a_correction(E, top, count, keep):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(E + top)
    T = 50
    z = (torch.randn(T, E + 3, generator=g) * 2.0).to(DEV)[:, 3:]        # a column slice
    for corr in (torch.randn(E, generator=g) * 0.3 - 0.5, torch.zeros(E)):
        idx, wts, margin = pg.route(z.double().cpu(), corr.double(), top, count, keep)
        choice, weights = kernels.group_router_choice(z, top, corr.to(DEV), count, keep)
        clear = margin > 1e-6
        assert torch.equal(choice.cpu().long()[clear], idx[clear]) and int(clear.sum()) >= T - 3
        _close(weights[clear.to(DEV)], wts[clear], 2e-6, "weights")
    ties = torch.zeros((2, E), device=DEV)                              # equal scores: the lowest indices, in order
    c, w = kernels.group_router_choice(ties, top, None, count, keep)
    assert c.cpu().tolist() == [list(range(top))] * 2 and torch.allclose(w.cpu(), torch.full((2, top), 1.0 / E))
    low = torch.full((E,), -5.0, device=DEV)                            # every choice score far below zero
    assert torch.equal(kernels.group_router_choice(z, top, low, count, keep)[0], kernels.group_router_choice(z, top, None, count, keep)[0])


@pytest.mark.parametrize("T,W,F,E,top", [(5, 96, 40, 6, 2), (200, 128, 64, 8, 3), (70, 84, 36, 3, 3), (3, 64, 16, 1, 1), (300, 256, 200, 5, 2)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_without_a_gate_in_rows_and_in_tiles(T, W, F, E, top, dtype):
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(T + W)
    x = torch.randn(T, W, generator=g).to(dtype)
    up = (torch.randn(E, F, W, generator=g) / W ** 0.5).to(dtype)
    down = (torch.randn(E, W, F, generator=g) / F ** 0.5).to(dtype)
    choice = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    wts = torch.rand(T, top, generator=g)
    y0 = torch.randn(T, W, generator=g)
    want = torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for s in range(top):
            e = int(choice[t, s])
            a = pg.square_relu(up[e].double() @ x[t].double())
            a = a.to(torch.bfloat16).double() if dtype == torch.bfloat16 else a
            want[t] += float(wts[t, s]) * (down[e].double() @ a)
    forms = [kernels.routed_experts_rows]
    if dtype == torch.bfloat16 and W % 8 == 0 and F % 8 == 0:
        forms.append(kernels.routed_experts_tiles)
    for form in forms:
        for acc in (True, False):
            y = y0.to(DEV).clone()
            form(x.to(DEV), up.to(DEV), down.to(DEV), choice.int().to(DEV), y, accumulate=acc, weights=wts.to(DEV), gated=False)
            _close(y, want + (y0.double() if acc else 0.0), 2e-5 if dtype == torch.float32 else 4e-3, f"{form.__name__} {acc}")


@pytest.mark.parametrize("M,K,N", [(1, 256, 256), (7, 96, 40), (16, 2048, 5632), (20, 160, 256), (64, 512, 96), (65, 256, 136),
                                   (300, 160, 256), (40, 84, 50), (129, 72, 17), (1000, 512, 1024)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_products_through_the_square_of_relu(M, K, N, dtype):
    """Every kernel that `linear` may pick for these rows; with and without a bias."""
    from tq_kv_b200 import kernels
    g = torch.Generator().manual_seed(M + K)
    x, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) / K ** 0.5).to(dtype)
    bias = torch.randn(N, generator=g)
    for b in (None, bias):
        z = x.double() @ w.double().T + (0.0 if b is None else b.double())
        got = kernels.linear(x.to(DEV), w.to(DEV), bias=None if b is None else b.to(DEV), activation=kernels.ACT_SQUARE_RELU)
        assert got.dtype == dtype
        _close(got, pg.square_relu(z), 2e-5 if dtype == torch.float32 else 6e-3, f"bias {b is not None}")
    with pytest.raises(kernels.KernelError):
        kernels.linear(x.to(DEV), w.to(DEV), out=torch.zeros(M, N, device=DEV), accumulate=True, activation=kernels.ACT_SQUARE_RELU)


def test_rows_that_ride_in_a_mixer_s_product_give_the_same_as_a_product_of_their_own():
    from tq_kv_b200.config import PartSpec, spec_from_config_dict
    from tq_kv_b200.engine.model import DecoderModel
    from gokapel_cases import CASES
    model = DecoderModel(spec_from_config_dict(CASES["a"])[2])
    riders = [(b.mixer.rider is not None, b.feed_forward is not None and b.feed_forward.rider is not None) for b in model.blocks]
    assert riders == [(True, True), (True, False), (True, False)]      # the dense feed-forward runs the gate's product itself
