"""Small Safurax configurations, weights with a spread that lets every
mechanism matter, and the plain implementation as oracle (cached)."""
from __future__ import annotations

import math
import os

import torch

import plain_safurax as ps
from furesun_cases import Want, check_rows, dense, tokens  # noqa: F401  (the bounds and token draws are the same)


def _rot(dims, base=10000.0, factor=None):
    rot = {"base": base, "dims": dims}
    if factor:
        rot["scaling"] = {"factor": factor}
    return rot


def latent(heads, dim, vdim, rank, q_rank, scale):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank,
                                                  "q_rank": q_rank, "scale": scale}}


def latent2(heads, dim, rot_dim, vdim, rank, window, scale, base=10000.0, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
         "rot": _rot(rot_dim, base)}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention_2", "mixer": m}


def diff(heads, kv, dim, vdim, scale, offset, dims=None, base=10000.0, factor=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                           "diff": offset, "rot": _rot(dim if dims is None else dims, base, factor)}}


def moe(ff, experts, top, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def model(vocab, width, eps, scale, layers):
    return {"architecture": "Safurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# A: a windowed latent whose rows a later layer reads with a WIDER window (the cache keeps the wider one), two maps of
#    20 entries over values of 12 (rows widened inside), a latent without positions between them; rotation over half a
#    map; experts with and without a shared one, a dense feed-forward, a layer without any.
S_A = model(310, 96, 1e-6, 2.0, [
    {**latent2(4, 24, 8, 40, 48, 33, 0.2, 5000.0), "mlp": moe(40, 6, 2, shared=56)},
    {**diff(6, 2, 20, 12, 0.3, 0.35, dims=10, base=5000.0, factor=8.0), "mlp": dense(136)},
    {**latent(3, 24, 20, 56, 40, 0.25), "mlp": None},
    {**latent2(2, 16, 8, 24, 48, 70, 0.25, 5000.0, kv_from=0), "mlp": moe(32, 4, 3)},
])
# B: sizes of the tensor-core kernels: maps of 64 over values of 128 and of 32 over 64, latents whose expanded heads are
#    128 and 64 wide and whose rows are 128 and 96 wide, windows of whole pages and around them, two readers of one
#    layer's rows (one with a narrower, one with a wider window).
S_B = model(392, 160, 1e-6, 1.5, [
    {**diff(4, 2, 64, 128, 0.125, 0.6, base=50000.0, factor=2.0), "mlp": moe(96, 4, 2, shared=64)},
    {**latent2(2, 96, 32, 128, 96, 128, 0.09, 50000.0), "mlp": None},
    {**latent2(4, 32, 32, 64, 96, 65, 0.11, 50000.0, kv_from=1), "mlp": dense(256)},
    {**latent(2, 128, 128, 128, 64, 0.09), "mlp": moe(64, 8, 1, shared=32)},
    {**latent2(2, 64, 32, 64, 96, 200, 0.1, 50000.0, kv_from=1), "mlp": None},
    {**diff(2, 1, 32, 64, 0.18, 0.2, dims=16, factor=16.0), "mlp": dense(96)},
])
# C: a width that is no multiple of 8, windows of 1 and 2 (a token sees itself only, or itself and one more) and none,
#    one expert in all and as many per token as there are, key heads == heads, one head, maps of 6 over values of 5,
#    one rotated pair, no scaling, an embedding that is not scaled.
S_C = model(130, 84, 1e-5, 1.0, [
    {**latent2(1, 16, 4, 24, 10, 2, 0.4), "mlp": moe(50, 1, 1)},
    {**diff(3, 3, 6, 5, 0.5, 0.4, dims=2), "mlp": moe(36, 3, 3, shared=20)},
    {**latent2(3, 8, 2, 8, 20, 1, 0.3), "mlp": dense(50)},
    {**diff(4, 1, 16, 72, 0.4, 0.1), "mlp": None},
    {**latent(1, 12, 36, 20, 6, 0.35), "mlp": dense(44)},
    {**latent2(2, 8, 4, 8, 12, None, 0.3), "mlp": moe(20, 5, 2, shared=12)},
])
# S: softmaxes that are sharp (a large scale on large keys): a single key, far back or at a window's edge, decides
#    a row's result.
S_S = model(150, 64, 1e-5, 2.5, [
    {**diff(2, 1, 32, 32, 1.5, 0.45, factor=3.0), "mlp": None},
    {**latent2(2, 16, 16, 16, 24, 90, 2.0), "mlp": None},
    {**latent(2, 24, 16, 40, 24, 1.5), "mlp": None},
    {**latent2(2, 16, 16, 16, 24, 40, 2.0, kv_from=1), "mlp": None},
])
CASES = {"a": S_A, "b": S_B, "c": S_C, "s": S_S}


def make_weights(cfg: dict, seed: int, sharp: bool | None = None, alike_experts: bool = False) -> dict:
    """bfloat16 tensors by name: matrices N(0, 1/fan_in) times a gain; norm weights around 1; sinks around the size of
    the scores' maximum, so that they take a share that matters; the maps' vectors wide enough that the factor of the
    second map differs from its offset.  `alike_experts`: as in the Furesun cases (the experts of a layer differ by a
    twentieth of their size only, so that a router's choice that bfloat16 turns moves a row little)."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    def matrix(out, inp, gain=1.0):
        return normal(out, inp, std=gain / inp ** 0.5)

    W, V = cfg["width"], cfg["vocab"]
    sharp = cfg is S_S if sharp is None else sharp
    # (rows with a mean of their own, so that a norm that forgets the mean shows)
    w = {"embed": normal(V, W, std=0.6) + normal(V, 1, std=0.4), "final.norm": normal(W, std=0.2, mean=1.0),
         "head": matrix(V, W, 2.0)}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        w[p + "norm1"] = normal(W, std=0.2, mean=1.0)
        m, q = layer["mixer"], p + "mix."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        gain = 4.0 if sharp else 1.5
        if layer["type"] == "attention":
            G = m["kv_heads"]
            w[q + "q"], w[q + "k"], w[q + "v"] = matrix(H * 2 * d, W, 1.5), matrix(G * 2 * d, W, 1.5), matrix(G * e, W, 1.5)
            w[q + "q.norm"] = normal(d, std=0.3, mean=1.5 if sharp else 1.2)
            w[q + "k.norm"] = normal(d, std=0.3, mean=1.5 if sharp else 1.2)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[q + n] = normal(d, std=0.8 / d ** 0.25)
            w[q + "g"], w[q + "o"] = matrix(H, W, 2.0), matrix(W, H * e)
        else:
            r = m.get("rot_dim", 0)
            n = m["kv_rank"]
            if layer["type"] == "latent_attention":
                w[q + "dq"], w[q + "dq.norm"] = matrix(m["q_rank"], W, 1.5), normal(m["q_rank"], std=0.2, mean=1.0)
                w[q + "uq"] = matrix(H * d, m["q_rank"], gain)
            else:
                w[q + "q"] = matrix(H * (d + r), W, gain)
                w[q + "sink"], w[q + "g"] = normal(H, std=1.5, mean=8.0 if sharp else 2.0), matrix(H, W, 2.0)
            if m.get("kv_from") is None:
                w[q + "dkv"], w[q + "dkv.norm"] = matrix(n + r, W, gain), normal(n, std=0.2, mean=1.0)
            w[q + "uk"], w[q + "uv"] = matrix(H * d, n, gain), matrix(H * e, n, 1.5)
            w[q + "o"] = matrix(W, H * e)
        f = layer["mlp"]
        if f is None:
            continue
        w[p + "norm2"] = normal(W, std=0.2, mean=1.0)
        q = p + "mlp."
        if f["kind"] == "dense":
            w[q + "gate"], w[q + "up"], w[q + "down"] = matrix(f["ff"], W, 1.5), matrix(f["ff"], W, 1.5), matrix(W, f["ff"], 1.5)
            continue
        n, E = f["expert"]["ff"], f["router"]["experts"]
        base = (matrix(n, W, 1.5).float(), matrix(n, W, 1.5).float(), matrix(W, n, 1.5).float())
        for x in range(E):
            own = (matrix(n, W, 1.5), matrix(n, W, 1.5), matrix(W, n, 1.5))
            if alike_experts:
                own = tuple((b + 0.05 * o.float()).to(torch.bfloat16) for b, o in zip(base, own))
            w[f"{q}e{x}.gate"], w[f"{q}e{x}.up"], w[f"{q}e{x}.down"] = own
        w[q + "router"], w[q + "router.b"] = matrix(E, W, 2.0), normal(E, std=1.0)
        if f.get("shared"):
            n = f["shared"]["ff"]
            w[q + "shared.gate"], w[q + "shared.up"], w[q + "shared.down"] = matrix(n, W, 1.5), matrix(n, W, 1.5), matrix(W, n, 1.5)
            w[q + "shared.sg"] = matrix(1, W, 2.0)
    return w


_folders: dict = {}
_wants: dict = {}


def folder(tmp_root, name: str, seed: int = 5, alike_experts: bool = False) -> str:
    key = (name, seed, alike_experts)
    if key not in _folders:
        c = CASES[name]
        _folders[key] = ps.write_folder(os.path.join(str(tmp_root), f"safurax_{name}_{seed}_{int(alike_experts)}"), c,
                                        make_weights(c, seed, alike_experts=alike_experts))
    return _folders[key]


def _bf16(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(t.dtype)


def oracle(path: str, toks: list[int]) -> Want:
    """The oracle's logits at every position and the noise of each row (cached)."""
    key = (path, tuple(toks))
    if key not in _wants:
        cfg, w = ps.read_folder(path)
        margins: list = []
        exact = ps.decoder(cfg, w, toks, torch.float64, margins_out=margins)
        rounded = ps.decoder(cfg, w, toks, torch.float64, rounding=_bf16)
        margin = torch.stack(margins).amin(dim=0) if margins else torch.full((len(toks),), math.inf, dtype=torch.float64)
        _wants[key] = Want(exact, (rounded - exact).abs().amax(dim=1), margin, bool(margins))
    return _wants[key]
