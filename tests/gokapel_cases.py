"""Small Gokapel configurations, weights with a spread that lets every mechanism matter, and the plain implementation
as oracle (cached).  Rows are compared as for the Furesun decoder (furesun_cases.Want, check_rows)."""
from __future__ import annotations

import math
import os

import torch

import plain_gokapel as pg
from furesun_cases import Want, check_rows, tokens  # noqa: F401


def delta(heads, kv, dim, vdim, conv):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def both(heads, kv, dim, vdim, chunk, scale, width, left=1.0, right=1.0, dims=None, base=10000.0):
    """A `parallel` layer: attention of these sizes beside a minGRU of `width` channels."""
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
         "rot": {"base": base, "dims": dim if dims is None else dims}}
    if chunk:
        m["mask"] = {"size": chunk}
    return {"type": "parallel", "mixer": {"left": m, "left_scale": left, "right": {"width": width}, "right_scale": right}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, shared=None):
    d = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    d["router"]["groups"] = {"count": groups[0], "keep": groups[1]} if groups else {"count": 1, "keep": 1}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def model(vocab, width, eps, streams, mult, scale, layers):
    return {"architecture": "Gokapel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "residual_mult": mult, "embedding": {"scale": scale}, "layers": layers}


# A: sizes that are no multiples of 8 or 4, several heads on one key head in both mixers, three streams, three groups
#    of which two take part, both kinds of layer run once more with another's tensors, a layer without a feed-forward.
G_A = model(300, 96, 1e-6, 3, 0.8, 3.0, [
    {**both(6, 2, 20, 12, 33, 0.3, 58, 0.7, 1.3, dims=10, base=5000.0), "mlp": moe(40, 6, 3, (3, 2), shared=56)},
    {**delta(6, 2, 20, 12, 3), "mlp": dense(136)},
    {**both(6, 2, 20, 12, 33, 0.3, 58, 0.7, 1.3, dims=10, base=5000.0), "mlp": moe(40, 6, 3, (3, 2), shared=56), "weights_of": 0},
    {**delta(6, 2, 20, 12, 3), "mlp": dense(136), "weights_of": 1},
    {**delta(3, 3, 18, 30, 5), "mlp": None},
])
# B: sizes that the tensor-core kernels take (heads of 64 and 128, inner widths from 64 on), chunks of whole pages and
#    one off, two streams, groups of two.
G_B = model(384, 160, 1e-6, 2, 0.6, 2.0, [
    {**delta(4, 2, 64, 64, 4), "mlp": moe(96, 8, 2, (4, 2), shared=64)},
    {**both(4, 2, 64, 64, 128, 0.15, 160, 0.9, 0.6), "mlp": dense(256)},
    {**both(2, 1, 128, 128, 65, 0.1, 96, 1.2, 0.8, base=50000.0), "mlp": moe(64, 12, 3, (2, 1))},
    {**delta(4, 2, 64, 64, 4), "mlp": moe(96, 8, 2, (4, 2), shared=64), "weights_of": 0},
    {**delta(1, 1, 128, 128, 2), "mlp": None},
    {**both(4, 4, 32, 32, None, 0.2, 128, 1.0, 1.0, dims=16), "mlp": dense(96)},
])
# C: one stream, a width that is no multiple of 8, a convolution of one tap, chunks of 1 and 2 positions, no mask, one
#    expert in all and as many per token as there are, a negative factor on a branch, factors of 1.
G_C = model(130, 84, 1e-5, 1, 1.0, 1.0, [
    {**both(1, 1, 24, 16, 1, 0.4, 30, 1.0, -0.5, dims=2), "mlp": moe(50, 1, 1)},
    {**delta(2, 1, 12, 36, 1), "mlp": moe(36, 3, 3, shared=20)},
    {**both(2, 2, 40, 24, 2, 0.25, 17, dims=20), "mlp": dense(50)},
    {**both(3, 1, 16, 8, None, 0.5, 84), "mlp": None},
    {**delta(1, 1, 8, 8, 7), "mlp": dense(44)},
])
# S: softmaxes that are sharp (a large scale on large keys): a single key, far back in its chunk or at the chunk's
#    edge, decides a row's result, or the sink takes it.
G_S = model(150, 64, 1e-5, 2, 0.7, 2.0, [
    {**both(2, 1, 32, 32, 90, 1.5, 16, 1.0, 0.3), "mlp": None},
    {**delta(2, 2, 16, 16, 4), "mlp": None},
    {**both(4, 2, 16, 16, 300, 1.5, 16, 1.0, 0.3), "mlp": None},
])
CASES = {"a": G_A, "b": G_B, "c": G_C, "s": G_S}
RANKS = (10, 14)                 # inner widths of the two-step projections, unless a weight set asks for others


def make_weights(cfg: dict, seed: int, sharp: bool | None = None, alike_experts: bool = False, ranks=None) -> dict:
    """bfloat16 tensors by name.  Matrices N(0, 1/fan_in) times a gain; decays spread from nearly one to nearly zero;
    corrections of both signs; sinks around the scores.  `alike_experts` as in furesun_cases.make_weights: experts
    that differ by a twentieth, so that a choice that bfloat16 turns moves a row by less than rounding does."""
    g = torch.Generator().manual_seed(seed)

    def normal(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    def matrix(out, inp, gain=1.0):
        return normal(out, inp, std=gain / inp ** 0.5)

    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    sharp = cfg is G_S if sharp is None else sharp
    if ranks is None:
        ranks = (64, 72) if cfg is G_B else RANKS

    def norm(name):
        return {name: normal(W, std=0.2, mean=1.0), name + ".b": normal(W, std=0.1),
                name + ".alpha": normal(1, std=0.1, mean=0.6).reshape(())}

    w = {"embed": normal(V, W, std=0.4), **norm("final.norm")}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p = f"l{i}."
        for q in (1, 2) if layer["mlp"] is not None else (1,):
            w.update(norm(f"{p}norm{q}"))
            w[f"{p}ls{q}"] = normal(W, std=0.3, mean=1.0)
            w[f"{p}rg{q}"], w[f"{p}rg{q}.b"] = matrix(W, W, 1.5), normal(W, std=0.5, mean=0.5)
            w[f"{p}hc{q}.in"] = normal(S, std=0.3, mean=1.0 / S)
            w[f"{p}hc{q}.out"] = normal(S, std=0.3, mean=1.0)
            w[f"{p}hc{q}.mix"] = (torch.eye(S) + torch.randn(S, S, generator=g) * 0.2).to(torch.bfloat16)
        m, q = layer["mixer"], p + "mix."
        if layer["type"] == "channel_delta":
            H, G, d, e, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                w[q + n] = matrix(rows, W, 1.5)
                w[q + n + ".conv"] = normal(rows, K, std=0.3) + torch.cat([torch.zeros(rows, K - 1), torch.ones(rows, 1)], 1).to(torch.bfloat16)
            w[q + "b"], w[q + "A_log"] = matrix(H, W, 2.0), normal(H, std=1.0, mean=-1.0)
            w[q + "a1"], w[q + "a2"] = matrix(ranks[0], W, 1.5), matrix(H * d, ranks[0], 2.0)
            w[q + "dt_bias"] = normal(H * d, std=2.0, mean=-2.0)
            w[q + "g1"], w[q + "g2"] = matrix(ranks[1], W, 1.5), matrix(H * e, ranks[1], 2.0)
            w[q + "norm"], w[q + "o"] = normal(e, std=0.2, mean=1.0), matrix(W, H * e)
        else:
            a, n = m["left"], m["right"]["width"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            w[q + "left.q"], w[q + "left.k"], w[q + "left.v"] = matrix(H * d, W, 1.5), matrix(G * d, W, 1.5), matrix(G * e, W, 1.5)
            w[q + "left.q.norm"] = normal(d, std=0.3, mean=2.0 if sharp else 1.2)
            w[q + "left.k.norm"] = normal(d, std=0.3, mean=2.0 if sharp else 1.2)
            w[q + "left.sink"] = normal(H, std=1.5, mean=8.0 if sharp else 1.0)
            w[q + "left.o"] = matrix(W, H * e, 1.5)
            for t in ("z", "x", "g"):
                w[f"{q}right.{t}"] = matrix(n, W, 1.5)
            w[q + "right.z.b"], w[q + "right.x.b"] = normal(n, std=1.5, mean=-1.5), normal(n, std=0.5)
            w[q + "right.o"] = matrix(W, n)
        f = layer["mlp"]
        if f is None:
            continue
        q = p + "mlp."
        if f["kind"] == "dense":
            w[q + "up"], w[q + "down"] = matrix(f["ff"], W, 1.5), matrix(W, f["ff"])
            continue
        n, E = f["expert"]["ff"], f["router"]["experts"]
        base = (matrix(n, W, 1.5).float(), matrix(W, n).float())
        for x in range(E):
            own = (matrix(n, W, 1.5), matrix(W, n))
            if alike_experts:
                own = tuple((b + 0.05 * o.float()).to(torch.bfloat16) for b, o in zip(base, own))
            w[f"{q}e{x}.up"], w[f"{q}e{x}.down"] = own
        w[q + "router"], w[q + "correction"] = matrix(E, W, 3.0), normal(E, std=0.3, mean=-0.2)
        if f.get("shared"):
            n = f["shared"]["ff"]
            w[q + "shared.up"], w[q + "shared.down"] = matrix(n, W, 1.5), matrix(W, n)
    return w


_folders: dict = {}
_wants: dict = {}
MARGIN_UNIT = 4.0         # a margin of a router here is a difference of probabilities; check_rows' bound is for logits


def folder(tmp_root, name: str, seed: int = 5, alike_experts: bool = False) -> str:
    key = (name, seed, alike_experts)
    if key not in _folders:
        c = CASES[name]
        _folders[key] = pg.write_folder(os.path.join(str(tmp_root), f"gokapel_{name}_{seed}_{int(alike_experts)}"), c,
                                        make_weights(c, seed, alike_experts=alike_experts))
    return _folders[key]


def _bf16(t: torch.Tensor) -> torch.Tensor:
    return t.to(torch.bfloat16).to(t.dtype)


def oracle(path: str, toks: list[int]) -> Want:
    """The oracle's logits at every position and the noise of each row (cached)."""
    key = (path, tuple(toks))
    if key not in _wants:
        cfg, w = pg.read_folder(path)
        margins: list = []
        exact = pg.decoder(cfg, w, toks, torch.float64, margins_out=margins)
        rounded = pg.decoder(cfg, w, toks, torch.float64, rounding=_bf16)
        margin = torch.full((len(toks),), math.inf, dtype=torch.float64)
        if margins:
            margin = torch.stack(margins).amin(dim=0) * MARGIN_UNIT
        _wants[key] = Want(exact, (rounded - exact).abs().amax(dim=1), margin, bool(margins))
    return _wants[key]
