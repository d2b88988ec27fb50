"""Plain, slow implementation of the Gokapel decoder: whole sequences, no
cache, one function per mechanism.  Nothing is imported from the product
package.  All math is done in the dtype asked for (float64 by default: the
anchor the product's float32 and bfloat16 paths are measured against).

Notation: T tokens, W model width, H heads, G key (or key/value) heads, d key
width per head, e value width per head, sigma(z) = 1 / (1 + exp(-z)).

The residual is S streams x_1 .. x_S, all equal to the embedding at the start.
A sublayer f with the tensors in, out, mix (of its connection), norm, gate
matrix R with bias r and scale vector l does, with a constant m of the model:

    u = sum_s in[s] x_s;   h = norm(u);   y = f(h) * l * sigma(R h + r)
    x_t <- sum_s mix[s, t] x_s + m out[t] y        (all t at once)

and the model reads the sum of the streams at the end.
"""
from __future__ import annotations

import math

import torch

from plain_zodosun import read_folder, write_folder  # noqa: F401  (the file format is the same)


# With a rounding function set (decoder(..., rounding=f)) the values that a 16-bit engine rounds are rounded here
# too: what a sublayer reads, q, k and v as the attention takes them, the inner vectors of the two-step projections,
# and what goes into an output or down product.
_rounding = [None]
_margins = [None]        # a list while decoder(..., margins_out=list) runs: per routed layer, each token's router margin


def _r(x):
    return x if _rounding[0] is None else _rounding[0](x)


# --------------------------------------------------------------------------
# mechanisms
# --------------------------------------------------------------------------
def dyt(x, alpha, weight, bias):
    """A norm without statistics: tanh(alpha x) * weight + bias."""
    return torch.tanh(alpha * x) * weight + bias


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(torch.clamp(z, max=30.0))))


def square_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def short_conv(x, taps):
    """y[t, c] = silu(sum_{j<K} taps[c, K-1-j] x[t-j, c]), zeros before the start.  x [T, C], taps [C, K]."""
    T, K = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for j in range(K):
        if j < T:
            y[j:] += x[:T - j] * taps[:, K - 1 - j]
    return silu(y)


def unit(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last dimension."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, g, beta):
    """Per head a d x e matrix S, zero at first:  S <- g * S (row i of S by g_i);  u = beta (v - S^T k);
    S <- S + k u^T;  o = S^T q.  q, k [T, G, d]; v [T, H, e]; g [T, H, d]; beta [T, H].  Returns [T, H, e]."""
    T, H, e = v.shape
    G, d = q.shape[1], q.shape[2]
    out = torch.zeros((T, H, e), dtype=v.dtype)
    for h in range(H):
        n = h // (H // G)
        S = torch.zeros((d, e), dtype=v.dtype)
        for t in range(T):
            S = g[t, h].reshape(d, 1) * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, n])
            S = S + k[t, n].reshape(d, 1) * u.reshape(1, e)
            out[t, h] = S.T @ q[t, n]
    return out


def channel_delta(x, w, p, c, eps):
    """Delta rule with a decay per head and key channel, convolved q, k, v, a low-rank output gate."""
    T = x.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (short_conv(x @ w[p + n].T, w[p + n + ".conv"]) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, d)) * d ** -0.5
    k = unit(k.reshape(T, G, d))
    beta = torch.sigmoid(x @ w[p + "b"].T)
    z = _r(x @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    g = torch.exp(-torch.exp(w[p + "A_log"]).reshape(1, H, 1) * softplus(z).reshape(T, H, d))
    o = rms(delta_scan(q, k, v.reshape(T, H, e), g, beta), eps) * w[p + "norm"]
    o = o.reshape(T, H * e) * torch.sigmoid(_r(x @ w[p + "g1"].T) @ w[p + "g2"].T)
    return _r(o) @ w[p + "o"].T


def rotate(x, positions, dims: int, base: float):
    """x [T, heads, n]: of the first `dims` entries of every head the neighbours (a, b) = (2i, 2i + 1) become
    (a cos t - b sin t, b cos t + a sin t), t = position * base^(-2i / dims).  The other entries pass."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / dims)
    ang = positions.to(torch.float64).reshape(-1, 1, 1) * f
    c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
    out = x.clone()
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def visible(T: int, chunk):
    """[T, T] bool: i reads j iff j <= i and both lie in the same chunk of `chunk` positions (None: every j <= i)."""
    i = torch.arange(T).reshape(-1, 1)
    j = torch.arange(T).reshape(1, -1)
    ok = j <= i
    if chunk:
        ok = ok & (i // chunk == j // chunk)
    return ok


def softmax_heads(q, k, v, scale, mask, sinks):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e].  Scores q . k * scale; weights
    exp(s_j) / (exp(sink_h) + sum exp(s))."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(~mask, -math.inf)
        m = torch.clamp(s.max(dim=-1, keepdim=True).values, min=float(sinks[h]))
        p = torch.exp(s - m)
        out[:, h] = (p / (p.sum(dim=-1, keepdim=True) + torch.exp(sinks[h] - m))) @ v[:, g]
    return out


def attention(x, w, p, c, positions, eps):
    """Grouped softmax attention in chunks: q and k normed head by head (weights shared by the heads), then turned
    in neighbouring pairs; a learned sink per head; W_o."""
    T = x.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    rot = c["rot"]
    q = rms((x @ w[p + "q"].T).reshape(T, H, d), eps) * w[p + "q.norm"]
    k = rms((x @ w[p + "k"].T).reshape(T, G, d), eps) * w[p + "k.norm"]
    q, k = rotate(q, positions, rot["dims"], rot["base"]), rotate(k, positions, rot["dims"], rot["base"])
    v = (x @ w[p + "v"].T).reshape(T, G, e)
    o = softmax_heads(_r(q), _r(k), _r(v), c["scale"], visible(T, (c.get("mask") or {}).get("size")), w[p + "sink"])
    return _r(o.reshape(T, H * e)) @ w[p + "o"].T


def gru_scan(z, cand):
    """S_t = (1 - z_t) S_{t-1} + z_t cand_t, S zero at first."""
    S = torch.zeros_like(z[0])
    out = torch.zeros_like(z)
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        out[t] = S
    return out


def min_gru(x, w, p):
    """One number of memory per channel, an update gate that does not look at it: z = sigma(W_z x + b_z), u = W_x x + b_x, the candidate
    is u + 1/2 for u >= 0 and sigma(u) below; result W_o (S * silu(W_g x))."""
    z = torch.sigmoid(x @ w[p + "z"].T + w[p + "z.b"])
    u = x @ w[p + "x"].T + w[p + "x.b"]
    s = gru_scan(z, torch.where(u >= 0, u + 0.5, torch.sigmoid(u)))
    return _r(s * silu(x @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(x, w, p, c, positions, eps):
    return (float(c["left_scale"]) * attention(x, w, p + "left.", c["left"], positions, eps)
            + float(c["right_scale"]) * min_gru(x, w, p + "right."))


def plain_ff(x, w, p):
    return _r(square_relu(x @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, top, count, keep):
    """Scores s = softmax(z); the choice goes by s + correction: the experts lie in `count` equal groups of
    neighbours, a group's score is the largest in it, only the `keep` best groups' experts can be chosen, of
    those the `top` best.  Returns indices [T, top], the chosen experts' s and each token's margin: how far the
    decision that was closest (between groups, or between experts) lies from turning."""
    s = torch.softmax(z, dim=-1)
    T, E = z.shape
    choice = s + correction
    per = E // count
    gs = choice.reshape(T, count, per).amax(dim=-1)
    order = torch.argsort(gs, dim=-1, descending=True, stable=True)
    allowed = torch.zeros((T, count), dtype=torch.bool)
    allowed.scatter_(1, order[:, :keep], True)
    masked = choice.masked_fill(~allowed.repeat_interleave(per, dim=1), -math.inf)
    idx = torch.argsort(masked, dim=-1, descending=True, stable=True)
    inf = torch.full((T,), math.inf, dtype=z.dtype)
    ms = torch.gather(masked, 1, idx)
    margin = ms[:, top - 1] - ms[:, top] if top < E else inf
    if keep < count:
        sg = torch.gather(gs, 1, order)
        margin = torch.minimum(margin, sg[:, keep - 1] - sg[:, keep])
    return idx[:, :top], torch.gather(s, 1, idx[:, :top]), margin


def routed_ff(x, w, p, c):
    r = c["router"]
    gr = r.get("groups") or {"count": 1, "keep": 1}
    idx, wts, margin = route(x @ w[p + "router"].T, w[p + "correction"], r["top"], gr["count"], gr["keep"])
    if _margins[0] is not None:
        _margins[0].append(margin)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(r["top"]):
            out[t] += wts[t, j] * plain_ff(x[t:t + 1], w, f"{p}e{int(idx[t, j])}.")[0]
    if c.get("shared"):
        out = out + plain_ff(x, w, p + "shared.")
    return out


def feed_forward(x, w, p, c):
    return plain_ff(x, w, p) if c["kind"] == "dense" else routed_ff(x, w, p, c)


def connect(xs, w, p, q: int, m: float, f):
    """One sublayer on the streams xs (a list): see the top of the file."""
    hc = f"{p}hc{q}."
    u = sum(w[hc + "in"][s] * xs[s] for s in range(len(xs)))
    n = f"{p}norm{q}"
    h = _r(dyt(u, w[n + ".alpha"], w[n], w[n + ".b"]))
    y = f(h) * w[f"{p}ls{q}"] * torch.sigmoid(h @ w[f"{p}rg{q}"].T + w[f"{p}rg{q}.b"])
    mix, out = w[hc + "mix"], w[hc + "out"]
    return [sum(mix[s, t] * xs[s] for s in range(len(xs))) + m * out[t] * y for t in range(len(xs))]


# --------------------------------------------------------------------------
# the decoder
# --------------------------------------------------------------------------
def decoder(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float64, layers_out=None, rounding=None,
            margins_out=None):
    """Logits [T, vocab] of a whole sequence.  `layers_out` (a list) receives the streams' sum after every layer.
    `rounding`: a function applied where a 16-bit engine rounds its activations.  `margins_out` (a list) receives,
    per routed feed-forward, each token's router margin (`route`): a small one is a choice that rounding can turn."""
    _rounding[0], _margins[0] = rounding, margins_out
    try:
        return _decoder(cfg, weights, tokens, dtype, layers_out)
    finally:
        _rounding[0] = _margins[0] = None


def _decoder(cfg, weights, tokens, dtype, layers_out):
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps, m = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    positions = torch.arange(len(tokens))
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    xs = [x.clone() for _ in range(int(cfg["streams"]))]
    for i, layer in enumerate(cfg["layers"]):
        i = i if layer.get("weights_of") is None else int(layer["weights_of"])      # another layer's tensors
        p, c = f"l{i}.", layer["mixer"]
        if layer["type"] == "channel_delta":
            xs = connect(xs, w, p, 1, m, lambda h: channel_delta(h, w, p + "mix.", c, eps))
        elif layer["type"] == "parallel":
            xs = connect(xs, w, p, 1, m, lambda h: parallel(h, w, p + "mix.", c, positions, eps))
        else:
            raise ValueError(f"unknown layer type {layer['type']}")
        if layer.get("mlp") is not None:
            xs = connect(xs, w, p, 2, m, lambda h: feed_forward(h, w, p + "mlp.", layer["mlp"]))
        if layers_out is not None:
            layers_out.append(sum(xs).clone())
    n = "final.norm"
    return _r(dyt(sum(xs), w[n + ".alpha"], w[n], w[n + ".b"])) @ w["embed"].T


def greedy(cfg: dict, weights: dict, prompt: list[int], n: int, dtype=torch.float64) -> list[int]:
    """n tokens after the prompt, each the arg-max (lowest id on a tie) of the logits of all tokens before it."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(decoder(cfg, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
