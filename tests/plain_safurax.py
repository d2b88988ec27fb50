"""Plain, slow implementation of the Safurax decoder: whole sequences, no
cache, one function per mechanism.  Nothing is imported from the product
package.  All math is done in the dtype asked for (float64 by default: the
anchor the product's float32 and bfloat16 paths are measured against).

Notation: T tokens, W model width, H query heads, G key/value heads, d key
width per head, e value width per head, sigma(z) = 1 / (1 + exp(-z)).
Position i may read position j <= i (with a window: i - j < window).

A layer is  x <- x + mixer(norm1(x));  x <- x + ff(norm2(x)),  the norms with
the mean taken off.
"""
from __future__ import annotations

import math

import torch

from plain_zodosun import read_folder, write_folder  # noqa: F401  (the file format is the same)


# With a rounding function set (decoder(..., rounding=f)) the values that a 16-bit engine rounds are rounded here
# too: what a sublayer reads, latents, q, k and v as the attention takes them, and what goes into an output or down
# product.
_rounding = [None]
_margins = [None]        # a list while decoder(..., margins_out=list) runs: per routed layer, each token's router margin


def _r(x):
    return x if _rounding[0] is None else _rounding[0](x)


# --------------------------------------------------------------------------
# mechanisms
# --------------------------------------------------------------------------
def layer_norm(x, weight, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * weight over the last dimension."""
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * weight


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def rotate(x, positions, dims: int, base: float, factor: float = 1.0):
    """x [T, heads, n]: entry i < dims/2 of every head is paired with entry i + dims/2; the pair (a, b) at position p
    turns by t = p * base^(-2i/dims) / factor into (a cos t - b sin t, b cos t + a sin t).  Entries from `dims` on
    pass."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    rate = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / dims) / factor
    ang = positions.to(torch.float64).reshape(-1, 1, 1) * rate
    c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
    out = x.clone()
    a, b = x[..., :half], x[..., half:dims]
    out[..., :half] = a * c - b * s
    out[..., half:dims] = b * c + a * s
    return out


def rot_args(c: dict):
    rot = c["rot"]
    return rot["dims"], rot["base"], float((rot.get("scaling") or {}).get("factor", 1.0))


def visible(T: int, window=None):
    """[T, T] bool: i reads j iff 0 <= i - j < window (no window: every j <= i)."""
    i = torch.arange(T).reshape(-1, 1)
    j = torch.arange(T).reshape(1, -1)
    ok = j <= i
    if window:
        ok = ok & (i - j < window)
    return ok


def softmax_head(q, k, v, scale, mask, sink=None):
    """One head: q [T, d], k [T, d], v [T, e] -> [T, e].  Weights exp(s_j) / (sum exp(s) [+ exp(sink): a key of
    that score that has no value]), s = q . k * scale over the visible keys."""
    s = ((q @ k.T) * scale).masked_fill(~mask, -math.inf)
    m = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        m = torch.clamp(m, min=float(sink))
    p = torch.exp(s - m)
    den = p.sum(dim=-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - m)
    return (p / den) @ v


def head_gate(o, x, w_g):
    """o [T, H, e] times sigma(W_g x) [T, H], one number per head."""
    return o * torch.sigmoid(x @ w_g.T).unsqueeze(-1)


def latent_of(x, w, p, c, positions, eps):
    """What a latent mixer caches: c = rms_norm of the first kv_rank rows of W_dkv x, and the other rot_dim rows
    turned (empty without a rotated part)."""
    n, r = c["kv_rank"], int(c.get("rot_dim") or 0)
    dkv = x @ w[p + "dkv"].T
    lat = rms_norm(dkv[:, :n], w[p + "dkv.norm"], eps)
    k_r = dkv[:, n:].reshape(x.shape[0], 1, r)
    if r:
        k_r = rotate(k_r, positions, *rot_args(c))
    return _r(lat), _r(k_r)


def latent_heads(q, lat, k_r, w, p, c, sinks=None):
    """q [T, H, d + r] (rotated part turned already) over the latents of one sequence: key_h = [U_k[h] c, k_r],
    value_h = U_v[h] c; softmax; [T, H, e]."""
    T = q.shape[0]
    H, d, e = c["heads"], c["dim"], c["vdim"]
    r = k_r.shape[-1]
    k_flat = _r(lat @ w[p + "uk"].T).reshape(T, H, d)
    val = _r(lat @ w[p + "uv"].T).reshape(T, H, e)
    mask = visible(T, (c.get("mask") or {}).get("size"))
    out = torch.zeros((T, H, e), dtype=q.dtype)
    for h in range(H):
        k = torch.cat([k_flat[:, h], k_r.reshape(T, r)], dim=-1)
        out[:, h] = softmax_head(_r(q[:, h]), k, val[:, h], c["scale"], mask, None if sinks is None else sinks[h])
    return out


def latent_attention(x, w, p, c, positions, eps):
    """Queries through a latent of their own, q = W_uq rms_norm(W_dq x); no positions; causal; W_o."""
    T, H, e = x.shape[0], c["heads"], c["vdim"]
    cq = _r(rms_norm(x @ w[p + "dq"].T, w[p + "dq.norm"], eps))
    q = (cq @ w[p + "uq"].T).reshape(T, H, c["dim"])
    lat, k_r = latent_of(x, w, p, c, positions, eps)
    o = latent_heads(q, lat, k_r, w, p, c)
    return _r(o.reshape(T, H * e)) @ w[p + "o"].T


def latent_attention_2(x, w, p, c, positions, eps, cached=None):
    """Queries projected directly, head by head [d plain | r turned]; a window, a sink, a gate per head; W_o.
    `cached`: another layer's latent and turned key part stand in for this layer's."""
    T = x.shape[0]
    H, d, r, e = c["heads"], c["dim"], c["rot_dim"], c["vdim"]
    q = (x @ w[p + "q"].T).reshape(T, H, d + r)
    q = torch.cat([q[..., :d], rotate(q[..., d:], positions, *rot_args(c))], dim=-1)
    lat, k_r = cached if cached is not None else latent_of(x, w, p, c, positions, eps)
    o = head_gate(latent_heads(q, lat, k_r, w, p, c, w[p + "sink"]), x, w[p + "g"])
    return _r(o.reshape(T, H * e)) @ w[p + "o"].T


def difference_factor(w, p, diff):
    """exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number for the layer."""
    return (torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff)


def differential_attention(x, w, p, c, positions, eps):
    """Two attention maps per head over the same values; head h reads key/value head h // (H / G).  q and k of each
    map: rms_norm over d with a weight that heads and maps share, then turned.  o = a1 - lambda a2, over its root mean
    square, times 1 - diff, times the head's gate; W_o."""
    T = x.shape[0]
    H, G, d, e = c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = (x @ w[p + "q"].T).reshape(T, H * 2, d)
    k = (x @ w[p + "k"].T).reshape(T, G * 2, d)
    v = _r((x @ w[p + "v"].T).reshape(T, G, e))
    q = _r(rotate(rms_norm(q, w[p + "q.norm"], eps), positions, *rot_args(c))).reshape(T, H, 2, d)
    k = _r(rotate(rms_norm(k, w[p + "k.norm"], eps), positions, *rot_args(c))).reshape(T, G, 2, d)
    lam = difference_factor(w, p, c["diff"])
    mask = visible(T)
    o = torch.zeros((T, H, e), dtype=x.dtype)
    for h in range(H):
        g = h // (H // G)
        a1, a2 = (softmax_head(q[:, h, m], k[:, g, m], v[:, g], c["scale"], mask) for m in (0, 1))
        o[:, h] = a1 - lam * a2
    o = head_gate(rms(o, eps) * (1.0 - c["diff"]), x, w[p + "g"])
    return _r(o.reshape(T, H * e)) @ w[p + "o"].T


def gated_ff(x, w, p):
    return _r(silu(x @ w[p + "gate"].T) * (x @ w[p + "up"].T)) @ w[p + "down"].T


def routed_ff(x, w, p, c):
    """Logits z = W_router x + b; the `top` largest are chosen, their softmax weighs the chosen experts' results.  A
    shared expert runs for every token, times sigma(W_sg x)."""
    top = c["router"]["top"]
    z = x @ w[p + "router"].T + w[p + "router.b"]
    val, idx = torch.topk(z, top, dim=-1)
    if _margins[0] is not None:
        # how far the last chosen logit lies above the first one left out, relative to the logits' root mean square
        zs = torch.sort(z, dim=-1, descending=True).values
        gap = zs[:, top - 1] - zs[:, top] if top < z.shape[1] else torch.full_like(zs[:, 0], math.inf)
        _margins[0].append(gap / (torch.sqrt((z * z).mean(dim=-1)) + 1e-9))
    wts = torch.softmax(val, dim=-1)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(top):
            out[t] += wts[t, j] * gated_ff(x[t:t + 1], w, f"{p}e{int(idx[t, j])}.")[0]
    if c.get("shared"):
        out = out + gated_ff(x, w, p + "shared.") * torch.sigmoid(x @ w[p + "shared.sg"].T)
    return out


def feed_forward(x, w, p, c):
    return gated_ff(x, w, p) if c["kind"] == "dense" else routed_ff(x, w, p, c)


# --------------------------------------------------------------------------
# the decoder
# --------------------------------------------------------------------------
def decoder(cfg: dict, weights: dict, tokens: list[int], dtype=torch.float64, layers_out=None, rounding=None,
            margins_out=None):
    """Logits [T, vocab] of a whole sequence.  `layers_out` (a list) receives the stream after every layer.
    `rounding`: a function applied where a 16-bit engine rounds its activations.  `margins_out` (a list) receives,
    per routed feed-forward, each token's router margin: the gap between the last chosen logit and the first one
    left out over the root mean square of the token's logits; a small margin is a choice that rounding can turn."""
    _rounding[0], _margins[0] = rounding, margins_out
    try:
        return _decoder(cfg, weights, tokens, dtype, layers_out)
    finally:
        _rounding[0] = _margins[0] = None


def _decoder(cfg, weights, tokens, dtype, layers_out):
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
    eps = float(cfg["norm"]["eps"])
    positions = torch.arange(len(tokens))
    x = w["embed"][torch.tensor(tokens, dtype=torch.long)] * float(cfg["embedding"]["scale"])
    kept: dict[int, tuple] = {}
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{i}.mix.", layer["mixer"]
        n = _r(layer_norm(x, w[f"l{i}.norm1"], eps))
        if layer["type"] == "latent_attention":
            y = latent_attention(n, w, p, c, positions, eps)
        elif layer["type"] == "latent_attention_2":
            if c.get("kv_from") is None:
                kept[i] = latent_of(n, w, p, c, positions, eps)
            y = latent_attention_2(n, w, p, c, positions, eps, kept[i if c.get("kv_from") is None else int(c["kv_from"])])
        elif layer["type"] == "attention":
            y = differential_attention(n, w, p, c, positions, eps)
        else:
            raise ValueError(f"unknown layer type {layer['type']}")
        x = x + y
        if layer.get("mlp") is not None:
            x = x + feed_forward(_r(layer_norm(x, w[f"l{i}.norm2"], eps)), w, f"l{i}.mlp.", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return _r(layer_norm(x, w["final.norm"], eps)) @ w["head"].T


def greedy(cfg: dict, weights: dict, prompt: list[int], n: int, dtype=torch.float64) -> list[int]:
    """n tokens after the prompt, each the arg-max (lowest id on a tie) of the logits of all tokens before it."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(torch.argmax(decoder(cfg, weights, toks, dtype)[-1])))
    return toks[len(prompt):]
