"""Plain statement of the Sapanex decoder: 64-bit, whole sequences, one function per mechanism.

Written from the design's equations and sharing no code with the engine.  `w` maps tensor names to
64-bit tensors, `cfg` is the parsed config.json.  Notation: T tokens, width W, residual multiplier A.

  norm          n(x) = x / sqrt(mean(x^2) + eps) * g
  layer         x <- n1(A x + mixer(x));  x <- n2(A x + ff(x))      (ff may be absent)
  rotation      pairs (i, i + d/2) of the first d elements of a head turned by p f_i, f_i = base^(-2i/d); with
                scaling, f_i is blended between f_i (fast pairs) and f_i / factor (slow pairs) along a ramp over the
                pair's number, and the turned pair is stretched by 0.1 ln(factor) + 1
  attention     q, k normed over all heads' rows at once, then turned; values turned over their whole size (no
                scaling); score q.k * scale over the last `size` tokens and over the means of aligned blocks of
                `pool` tokens that lie wholly before them; one softmax; the sum of values turned back; O
  delta rule    S_t = diag(w) S_{t-1} - (a u)(u^T S_{t-1}) + k v^T; o = S_t^T r per head; o / rms(o); times a weight
                and sigmoid(G x); O
  dense ff      Dn relu(Up x)^2
  output        E n(x), E the token table without its multiplier
"""
from __future__ import annotations

import math

import torch

UNIT_EPS = 1e-6           # what joins the sum of squares under a unit key's root
LOG_DECAY = math.exp(-0.5)


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(base, dims, scaling=None):
    """Angular frequencies of the pairs and what cos and sin are multiplied by."""
    f = [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor = float(scaling["factor"])

    def place(turns):                  # the (fractional) pair number whose wave turns that often over the original length
        return dims * math.log(float(scaling["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))

    lo = max(math.floor(place(float(scaling["fast"]))), 0)
    hi = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def turn(x, positions, freq, stretch=1.0, sign=1.0):
    """x [T, heads, size]: the first 2 * len(freq) elements of each head are turned, pairs (i, i + len(freq))."""
    n = freq.numel()
    ang = sign * positions.to(torch.float64)[:, None] * freq[None, :]
    c, s = (torch.cos(ang) * stretch)[:, None, :], (torch.sin(ang) * stretch)[:, None, :]
    u, v = x[..., :n], x[..., n: 2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], dim=-1)


def block_means(x, pool):
    """x [T, heads, size] -> [T // pool, heads, size]: means of the complete blocks."""
    n = x.shape[0] // pool
    return x[: n * pool].reshape(n, pool, *x.shape[1:]).mean(1)


def visible(T, size, pool):
    """(tokens [T, T], blocks [T, T // pool]) booleans: what position i sees."""
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    b = torch.arange(T // pool)[None, :]
    return (j <= i) & (i - j < size), b * pool + pool - 1 <= i - size


def pooled_window_attention(q, k, v, scale, size, pool):
    """q [T, H, d], k [T, G, d], v [T, G, dv] (normed, turned): the sum of values [T, H, dv].  `size` None: every earlier token."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    if size is None:
        tok, blk = torch.tril(torch.ones(T, T, dtype=torch.bool)), torch.zeros(T, 0, dtype=torch.bool)
        kb, vb = k[:0], v[:0]
    else:
        tok, blk = visible(T, size, pool)
        kb, vb = block_means(k, pool), block_means(v, pool)
    seen = torch.cat([tok, blk], dim=1)
    keys, values = torch.cat([k, kb]), torch.cat([v, vb])
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ keys[:, g].T) * scale
        out[:, h] = torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ values[:, g]
    return out


def attention(w, p, m, h, eps):
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    positions = torch.arange(T)
    q = (rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"]).view(T, H, d)
    k = (rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"]).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    rot = m.get("rot")
    if rot is not None:
        freq, stretch = frequencies(rot["base"], int(rot["dims"]), rot.get("scaling"))
        vfreq, _ = frequencies(rot["base"], dv)
        q, k = turn(q, positions, freq, stretch), turn(k, positions, freq, stretch)
        v = turn(v, positions, vfreq)
    mask = m.get("mask")
    o = pooled_window_attention(q, k, v, float(m["scale"]), None if mask is None else int(mask["size"]),
                                None if mask is None else int(mask["pool"]))
    if rot is not None:
        o = turn(o, positions, vfreq, sign=-1.0)
    return o.reshape(T, H * dv) @ w[p + "o"].T


def delta_rule(decay, removal, k, v, r, state=None):
    """decay, removal, k, r [T, H, d], v [T, H, dv] -> (o [T, H, dv], state [H, d, dv])."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[2], dtype=k.dtype) if state is None else state.clone()
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + UNIT_EPS)
    out = torch.zeros(T, H, v.shape[2], dtype=k.dtype)
    for t in range(T):
        read = torch.einsum("hd,hde->he", u[t], S)
        S = decay[t][:, :, None] * S - (removal[t] * u[t])[:, :, None] * read[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hd,hde->he", r[t], S)
    return out, S


def general_delta(w, p, m, h, eps):
    T, H, d = h.shape[0], int(m["heads"]), int(m["dim"])
    heads = lambda x: x.view(T, H, d)
    r, k, v = heads(h @ w[p + "r"].T), heads(h @ w[p + "k"].T), heads(h @ w[p + "v"].T)
    decay = torch.exp(-LOG_DECAY * torch.sigmoid(torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))
    removal = torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"])
    o, _ = delta_rule(heads(decay), heads(removal), k, v, r)
    o = rms(o, eps).reshape(T, H * d) * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def dense_ff(w, p, h):
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def forward(w, cfg, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; `layers_out` collects the stream after every layer."""
    eps, A = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    x = w["embed"][torch.tensor(tokens)] * float(cfg["embedding"]["scale"])
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        mixer = attention if layer["type"] == "attention" else general_delta
        x = rms(A * x + mixer(w, p + "mix.", layer["mixer"], x, eps), eps) * w[p + "norm1"]
        if layer.get("mlp"):
            x = rms(A * x + dense_ff(w, p + "mlp.", x), eps) * w[p + "norm2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps) * w["final.norm"] @ w["embed"].T
