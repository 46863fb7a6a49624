"""Plain statement of the Tamovik decoder: 64-bit, whole sequences, one function per mechanism.

Written from the design's equations and sharing no code with the engine.  `w` maps tensor names to 64-bit tensors,
`cfg` is the parsed config.json.  rms(x) = x / sqrt(mean(x^2) + eps) over the last dimension.

  embedding     E[tok] + B[(tok_before * mul_prev + tok * mul_cur) mod buckets]; B's last row for the first token
  layer         x <- x + n1(mixer(x));  x <- x + n2(ff(x));  n = rms times a weight
  latent        q = Wq h (head: [plain | turned]);  W_dkv h = [c | r], c <- rms(c) g, r turned, one r for all heads
                s_ij = scale (qp_i . Uk c_j + qr_i . r_j), j <= i; softmax; values Uv c; O
  rotation      pairs (i, i + d/2) of the first d elements, angle p f_i; f_i blended along a ramp over i between
                f_i and f_i / factor; cos and sin times 0.1 ln(factor) + 1
  chunked       q, k = short causal convolution of Wq h, Wk h; v = k; q, k <- rms over ALL heads' elements, weighted;
                s_ij = scale q_i . k_j for j <= i in i's aligned chunk; softmax; times sigmoid(G h) by element; O
  mlstm         log gates i = cap tanh(./cap), f = logsigmoid(cap tanh(./cap)); m_t = max(f + m_{t-1}, i), m_0 = 0;
                S_t = e^(f + m_{t-1} - m_t) S_{t-1} + e^(i - m_t) k v^T, n_t the same with k alone;
                o = S^T q / (max(|n . q|, e^(-m)) + 1e-6); rms per head; times a weight and sigmoid(G h); O
  parallel      (rms(chunked(h)) w_left + rms(mlstm(h)) w_right) / 2
  dense ff      Dn (gelu(Gt h) * Up h)
  experts       s = sigmoid(R h); ranked by s + corr; a group of neighbours ranks by its two best together, the best
                `keep` groups stay; the `top` best of them, weighted by s alone;
                expert: g = min(Gt h, L), u = clamp(Up h, -L, L); Dn (g sigmoid(1.702 g) (u + 1))
  output        H n(x)
"""
from __future__ import annotations

import math

import torch

GATE_SHARPNESS = 1.702
DENOMINATOR_EPS = 1e-6


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, weight, eps):
    return rms(x, eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def embedding(w, cfg, tokens):
    x = w["embed"][torch.tensor(tokens)]
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        n = int(b["buckets"])
        rows = [n] + [(p * int(b["mul_prev"]) + t * int(b["mul_cur"])) % n for p, t in zip(tokens, tokens[1:])]
        x = x + w["bigram"][torch.tensor(rows)]
    return x


def frequencies(rot):
    """(frequency of every pair, multiplier of cos and sin)."""
    d, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / d) for i in range(d // 2)]
    if not sc:
        return torch.tensor(f, dtype=torch.float64), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])
    place = lambda t: d * math.log(original / (2 * math.pi * t)) / (2 * math.log(base))
    lo = max(math.floor(place(float(sc["fast"]))), 0)
    hi = min(math.ceil(place(float(sc["slow"]))), d - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / factor * r + fi * (1 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(factor) + 1.0


def turn(x, positions, rot):
    """x [T, ..., size]: the first rot.dims elements turned in pairs (i, i + dims/2) by the row's position."""
    d = int(rot["dims"])
    f, stretch = frequencies(rot)
    a = positions.double()[:, None] * f[None, :]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (d // 2,)
    c, s = (torch.cos(a) * stretch).view(shape), (torch.sin(a) * stretch).view(shape)
    u, v = x[..., : d // 2], x[..., d // 2: d]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., d:]], dim=-1)


def softmax_attention(q, k, v, scale, seen):
    """q [T, H, d], k [T, G, d], v [T, G, dv], seen [T, T] -> [T, H, dv]; query head h reads head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        out.append(torch.softmax(s.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g])
    return torch.stack(out, dim=1)


def causal(n):
    return torch.tril(torch.ones(n, n, dtype=torch.bool))


def same_chunk(n, size):
    c = torch.arange(n) // size
    return causal(n) & (c[:, None] == c[None, :])


def latent_attention(w, p, m, h, positions, eps):
    H, d, t, dv, r = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    T = h.shape[0]
    q = (h @ w[p + "q"].T).view(T, H, d + t)
    down = h @ w[p + "dkv"].T
    c = norm(down[:, :r], w[p + "dkv.norm"], eps)
    tail = turn(down[:, r:], positions, m["rot"])
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    qt = turn(q[..., d:], positions, m["rot"])
    full_q = torch.cat([q[..., :d], qt], dim=-1)
    full_k = torch.cat([k, tail[:, None, :].expand(T, H, t)], dim=-1)
    o = softmax_attention(full_q, full_k, v, float(m["scale"]), causal(T))
    return o.reshape(T, H * dv) @ w[p + "o"].T


def short_conv(u, weight):
    """y_t = sum_j weight[:, j] u_{t - taps + 1 + j}, zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u])
    return sum(weight[:, j] * padded[j: j + u.shape[0]] for j in range(taps))


def chunked_attention(w, p, m, h, eps):
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    T = h.shape[0]
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    if m.get("conv"):
        q, k = short_conv(q, w[p + "q.conv"]), short_conv(k, w[p + "k.conv"])
    v = k.view(T, G, d)
    q, k = norm(q, w[p + "q.norm"], eps).view(T, H, d), norm(k, w[p + "k.norm"], eps).view(T, G, d)
    mask = m.get("mask")
    seen = same_chunk(T, int(mask["size"])) if mask else causal(T)
    o = softmax_attention(q, k, v, float(m["scale"]), seen).reshape(T, H * d)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mlstm_gates(w, p, m, h):
    cap = float(m["gate_cap"])
    i = cap * torch.tanh((h @ w[p + "i"].T + w[p + "i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w[p + "f"].T + w[p + "f.b"]) / cap))
    return i, f


def matrix_memory(q, k, v, i, f, terms=None):
    """q, k [T, H, d], v [T, H, dv], log gates i, f [T, H] -> o [T, H, dv], token by token from zero.  `terms` collects, per
    token, what the read-out's two sums are made of: (sum of |k||q||v| weighted, sum of |k||q| weighted, denominator)."""
    T, H, d = q.shape
    S, n = torch.zeros(H, d, v.shape[2], dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    out = []
    Sa, na = S.clone(), n.clone()
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + DENOMINATOR_EPS
        out.append(torch.einsum("hde,hd->he", S, q[t]) / den[:, None])
        if terms is not None:
            Sa = keep[:, None, None] * Sa + add[:, None, None] * (k[t][:, :, None] * v[t][:, None, :]).abs()
            na = keep[:, None] * na + add[:, None] * k[t].abs()
            terms.append((torch.einsum("hde,hd->he", Sa, q[t].abs()), (na * q[t].abs()).sum(-1), den))
    return torch.stack(out)


def mlstm(w, p, m, h, eps):
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    T = h.shape[0]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ w[p + "k"].T).view(T, H, d), (h @ w[p + "v"].T).view(T, H, dv)
    i, f = mlstm_gates(w, p, m, h)
    o = rms(matrix_memory(q, k, v, i, f), eps).reshape(T, H * dv)
    return (o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel_mixer(w, p, m, h, eps):
    left, right = chunked_attention(w, p + "left.", m["left"], h, eps), mlstm(w, p + "right.", m["right"], h, eps)
    return 0.5 * (norm(left, w[p + "left.out"], eps) + norm(right, w[p + "right.out"], eps))


def dense_ff(w, p, h):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def expert(w, p, limit, h):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(GATE_SHARPNESS * g) * (u + 1.0)) @ w[p + "down"].T


def group_scores(choice, count):
    """[T, E] -> [T, count]: a group's two largest choice scores together."""
    c = choice.view(choice.shape[0], count, -1)
    return torch.topk(c, min(2, c.shape[-1]), dim=-1).values.sum(-1)


def route(scores, correction, top, groups):
    """-> chosen experts [T, top] (best first, ties to the lower number) and their weights."""
    choice = scores + correction
    if groups:
        count, keep = int(groups["count"]), int(groups["keep"])
        best = torch.argsort(group_scores(choice, count), dim=-1, descending=True, stable=True)[:, :keep]
        allowed = torch.zeros(choice.shape[0], count, dtype=torch.bool).scatter_(1, best, True)
        choice = choice.masked_fill(~allowed.repeat_interleave(choice.shape[1] // count, dim=1), float("-inf"))
    chosen = torch.argsort(choice, dim=-1, descending=True, stable=True)[:, :top]
    return chosen, scores.gather(1, chosen)


def routing_margin(w, p, f, h):
    """How far each token's routing is from another outcome (in choice scores)."""
    r = f["router"]
    choice = torch.sigmoid(h @ w[p + "router"].T) + w[p + "correction"]
    T, E = choice.shape
    margin = torch.full((T,), float("inf"), dtype=torch.float64)
    if r.get("groups"):
        count, keep = int(r["groups"]["count"]), int(r["groups"]["keep"])
        s, order = torch.sort(group_scores(choice, count), dim=-1, descending=True, stable=True)
        if keep < count:
            margin = torch.minimum(margin, s[:, keep - 1] - s[:, keep])
        allowed = torch.zeros(T, count, dtype=torch.bool).scatter_(1, order[:, :keep], True)
        choice = choice.masked_fill(~allowed.repeat_interleave(E // count, dim=1), float("-inf"))
    ranked = torch.sort(choice, dim=-1, descending=True).values
    top = int(r["top"])
    if top < E and bool(torch.isfinite(ranked[:, top]).all()):
        margin = torch.minimum(margin, ranked[:, top - 1] - ranked[:, top])
    return margin


def experts_ff(w, p, f, h):
    r = f["router"]
    scores = torch.sigmoid(h @ w[p + "router"].T)
    chosen, weights = route(scores, w[p + "correction"], int(r["top"]), r.get("groups"))
    out = torch.zeros_like(h)
    for e in range(int(r["experts"])):
        t, j = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            out[t] += weights[t, j][:, None] * expert(w, f"{p}e{e}.", float(f["expert"]["limit"]), h[t])
    return out


def feed_forward(w, p, f, h):
    return dense_ff(w, p, h) if f["kind"] == "dense" else experts_ff(w, p, f, h)


def forward(w, cfg, tokens, layers_out=None, margins=None):
    """Logits [T, vocab] of one sequence; `layers_out` collects the stream after every layer, `margins` the routing
    margins [T] of every routed layer."""
    eps = float(cfg["norm"]["eps"])
    positions = torch.arange(len(tokens))
    x = embedding(w, cfg, list(tokens))
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] == "parallel":
            y = parallel_mixer(w, p + "mix.", layer["mixer"], x, eps)
        else:
            y = latent_attention(w, p + "mix.", layer["mixer"], x, positions, eps)
        x = x + norm(y, w[p + "norm1"], eps)
        f = layer.get("mlp")
        if f:
            if margins is not None and f["kind"] == "moe":
                margins.append(routing_margin(w, p + "mlp.", f, x))
            x = x + norm(feed_forward(w, p + "mlp.", f, x), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, w["final.norm"], eps) @ w["head"].T
