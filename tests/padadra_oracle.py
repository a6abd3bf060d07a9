"""Plain, slow Padadra in float64: one function per mechanism, whole sequences only, no cache.  Used by the tests as the
independent statement of the architecture; it shares no code with the framework.

``cfg`` is the dict a config.json holds, ``W`` maps tensor names to tensors (any dtype; everything is computed in float64).
"""
import math

import torch

F64 = torch.float64
sigmoid = torch.sigmoid


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0.0)


def embed(ids, W, e):
    """Scaled token rows plus the row of the pair (token before, token), hashed; the first token takes the last row."""
    rows = []
    for t, tok in enumerate(ids):
        x = W["embed"][tok] * e["scale"]
        b = e.get("bigram")
        if b:
            x = x + W["bigram"][b["buckets"] if t == 0 else (ids[t - 1] * b["mul_prev"] + tok * b["mul_cur"]) % b["buckets"]]
        rows.append(x)
    return torch.stack(rows)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: the last tap meets the current token."""
    T, taps = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += w[:, j] * u[t - taps + 1 + j]
    return out


def frequencies(dims, base, scaling=None):
    """Angle per position of every pair; ``scaling`` slows the long waves down."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if scaling:
            wave, size = 2.0 * math.pi / f, scaling["original"]
            if wave > size / scaling["low"]:
                f = f / scaling["factor"]
            elif wave >= size / scaling["high"]:
                s = (size / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return out


def rotate(x, freq, sign=1.0):
    """x [T, ..., n]: pair (2i, 2i + 1) turns by sign * position * freq[i]; entries beyond the pairs pass."""
    T = x.shape[0]
    out = x.clone()
    for i, f in enumerate(freq):
        ang = sign * torch.arange(T, dtype=F64) * f
        c, s = (t.view([T] + [1] * (x.dim() - 2)) for t in (torch.cos(ang), torch.sin(ang)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def window_softmax(s, v, size, sink):
    """Scores s [T, T] of one head, v [T, E]: row i sees itself and the size - 1 rows before; ``sink`` is a logit without value."""
    out = torch.zeros(s.shape[0], v.shape[1], dtype=F64)
    for i in range(s.shape[0]):
        j = max(0, i - size + 1)
        row = s[i, j:i + 1]
        top = max(float(row.max()), float(sink))
        e = torch.exp(row - top)
        out[i] = (e / (math.exp(float(sink) - top) + e.sum())) @ v[j:i + 1]
    return out


def windowed_attention(h, W, p, m, eps):
    """Grouped heads behind biased projections and a short convolution, normed whole, rotated; values turn with their position
    and back at the reader's."""
    T, H, G, D, E, rot = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    q, k, v = (causal_conv(h @ W[p + n].T + W[p + n + ".b"], W[p + n + ".conv"]) for n in "qkv")
    q, k = over_rms(q, eps) * W[p + "q.norm"], over_rms(k, eps) * W[p + "k.norm"]
    freq, turn = frequencies(rot["dims"], rot["base"], rot.get("scaling")), frequencies(E, rot["base"])
    q, k, v = rotate(q.view(T, H, D), freq), rotate(k.view(T, G, D), freq), rotate(v.view(T, G, E), turn)
    out = []
    for a in range(H):
        g = a // (H // G)
        out.append(window_softmax((q[:, a] @ k[:, g].T) * m["scale"], v[:, g], m["mask"]["size"], W[p + "sink"][a]))
    return rotate(torch.stack(out, dim=1), turn, -1.0).reshape(T, H * E) @ W[p + "o"].T


def forget_write(q, v, f):
    """One head, q and f [T, D], v [T, E]: S <- diag(f) S + (1 - f) v^T, then S^T q."""
    S, out = torch.zeros(q.shape[1], v.shape[1], dtype=F64), []
    for t in range(q.shape[0]):
        S = f[t].unsqueeze(1) * S + torch.outer(1.0 - f[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out)


def hgrn2(h, W, p, m, eps):
    T, H, D, E = h.shape[0], m["heads"], m["dim"], m["vdim"]
    low = W[p + "lower"]
    q = silu(h @ W[p + "q"].T).view(T, H, D)
    f = (low + (1.0 - low) * sigmoid(h @ W[p + "f"].T + W[p + "f.b"])).view(T, H, D)
    v = (h @ W[p + "v"].T).view(T, H, E)
    o = torch.stack([forget_write(q[:, a], v[:, a], f[:, a]) for a in range(H)], dim=1)
    return (over_rms(o, eps) * W[p + "norm"]).reshape(T, H * E) @ W[p + "o"].T


def parallel(h, W, p, m, eps):
    a = over_rms(windowed_attention(h, W, p + "left.", m["left"], eps), eps) * W[p + "left.out"]
    b = over_rms(hgrn2(h, W, p + "right.", m["right"], eps), eps) * W[p + "right.out"]
    return 0.5 * (a + b)


def channel_delta_rule(q, k, v, g, beta):
    """One head, q, k and decays g [T, D], v [T, E], beta [T]: decay, then write what is missing of v at k, then read."""
    S, out = torch.zeros(q.shape[1], v.shape[1], dtype=F64), []
    for t in range(q.shape[0]):
        S = g[t].unsqueeze(1) * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.T @ q[t])
    return torch.stack(out)


def channel_delta(h, W, p, m, eps):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv")
    q, k, v = q.view(T, G, D), k.view(T, G, D), v.view(T, H, E)
    q, k = (z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6) for z in (q, k))
    q = q * D ** -0.5
    beta = sigmoid(h @ W[p + "b"].T)
    z = ((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "dt_bias"]).view(T, H, D)
    g = torch.exp(-torch.exp(W[p + "A_log"]).view(1, H, 1) * softplus(z))
    o = torch.stack([channel_delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], g[:, a], beta[:, a]) for a in range(H)], dim=1)
    o = (over_rms(o, eps) * W[p + "norm"]).reshape(T, H * E) * sigmoid((h @ W[p + "g1"].T) @ W[p + "g2"].T)
    return o @ W[p + "o"].T


MIXERS = {"parallel": parallel, "channel_delta": channel_delta}


def feed_forward(h, W, p):
    return (h @ W[p + "up"].T).clamp(min=0.0) ** 2 @ W[p + "down"].T


def forward(cfg, weights, ids, per_layer=None):
    """Logits [T, vocab] of one sequence; ``per_layer`` (a list) receives the residual stream after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = embed([int(i) for i in ids], W, cfg["embedding"])
    for li, L in enumerate(cfg["layers"]):
        p = f"l{li}."
        y = MIXERS[L["type"]](over_rms(x, eps) * W[p + "norm1"], W, p + "mix.", L["mixer"], eps)
        if L["mlp"] is not None:
            y = y + feed_forward(over_rms(x, eps) * W[p + "norm2"], W, p + "mlp.")
        x = x + cfg["residual_mult"] * y
        if per_layer is not None:
            per_layer.append(x)
    return (over_rms(x, eps) * W["final.norm"]) @ W["head"].T
