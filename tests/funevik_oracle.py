"""Plain, slow Funevik in float64: one function per mechanism, whole sequences only, no cache.  Used by the tests as the
independent statement of the architecture; it shares no code with the framework.

``cfg`` is the dict a config.json holds, ``W`` maps tensor names to tensors (any dtype; everything is computed in float64).
"""
import math

import torch

F64 = torch.float64
sigmoid = torch.sigmoid


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def log_sigmoid(z):
    return -torch.log1p(torch.exp(-z.abs())) + z.clamp(max=0.0)


def matrix_memory(q, k, v, i, f):
    """One head, q and k [T, D], v [T, E], log gates i and f [T] -> [T, E].  With a running maximum m: decay exp(f + m_old - m),
    input weight exp(i - m); the read-out is divided by max(|n.q|, exp(-m)) + 1e-6."""
    T, D = q.shape
    S, n, m = torch.zeros(D, v.shape[1], dtype=F64), torch.zeros(D, dtype=F64), 0.0
    out = torch.zeros(T, v.shape[1], dtype=F64)
    for t in range(T):
        top = max(float(f[t]) + m, float(i[t]))
        keep, add = math.exp(float(f[t]) + m - top), math.exp(float(i[t]) - top)
        S = keep * S + add * torch.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = top
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(h, W, p, m, eps):
    T, H, D, E, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ W[p + "q"].T).view(T, H, D) * D ** -0.5
    k, v = (h @ W[p + "k"].T).view(T, H, D), (h @ W[p + "v"].T).view(T, H, E)
    i = cap * torch.tanh((h @ W[p + "i"].T + W[p + "i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((h @ W[p + "f"].T + W[p + "f.b"]) / cap))
    o = torch.stack([matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(H)], dim=1)
    o = over_rms(o, eps).reshape(T, H * E) * W[p + "norm"] * sigmoid(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def rotate(x, base, dims):
    """x [T, ..., n]: pairs (2i, 2i + 1) of the first ``dims`` entries turn by position / base^(2i / dims)."""
    T = x.shape[0]
    out = x.clone()
    for a in range(dims // 2):
        ang = torch.arange(T, dtype=F64) * base ** (-2.0 * a / dims)
        c, s = (t.view([T] + [1] * (x.dim() - 2)) for t in (torch.cos(ang), torch.sin(ang)))
        u, v = x[..., 2 * a], x[..., 2 * a + 1]
        out[..., 2 * a], out[..., 2 * a + 1] = u * c - v * s, v * c + u * s
    return out


def window_softmax(s, v, first, extra):
    """Scores s [T, T] of one head, v [T, E]: row i sees positions first(i)..i; ``extra`` is a logit in the sum without value."""
    out = torch.zeros(s.shape[0], v.shape[1], dtype=F64)
    for i in range(s.shape[0]):
        j = max(0, first(i))
        row = s[i, j:i + 1]
        top = max(float(row.max()), float(extra))
        e = torch.exp(row - top)
        out[i] = (e / (math.exp(float(extra) - top) + e.sum())) @ v[j:i + 1]
    return out


def latent_attention(h, W, p, m, eps):
    T, H, D, E, R, r = h.shape[0], m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["rot_dim"]
    q = ((over_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, D + r)
    down = h @ W[p + "dkv"].T
    c = over_rms(down[:, :R], eps) * W[p + "dkv.norm"]
    k, v = (c @ W[p + "uk"].T).view(T, H, D), (c @ W[p + "uv"].T).view(T, H, E)
    k_rot = rotate(down[:, R:], m["rot"]["base"], r)
    q_rot = rotate(q[..., D:], m["rot"]["base"], r)
    size, out = m["mask"]["size"], []
    for a in range(H):
        s = (q[:, a, :D] @ k[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]
        out.append(window_softmax(s, v[:, a], lambda i: i - size + 1, W[p + "sink"][a]))
    return torch.stack(out, dim=1).reshape(T, H * E) @ W[p + "o"].T


def causal_conv(u, w):
    """u [T, C], w [C, taps]: the last tap meets the current token."""
    T, taps = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                out[t] += w[:, j] * u[t - taps + 1 + j]
    return out


def attention(h, W, p, m, eps):
    T, H, G, D, E = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(h @ W[p + n].T, W[p + n + ".conv"]) for n in "qkv")
    q = rotate(q.view(T, H, D), m["rot"]["base"], m["rot"]["dims"])
    k = rotate(k.view(T, G, D), m["rot"]["base"], m["rot"]["dims"])
    v, cap, out = v.view(T, G, E), m["softcap"], []
    for a in range(H):
        g = a // (H // G)
        s = cap * torch.tanh((q[:, a] @ k[:, g].T) * m["scale"] / cap)
        out.append(window_softmax(s, v[:, g], lambda i: 0, 0.0))
    o = torch.stack(out, dim=1) * sigmoid(h @ W[p + "g"].T).unsqueeze(-1)
    return o.reshape(T, H * E) @ W[p + "o"].T


MIXERS = {"mlstm": mlstm, "latent_attention": latent_attention, "attention": attention}


def gated(h, W, p, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def experts(h, W, p, top):
    z = h @ W[p + "router"].T + W[p + "router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = sorted(range(z.shape[1]), key=lambda e: -float(z[t, e]))[:top]
        w = torch.softmax(z[t, best], dim=0)
        for e, g in zip(best, w):
            out[t] += g * gated(h[t:t + 1], W, f"{p}e{e}.", silu)[0]
    return out


def feed_forward(h, W, p, f):
    if f["kind"] == "dense":
        return gated(h, W, p, gelu_tanh)
    y = experts(h, W, p, f["router"]["top"])
    if f.get("shared"):
        y = y + gated(h, W, p + "shared.", silu) * sigmoid(h @ W[p + "shared.sg"].T)
    return y


def forward(cfg, weights, ids, per_layer=None):
    """Logits [T, vocab] of one sequence; ``per_layer`` (a list) receives the residual stream after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(ids, dtype=torch.long)] * cfg["embedding"]["scale"]
    for li, L in enumerate(cfg["layers"]):
        p = f"l{li}."
        y = MIXERS[L["type"]](over_rms(x, eps) * W[p + "norm1"], W, p + "mix.", L["mixer"], eps) * W[p + "ls1"]
        if L["mlp"] is not None:
            y = y + feed_forward(over_rms(x, eps) * W[p + "norm2"], W, p + "mlp.", L["mlp"]) * W[p + "ls2"]
        x = x + y
        if per_layer is not None:
            per_layer.append(x)
    return (over_rms(x, eps) * W["final.norm"]) @ W["head"].T
