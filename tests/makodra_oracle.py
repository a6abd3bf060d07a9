"""Plain, slow Makodra in float64: one function per mechanism, whole sequences only, no cache.  Used by the tests as the
independent statement of the architecture; it shares no code with the framework.

``cfg`` is the dict a config.json holds, ``W`` maps tensor names to tensors (any dtype; everything is computed in float64).
"""
import math

import torch

F64 = torch.float64


def over_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sinusoid(T, d):
    """[T, d]: even entries sine, odd entries cosine of p / 10000^(even index / d)."""
    out = torch.zeros(T, d, dtype=F64)
    for c in range(d):
        ang = torch.arange(T, dtype=F64) * 10000.0 ** (-(c - c % 2) / d)
        out[:, c] = torch.cos(ang) if c % 2 else torch.sin(ang)
    return out


def chunk_attention(q, k, v, scale, r1, r2, size):
    """q [T, H, D], k [T, G, D], v [T, G, V] -> [T, H, V]: scores scale q.k - r1 ln(1 + r2 distance) inside chunks of
    ``size`` positions, weights exp(s) / (1 + sum exp(s))."""
    T, H, D = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        j0 = i // size * size
        dist = torch.arange(i - j0, -1, -1, dtype=F64)
        for h in range(H):
            g = h // (H // G)
            s = (k[j0:i + 1, g] @ q[i, h]) * scale - r1[h] * torch.log(1.0 + r2[h] * dist)
            top = max(float(s.max()), 0.0)
            e = torch.exp(s - top)
            out[i, h] = (e / (math.exp(-top) + e.sum())) @ v[j0:i + 1, g]
    return out


def attention(h, W, p, m, eps, v_first):
    """-> (mixer output [T, d], this layer's own values [T, G, V])."""
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms((h @ W[p + "q"].T).view(T, H, D), eps)
    k = over_rms((h @ W[p + "k"].T).view(T, G, D), eps)
    own = (h @ W[p + "v"].T).view(T, G, V)
    v = own
    if m["v_mix"] and v_first is not None:
        lam = W[p + "vmix"]
        v = (1.0 - lam) * own + lam * v_first
    o = chunk_attention(q, k, v, m["scale"], W[p + "r1"], W[p + "r2"], m["mask"]["size"]).reshape(T, H * V)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T, own


def delta_rule(r, w, k, v, a):
    """One head, all [T, D]: S <- diag(w) S - (a u)(u^T S) + k v^T with u = k / |k|; read out with r after the update."""
    T, D = r.shape
    S = torch.zeros(D, v.shape[1], dtype=F64)
    out = torch.zeros(T, v.shape[1], dtype=F64)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        S = w[t][:, None] * S - torch.outer(a[t] * u, u @ S) + torch.outer(k[t], v[t])
        out[t] = S.T @ r[t]
    return out


def general_delta(h, W, p, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    sig = torch.sigmoid
    w = torch.exp(-math.exp(-0.5) * sig(torch.tanh(h @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).view(T, H, D)
    a = sig(h @ W[p + "a"].T + W[p + "a.b"]).view(T, H, D)
    r, k, v = ((h @ W[p + n].T).view(T, H, D) for n in "rkv")
    o = torch.stack([delta_rule(r[:, i], w[:, i], k[:, i], v[:, i], a[:, i]) for i in range(H)], dim=1)
    o = over_rms(o, eps).reshape(T, H * D) * W[p + "norm"] * sig(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def bonus_memory(r, w, k, v, u):
    """One head: read out before the update, the current token's own k v^T weighted by the bonus u; S <- diag(w) S + k v^T."""
    T, D = r.shape
    S = torch.zeros(D, v.shape[1], dtype=F64)
    out = torch.zeros(T, v.shape[1], dtype=F64)
    for t in range(T):
        kv = torch.outer(k[t], v[t])
        out[t] = (S + u[:, None] * kv).T @ r[t]
        S = w[t][:, None] * S + kv
    return out


def shifted(h):
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv(h, W, p, m, eps):
    T, H, D = h.shape[0], m["heads"], m["dim"]
    back = shifted(h) - h
    x = {s: h + back * W[p + "mu." + s] for s in "rkvgw"}
    r, k, v = ((x[s] @ W[p + s].T).view(T, H, D) for s in "rkv")
    gate = x["g"] @ W[p + "g"].T
    gate = gate * torch.sigmoid(gate)
    w = torch.exp(-torch.exp(torch.tanh(x["w"] @ W[p + "w1"].T) @ W[p + "w2"].T + W[p + "w0"])).view(T, H, D)
    u = W[p + "u"].view(H, D)
    o = torch.stack([bonus_memory(r[:, i], w[:, i], k[:, i], v[:, i], u[i]) for i in range(H)], dim=1)
    return (over_rms(o, eps).reshape(T, H * D) * W[p + "norm"] * gate) @ W[p + "o"].T


def swiglu(h, W, p):
    g = h @ W[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, weights, ids, per_layer=None):
    """Logits [T, vocab] of one sequence; ``per_layer`` (a list) receives the residual stream after every layer."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(ids, dtype=torch.long)
    x = W["embed"][ids] + sinusoid(ids.numel(), cfg["width"])
    v_first = None
    for li, L in enumerate(cfg["layers"]):
        p, m = f"l{li}.", L["mixer"]
        if L["type"] == "attention":
            y, own = attention(x, W, p + "mix.", m, eps, v_first)
            if m["v_mix"] and v_first is None:
                v_first = own
        else:
            y = {"general_delta": general_delta, "wkv": wkv}[L["type"]](x, W, p + "mix.", m, eps)
        x = x + over_rms(y, eps) * W[p + "norm1"]
        if L["mlp"] is not None:
            x = x + over_rms(swiglu(x, W, p + "mlp."), eps) * W[p + "norm2"]
        if per_layer is not None:
            per_layer.append(x)
    z = (over_rms(x, eps) * W["final.norm"]) @ W["embed"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
