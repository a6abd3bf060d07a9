"""Plain, slow Pasizen in float64: one function per mechanism, whole sequences only, no cache.  Used by the tests as the
independent statement of the architecture; it shares no code with the framework.

``cfg`` is the dict a config.json holds, ``W`` maps tensor names to tensors (any dtype; everything is computed in float64).
"""
import torch

F64 = torch.float64


def rms_normalise(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def causal_short_conv(h, w):
    """h [T, C], w [C, taps]: out[t] = sum_j w[:, j] * h[t - taps + 1 + j], zero history."""
    T, C = h.shape
    taps = w.shape[1]
    out = torch.zeros_like(h)
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += w[:, j] * h[s]
    return out


def latent_attention(h, W, p, m, eps, trace=None):
    """h [T, d] -> [T, d]; keys and values are expanded from the latent, head by head."""
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, D)
    c = rms_normalise(h @ W[p + "dkv"].T, eps) * W[p + "dkv.norm"]
    k = (c @ W[p + "uk"].T).view(T, H, D)
    v = (c @ W[p + "uv"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    for i in range(H):
        s = (q[:, i] @ k[:, i].T) * m["scale"]
        pr = torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1)
        if trace is not None:
            trace.append(pr)
        out[:, i] = pr @ v[:, i]
    return out.reshape(T, H * V) @ W[p + "o"].T


def poly_norm(z, abce, eps):
    a, b, c, e = [float(x) for x in abce]
    return a * rms_normalise(z, eps) + b * rms_normalise(z ** 2, eps) + c * rms_normalise(z ** 3, eps) + e


def dense_ff(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def clamped_glu(gate, up, limit):
    g = torch.minimum(gate, torch.full_like(gate, limit))
    u = up.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def glu_ff(h, W, p, limit):
    return clamped_glu(h @ W[p + "gate"].T, h @ W[p + "up"].T, limit) @ W[p + "down"].T


def route(z, r):
    """Router logits z [T, E] -> (chosen experts [T, top], weights [T, top])."""
    s = torch.softmax(z, dim=-1)
    T, E = s.shape
    n, keep = r["groups"]["count"], r["groups"]["keep"]
    best = s.view(T, n, E // n).amax(-1)
    kept = torch.zeros(T, n, dtype=torch.bool)
    kept.scatter_(1, best.topk(keep, dim=-1).indices, True)
    allowed = kept.repeat_interleave(E // n, dim=1)
    idx = s.masked_fill(~allowed, -1.0).topk(r["top"], dim=-1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20)


def moe_ff(h, W, p, mlp):
    idx, w = route(h @ W[p + "router"].T, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(idx.shape[1]):
            e = int(idx[t, j])
            out[t] += w[t, j] * glu_ff(h[t:t + 1], W, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        out = out + glu_ff(h, W, p + "shared.", mlp["shared"]["limit"])
    return out


def hyper_step(x, w_in, w_mix, w_out, f):
    """x: list of streams.  One sublayer f between its read and its write."""
    s = len(x)
    u = sum(w_in[i] * x[i] for i in range(s))
    y = f(u)
    return [sum(w_mix[i, t] * x[i] for i in range(s)) + w_out[t] * y for t in range(s)]


def layer_order(cfg):
    n = len(cfg["layers"])
    lp = cfg.get("loop")
    if not lp:
        return list(range(n))
    a, b = lp["start"], lp["stop"]
    return list(range(a)) + list(range(a, b)) * lp["times"] + list(range(b, n))


def forward(cfg, weights, ids, per_layer=None):
    """Logits [T, vocab] of one sequence; ``per_layer`` (a list) receives the residual stream after every layer run."""
    W = {k: v.to(F64) if v.is_floating_point() else v for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    ids = torch.as_tensor(ids, dtype=torch.long)
    T = ids.numel()
    e = W["embed"][ids] + W["pos"][:T]
    x = [e.clone() for _ in range(cfg["streams"])]
    for li in layer_order(cfg):
        L, p = cfg["layers"][li], f"l{li}."

        def mix(u):
            h = rms_normalise(u, eps) * W[p + "norm1"]
            h = h + causal_short_conv(h, W[p + "canon1"])
            return latent_attention(h, W, p + "mix.", L["mixer"], eps)
        x = hyper_step(x, W[p + "hc1.in"], W[p + "hc1.mix"], W[p + "hc1.out"], mix)
        mlp = L["mlp"]
        if mlp is not None:
            def ff(u):
                h = rms_normalise(u, eps) * W[p + "norm2"]
                return dense_ff(h, W, p + "mlp.", eps) if mlp["kind"] == "dense" else moe_ff(h, W, p + "mlp.", mlp)
            x = hyper_step(x, W[p + "hc2.in"], W[p + "hc2.mix"], W[p + "hc2.out"], ff)
        if per_layer is not None:
            per_layer.append(sum(x))
    return (rms_normalise(sum(x), eps) * W["final.norm"]) @ W["head"].T
