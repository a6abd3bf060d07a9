"""Small Padadra models with weights chosen so that faults show: in every layer the queries of the token SEEKER single out the keys
of the token SOUGHT, whatever their distance, which every memory writes down loudly and partly never forgets; every constant
differs from a neutral value."""
import json
import os

import torch

from pasizen_models import far_effect, row_error  # noqa: F401  (the suite takes them from the family's module)


def pair(cfg):
    """(SOUGHT, SEEKER): the last two ids."""
    return cfg["vocab"] - 2, cfg["vocab"] - 1


def tokens(cfg, n, seed=0):
    """Random ids, the first the sought token and the last its seeker; neither occurs elsewhere."""
    ids = torch.randint(0, cfg["vocab"] - 2, (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
    ids[-1] = pair(cfg)[1]
    if n > 1:
        ids[0] = pair(cfg)[0]
    return ids


def delta(heads, kv_heads, dim, vdim, conv=4):
    return "channel_delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


SLOWED = {"factor": 5.0, "low": 1.0, "high": 3.5, "original": 90}


def attn(heads, kv_heads, dim, vdim, rot, window, conv=3, base=900.0, scale=None, scaling=SLOWED):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window},
            "rot": {"base": base, "dims": rot, "scaling": scaling}, "scale": 8.0 / dim if scale is None else scale}


def both(left, heads, dim, vdim):
    return "parallel", {"left": left, "right": {"heads": heads, "dim": dim, "vdim": vdim}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


PAIRS = {"buckets": 89, "mul_prev": 37, "mul_cur": 11}


def config(width, layers, vocab=211, eps=1e-5, scale=5.0, mult=0.7, pairs=PAIRS, quiet=False):
    """``layers``: (mixer, feed-forward or None); ``quiet``: the memories beside attention hold nothing."""
    return {"architecture": "Padadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale, "bigram": pairs},
            "residual_mult": mult, "quiet": quiet, "layers": [{"type": kind, "mixer": mixer, "mlp": f} for (kind, mixer), f in layers]}


CONFIGS = {
    "all_kinds": config(136, [(both(attn(6, 3, 24, 40, 12, 48), 3, 40, 24), dense(96)), (delta(4, 2, 40, 24), None),
                              (both(attn(4, 1, 40, 24, 40, 200, conv=1, base=3000.0, scaling=None), 5, 24, 56), None),
                              (delta(5, 5, 24, 56, conv=2), dense(200))]),
    "odd_sizes": config(100, [(delta(6, 2, 18, 22, conv=3), dense(77)), (both(attn(5, 5, 28, 44, 2, 21, conv=5), 1, 70, 33), dense(130)),
                              (delta(1, 1, 70, 34, conv=1), None), (both(attn(3, 1, 20, 12, 20, 33, conv=2), 3, 13, 7), None)],
                        eps=1e-3, vocab=97, scale=0.7, mult=1.3, pairs={"buckets": 13, "mul_prev": 1, "mul_cur": 1}),
    "delta_only": config(64, [(delta(4, 1, 16, 16), None), (delta(2, 2, 64, 130, conv=8), dense(50))], vocab=300, mult=1.0),
    "parallel_only": config(96, [(both(attn(2, 2, 32, 16, 16, 33), 2, 130, 40), dense(64)), (both(attn(8, 4, 16, 24, 8, 70), 4, 16, 16), None)],
                            pairs={"buckets": 1000, "mul_prev": 2000003, "mul_cur": 999}),
}

GAIN = 2.5


def make_weights(cfg, seed=0):
    """name -> bf16 tensor."""
    g = torch.Generator().manual_seed(seed)
    d, V, pairs = cfg["width"], cfg["vocab"], cfg["embedding"]["bigram"]
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    gainful = lambda n: 1.0 + 0.3 * r(n)
    one = lambda: 1.0 + 0.3 * torch.rand((), generator=g)
    embed = r(V, d)
    embed[:, 0] = 2.0                                          # what all tokens share: maps without a bias get theirs from it
    W = {"embed": embed / cfg["embedding"]["scale"], "head": lin(V, d), "final.norm": one()}
    if pairs:
        W["bigram"] = 0.4 * r(pairs["buckets"] + 1, d)
        W["bigram"][:, 0] = 0.0
    unit = lambda v: v / v.pow(2).mean().sqrt()
    sought, seeker = (unit(embed[t]) for t in pair(cfg))
    loud = sought.clone()
    loud[0] = 0.0
    loud = loud / loud.pow(2).sum()

    def seek(q, k):
        """Query map [H, D, d] to which the seeker gives ``GAIN`` times what the key map makes of the sought token."""
        return q + GAIN * torch.einsum("hdn,n,m->hdm", k, sought, seeker / seeker.pow(2).sum())

    def conv(n, taps):
        w = 0.3 * r(n, taps)
        w[:, -1] = 1.0 + 0.1 * r(n)
        return w

    def queries(H, G, D):
        k = lin(G * D, d)
        return k, seek(0.6 * lin(H * D, d).view(H, D, d), k.view(G, D, d).repeat_interleave(H // G, 0)).reshape(H * D, d)

    def shared_conv(H, G, D, taps):
        ck = conv(G * D, taps)
        return ck, ck.view(G, 1, D, taps).repeat(1, H // G, 1, 1).reshape(H * D, taps)
    for li, L in enumerate(cfg["layers"]):
        p, m = f"l{li}.", L["mixer"]
        x = p + "mix."
        W[p + "norm1"] = one()
        if L["type"] == "channel_delta":
            H, G, D, E, taps = (m[n] for n in ("heads", "kv_heads", "dim", "vdim", "conv"))
            k, q = queries(G, G, D)
            ck, cq = shared_conv(G, G, D, taps)
            ra, rg = 5 + li, 19 - li
            b = 0.3 * lin(H, d)
            b[:, 0] -= 1.5                                     # others write little, the sought token all of itself
            slow = torch.rand(H, generator=g) < 0.6            # these heads keep what they hold
            slow[0] = True
            W.update({x + "q": q, x + "k": k, x + "v": lin(H * E, d), x + "q.conv": cq, x + "k.conv": ck, x + "v.conv": conv(H * E, taps),
                      x + "b": b + 8.0 * loud, x + "A_log": 0.5 * r(H), x + "a1": lin(ra, d), x + "a2": 0.5 * lin(H * D, ra),
                      x + "dt_bias": (torch.where(slow, -9.0, -2.0).view(H, 1) + 0.3 * r(H, D)).reshape(-1), x + "g1": lin(rg, d),
                      x + "g2": lin(H * E, rg), x + "norm": gainful(E), x + "o": lin(d, H * E)})
        else:
            a, b, l, rt = m["left"], m["right"], x + "left.", x + "right."
            H, G, D, E, taps = (a[n] for n in ("heads", "kv_heads", "dim", "vdim", "conv"))
            k, q = queries(H, G, D)
            ck, cq = shared_conv(H, G, D, taps)
            W.update({l + "q": q, l + "k": k, l + "v": lin(G * E, d), l + "q.b": 0.2 * r(H * D), l + "k.b": 0.2 * r(G * D), l + "v.b": 0.3 * r(G * E),
                      l + "q.norm": gainful(H * D), l + "k.norm": gainful(G * D), l + "q.conv": cq, l + "k.conv": ck, l + "v.conv": conv(G * E, taps),
                      l + "sink": 1.0 + r(H), l + "o": lin(d, H * E), l + "out": gainful(d)})
            H, D, E = (b[n] for n in ("heads", "dim", "vdim"))
            slow = torch.rand(H, generator=g) < 0.6
            slow[0] = True
            W.update({rt + "q": lin(H * D, d), rt + "f": 0.5 * lin(H * D, d) - 14.0 * loud, rt + "v": lin(H * E, d) * (not cfg["quiet"]),
                      rt + "f.b": (torch.where(slow, 9.0, 2.0).view(H, 1) + 0.5 * r(H, D)).reshape(-1), rt + "lower": 0.4 * torch.rand(H * D, generator=g),
                      rt + "norm": gainful(E), rt + "o": lin(d, H * E), rt + "out": gainful(d)})
        if L["mlp"] is not None:
            ff = L["mlp"]["ff"]
            W.update({p + "norm2": one(), p + "mlp.up": lin(ff, d), p + "mlp.down": lin(d, ff)})
    return {k: v.to(torch.bfloat16) for k, v in W.items()}


def save_model(path, name, seed=0):
    """Writes config.json and model.safetensors; returns (folder, configuration, weights)."""
    from smcsd_b200.models.loader import save_safetensors
    cfg = CONFIGS[name] if isinstance(name, str) else name
    W = make_weights(cfg, seed)
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(W, os.path.join(path, "model.safetensors"))
    return str(path), cfg, W
