"""Small Makodra models with weights chosen so that faults show: equal tokens attract each other (receptances and queries are
the keys' own map), a part of every recurrent memory hardly decays, and every constant differs from a neutral value."""
import json
import os

import torch

from pasizen_models import row_error, tokens  # noqa: F401  (the suite takes both from the family's module)


def attn(heads, kv_heads, dim, vdim, chunk, v_mix=True, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "v_mix": v_mix, "mask": {"size": chunk},
                         "scale": 7.0 / dim if scale is None else scale}


def delta(heads, dim):
    return "general_delta", {"heads": heads, "dim": dim}


def wkv(heads, dim):
    return "wkv", {"heads": heads, "dim": dim}


def config(width, layers, vocab=211, eps=1e-5, cap=17.0, ff=96):
    """``layers``: mixers, or (mixer, ff) with ff None for a layer without feed-forward."""
    out = []
    for m in layers:
        (kind, mixer), f = m if isinstance(m[0], tuple) else (m, ff)
        out.append({"type": kind, "mixer": mixer, "mlp": None if f is None else {"kind": "dense", "ff": f}})
    return {"architecture": "Makodra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_softcap": cap, "layers": out}


CONFIGS = {
    "all_kinds": config(136, [delta(3, 40), attn(6, 2, 24, 40, 48), wkv(5, 24), attn(4, 2, 72, 40, 33)]),
    "odd_sizes": config(100, [(wkv(2, 50), 77), (attn(3, 1, 20, 12, 21, v_mix=False), None), (delta(1, 70), 130), (attn(5, 5, 12, 28, 100), 40)],
                        eps=1e-3, cap=None, vocab=97),
    "attention_only": config(96, [(attn(2, 2, 32, 16, 64), None)], vocab=300),
    "memory_only": config(64, [(delta(4, 16), None), (wkv(1, 64), 50), (wkv(8, 8), None), delta(2, 130)], cap=5.0),
}


def make_weights(cfg, seed=0, gain=1.5):
    """name -> bf16 tensor."""
    g = torch.Generator().manual_seed(seed)
    d, V = cfg["width"], cfg["vocab"]
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    gainful = lambda n: 1.0 + 0.3 * r(n)
    W = {"embed": 2.0 * r(V, d), "final.norm": 0.3 * gainful(d)}
    for li, L in enumerate(cfg["layers"]):
        p, m, f = f"l{li}.", L["mixer"], L["mlp"]
        x, H, D = p + "mix.", m["heads"], m["dim"]
        W[p + "norm1"] = 1.5 * gainful(d)
        if L["type"] == "attention":
            G, Vd = m["kv_heads"], m["vdim"]
            k = lin(G * D, d)
            W.update({x + "q": k.view(G, 1, D, d).repeat(1, H // G, 1, 1).reshape(H * D, d) + 0.2 * lin(H * D, d), x + "k": k,
                      x + "v": lin(G * Vd, d), x + "g": lin(H * Vd, d), x + "o": lin(d, H * Vd),
                      x + "r1": 0.2 + 0.3 * torch.rand(H, generator=g), x + "r2": 0.1 + torch.rand(H, generator=g)})
            if m["v_mix"]:
                W[x + "vmix"] = torch.tensor(0.35 + 0.05 * li)
        else:
            n, delta_rule = H * D, L["type"] == "general_delta"
            rank = 12 if li % 2 else 20
            k = lin(n, d) * D ** -0.5
            slow = torch.rand(n, generator=g) < 0.5            # these channels keep what they hold
            W.update({x + "k": k, x + "r": gain * k + 0.2 * lin(n, d) * D ** -0.5, x + "v": lin(n, d), x + "g": 0.5 * lin(n, d),
                      x + "w1": lin(rank, d), x + "w2": 0.3 * lin(n, rank), x + "norm": gainful(n), x + "o": lin(d, n),
                      x + "w0": torch.where(slow, torch.tensor(-9.0), torch.tensor(-1.0)) + 0.3 * r(n)})
            if delta_rule:
                W.update({x + "a": 0.3 * lin(n, d), x + "a.b": -3.0 + 0.5 * r(n)})
            else:
                W[x + "u"] = 0.5 + 0.5 * r(H, D)
                for s in "rkvgw":
                    W[x + "mu." + s] = 0.3 + 0.2 * r(d)
        if f is not None:
            W.update({p + "norm2": gainful(d), p + "mlp.gate": lin(f["ff"], d), p + "mlp.up": lin(f["ff"], d), p + "mlp.down": lin(d, f["ff"])})
    return {k: v.to(torch.bfloat16) for k, v in W.items()}


def save_model(path, name, seed=0, **changed):
    """Writes config.json and model.safetensors; returns (folder, configuration, weights).  ``changed`` multiplies all weights
    with a leaf name by a factor."""
    from smcsd_b200.models.loader import save_safetensors
    cfg = CONFIGS[name] if isinstance(name, str) else name
    W = make_weights(cfg, seed)
    W = {k: w * changed.get(k.rsplit(".", 1)[-1], 1.0) for k, w in W.items()}
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_safetensors(W, os.path.join(path, "model.safetensors"))
    return str(path), cfg, W
