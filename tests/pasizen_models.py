"""Small Pasizen models with weights chosen so that faults show: equal tokens attract each other whatever their distance
(queries are the keys' own map of the latent), attention is sharp, and every constant differs from a neutral value."""
import json
import os

import torch


def mixer(heads, dim, vdim, rank, scale=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": dim ** -0.5 if scale is None else scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, count, keep, ff, limit, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}},
         "expert": {"ff": ff, "limit": limit}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def config(width, layers, streams, taps, loop=None, vocab=211, positions=700, eps=1e-5):
    c = {"architecture": "Pasizen", "vocab": vocab, "width": width, "max_positions": positions, "norm": {"eps": eps},
         "canon": {"taps": taps}, "streams": streams,
         "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CONFIGS = {
    "looped_mix": config(136, [(mixer(3, 40, 24, 48), dense(200)), (mixer(2, 32, 56, 72), moe(8, 2, 4, 2, 40, 0.9, (72, 1.3))),
                               (mixer(3, 40, 24, 48), None)], streams=2, taps=3, loop=(1, 3, 2)),
    "odd_sizes": config(100, [(mixer(5, 20, 72, 130, 0.31), moe(6, 3, 1, 1, 33, 0.7)), (mixer(1, 12, 28, 20), dense(77))],
                        streams=4, taps=2, eps=1e-3),
    "one_layer": config(64, [(mixer(4, 16, 16, 64), dense(96))], streams=1, taps=1, vocab=97),
    "looped_all": config(192, [(mixer(6, 24, 40, 96), moe(6, 1, 3, 1, 64, 2.5, (128, 0.6))), (mixer(12, 64, 32, 200), dense(256))],
                         streams=3, taps=5, loop=(0, 2, 3), vocab=300),
}


def make_weights(cfg, seed=0, gain=8.0):
    """name -> bf16 tensor."""
    g = torch.Generator().manual_seed(seed)
    d, S, V = cfg["width"], cfg["streams"], cfg["vocab"]
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    gainful = lambda n: 1.0 + 0.3 * r(n)
    W = {"embed": r(V, d), "pos": 0.2 * r(cfg["max_positions"], d), "final.norm": gainful(d), "head": lin(V, d)}
    for li, L in enumerate(cfg["layers"]):
        p, m, f = f"l{li}.", L["mixer"], L["mlp"]
        H, D, R = m["heads"], m["dim"], m["kv_rank"]
        dkv, uk = lin(R, d), lin(H * D, R)
        c_norm = gainful(R)
        q = (gain / (m["scale"] * D) * (uk * c_norm).view(H, D, R) @ dkv).reshape(H * D, d) * (D / R) ** 0.5
        W.update({p + "norm1": gainful(d), p + "canon1": r(d, cfg["canon"]["taps"]) * 0.3, p + "mix.q": q, p + "mix.dkv": dkv,
                  p + "mix.dkv.norm": c_norm, p + "mix.uk": uk, p + "mix.uv": lin(H * m["vdim"], R), p + "mix.o": 3.0 * lin(d, H * m["vdim"])})
        for k in ("hc1.", "hc2.")[:1 if f is None else 2]:
            W.update({p + k + "in": 1.0 / S + 0.2 * r(S), p + k + "out": 1.0 + 0.3 * r(S),
                      p + k + "mix": 0.8 * torch.eye(S) + 0.2 * r(S, S) / S ** 0.5})
        if f is None:
            continue
        W[p + "norm2"] = gainful(d)

        def glu(name, ff):
            W.update({name + "gate": lin(ff, d), name + "up": lin(ff, d), name + "down": lin(d, ff)})
        if f["kind"] == "dense":
            W.update({p + "mlp.up": lin(f["ff"], d), p + "mlp.down": lin(d, f["ff"]), p + "mlp.act": torch.tensor([0.7, -0.4, 0.3, 0.15])})
        else:
            W[p + "mlp.router"] = 8.0 * lin(f["router"]["experts"], d)
            for e in range(f["router"]["experts"]):
                glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
            if f.get("shared"):
                glu(p + "mlp.shared.", f["shared"]["ff"])
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


def tokens(cfg, n, seed=0):
    """Random ids; the last token equals the first, which occurs nowhere else (a far key that the last query singles out)."""
    ids = torch.randint(0, cfg["vocab"] - 1, (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()
    ids[0] = ids[-1] = cfg["vocab"] - 1
    return ids


def far_effect(forward, cfg, ids, ref):
    """How far the last row moves when only the first token changes; ``forward(ids)`` gives logits."""
    return row_error(forward([ids[0] - 1] + ids[1:])[-1:], ref[-1:]).item()


def row_error(got, ref):
    """Per row: rms difference after taking the mean off, over the spread of the reference logits."""
    d = got.double().cpu() - ref.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / ref.double().cpu().std(-1).mean()
