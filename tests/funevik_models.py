"""Small Funevik models with weights chosen so that faults show: in every layer the queries of the token SEEKER single out the keys
of the token SOUGHT, whatever their distance, a part of every memory hardly decays, and every constant differs from a neutral
value."""
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


def mem(heads, dim, vdim, cap=9.0):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def latent(heads, dim, vdim, kv_rank, q_rank, rot, window, base=3000.0, scale=None):
    return "latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot_dim": rot,
                                "rot": {"base": base, "dims": rot}, "mask": {"size": window}, "scale": 4.0 / dim if scale is None else scale}


def attn(heads, kv_heads, dim, vdim, rot, conv=3, cap=21.0, base=900.0, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "softcap": cap,
                         "rot": {"base": base, "dims": rot}, "scale": 4.0 / dim if scale is None else scale}


def moe(experts, top, ff, shared):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(width, layers, vocab=211, eps=1e-5, scale=5.0):
    """``layers``: (mixer, feed-forward or None)."""
    return {"architecture": "Funevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": [{"type": kind, "mixer": mixer, "mlp": f} for (kind, mixer), f in layers]}


CONFIGS = {
    "all_kinds": config(136, [(latent(6, 24, 40, 56, 72, 8, 48), dense(96)), (mem(3, 40, 24), moe(8, 3, 48, 40)),
                              (attn(4, 2, 40, 24, 12), moe(5, 2, 64, 72)), (mem(5, 24, 56), None)]),
    "odd_sizes": config(100, [(attn(3, 1, 20, 12, 20, conv=1, cap=9.0), None), (mem(1, 70, 33, 4.0), dense(77)),
                              (latent(5, 18, 12, 30, 21, 6, 21), moe(3, 1, 20, None)), (attn(5, 5, 28, 44, 2, conv=5), dense(130))],
                        eps=1e-3, vocab=97, scale=0.7),
    "latent_only": config(96, [(latent(2, 32, 16, 64, 40, 16, 33), dense(64)), (latent(8, 16, 24, 100, 130, 32, 70), None)], vocab=300),
    "memory_only": config(64, [(mem(4, 16, 16), None), (mem(1, 64, 130), dense(50)), (mem(2, 130, 40, 20.0), moe(4, 2, 24, 16))]),
}


GAIN = 2.5


def make_weights(cfg, seed=0):
    """name -> bf16 tensor."""
    g = torch.Generator().manual_seed(seed)
    d, V = cfg["width"], cfg["vocab"]
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    gainful = lambda n: 1.0 + 0.3 * r(n)
    W = {"embed": r(V, d) / cfg["embedding"]["scale"], "head": lin(V, d), "final.norm": gainful(d)}
    unit = lambda v: v / v.pow(2).mean().sqrt()
    sought, seeker = (unit(W["embed"][t]) for t in pair(cfg))

    def seek(q, k, hears, wants):
        """Query map [H, D, n] to which ``hears`` [n] gives ``GAIN`` times what the key map [H, D, n'] makes of ``wants``."""
        return q + GAIN * torch.einsum("hdn,n,m->hdm", k, wants, hears / hears.pow(2).sum())
    for li, L in enumerate(cfg["layers"]):
        p, m, f = f"l{li}.", L["mixer"], L["mlp"]
        x, H, D, E = p + "mix.", m["heads"], m["dim"], m["vdim"]
        W.update({p + "norm1": gainful(d), p + "ls1": 0.8 * gainful(d)})
        if L["type"] == "mlstm":
            k = lin(H * D, d)
            slow = torch.rand(H, generator=g) < 0.6            # these heads keep what they hold
            slow[0] = True
            loud = sought * W[p + "norm1"]                     # and this token enters with more weight
            q = seek(lin(H * D, d).view(H, D, d), k.view(H, D, d), seeker * W[p + "norm1"], sought * W[p + "norm1"])
            W.update({x + "k": k, x + "q": q.reshape(H * D, d), x + "v": lin(H * E, d), x + "g": 0.5 * lin(H * E, d),
                      x + "i": lin(H, d) + 6.0 * loud / loud.pow(2).sum(), x + "i.b": -2.0 + 0.5 * r(H), x + "f": 0.3 * lin(H, d), x + "f.b": torch.where(slow, 30.0, 1.0) + 0.3 * r(H),
                      x + "norm": gainful(H * E), x + "o": lin(d, H * E)})
        elif L["type"] == "latent_attention":
            R, Q, rot, n1 = m["kv_rank"], m["q_rank"], m["rot_dim"], W[p + "norm1"]
            dkv, uk, dq, uq = lin(R + rot, d), lin(H * D, R), lin(Q, d), lin(H * (D + rot), Q).view(H, D + rot, Q)
            qn, cn = gainful(Q), gainful(R)
            c = unit(dkv[:R] @ (sought * n1)) * cn
            uq[:, :D] = seek(uq[:, :D], uk.view(H, D, R), unit(dq @ (seeker * n1)) * qn, c)
            W.update({x + "dq": dq, x + "dq.norm": qn, x + "uq": uq.reshape(H * (D + rot), Q), x + "dkv": dkv, x + "dkv.norm": cn,
                      x + "uk": uk, x + "uv": lin(H * E, R), x + "sink": 1.0 + r(H), x + "o": lin(d, H * E)})
        else:
            G, taps = m["kv_heads"], m["conv"]
            k = lin(G * D, d)

            def conv(n):
                w = 0.3 * r(n, taps)
                w[:, -1] = 1.0 + 0.1 * r(n)
                return w
            ck = conv(G * D)
            q = seek(lin(H * D, d).view(H, D, d), k.view(G, D, d).repeat_interleave(H // G, 0), seeker * W[p + "norm1"], sought * W[p + "norm1"])
            W.update({x + "k": k, x + "q": q.reshape(H * D, d), x + "v": lin(G * E, d), x + "k.conv": ck, x + "v.conv": conv(G * E),
                      x + "q.conv": ck.view(G, 1, D, taps).repeat(1, H // G, 1, 1).reshape(H * D, taps), x + "g": lin(H, d), x + "o": lin(d, H * E)})
        if f is None:
            continue
        W.update({p + "norm2": gainful(d), p + "ls2": 0.6 * gainful(d)})

        def glu(name, ff):
            W.update({name + "gate": lin(ff, d), name + "up": lin(ff, d), name + "down": lin(d, ff)})
        if f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
            continue
        n = f["router"]["experts"]
        W.update({p + "mlp.router": 8.0 * lin(n, d), p + "mlp.router.b": 2.0 * r(n)})
        for e in range(n):
            glu(f"{p}mlp.e{e}.", f["expert"]["ff"])
        if f["shared"]:
            glu(p + "mlp.shared.", f["shared"]["ff"])
            W[p + "mlp.shared.sg"] = lin(1, d)
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
