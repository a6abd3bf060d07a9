"""Prefill and decode of a layer-by-layer family beside existing models of equal size, whole forwards and kernel by kernel.

    python -m smcsd_b200.bench.layered --width 2048 --family makodra
    (or: python bench.py --layered 2048,1024 --layered-family makodra)

Pasizen runs beside a dense Llama-style model, Makodra beside that and a Gated-DeltaNet hybrid with as many attention layers,
Funevik beside a dense model, Makodra (memories, attention over heads) and Pasizen (latent attention, experts), Padadra beside a
dense model, the hybrid and Makodra.
All run random weights through their kernel chains: the same width, heads, layer count, head and feed-forward weights per
layer; the dense models cache as many bytes per token as their KV heads take.  A forward is captured in a CUDA
graph and timed with CUDA events (weights of all layers exceed L2; the cached keys come on top).  For the kernel table every
launch of one forward is recorded and the launches of one kind - the same kernel in all layers, so that the weights rotate -
are captured and timed together.  Fraction = (the larger of bytes / measured copy bandwidth and FLOPs / measured bf16 rate)
/ measured time; recurrent memories held to fp32 are set against the CUDA cores' fp32 rate instead.
"""
from __future__ import annotations

import argparse
import ctypes
import json
from collections import OrderedDict
from typing import Dict, List, Tuple

import torch

from ..models.config import (ChunkAttentionSpec, FeedForwardSpec, GluSpec, GroupedAttentionSpec, LatentAttentionSpec, LayerSpec, ModelConfig,
                             ParallelSpec, RecurrentSpec, RotarySpec, RouterSpec)
from ..utils.roofline import measured_peaks

VOCAB = 32768
F32_TFLOPS = 148 * 128 * 2 * 1.965e-3        # CUDA cores at the highest clock


def pasizen_config(width: int, layers: int, kv_rank: int, experts: bool) -> ModelConfig:
    H, ff = width // 128, 3 * width
    mixer = LatentAttentionSpec(heads=H, dim=128, vdim=128, kv_rank=kv_rank, scale=128 ** -0.5)
    dense = LayerSpec(mixer, FeedForwardSpec("dense", ff=ff))
    moe = LayerSpec(mixer, FeedForwardSpec("moe", expert=GluSpec(ff // 8, 7.0), router=RouterSpec(32, 4, 8, 4), shared=GluSpec(ff // 6, 7.0)))
    return ModelConfig(arch="pasizen", vocab_size=VOCAB, hidden_size=width, n_layers=layers, n_heads=H, n_kv_heads=1, head_dim=kv_rank,
                       ffn_size=0, rms_eps=1e-6, max_position=8192, layers=[moe if experts else dense] * layers, streams=4,
                       conv_taps=4, name=f"pasizen-{width}-{'experts' if experts else 'dense'}")


def dense_config(width: int, layers: int) -> ModelConfig:
    """The closest existing family: gate / up / down of the same number of weights as the two PolyNorm matrices."""
    return ModelConfig(arch="llama", vocab_size=VOCAB, hidden_size=width, n_layers=layers, n_heads=width // 128,
                       n_kv_heads=max(1, width // 512), head_dim=128, ffn_size=2 * width, rms_eps=1e-6, max_position=8192,
                       name=f"llama-{width}")


def hybrid_config(width: int, layers: int) -> ModelConfig:
    """Two Gated-DeltaNet layers to one attention layer, the feed-forward of ``makodra_config``."""
    H = width // 128
    return ModelConfig(arch="hybrid_gdn", vocab_size=VOCAB, hidden_size=width, n_layers=layers, n_heads=H, n_kv_heads=max(1, width // 512),
                       head_dim=128, ffn_size=2 * width, rms_eps=1e-6, max_position=8192, layer_types=["linear_attention", "linear_attention",
                       "full_attention"] * (layers // 3), gdn_n_k_heads=H, gdn_n_v_heads=H, gdn_head_k_dim=128, gdn_head_v_dim=128,
                       gdn_conv_width=4, partial_rotary=0.25, attn_output_gate=True, qk_norm=True, norm_plus_one=True,
                       name=f"hybrid-gdn-{width}")


def makodra_config(width: int, layers: int, memory_dim: int = 64, chunk: int = 8192) -> ModelConfig:
    """Delta rule, wkv and attention in turn; the chunk holds every sequence of the comparison, so that all keys are seen."""
    mlp, H = FeedForwardSpec("swiglu", ff=2 * width), width // memory_dim
    trio = [LayerSpec(RecurrentSpec("general_delta", H, memory_dim), mlp), LayerSpec(RecurrentSpec("wkv", H, memory_dim), mlp),
            LayerSpec(ChunkAttentionSpec(width // 128, max(1, width // 512), 128, 128, 11.3, chunk, True), mlp)]
    return ModelConfig(arch="makodra", vocab_size=VOCAB, hidden_size=width, n_layers=layers, n_heads=H, n_kv_heads=H, head_dim=memory_dim,
                       ffn_size=0, rms_eps=1e-6, max_position=1 << 20, tie_embeddings=True, logit_softcap=30.0, layers=trio * (layers // 3),
                       name=f"makodra-{width}-heads{memory_dim}")


def funevik_config(width: int, layers: int, kv_rank: int, experts: bool, window: int = 1024) -> ModelConfig:
    """Two memories, one latent and one full attention in turn; feed-forwards as in ``makodra_config`` or ``pasizen_config``."""
    H, rot = width // 128, RotarySpec(64, 10000.0)
    mlp = FeedForwardSpec("geglu", ff=2 * width)
    if experts:
        ff = 3 * width
        mlp = FeedForwardSpec("moe", expert=GluSpec(ff // 8), router=RouterSpec(32, 4, bias=True), shared=GluSpec(ff // 6), shared_gate=True)
    mem = RecurrentSpec("mlstm", max(1, width // 256), 128, 256, 15.0)
    four = [mem, mem, LatentAttentionSpec(H, 128, 128, kv_rank, 192 ** -0.5, 3 * width // 8, rot, window, True),
            GroupedAttentionSpec(H, max(1, H // 4), 128, 128, 128 ** -0.5, 4, rot, 50.0)]
    return ModelConfig(arch="funevik", vocab_size=VOCAB, hidden_size=width, n_layers=layers, n_heads=H, n_kv_heads=max(1, H // 4), head_dim=128,
                       ffn_size=0, rms_eps=1e-6, max_position=1 << 20, embed_scale=width ** 0.5, layers=[LayerSpec(m, mlp) for m in four * (layers // 4)],
                       name=f"funevik-{width}-{'experts' if experts else 'dense'}")


def padadra_config(width: int, layers: int, window: int = 1024) -> ModelConfig:
    """Two delta rules to one layer of attention beside a memory; the feed-forward has as many weights as ``makodra_config``'s."""
    H, rot = width // 128, RotarySpec(64, 500000.0, (8.0, 1.0, 4.0, 8192.0))
    mlp, delta = FeedForwardSpec("relu2", ff=3 * width), RecurrentSpec("channel_delta", H, 128, 128, kv_heads=max(1, H // 2), conv=4)
    both = ParallelSpec(GroupedAttentionSpec(H, max(1, H // 4), 128, 128, 128 ** -0.5, 4, rot, gate=False, window=window, learned_sink=True,
                                             bias=True, row_norm=True, turn_values=RotarySpec(128, rot.base)), RecurrentSpec("hgrn2", H, 128, 128))
    return ModelConfig(arch="padadra", vocab_size=VOCAB, hidden_size=width, n_layers=layers, n_heads=H, n_kv_heads=max(1, H // 4), head_dim=128,
                       ffn_size=0, rms_eps=1e-6, max_position=1 << 20, bigram=(32749, 31013, 4099), residual_mult=0.4,
                       layers=[LayerSpec(m, mlp) for m in [delta, delta, both] * (layers // 3)], name=f"padadra-{width}")


class Rig:
    """One model with its chain, caches filled with noise, and step inputs."""

    def __init__(self, cfg: ModelConfig, bs: int, ctx: int, prompt: int, n_prompts: int):
        from ..memory.pools import KVPool, StatePool
        from ..models import build_model
        from ..ops.native_backend import NativeLlama
        from ..ops.native_funevik import NativeFunevik
        from ..ops.native_hybrid import NativeHybrid
        from ..ops.native_makodra import NativeMakodra
        from ..ops.native_padadra import NativePadadra
        from ..ops.native_pasizen import NativePasizen
        dev = self.dev = torch.device("cuda", 0)
        self.cfg, self.bs, self.ctx, self.prompt, self.n_prompts = cfg, bs, ctx, prompt, n_prompts
        m = self.m = build_model(cfg, torch.bfloat16, dev, seed=3)
        span = max(ctx + 1, prompt)
        rows = max(bs, n_prompts)
        kv = self.kv = KVPool(m.kv_spec(torch.bfloat16), rows * span, dev)
        for t in list(kv.k) + list(kv.v):
            t.normal_(0, 0.5)
        perm = (torch.randperm(rows * span, generator=torch.Generator().manual_seed(1)) + 1).to(torch.int32)
        self.bt = perm.view(rows, span).to(dev).contiguous()               # scattered pages: the worst case for both
        self.status = torch.zeros(1, dtype=torch.int32, device=dev)
        T = n_prompts * prompt
        if cfg.arch != "llama":
            self.state = StatePool(m.state_spec(), rows, dev)
            Chain = {"pasizen": NativePasizen, "makodra": NativeMakodra, "funevik": NativeFunevik, "padadra": NativePadadra,
                     "hybrid_gdn": NativeHybrid}[cfg.arch]
            make = lambda t, lr: Chain(m, kv, self.bt, t, lr, 16, self.status, True, state=self.state)
        else:
            make = lambda t, lr: NativeLlama(m, kv, self.bt, t, lr, 16, self.status, True)
        self.dec, self.pre = make(bs, bs), make(T, 8)
        g = torch.Generator().manual_seed(2)
        i32 = lambda v: torch.as_tensor(v, dtype=torch.int32).to(dev)
        self.ids = i32(torch.randint(0, VOCAB, (bs,), generator=g))
        self.pos, self.rows, self.pref = i32([ctx] * bs), i32(list(range(bs))), i32([ctx] * bs)
        self.locs = self.bt[:bs, ctx].contiguous()
        self.p_ids = torch.randint(0, VOCAB, (T,), generator=g).tolist()
        self.dec.set_context(ctx + 1, bs, (1,))
        self.ragged = getattr(self.pre, "ragged", False)
        if self.ragged:
            from ..ops.ragged import Portion, pack_ragged
            portions = [Portion(r, 0, self.p_ids[r * prompt:(r + 1) * prompt]) for r in range(n_prompts)]
            self.plan = next(pack_ragged(portions, T, self.pre.BLOCK, self.bt))
        else:
            B = 16
            nb = prompt // B
            self.p_args = (i32(self.p_ids), i32(list(range(prompt)) * n_prompts), self.bt[:n_prompts, :prompt].reshape(-1).contiguous(),
                           i32([r for r in range(n_prompts) for _ in range(nb)]), i32([j * B for _ in range(n_prompts) for j in range(nb)]))
            self.pre.set_context(prompt, n_prompts * nb)
            self.seqs = {} if cfg.arch == "llama" else {"seqs": {
                "rows": i32(list(range(n_prompts))), "off": i32([r * prompt for r in range(n_prompts)]), "len": i32([prompt] * n_prompts),
                "n": n_prompts, "max": prompt}}

    def decode(self) -> None:
        self.dec.forward(self.ids, self.pos, self.locs, self.rows, self.pref, self.bs, 1)

    def prefill(self) -> None:
        if self.ragged:
            self.pre.forward_plan(self.plan)
        else:
            self.pre.forward(*self.p_args, self.n_prompts * self.prompt // 16, 16, two_pass=True, **self.seqs)


def timed(fn, reps: int = 20) -> float:
    """Microseconds per call, captured in a graph (so that host launch time is out)."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        fn()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    gr = torch.cuda.CUDAGraph()
    with torch.cuda.graph(gr):
        fn()
    for _ in range(3):
        gr.replay()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(reps):
        gr.replay()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / reps * 1e3


# ---------------------------------------------------------------------------------- kernel by kernel
RECORDED = ("gemm_skinny", "gemm_skinny_norm", "gemm_grouped", "add_rmsnorm", "attention_fused", "rope_kv_write", "hyper_step",
            "short_conv", "poly_norm", "route", "dispatch", "gather_rows", "latent_new", "latent_attention_tc", "gdn_step",
            "rope_kv_write_heads", "post_norm_step", "token_shift", "heads_new", "chunk_attention", "chunk_attention_tc", "memory_scan",
            "tanh_rows", "low_rank", "side_step", "conv_heads", "rotate_heads", "gated_step", "gated_chunk",
            "normed_heads", "conv_act", "memory_step")


def record(fn) -> List[Tuple[str, tuple, dict]]:
    """Every kernel call of one forward (structures copied: the chain reuses them)."""
    from ..ops import native as K
    calls, saved = [], {}

    def keep(x):
        return type(x).from_buffer_copy(x) if isinstance(x, ctypes.Structure) else x
    for name in RECORDED:
        real = saved[name] = getattr(K, name)

        def wrapped(*a, _real=real, _name=name, **kw):
            calls.append((_name, tuple(keep(x) for x in a), {k: keep(v) for k, v in kw.items()}))
            return _real(*a, **kw)
        setattr(K, name, wrapped)
    try:
        fn()
        torch.cuda.synchronize()
    finally:
        for name, real in saved.items():
            setattr(K, name, real)
    return calls


def work_of(rig: Rig, name: str, a: tuple, kw: dict, T: int, keys: float, seqs: int) -> Tuple[str, float, float]:
    """(kind, bytes, FLOPs) of a recorded call; ``keys``: cached rows an average token attends to; ``seqs``: sequences."""
    cfg = rig.cfg
    d = cfg.hidden_size
    if name in ("gemm_skinny", "gemm_skinny_norm", "gemm_grouped"):
        W, X, out = a[:3]
        M, N, Kd = kw["M"], (kw["N"] if "N" in kw else W.shape[0]), W.shape[-1]
        link = kw.get("link")
        groups = link.groups if link is not None and link.mode == 1 else 1
        wbytes = W.numel() * 2
        if link is not None and link.mode == 2:                # experts that some token chose (uniform choices)
            wbytes = wbytes * (1.0 - (1.0 - 1.0 / link.groups) ** M)
        flops = 2.0 * M * N * Kd * groups
        epi = kw["epi"]
        per_out = {1: 2, 2: 1, 3: 4, 4: 8, 8: 2}[epi]                # bytes per product (gated pairs leave half a bf16 value each)
        kind = f"gemm {N}x{Kd}" + (" relu2" if epi == 8 else "") + (f" x{groups} heads" if groups > 1 else "") + (" experts" if link is not None and link.mode == 2 else "")
        return kind, wbytes + M * Kd * 2 * groups + M * N * groups * per_out, flops
    if name == "latent_attention_tc":
        s = a[0]
        seen, held = keys, rig.ctx if T == rig.bs else rig.prompt
        if s.window:
            seen, held = min(keys, s.window), min(held, s.window) if T == rig.bs else held
        return ("latent " if rig.cfg.arch == "funevik" else "") + "attention", T * s.H * s.ldc * 4 + seqs * held * s.ldc * 2, 4.0 * T * s.H * seen * s.ldc
    if name == "attention_fused":
        H, Hkv, D = kw["Hq"], kw["Hkv"], kw["D"]
        fl = 2.0 * 2 * T * H * keys * D
        return "attention", T * H * D * 6 + seqs * (rig.ctx if T == rig.bs else rig.prompt) * Hkv * D * 4, fl
    if name in ("chunk_attention", "chunk_attention_tc"):
        s = a[0]
        seen, held = keys, rig.ctx if T == rig.bs else rig.prompt
        if s.window:
            seen, held = min(keys, s.window), min(held, s.window) if T == rig.bs else held
        fl = 2.0 * T * s.H * seen * (s.D + s.V)
        return "attention", T * s.H * (2 * s.D + (6 if s.gate else 2) * s.V) + seqs * held * s.G * (s.D + s.V) * 2, fl
    if name == "gated_chunk":                    # intra-chunk products and two with the state per token, at the bf16 rate
        s = a[0]
        return "memory gated (chunked)", T * s.H * (s.D * 8 + s.V * 10) + seqs * s.H * s.V * s.D * 8, 2.0 * T * s.H * (2 * s.V * s.D + 32 * (s.D + s.V))
    if name in ("memory_scan", "gated_step", "memory_step"):
        s, kind = a[0], 2 if name == "gated_step" else a[1]
        HD, HV = s.H * s.D, s.H * s.V
        # fp32 multiply-adds per matrix element and token, as bf16-rate equivalents (the floor divides by the bf16 rate)
        fl = 2.0 * (3, 5, 3, 4, 3)[kind] * T * HV * s.D * measured_peaks()[1] / F32_TFLOPS
        name = ("wkv", "delta", "gated", "channel delta", "hgrn2")[kind]
        return "memory " + name, T * (HD * 4 * (3, 4, 2, 2, 2)[kind] + HV * (10, 10, 10, 10, 6)[kind]) + seqs * HV * s.D * 8, fl
    if name == "side_step":
        s = a[0]
        by = T * d * (4 * (s.ids is None) + 4 * (not s.final) + 4 * bool(s.y1) + 4 * bool(s.y2) + 4 * bool(s.yb) + 4 * s.top + 2 + 2 * bool(s.w2) + 4 * bool(s.n2))
        return ("embedding + norms" if s.ids else "stream + final norm" if s.final else "stream + norms") + (" + experts" if s.top else "") + (" + pair" if s.yb else ""), by, 0.0
    if name == "conv_act":
        s = a[0]
        low = T * (s.k1 + s.k2) * 6 if s.low else (s.n1 * s.k1 + s.n2 * s.k2) * 2 + T * (s.k1 + s.k2 + s.n1 + s.n2) * 4
        return "conv + silu" + ("" if s.low else " + low-rank maps"), T * s.C * 8 + low, 0.0 if s.low else 2.0 * T * (s.n1 * s.k1 + s.n2 * s.k2)
    if name in ("conv_heads", "normed_heads"):
        s = a[0]
        return "conv + " + ("norms + " if name == "normed_heads" else "") + "rotation + new heads", T * ((s.H + s.G) * s.D + s.G * s.V) * 6, 0.0
    if name == "rotate_heads":
        return "rotate queries", T * kw["heads"] * kw["width"] * 6, 0.0
    if name == "gdn_step":
        Hv, dk, dv = kw["Hv"], kw["dk"], kw["dv"]
        conv = 2 * kw["Hk"] * dk + Hv * dv
        return "memory gdn + conv", T * (conv * 12 + Hv * dv * 6) + seqs * Hv * dk * dv * 8, 2.0 * 4 * T * Hv * dk * dv
    if name == "post_norm_step":
        s = a[0]
        return "norm + residual" + (" + shift" if s.mu else ""), T * d * (4 + 8 + (2 if s.xa else 0) + (8 + 2 * s.n_mix if s.mu else 0)), 0.0
    if name == "token_shift":
        return "token shift", T * d * (4 + 2 * a[1].shape[0]), 0.0
    if name == "heads_new":
        s = a[0]
        return "new heads", T * ((s.H + s.G) * s.D * 6 + s.G * s.V * (6 + 4 * bool(s.v_first))), 0.0
    if name == "low_rank":
        W = a[1]
        return "decay logits", W.numel() * 2 + T * (W.shape[0] + W.shape[1]) * 4, 2.0 * T * W.numel()
    if name == "tanh_rows":
        return "tanh", T * kw["n"] * 6, 0.0
    if name == "hyper_step":
        s = a[0]
        S = s.S
        by = T * d * (4 * S * (1 + (s.w_in is not None)) + 4 * (s.y is not None) + 4 * s.top + 4 * (s.n_out is not None) + 2 * (s.xa is not None))
        return "streams + norm" + (" + conv" if s.conv_w else "") + (" + experts" if s.top else ""), by, 0.0
    sizes = {"add_rmsnorm": T * d * 10, "short_conv": T * d * 6, "rope_kv_write": T * (cfg.q_size + 2 * cfg.kv_size) * 6,
             "rope_kv_write_heads": T * (cfg.q_size + 2 * cfg.kv_size) * 6}
    if name == "poly_norm":
        return "PolyNorm", T * kw["ff"] * 6, 0.0
    if name == "latent_new":
        s = a[0]
        return "latent_new", T * (s.nq + s.R + s.rot) * 6, 0.0
    if name == "gather_rows":
        return "gather_rows", kw["n"] * a[2].shape[1] * 4, 0.0
    if name == "route":
        return "route", T * kw["d"] * 4 + a[1].numel() * 2, 2.0 * T * kw["d"] * a[1].shape[0]
    if name == "dispatch":
        return "dispatch", kw["n"] * 12, 0.0
    return name, float(sizes[name]), 0.0


def kernel_table(rig: Rig, fn, T: int, keys: float, seqs: int) -> List[dict]:
    from ..ops import native as K
    hbm, tflops, _ = measured_peaks()
    kinds: Dict[str, dict] = OrderedDict()
    for name, a, kw in record(fn):
        kind, by, fl = work_of(rig, name, a, kw, T, keys, seqs)
        k = kinds.setdefault(kind, {"kernel": kind, "calls": [], "bytes": by, "flops": fl})
        k["calls"].append((getattr(K, name), a, kw))
    out = []
    for k in kinds.values():
        calls = k.pop("calls")
        us = timed(lambda: [f(*a, **kw) for f, a, kw in calls], reps=8) / len(calls)
        floor = max(k["bytes"] / (hbm * 1e3), k["flops"] / (tflops * 1e6))
        out.append({**k, "launches": len(calls), "us": round(us, 2), "floor_us": round(floor, 2), "fraction": round(floor / us, 3)})
    return out


def run(width: int, layers: int = 12, bs: int = 8, ctx: int = 1024, prompt: int = 1024, n_prompts: int = 4, kv_rank: int = 256,
        tables: bool = True, family: str = "pasizen") -> dict:
    import gc
    rec = {"width": width, "layers": layers, "decode": {"sequences": bs, "context": ctx}, "prefill": {"prompts": n_prompts, "tokens": prompt},
           "kv_rank": kv_rank if family in ("pasizen", "funevik") else None, "pages": "scattered", "weights": "random, bf16", "models": []}
    own = {"pasizen": lambda: [pasizen_config(width, layers, kv_rank, False), pasizen_config(width, layers, kv_rank, True)],
           "makodra": lambda: [hybrid_config(width, layers), makodra_config(width, layers), makodra_config(width, layers, 128)],
           "funevik": lambda: [makodra_config(width, layers, 128), pasizen_config(width, layers, kv_rank, True),
                               funevik_config(width, layers, kv_rank, False), funevik_config(width, layers, kv_rank, True)],
           "padadra": lambda: [hybrid_config(width, layers), makodra_config(width, layers, 128), padadra_config(width, layers)]}[family]()
    for cfg in [dense_config(width, layers)] + own:
        rig = Rig(cfg, bs, ctx, prompt, n_prompts)
        T = n_prompts * prompt
        dec, pre = timed(rig.decode), timed(rig.prefill, reps=8)
        one = {"model": cfg.name, "weight_mb": rig.m.weight_bytes() / 1e6, "decode_us": round(dec, 1), "decode_tok_s": round(bs / dec * 1e6),
               "prefill_us": round(pre, 1), "prefill_tok_s": round(T / pre * 1e6)}
        if tables:
            one["decode_kernels"] = kernel_table(rig, rig.decode, bs, ctx + 1, bs)
            one["prefill_kernels"] = kernel_table(rig, rig.prefill, T, (prompt + 1) / 2, n_prompts)
        one["device_status"] = int(rig.status.item())
        rec["models"].append(one)
        del rig
        gc.collect()
        torch.cuda.empty_cache()
    return rec


def show(rec: dict) -> str:
    lines = [f"width {rec['width']}, {rec['layers']} layers{', kv_rank ' + str(rec['kv_rank']) if rec['kv_rank'] else ''}; decode {rec['decode']}, prefill {rec['prefill']}, "
             f"pages {rec['pages']}"]
    for m in rec["models"]:
        lines.append(f"{m['model']}: {m['weight_mb']:.0f} MB  decode {m['decode_us']} us ({m['decode_tok_s']} tok/s)  prefill "
                     f"{m['prefill_us']} us ({m['prefill_tok_s']} tok/s)  status {m['device_status']}")
        for part in ("decode_kernels", "prefill_kernels"):
            for k in m.get(part, []):
                lines.append(f"  {part[:7]:8}{k['kernel']:34}{k['launches']:4} x {k['us']:9.2f} us  floor {k['floor_us']:8.2f}  {k['fraction']:.3f}")
    return "\n".join(lines)


def main(argv=None) -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--width", type=int, default=2048)
    ap.add_argument("--layers", type=int, default=12)
    ap.add_argument("--bs", type=int, default=8)
    ap.add_argument("--ctx", type=int, default=1024)
    ap.add_argument("--prompt", type=int, default=1024)
    ap.add_argument("--kv-rank", type=int, default=256)
    ap.add_argument("--family", default="pasizen", choices=["pasizen", "makodra", "funevik", "padadra"])
    ap.add_argument("--no-tables", action="store_true")
    ap.add_argument("--json", default=None)
    ns = ap.parse_args(argv)
    rec = run(ns.width, ns.layers, ns.bs, ns.ctx, ns.prompt, kv_rank=ns.kv_rank, tables=not ns.no_tables, family=ns.family)
    print(show(rec))
    if ns.json:
        with open(ns.json, "w") as f:
            json.dump(rec, f)


if __name__ == "__main__":
    main()
