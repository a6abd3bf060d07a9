"""Kernel-chain forward of Funevik on sm_100a, in bf16 (tensor cores) or in 32-bit.

A layer, between two steps of the residual stream (both outputs added, the new row under the next layer's two norms):
  mlstm      projections -> scan (gates, normaliser, norm and output gate) -> output
  attention  projections -> convolution, rotation, new keys and values to the cache -> soft-capped attention with the head
             gates -> output
  latent     projections -> query latent normed, cached latent and rotated key to the cache -> queries -> rotation -> queries into
             latent space (one product per head, the rotated part passed on) -> windowed attention with sinks over cached rows
             -> value expansion -> output
  geglu      gate / up with the gated epilogue -> down
  experts    router (with the shared expert's gate) -> dispatch -> gather -> gate / up -> down, all experts in one launch each,
             beside the shared expert; the next step of the stream adds the weighted rows
Sequences may bring any number of new tokens each (``ops/ragged.py``); a uniform batch runs without index arrays and can be
captured in a graph.
"""
from __future__ import annotations

import math
from contextlib import nullcontext
from typing import Dict, List, Optional

import torch

from ..models.config import RotarySpec
from ..models.funevik import conv_channels, latent_row
from ..models.layered import GU_BLOCK, round_up
from ..models.layers import NORMALISER_EPS
from . import native as K
from .native_layered import NativeLayered, env_flag


class NativeFunevik(NativeLayered):
    CHUNK_MIN_TOKENS = 32                 # portions at least this long take the chunked form of the memories

    def __init__(self, model, kv, block_table: torch.Tensor, max_tokens: int, max_logit_rows: int, attn_splits: int,
                 status: torch.Tensor, pdl: bool, state=None):
        super().__init__(model, kv, block_table, max_tokens, max_logit_rows, attn_splits, status, pdl, state)
        T, ls, d = max_tokens, model.layers, self.d
        most = lambda it: max(it, default=0)
        kinds = lambda k: [L.spec.mixer for L in ls if L.kind == k]
        mlps = [L.spec.mlp for L in ls if L.spec.mlp is not None]
        moe, dense = [f for f in mlps if f.kind == "moe"], [f.ff for f in mlps if f.kind != "moe"]
        self.x = torch.zeros(T, d, dtype=torch.float32, device=self.dev)
        self.xb = torch.zeros(T, self.d8, dtype=self.dt, device=self.dev)       # rows under the feed-forward's norm
        self._room("n2", T * d if moe else 0, torch.float32)
        self._room("proj", T * most(L.win.shape[0] for L in ls), torch.float32)
        self._room("vo", T * most(L.wo.shape[1] for L in ls), self.dt)
        self._room("q", T * most([m.heads * round_up(m.dim, 8) for m in kinds("attention")] +
                                 [L.wuq.shape[0] for L in ls if L.kind == "latent"]), self.dt)
        self._room("cq", T * most(L.wuq.shape[1] for L in ls if L.kind == "latent"), self.dt)
        self._room("qf", T * most(L.wuq.shape[0] for L in ls if L.kind == "latent"), torch.float32)
        for name in ("lat", "ctx"):
            self._room(name, T * most(m.heads * latent_row(m) for m in kinds("latent")), self.dt)
        for name in ("y1", "y2"):
            self._room(name, T * d, torch.float32)
        self._room("act", T * most(round_up(n, GU_BLOCK) for n in dense + [f.shared.ff for f in moe if f.shared]), self.dt)
        self._room("sg", T if any(f.shared for f in moe) else 0, torch.float32)
        self._room_experts(moe)
        self._room_gate_up(dense, moe)
        self.attn_tc = not self.f32
        self.memory_tc = not self.f32 and env_flag("SMC_GATED_CHUNK", True)
        self.beside = env_flag("SMC_BESIDE", True)
        self.freq: Dict[RotarySpec, torch.Tensor] = {}
        for rot in {L.spec.mixer.rot for L in ls if L.kind != "mlstm"}:
            self.freq[rot] = rot.base ** (-torch.arange(0, rot.dims, 2, dtype=torch.float64, device=self.dev) / rot.dims)
        self.taps = [L.conv.t().contiguous() if L.conv is not None else None for L in ls]
        self._steps = self._build_steps()

    def _build_steps(self) -> List["K.SideArgs"]:
        """Arguments of the stream step in front of every layer, and of the last one, which ends with the final norm."""
        m, steps, flat = self.m, [], self._flat
        for before, L in zip([None] + m.layers, m.layers + [None]):
            a = K.SideArgs(x=K.ptr(self.x), d=self.d, vocab=self.c.vocab_size, eps=self.c.rms_eps, ldy=self.d, ldye=self.d, xa=K.ptr(self.xa),
                           ldxa=self.d8, status=K.ptr(self.status), pdl=int(self.pdl))
            if before is None:
                a.embed, a.embed_scale = K.ptr(m.embed), self.c.embed_scale
            else:
                f = before.spec.mlp
                a.y1, a.s1, a.s2 = K.ptr(flat["y1"]), K.ptr(before.ls1), K.ptr(before.ls2)
                if f is not None and f.kind == "moe":
                    a.ye, a.top = K.ptr(flat["ye"]), f.router.top
                    a.route_slot, a.route_w = K.ptr(flat["slot"]), K.ptr(flat["wgt"])
                    if f.shared is not None:
                        a.y2, a.gate = K.ptr(flat["y2"]), K.ptr(flat["sg"])
                elif f is not None:
                    a.y2 = K.ptr(flat["y2"])
            if L is None:
                a.w1, a.final = K.ptr(m.final_norm), 1
            else:
                a.w1 = K.ptr(L.norm1)
                if L.spec.mlp is not None:
                    a.w2, a.xb = K.ptr(L.norm2), K.ptr(self.xb)
                    if L.spec.mlp.kind == "moe":
                        a.n2 = K.ptr(flat["n2"])
            steps.append(a)
        return steps

    # ---- planning -----------------------------------------------------------------------
    def set_context(self, ctx: int, bs: int, Es=(1, 2)) -> tuple:
        """Record the context-length hint; returns what it decides about the launch grids (part of a graph's identity)."""
        self.ctx_hint = int(ctx)
        out = []
        for E in Es:
            for i, L in enumerate(self.m.layers):
                m = L.spec.mixer
                if L.kind == "latent":
                    blocks = bs * ((E + self.BLOCK - 1) // self.BLOCK)
                    out.append((E, i, self._latent_splits(blocks, min(E, self.BLOCK), m.heads, latent_row(m), m.window)))
                elif L.kind == "attention":
                    out.append((E, i, self._chunk_splits(bs * E, m, 0)))
        return tuple(out)

    # ---- mixers -------------------------------------------------------------------------
    def _memory(self, i: int, L, T: int, positions, locs, work: "K.Ragged", longest: int) -> torch.Tensor:
        m = L.spec.mixer
        H, D, E, ldo = m.heads, m.dim, m.values, L.wo.shape[1]
        proj, vo = self._rows("proj", T, L.win.shape[0]), self._rows("vo", T, ldo)
        S, top = self.state.matrix(L.state), self.state.matrix(L.state + 1)
        a = K.ScanArgs(proj=K.ptr(proj), ldp=proj.stride(0), r_off=0, k_off=H * D, v_off=2 * H * D, g_off=H * (2 * D + E),
                       a_off=2 * H * (D + E), a_bias=K.ptr(L.gate_bias), onorm=K.ptr(L.onorm), state=K.ptr(S), row_stride=S.stride(0),
                       n_rows=S.shape[0], out=K.ptr(vo), ldo=ldo, H=H, D=D, V=E, eps=self.c.rms_eps, unit_eps=NORMALISER_EPS, top=K.ptr(top),
                       gate_cap=m.gate_cap, r_scale=D ** -0.5, r=work, status=K.ptr(self.status), pdl=int(self.pdl))
        if longest == 1 and K.gated_step_takes(D, E):
            K.gated_step(a, self.f32)
        elif self.memory_tc and longest >= self.CHUNK_MIN_TOKENS and K.gated_chunk_takes(D, E):
            K.gated_chunk(a)
        else:
            K.memory_scan(a, K.SCAN_GATED, self.f32)
        return vo

    def _attention(self, i: int, L, T: int, positions, locs, work: "K.Ragged", longest: int) -> torch.Tensor:
        m, pdl, st = L.spec.mixer, int(self.pdl), K.ptr(self.status)
        H, G, D, V, C = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8), conv_channels(m)
        kp, vp = self.kv.k[L.cache], self.kv.v[L.cache]
        proj, q, vo = self._rows("proj", T, L.win.shape[0]), self._rows("q", T, H * D), self._rows("vo", T, H * V)
        hist = self.state.matrix(L.state) if m.conv > 1 else None
        K.conv_heads(K.ConvHeadsArgs(proj=K.ptr(proj), ldp=proj.stride(0), H=H, G=G, D=D, V=V, rot=m.rot.dims, conv=K.ptr(self.taps[i]),
                                     taps=m.conv, hist=K.ptr(hist), row_stride=hist.stride(0) if hist is not None else 0,
                                     n_rows=hist.shape[0] if hist is not None else 0, freq=K.ptr(self.freq[m.rot]),
                                     positions=K.ptr(positions), q=K.ptr(q), kpool=K.ptr(kp), vpool=K.ptr(vp), n_pages=kp.shape[0] - 1,
                                     locs=K.ptr(locs), r=work, status=st, pdl=pdl), self.f32)
        a = K.ChunkAttnArgs(q=K.ptr(q), kpool=K.ptr(kp), vpool=K.ptr(vp), out=K.ptr(vo), gate=K.ptr(proj[:, C:]), ldg=proj.stride(0),
                            gate_heads=1, block_table=K.ptr(self.bt), bt_stride=self.bt.stride(0), bt_rows=self.bt.shape[0],
                            n_pages=kp.shape[0] - 1, H=H, G=G, D=D, V=V, chunk=1 << 30, scale=m.scale, softcap=m.softcap, sink=1, r=work,
                            status=st, pdl=pdl)
        self._chunk_attention(a, m, 0, T, longest)
        return vo

    def _latent(self, i: int, L, T: int, positions, locs, work: "K.Ragged", longest: int) -> torch.Tensor:
        m, pdl = L.spec.mixer, int(self.pdl)
        H, D, R, r, Rp = m.heads, m.dim, m.kv_rank, m.rot.dims, latent_row(m)
        Q8, K8, pool, freq = L.wuq.shape[1], L.wuk_t.shape[1], self.kv.k[L.cache], self.freq[m.rot]
        proj, cq = self._rows("proj", T, L.win.shape[0]), self._rows("cq", T, Q8)
        K.latent_new(K.LatentNewArgs(proj=K.ptr(proj), ldp=proj.stride(0), nq=Q8, c_off=Q8, R=R, rot=r, q_norm=K.ptr(L.q_norm),
                                     nq_real=m.q_rank, c_norm=K.ptr(L.c_norm), eps=self.c.rms_eps, freq=K.ptr(freq),
                                     positions=K.ptr(positions), q=K.ptr(cq), ldq=Q8, pool=K.ptr(pool), ldc=Rp, n_pages=pool.shape[0] - 1,
                                     locs=K.ptr(locs), status=K.ptr(self.status), pdl=pdl), T, self.f32)
        qf, q = self._rows("qf", T, H * K8), self._rows("q", T, H * K8)
        self._gemm(L.wuq, cq, qf, T)
        K.rotate_heads(qf, q, freq, positions, heads=H, width=K8, first=D, rot=r, M=T, f32=self.f32, pdl=self.pdl)
        lat, ctx, vo = self._rows("lat", T, H * Rp), self._rows("ctx", T, H * Rp), self._rows("vo", T, L.wo.shape[1])
        self._per_head(L.wuk_t, q, lat, T, H, K8, Rp)
        self._latent_attention(lat, pool, ctx, H, m.scale, T, work, longest, m.window, L.sink)
        self._per_head(L.wuv, ctx, vo, T, H, Rp, m.vdim)
        return vo

    # ---- feed-forward -------------------------------------------------------------------
    def _unit(self, W: torch.Tensor, X: torch.Tensor, act: torch.Tensor, M: int, link: "K.GroupLink", kind: int = K.ACT_SILU) -> None:
        link.act, link.limit, link.slope = kind, math.inf, 1.0
        self._gated_gemm(W, X, act, M, GU_BLOCK, link, shift=0.0)

    def _feed_forward(self, L, T: int, forked: bool) -> None:
        """All of the feed-forward but a shared expert; ``forked``: first work of a stream that has just been forked."""
        f = L.spec.mlp
        first = self._full_order if forked else nullcontext
        if f.kind != "moe":
            act = self._rows("act", T, L.wdown.shape[1])
            with first():
                self._unit(L.wgu, self.xb, act, T, K.GroupLink(), K.ACT_GELU)
            self._gemm(L.wdown, act, self._rows("y2", T, self.d), T)
            return
        with first():
            K.route(self._flat["n2"], L.router, self._flat["idx"], self._flat["wgt"], d=self.d, top=f.router.top, groups=1, keep=1, T=T,
                    f32=self.f32, bias=L.router_bias, gate=self._flat["sg"] if f.shared is not None else None, pdl=self.pdl)
        self._expert_rows(L, f, self.xb, T, lambda W, X, out, M, spec, link: self._unit(W, X, out, M, link))

    def _shared_expert(self, L, T: int) -> None:
        act = self._rows("act", T, L.s_down.shape[1])
        self._unit(L.s_gu, self.xb, act, T, K.GroupLink())
        self._gemm(L.s_down, act, self._rows("y2", T, self.d), T)

    # ---- forward ------------------------------------------------------------------------
    def _run(self, ids, positions, locs, T: int, work: "K.Ragged", single_rows: Optional[torch.Tensor], longest: int) -> torch.Tensor:
        assert T <= self.T and (self.state is not None or not self.m.has_state)
        work = self._walk(work, longest)
        self._steps[0].ids = K.ptr(ids)
        mixers = {"mlstm": self._memory, "attention": self._attention, "latent": self._latent}
        beside = self.beside and not self.f32
        joined = False
        for i, L in enumerate(self.m.layers):
            self._step(i, T, joined)
            f = L.spec.mlp
            joined = beside and f is not None
            if joined:
                with torch.cuda.stream(self._fork()):
                    self._feed_forward(L, T, True)
            self._gemm(L.win, self.xa, self._rows("proj", T, L.win.shape[0]), T)
            vo = mixers[L.kind](i, L, T, positions, locs, work, longest)
            self._gemm(L.wo, vo, self._rows("y1", T, self.d), T)
            if f is not None and f.shared is not None:
                self._shared_expert(L, T)
            if joined:
                self._join()
            elif f is not None:
                self._feed_forward(L, T, False)
        self._step(len(self.m.layers), T, joined)
        return self.xa

    def _step(self, i: int, T: int, joined: bool) -> None:
        a = self._steps[i]
        a.pdl = int(self.pdl and not joined)
        K.side_step(a, T, self.f32)
