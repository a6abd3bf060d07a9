"""Kernel-chain forward of Pasizen on sm_100a, in bf16 (tensor cores) or in 32-bit.

A layer run, between two steps of the hyper-connected streams:
  mixer         [streams + norm (+ convolution) ] -> query / latent projection -> new latents to the cache -> queries into
                latent space (one product per head) -> attention over cached latents -> value expansion -> output projection
  dense         [streams + norm] -> up -> PolyNorm -> down
  experts       [streams + norm] -> router -> dispatch -> gather -> gate/up with the gated epilogue -> down, all experts in
                one launch each, beside the shared expert; the next step of the streams adds the weighted rows
Sequences may bring any number of new tokens each (``ops/ragged.py``); a uniform batch runs without index arrays and can be
captured in a graph.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..models.layers import GLU_SIGMOID_SLOPE
from ..models.layered import GU_BLOCK, round_up
from . import native as K
from .native_layered import NativeLayered, env_flag


class NativePasizen(NativeLayered):
    def __init__(self, model, kv, block_table: torch.Tensor, max_tokens: int, max_logit_rows: int, attn_splits: int,
                 status: torch.Tensor, pdl: bool, state=None):
        super().__init__(model, kv, block_table, max_tokens, max_logit_rows, attn_splits, status, pdl, state)
        c = self.c
        self.S = c.streams
        mixers = [L.mixer for L in c.layers]
        mlps = [L.mlp for L in c.layers if L.mlp is not None]
        dense, moe = [f for f in mlps if f.kind == "dense"], [f for f in mlps if f.kind == "moe"]
        most = lambda it: max(it, default=0)
        T = max_tokens
        self.x = torch.zeros(T, self.S, self.d, dtype=torch.float32, device=self.dev)
        self.n = torch.zeros(T, self.d, dtype=torch.float32, device=self.dev)
        self._room("proj", T * most(m.heads * round_up(m.dim, 8) + m.kv_rank for m in mixers), torch.float32)
        self._room("q", T * most(m.heads * round_up(m.dim, 8) for m in mixers), self.dt)
        self._room("lat", T * most(m.heads * round_up(m.kv_rank, 64) for m in mixers), self.dt)
        self._room("ctx", T * most(m.heads * round_up(m.kv_rank, 64) for m in mixers), self.dt)
        self._room("vo", T * most(round_up(m.heads * m.vdim, 8) for m in mixers), self.dt)
        self._room("y", T * self.d, torch.float32)
        self._room("z", T * most(round_up(f.ff, 8) for f in dense), torch.float32)
        self._room("act", T * most([round_up(f.ff, 8) for f in dense] +
                                   [round_up(f.shared.ff, GU_BLOCK) for f in moe if f.shared]), self.dt)
        self._room_experts(moe)
        self._room_gate_up([], moe)
        self.attn_tc = not self.f32 and env_flag("SMC_LATENT_TC", True)
        self._steps = self._build_steps()

    def _build_steps(self) -> List[dict]:
        """The sublayers of every layer run in execution order, each with the prepared arguments of the stream step that
        leads into it (the last entry is the final norm)."""
        c, m = self.c, self.m
        steps: List[dict] = []
        prev = None                       # (hyper weights, feed-forward spec or None) of the sublayer before
        for run, li in enumerate(m.runs):
            L = m.layers[li]
            subs = [("mix", L.hc1, L.norm1)] + ([("ff", L.hc2, L.norm2)] if L.spec.mlp is not None else [])
            for kind, hc, norm in subs:
                steps.append({"kind": kind, "run": run, "L": L, "hc": hc, "norm": norm, "prev": prev})
                prev = (hc, L.spec.mlp if kind == "ff" else None)
        steps.append({"kind": "final", "norm": m.final_norm, "hc": None, "prev": prev})
        for s in steps:
            a = K.HyperArgs(x=K.ptr(self.x), S=self.S, d=self.d, vocab=c.vocab_size, max_pos=c.max_position, ldy=self.d, ldye=self.d,
                            norm_w=K.ptr(s["norm"]), eps=c.rms_eps, ldxa=self.d8, status=K.ptr(self.status), pdl=int(self.pdl))
            if s["hc"] is not None:
                a.w_in = K.ptr(s["hc"].w_in)
            if s["prev"] is None:
                a.embed, a.pos = K.ptr(m.embed), K.ptr(m.pos)
            else:
                hc, f = s["prev"]
                a.w_mix, a.w_out = K.ptr(hc.w_mix), K.ptr(hc.w_out)
                moe = f is not None and f.kind == "moe"
                if not moe or f.shared is not None:
                    a.y = K.ptr(self._flat["y"])
                if moe:
                    a.ye, a.top = K.ptr(self._flat["ye"]), f.router.top
                    a.route_slot, a.route_w = K.ptr(self._flat["slot"]), K.ptr(self._flat["wgt"])
            s["args"] = a
        return steps

    # ---- planning -----------------------------------------------------------------------
    def set_context(self, ctx: int, bs: int, Es=(1, 2)) -> tuple:
        """Record the context-length hint; returns what it decides about the launch grids (part of a graph's identity)."""
        self.ctx_hint = int(ctx)
        shapes = sorted({(L.mixer.heads, round_up(L.mixer.kv_rank, 64)) for L in self.c.layers})
        return tuple(self._latent_splits(bs * ((E + self.BLOCK - 1) // self.BLOCK), min(E, self.BLOCK), H, Rp) for E in Es for H, Rp in shapes)

    # ---- products -----------------------------------------------------------------------
    def _glu_gemm(self, W: torch.Tensor, X: torch.Tensor, act: torch.Tensor, M: int, limit: float, link: "K.GroupLink") -> None:
        """act = clamped gated unit of the interleaved gate / up product."""
        link.act, link.limit, link.slope = K.ACT_CLAMPED, limit, GLU_SIGMOID_SLOPE
        self._gated_gemm(W, X, act, M, GU_BLOCK, link, shift=1.0)

    # ---- sublayers ----------------------------------------------------------------------
    def _mixer(self, s: dict, T: int, locs: torch.Tensor, work: "K.Ragged", longest: int) -> None:
        L, run = s["L"], s["run"]
        m, pdl = L.spec.mixer, self.pdl
        H, D8, R, Rp = m.heads, round_up(m.dim, 8), m.kv_rank, round_up(m.kv_rank, 64)
        nq, ov = H * D8, round_up(H * m.vdim, 8)
        proj = self._rows("proj", T, nq + R)
        self._gemm(L.wqc, self.xa, proj, T)
        pool = self.kv.k[run]
        q = None if self.f32 else self._rows("q", T, nq)
        K.latent_new(K.LatentNewArgs(proj=K.ptr(proj), ldp=proj.stride(0), nq=nq, c_off=nq, R=R, c_norm=K.ptr(L.c_norm), eps=self.c.rms_eps,
                                     q=K.ptr(q), ldq=nq, pool=K.ptr(pool), ldc=Rp, n_pages=pool.shape[0] - 1, locs=K.ptr(locs),
                                     status=K.ptr(self.status), pdl=int(pdl)), T, self.f32)
        lat, ctx, vo = self._rows("lat", T, H * Rp), self._rows("ctx", T, H * Rp), self._rows("vo", T, ov)
        self._per_head(L.wuk_t, proj if q is None else q, lat, T, H, D8, Rp)
        self._latent_attention(lat, pool, ctx, H, m.scale, T, work, longest)
        self._per_head(L.wuv, ctx, vo, T, H, Rp, m.vdim)
        self._gemm(L.wo, vo, self._rows("y", T, self.d), T)

    def _dense(self, s: dict, T: int) -> None:
        L, f = s["L"], s["L"].spec.mlp
        f8 = round_up(f.ff, 8)
        z, act = self._rows("z", T, f8), self._rows("act", T, f8)
        self._gemm(L.wup, self.xa, z, T)
        K.poly_norm(z, L.poly, act, ff=f.ff, M=T, eps=self.c.rms_eps, f32=self.f32, pdl=self.pdl)
        self._gemm(L.wdown, act, self._rows("y", T, self.d), T)

    def _experts(self, s: dict, T: int) -> None:
        L, f, pdl = s["L"], s["L"].spec.mlp, self.pdl
        r = f.router
        K.route(self.n, L.router, self._flat["idx"], self._flat["wgt"], d=self.d, top=r.top, groups=r.groups, keep=r.keep, T=T, f32=self.f32,
                pdl=pdl)
        self._expert_rows(L, f, self.xa, T, lambda W, X, out, M, unit, link: self._glu_gemm(W, X, out, M, unit.limit, link))
        if f.shared is not None:
            sa = self._rows("act", T, L.s_down.shape[1])
            self._glu_gemm(L.s_gu, self.xa, sa, T, f.shared.limit, K.GroupLink())
            self._gemm(L.s_down, sa, self._rows("y", T, self.d), T)

    # ---- forward ------------------------------------------------------------------------
    def _run(self, ids, positions, locs, T: int, work: "K.Ragged", single_rows: Optional[torch.Tensor], longest: int) -> torch.Tensor:
        assert T <= self.T and self.state is not None
        for s in self._steps:
            a, kind = s["args"], s["kind"]
            if s["prev"] is None:
                a.ids, a.positions = K.ptr(ids), K.ptr(positions)
            conv = kind == "mix"
            folded = conv and single_rows is not None
            a.n_out = K.ptr(self.n) if (conv and not folded) or (kind == "ff" and s["L"].spec.mlp.kind == "moe") else None
            a.xa = None if conv and not folded else K.ptr(self.xa)
            if folded:
                hist = self.state.conv[s["run"]]
                a.conv_w, a.hist, a.rows = K.ptr(s["L"].conv_w), K.ptr(hist), K.ptr(single_rows)
                a.taps, a.n_rows = self.c.conv_taps, hist.shape[0]
            else:
                a.conv_w = None
            K.hyper_step(a, T, self.f32)
            if conv:
                if not folded:
                    K.short_conv(self.n, self.xa, s["L"].conv_w, self.state.conv[s["run"]], work, status=self.status, f32=self.f32,
                                 pdl=self.pdl)
                self._mixer(s, T, locs, work, longest)
            elif kind == "ff":
                (self._dense if s["L"].spec.mlp.kind == "dense" else self._experts)(s, T)
        return self.xa
