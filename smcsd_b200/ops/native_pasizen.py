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
        pairs = T * most(f.router.top for f in moe)
        self._room("idx", pairs, torch.int32)
        self._room("wgt", pairs, torch.float32)
        self._room("slot", pairs, torch.int32)
        self._room("src", pairs, torch.int32)
        self._room("tiles", 4 * most(f.router.experts for f in moe) + 4 * (pairs // 16 + 1), torch.int32)
        self._room("xe", pairs * self.d8, self.dt)
        self._room("ea", pairs * most(round_up(f.expert.ff, GU_BLOCK) for f in moe), self.dt)
        self._room("ye", pairs * self.d, torch.float32)
        if self.f32:
            self._room("gu", max([pairs * 2 * round_up(f.expert.ff, GU_BLOCK) for f in moe] +
                                 [T * 2 * round_up(f.shared.ff, GU_BLOCK) for f in moe if f.shared], default=0), torch.float32)
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
        return tuple(self._ks(bs * ((E + self.BLOCK - 1) // self.BLOCK), min(E, self.BLOCK), H, Rp) for E in Es for H, Rp in shapes)

    def _ks(self, n_blk: int, tokens: int, H: int, Rp: int) -> int:
        """Key splits of one layer's attention: ``n_blk`` blocks of at most ``tokens`` tokens."""
        if not self.attn_tc or Rp > K.latent_tc_max_width():
            return 1
        ks = K.latent_tc_splits(n_blk * ((tokens * H + 127) // 128), Rp, self.ctx_hint)
        cap = max(1, int(self.attn_splits))
        while ks > cap:
            ks //= 2
        return ks

    # ---- products -----------------------------------------------------------------------
    def _per_head(self, W: torch.Tensor, X: torch.Tensor, out: torch.Tensor, M: int, H: int, x_cols: int, out_cols: int) -> None:
        """Head h: out[:, h * out_cols ..] = X[:, h * x_cols ..] W_h^T, in the activation type."""
        link = K.GroupLink(mode=K.GROUP_BATCHED, groups=H, w_rows=out_cols, x_cols=x_cols, out_cols=out_cols)
        if self.f32:
            K.gemm_f32(W, X, out, N=out_cols, M=M, link=link, pdl=self.pdl)
        else:
            K.gemm_grouped(W, X, out, N=out_cols, M=M, splits=1, epi=K.EPI_BF16, link=link, status=self.status, pdl=self.pdl)

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
        K.latent_new(proj, q, pool, L.c_norm, locs, nq=nq, R=R, eps=self.c.rms_eps, M=T, status=self.status, f32=self.f32, pdl=pdl)
        lat, ctx, vo = self._rows("lat", T, H * Rp), self._rows("ctx", T, H * Rp), self._rows("vo", T, ov)
        self._per_head(L.wuk_t, proj if q is None else q, lat, T, H, D8, Rp)
        a = K.LatentArgs(q=K.ptr(lat), pool=K.ptr(pool), out=K.ptr(ctx), block_table=K.ptr(self.bt), bt_stride=self.bt.stride(0),
                         bt_rows=self.bt.shape[0], n_pages=pool.shape[0] - 1, H=H, ldc=Rp, scale=m.scale, r=work,
                         status=K.ptr(self.status), pdl=int(pdl))
        if self.attn_tc and Rp <= K.latent_tc_max_width():
            tokens = min(longest, self.BLOCK)
            ks = self._ks(work.n_blk, tokens, H, Rp)
            K.latent_attention_tc(a, tokens=T, blk_rows=tokens * H, splits=ks)
        else:
            K.latent_attention(a, self.f32)
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
        r, E, top = f.router, f.router.experts, f.router.top
        n = T * top
        idx, wgt, slot, src, tiles = (self._flat[k] for k in ("idx", "wgt", "slot", "src", "tiles"))
        K.route(self.n, L.router, idx, wgt, d=self.d, top=top, groups=r.groups, keep=r.keep, T=T, f32=self.f32, pdl=pdl)
        avg = (n + E - 1) // E
        bn = 64 if self.f32 else 16 if avg <= 16 else 32 if avg <= 32 else 64 if avg <= 64 else 128
        max_tiles = n // bn + min(E, n)
        K.dispatch(idx, slot, src, tiles, n=n, top=top, experts=E, rows=bn, max_tiles=max_tiles, status=self.status, pdl=pdl)
        xe, ffp = self._rows("xe", n, self.d8), L.e_down.shape[-1]
        K.gather_rows(self.xa, src, xe, n=n, n_src=T, status=self.status, pdl=pdl)
        ea, ye = self._rows("ea", n, ffp), self._rows("ye", n, self.d)
        link = K.GroupLink(mode=K.GROUP_TILED, groups=E, w_rows=2 * ffp, tiles=K.ptr(tiles), max_tiles=max_tiles, bn=bn)
        self._glu_gemm(L.e_gu, xe, ea, n, f.expert.limit, link)
        link = K.GroupLink(mode=K.GROUP_TILED, groups=E, w_rows=self.d, tiles=K.ptr(tiles), max_tiles=max_tiles, bn=bn)
        if self.f32:
            K.gemm_f32(L.e_down, ea, ye, N=self.d, M=n, link=link, pdl=pdl)
        else:
            units, slabs, kb, sp = min(E, n), (self.d + 127) // 128, (ffp + 63) // 64, 1
            while sp < 8 and units * slabs * sp * 2 <= 256 and kb // (sp * 2) >= 2:
                sp *= 2
            K.gemm_grouped(L.e_down, ea, ye, N=self.d, M=n, splits=sp, epi=K.EPI_STORE_F32, link=link, status=self.status, pdl=pdl)
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
