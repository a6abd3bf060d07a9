"""Kernel-chain forward of Makodra on sm_100a, in bf16 (tensor cores) or in 32-bit.

A layer, between two steps of the residual stream (x <- x + norm(y), the next sublayer's operand, and for single tokens the
shifted inputs of a wkv mixer):
  attention      [step] -> projections -> new keys and values to the cache -> chunked attention with the output gate -> output
  general_delta  [step] -> projections -> tanh -> decay logits -> scan (with norm and gate) -> output
  wkv            [step (+ token shift)] -> one product per shifted input -> decay input -> tanh -> decay logits -> scan -> output
  swiglu         [step] -> gate / up with the gated epilogue -> down
Sequences may bring any number of new tokens each (``ops/ragged.py``); a uniform batch runs without index arrays and can be
captured in a graph.
"""
from __future__ import annotations

from typing import List, Optional

import torch

from ..models.layered import GU_BLOCK, round_up
from ..models.layers import DELTA_UNIT_EPS
from ..models.makodra import DELTA_LOG_DECAY, SHIFTED
from . import native as K
from .native_layered import NativeLayered, env_flag


class NativeMakodra(NativeLayered):
    LOW_RANK_TOKENS = 32                  # steps up to this long expand the decay logits in one launch

    def __init__(self, model, kv, block_table: torch.Tensor, max_tokens: int, max_logit_rows: int, attn_splits: int,
                 status: torch.Tensor, pdl: bool, state=None):
        super().__init__(model, kv, block_table, max_tokens, max_logit_rows, attn_splits, status, pdl, state)
        T, ls = max_tokens, model.layers
        most = lambda it: max(it, default=0)
        attn = [L.spec.mixer for L in ls if L.kind == "attention"]
        d = self.d
        self.x = torch.zeros(T, d, dtype=torch.float32, device=self.dev)
        self.freq = 10000.0 ** (-2.0 * torch.arange((d + 1) // 2, dtype=torch.float64, device=self.dev) / d)
        self._room("proj", T * most(L.win.shape[0] for L in ls), torch.float32)
        self._room("q", T * most(m.heads * round_up(m.dim, 8) for m in attn), self.dt)
        self._room("v_first", T * most(m.kv_heads * round_up(m.vdim, 8) for m in attn), torch.float32)
        self._room("vo", T * most(L.wo.shape[1] for L in ls), self.dt)
        self._room("mix", T * (len(SHIFTED) * self.d8 if any(L.mu is not None for L in ls) else 0), self.dt)
        self._room("low_in", T * most(L.w1.shape[0] for L in ls if L.w1 is not None), torch.float32)
        self._room("low", T * most(L.w2.shape[1] for L in ls if L.w2 is not None), self.dt)
        self._room("z", T * most(L.w2.shape[0] for L in ls if L.w2 is not None), torch.float32)
        self._room("y", T * d, torch.float32)
        ff = most(L.wdown.shape[1] for L in ls if L.wdown is not None)
        self._room("act", T * ff, self.dt)
        if self.f32:
            self._room("gu", T * 2 * ff, torch.float32)
        self.attn_tc = not self.f32 and env_flag("SMC_CHUNK_TC", True)
        self._steps = self._build_steps()

    def _build_steps(self) -> List[dict]:
        """The sublayers in execution order, each with the prepared arguments of the stream step that leads into it (the
        last entry is the final norm)."""
        m = self.m
        steps: List[dict] = []
        prev = None                       # norm weight of the sublayer before
        for L in m.layers:
            steps.append({"kind": L.kind, "L": L, "prev": prev})
            prev = L.norm1
            if L.spec.mlp is not None:
                steps.append({"kind": "ff", "L": L, "prev": prev})
                prev = L.norm2
        steps.append({"kind": "final", "L": None, "prev": prev})
        for s in steps:
            a = K.PostNormArgs(x=K.ptr(self.x), d=self.d, vocab=self.c.vocab_size, eps=self.c.rms_eps, ldxa=self.d8, ldy=self.d,
                               status=K.ptr(self.status), pdl=int(self.pdl))
            if s["prev"] is None:
                a.embed, a.freq = K.ptr(m.embed), K.ptr(self.freq)
            else:
                a.y, a.w = K.ptr(self._flat["y"]), K.ptr(s["prev"])
            if s["kind"] == "final":
                a.w_final = K.ptr(m.final_norm)
            if s["kind"] != "wkv":
                a.xa = K.ptr(self.xa)
            s["args"] = a
        return steps

    # ---- planning -----------------------------------------------------------------------
    def set_context(self, ctx: int, bs: int, Es=(1, 2)) -> tuple:
        """Record the context-length hint; returns what it decides about the launch grids (part of a graph's identity)."""
        self.ctx_hint = int(ctx)
        mixers = {L.spec.mixer for L in self.m.layers if L.kind == "attention"}
        return tuple(sorted((E, m.chunk, m.heads, self._chunk_splits(bs * E, m, m.chunk)) for E in Es for m in mixers))

    # ---- sublayers ----------------------------------------------------------------------
    def _attention(self, L, T: int, locs: torch.Tensor, work: "K.Ragged", longest: int) -> None:
        m, pdl, st = L.spec.mixer, int(self.pdl), K.ptr(self.status)
        H, G, D, V = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8)
        kp, vp = self.kv.k[L.index], self.kv.v[L.index]
        proj, q, vo = self._rows("proj", T, L.win.shape[0]), self._rows("q", T, H * D), self._rows("vo", T, H * V)
        self._gemm(L.win, self.xa, proj, T)
        mixing = K.ptr(self._flat["v_first"]) if L.gives_values or L.lam != 0.0 else None
        K.heads_new(K.HeadsNewArgs(proj=K.ptr(proj), ldp=proj.stride(0), H=H, G=G, D=D, V=V, dim=m.dim, eps=self.c.rms_eps, q=K.ptr(q),
                                   kpool=K.ptr(kp), vpool=K.ptr(vp), n_pages=kp.shape[0] - 1, locs=K.ptr(locs), lam=L.lam,
                                   v_first=mixing, gives=int(L.gives_values), status=st, pdl=pdl), T, self.f32)
        gate = proj[:, (H + G) * D + G * V:]
        a = K.ChunkAttnArgs(q=K.ptr(q), kpool=K.ptr(kp), vpool=K.ptr(vp), out=K.ptr(vo), gate=K.ptr(gate), ldg=proj.stride(0),
                            block_table=K.ptr(self.bt), bt_stride=self.bt.stride(0), bt_rows=self.bt.shape[0],
                            n_pages=kp.shape[0] - 1, H=H, G=G, D=D, V=V, chunk=m.chunk, scale=m.scale, r1=K.ptr(L.r1), r2=K.ptr(L.r2),
                            sink=1, r=work, status=st, pdl=pdl)
        self._chunk_attention(a, m, m.chunk, T, longest)
        self._gemm(L.wo, vo, self._rows("y", T, self.d), T)

    def _recurrent(self, L, T: int, work: "K.Ragged", single: bool) -> None:
        m, pdl = L.spec.mixer, int(self.pdl)
        HD, delta, d8 = m.heads * m.dim, L.kind == "general_delta", self.d8
        proj, rank = self._rows("proj", T, L.win.shape[0]), L.w2.shape[1]
        low, z = self._rows("low", T, rank), self._rows("z", T, HD)
        if delta:
            self._gemm(L.win, self.xa, proj, T)
            low_in = proj[:, 5 * HD:]
        else:
            mix, n = self._rows("mix", T, len(SHIFTED) * d8), len(SHIFTED) - 1
            if not single:
                K.token_shift(self.x[:T], L.mu, mix, self.state.conv[L.shift_index].squeeze(-1), work, ldm=d8, status=self.status,
                              f32=self.f32, pdl=self.pdl)
            proj = self._rows("proj", T, n * HD)
            link = K.GroupLink(mode=K.GROUP_BATCHED, groups=n, w_rows=HD, x_cols=d8, out_cols=HD)
            if self.f32:
                K.gemm_f32(L.win, mix, proj, N=HD, M=T, link=link, pdl=self.pdl)
            else:
                K.gemm_grouped(L.win, mix, proj, N=HD, M=T, splits=self._cluster(n * HD, d8, T), epi=K.EPI_STORE_F32, link=link,
                               status=self.status, pdl=self.pdl)
            low_in = self._rows("low_in", T, rank)
            self._gemm(L.w1, mix[:, n * d8:], low_in, T, ldx=mix.stride(0))
        if T <= self.LOW_RANK_TOKENS:
            K.low_rank(low_in, L.w2, z, M=T, f32=self.f32, pdl=self.pdl)
        else:
            K.tanh_rows(low_in, low, n=rank, M=T, f32=self.f32, pdl=self.pdl)
            self._gemm(L.w2, low, z, T)
        S, ldo = self.state.matrix(L.index), L.wo.shape[1]
        vo = self._rows("vo", T, ldo)
        K.memory_scan(K.ScanArgs(proj=K.ptr(proj), ldp=proj.stride(0), r_off=0, k_off=HD, v_off=2 * HD, g_off=3 * HD, a_off=4 * HD,
                                 z=K.ptr(z), ldz=HD, w0=K.ptr(L.w0), a_bias=K.ptr(L.a_bias), bonus=K.ptr(L.bonus), onorm=K.ptr(L.onorm),
                                 state=K.ptr(S), row_stride=S.stride(0), n_rows=S.shape[0], out=K.ptr(vo), ldo=ldo, H=m.heads, D=m.dim, V=m.dim,
                                 eps=self.c.rms_eps, unit_eps=DELTA_UNIT_EPS, log_decay=DELTA_LOG_DECAY, r=work,
                                 status=K.ptr(self.status), pdl=pdl), K.SCAN_DELTA if delta else K.SCAN_BONUS, self.f32)
        self._gemm(L.wo, vo, self._rows("y", T, self.d), T)

    def _swiglu(self, L, T: int) -> None:
        act = self._rows("act", T, L.wdown.shape[1])
        self._gated_gemm(L.wgu, self.xa, act, T, GU_BLOCK, K.GroupLink(act=K.ACT_SILU, limit=float("inf"), slope=1.0), shift=0.0)
        self._gemm(L.wdown, act, self._rows("y", T, self.d), T)

    # ---- forward ------------------------------------------------------------------------
    def _run(self, ids, positions, locs, T: int, work: "K.Ragged", single_rows: Optional[torch.Tensor], longest: int) -> torch.Tensor:
        assert T <= self.T and (self.state is not None or not self.m.has_state)
        work = self._walk(work, longest)
        for s in self._steps:
            a, L, kind = s["args"], s["L"], s["kind"]
            if s["prev"] is None:
                a.ids, a.positions = K.ptr(ids), K.ptr(positions)
            if kind == "wkv":
                if single_rows is not None:
                    hist = self.state.conv[L.shift_index]
                    a.mu, a.mix, a.n_mix, a.rows = K.ptr(L.mu), K.ptr(self._flat["mix"]), len(SHIFTED), K.ptr(single_rows)
                    a.hist, a.ldh, a.n_rows = K.ptr(hist), hist.shape[1], hist.shape[0]
                else:
                    a.mu = None
            K.post_norm_step(a, T, self.f32)
            if kind == "attention":
                self._attention(L, T, locs, work, longest)
            elif kind == "ff":
                self._swiglu(L, T)
            elif kind != "final":
                self._recurrent(L, T, work, single_rows is not None)
        return self.xa
