"""Kernel-chain forward of Padadra on sm_100a, in bf16 (tensor cores) or in 32-bit.

The chain starts with the embedding (token and pair rows) and the step's sines and cosines, which all layers share.  A layer,
between two steps of the residual stream (outputs added, the new row under the next layer's two norms):
  channel_delta  projections -> convolution, silu and low-rank maps (of prompts: their operands -> two products) -> memory with
                 norm and output gate -> output
  parallel       projections of both mixers in one product, then side by side
                   attention: convolution, norms, rotation, new keys and values to the cache -> windowed attention with sinks, heads
                              turned back -> output
                   memory:    scan or step from the projections, with norm -> output
                 the next step of the stream norms and averages the two
  feed-forward   up with the squared relu in the epilogue -> down, beside the mixer
Sequences may bring any number of new tokens each (``ops/ragged.py``); a uniform batch runs without index arrays and can be
captured in a graph.
"""
from __future__ import annotations

from contextlib import nullcontext
from typing import Dict, List, Optional

import torch

from ..models.config import RotarySpec
from ..models.layered import round_up
from ..models.padadra import UNIT_EPS, attention_columns, delta_columns, frequencies
from . import native as K
from .native_layered import NativeLayered, env_flag


class NativePadadra(NativeLayered):
    LOW_RANK_TOKENS = 32                  # steps up to this long expand the low-rank maps beside the convolution
    FEED_FORWARD, MEMORY = 0, 1           # streams beside the main one

    def __init__(self, model, kv, block_table: torch.Tensor, max_tokens: int, max_logit_rows: int, attn_splits: int,
                 status: torch.Tensor, pdl: bool, state=None):
        super().__init__(model, kv, block_table, max_tokens, max_logit_rows, attn_splits, status, pdl, state)
        T, ls, d = max_tokens, model.layers, self.d
        most = lambda it: max(it, default=0)
        pairs, deltas = [L for L in ls if L.parallel], [L for L in ls if not L.parallel]
        self.x = torch.zeros(T, d, dtype=torch.float32, device=self.dev)
        self.xb = torch.zeros(T, self.d8, dtype=self.dt, device=self.dev)       # rows under the feed-forward's norm
        self._room("proj", T * most(L.win.shape[0] for L in ls), torch.float32)
        self._room("q", T * most(L.spec.mixer.left.heads * round_up(L.spec.mixer.left.dim, 8) for L in pairs), self.dt)
        self._room("vo", T * most(L.wo.shape[1] for L in ls), self.dt)
        self._room("vo2", T * most(L.wo2.shape[1] for L in pairs), self.dt)
        self._room("conv", T * most(delta_columns(L.spec.mixer) for L in deltas), torch.float32)
        self._room("low", T * most(L.wa.shape[1] + L.wg.shape[1] for L in deltas), self.dt)
        self._room("z", T * most(L.wa.shape[0] for L in deltas), torch.float32)
        self._room("gate", T * most(L.wg.shape[0] for L in deltas), torch.float32)
        for name in ("y1", "y2", "yb"):
            self._room(name, T * d, torch.float32)
        self._room("act", T * most(L.wup.shape[0] for L in ls if L.wup is not None), self.dt)
        self.attn_tc = not self.f32 and env_flag("SMC_CHUNK_TC", True)
        self.beside = env_flag("SMC_BESIDE", True) and not self.f32
        # one table of angles per step: the pairs of all rotations of the model behind one another
        self.first_pair: Dict[RotarySpec, int] = {}
        freq: List[torch.Tensor] = []
        for rot in (r for L in pairs for r in (L.spec.mixer.left.rot, L.spec.mixer.left.turn_values)):
            if rot not in self.first_pair:
                self.first_pair[rot] = sum(f.numel() for f in freq)
                freq.append(frequencies(rot))
        self.freq = torch.cat(freq).to(self.dev) if freq else None
        self.n_pairs = self.freq.numel() if freq else 0
        self._room("angles", T * self.n_pairs * 2, torch.float32)
        self.taps = [L.conv.t().contiguous() for L in ls]
        self._steps = self._build_steps()

    def _build_steps(self) -> List["K.SideArgs"]:
        """Arguments of the stream step in front of every layer, and of the last one, which ends with the final norm."""
        m, c, steps, flat = self.m, self.c, [], self._flat
        for before, L in zip([None] + m.layers, m.layers + [None]):
            a = K.SideArgs(x=K.ptr(self.x), d=self.d, vocab=c.vocab_size, eps=c.rms_eps, ldy=self.d, ldye=self.d, xa=K.ptr(self.xa), ldxa=self.d8,
                           one_weight=1, mult=c.residual_mult, status=K.ptr(self.status), pdl=int(self.pdl))
            if before is None:
                a.embed, a.embed_scale = K.ptr(m.embed), c.embed_scale
                if m.bigram is not None:
                    kept = self.state.matrix(0)
                    a.pairs, (a.buckets, a.mul_prev, a.mul_cur) = K.ptr(m.bigram), c.bigram
                    a.before, a.before_stride, a.n_rows = K.ptr(kept), kept.stride(0), kept.shape[0]
                if self.freq is not None:
                    a.freq, a.n_freq, a.angles = K.ptr(self.freq), self.n_pairs, K.ptr(flat["angles"])
            else:
                a.y1 = K.ptr(flat["y1"])
                if before.parallel:
                    a.yb, a.o1, a.o2 = K.ptr(flat["yb"]), K.ptr(before.out1), K.ptr(before.out2)
                if before.spec.mlp is not None:
                    a.y2 = K.ptr(flat["y2"])
            if L is None:
                a.w1, a.final = K.ptr(m.final_norm), 1
            else:
                a.w1 = K.ptr(L.norm1)
                if L.spec.mlp is not None:
                    a.w2, a.xb = K.ptr(L.norm2), K.ptr(self.xb)
            steps.append(a)
        return steps

    # ---- planning -----------------------------------------------------------------------
    def set_context(self, ctx: int, bs: int, Es=(1, 2)) -> tuple:
        """Record the context-length hint; returns what it decides about the launch grids (part of a graph's identity)."""
        self.ctx_hint = int(ctx)
        mixers = {L.spec.mixer.left for L in self.m.layers if L.parallel}
        return tuple(sorted((E, m.window, m.heads, self._chunk_splits(bs * E, m, m.window)) for E in Es for m in mixers))

    # ---- mixers -------------------------------------------------------------------------
    def _memory(self, a: "K.ScanArgs", kind: int, T: int, longest: int) -> None:
        if longest == 1 and K.memory_step_takes(a.D, a.V):
            K.memory_step(a, kind, self.f32)
        else:
            K.memory_scan(a, kind, self.f32, T)

    def _scan_args(self, L, m, proj: torch.Tensor, out: torch.Tensor, work: "K.Ragged", **kw) -> "K.ScanArgs":
        S = self.state.matrix(L.state + 1)
        return K.ScanArgs(proj=K.ptr(proj), ldp=proj.stride(0), onorm=K.ptr(L.onorm), state=K.ptr(S), row_stride=S.stride(0), n_rows=S.shape[0],
                          out=K.ptr(out), ldo=out.stride(0), H=m.heads, D=m.dim, V=m.values, eps=self.c.rms_eps, unit_eps=UNIT_EPS, r=work,
                          status=K.ptr(self.status), pdl=int(self.pdl), **kw)

    def _history(self, L, taps: int) -> dict:
        hist = self.state.matrix(L.state) if taps > 1 else None
        return dict(hist=K.ptr(hist), row_stride=hist.stride(0) if hist is not None else 0, n_rows=hist.shape[0] if hist is not None else 0)

    def _delta(self, i: int, L, T: int, work: "K.Ragged", longest: int) -> torch.Tensor:
        m, pdl, st = L.spec.mixer, int(self.pdl), K.ptr(self.status)
        H, G, D, E, C = m.heads, m.kv_heads, m.dim, m.values, delta_columns(m)
        C8, (HD, ra), (HE, rg) = round_up(C, 8), L.wa.shape, L.wg.shape
        proj, u, vo = self._rows("proj", T, L.win.shape[0]), self._rows("conv", T, C), self._rows("vo", T, L.wo.shape[1])
        z, gate, low = self._rows("z", T, HD), self._rows("gate", T, HE), self._rows("low", T, ra + rg)
        few = T <= self.LOW_RANK_TOKENS
        K.conv_act(K.ConvActArgs(proj=K.ptr(proj), ldp=proj.stride(0), C=C, conv=K.ptr(self.taps[i]), taps=m.conv, **self._history(L, m.conv),
                                 out=K.ptr(u), ldo=C, low_off=C8 + round_up(H, 8), k1=ra, k2=rg, low=None if few else K.ptr(low), w1=K.ptr(L.wa),
                                 w2=K.ptr(L.wg), z1=K.ptr(z), z2=K.ptr(gate), n1=HD, n2=HE, r=work, status=st, pdl=pdl), self.f32)
        if not few:
            self._gemm(L.wa, low, z, T, ldx=ra + rg)
            self._gemm(L.wg, low[:, ra:], gate, T, ldx=ra + rg)
        self._memory(self._scan_args(L, m, u, vo, work, r_off=0, k_off=G * D, v_off=2 * G * D, z=K.ptr(z), ldz=HD, w0=K.ptr(L.dt_bias),
                                     r_scale=D ** -0.5, beta=K.ptr(proj[:, C8:]), ldb=proj.stride(0), gate=K.ptr(gate), ldg=HE, a_log=K.ptr(L.a_log),
                                     rep=H // G), K.SCAN_CHANNEL, T, longest)
        return vo

    def _attention(self, i: int, L, T: int, locs, work: "K.Ragged", longest: int) -> torch.Tensor:
        m, pdl, st = L.spec.mixer.left, int(self.pdl), K.ptr(self.status)
        H, G, D, V = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8)
        kp, vp, angles, turn = self.kv.k[L.cache], self.kv.v[L.cache], K.ptr(self._flat["angles"]), self.first_pair[m.turn_values]
        proj, q, vo = self._rows("proj", T, L.win.shape[0]), self._rows("q", T, H * D), self._rows("vo", T, H * V)
        K.normed_heads(K.ConvHeadsArgs(proj=K.ptr(proj), ldp=proj.stride(0), H=H, G=G, D=D, V=V, rot=m.rot.dims, conv=K.ptr(self.taps[i]),
                                       taps=m.conv, **self._history(L, m.conv), q=K.ptr(q), kpool=K.ptr(kp), vpool=K.ptr(vp),
                                       n_pages=kp.shape[0] - 1, locs=K.ptr(locs), bias=K.ptr(L.bias), qk_norm=K.ptr(L.qk_norm), dim=m.dim,
                                       eps=self.c.rms_eps, angles=angles, ld_angles=self.n_pairs, qk_first=self.first_pair[m.rot], v_first=turn,
                                       turn=m.vdim, r=work, status=st, pdl=pdl), self.f32)
        a = K.ChunkAttnArgs(q=K.ptr(q), kpool=K.ptr(kp), vpool=K.ptr(vp), out=K.ptr(vo), block_table=K.ptr(self.bt), bt_stride=self.bt.stride(0),
                            bt_rows=self.bt.shape[0], n_pages=kp.shape[0] - 1, H=H, G=G, D=D, V=V, scale=m.scale, sink=1,
                            sink_logit=K.ptr(L.sink), window=m.window, angles=angles, ld_angles=self.n_pairs, angle_first=turn, turn=m.vdim, r=work,
                            status=st, pdl=pdl)
        self._chunk_attention(a, m, m.window, T, longest)
        return vo

    def _forget(self, L, T: int, work: "K.Ragged", longest: int) -> torch.Tensor:
        m, C = L.spec.mixer.right, attention_columns(L.spec.mixer.left)
        proj, vo, HD = self._rows("proj", T, L.win.shape[0]), self._rows("vo2", T, L.wo2.shape[1]), m.heads * m.dim
        self._memory(self._scan_args(L, m, proj, vo, work, r_off=C, a_off=C + HD, v_off=C + 2 * HD, a_bias=K.ptr(L.f_bias), lower=K.ptr(L.lower)),
                     K.SCAN_FORGET, T, longest)
        return vo

    # ---- forward ------------------------------------------------------------------------
    def _run(self, ids, positions, locs, T: int, work: "K.Ragged", single_rows: Optional[torch.Tensor], longest: int) -> torch.Tensor:
        assert T <= self.T and self.state is not None
        work = self._walk(work, longest)
        first = self._steps[0]
        first.ids, first.positions, first.r = K.ptr(ids), K.ptr(positions), work
        joined = False
        for i, L in enumerate(self.m.layers):
            self._step(i, T, joined)
            joined = self.beside and (L.parallel or L.spec.mlp is not None)
            if L.spec.mlp is not None:
                with torch.cuda.stream(self._fork(self.FEED_FORWARD)) if self.beside else nullcontext():
                    self._feed_forward(L, T)
            self._gemm(L.win, self.xa, self._rows("proj", T, L.win.shape[0]), T)
            y1 = self._rows("y1", T, self.d)
            if L.parallel:
                with torch.cuda.stream(self._fork(self.MEMORY)) if self.beside else nullcontext():
                    with self._full_order() if self.beside else nullcontext():
                        vo2 = self._forget(L, T, work, longest)
                    self._gemm(L.wo2, vo2, self._rows("yb", T, self.d), T)
                self._gemm(L.wo, self._attention(i, L, T, locs, work, longest), y1, T)
                if self.beside:
                    self._join(self.MEMORY)
            else:
                self._gemm(L.wo, self._delta(i, L, T, work, longest), y1, T)
            if self.beside and L.spec.mlp is not None:
                self._join(self.FEED_FORWARD)
        self._step(len(self.m.layers), T, joined)
        return self.xa

    def _feed_forward(self, L, T: int) -> None:
        act = self._rows("act", T, L.wup.shape[0])
        with self._full_order() if self.beside else nullcontext():       # first work of a stream that has just been forked
            self._relu2_gemm(L.wup, self.xb, act, T)
        self._gemm(L.wdown, act, self._rows("y2", T, self.d), T)

    def _step(self, i: int, T: int, joined: bool) -> None:
        a = self._steps[i]
        a.pdl = int(self.pdl and not joined)
        K.side_step(a, T, self.f32)
