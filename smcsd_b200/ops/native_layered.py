"""What the kernel chains of the layer-by-layer families share: buffers viewed per layer with that layer's own widths, products
in bf16 (tensor cores) or in 32-bit, steps over sequences of unequal length (``ops/ragged.py``) or over a uniform batch that
can be captured in a graph, and the head."""
from __future__ import annotations

import os
from contextlib import contextmanager
from typing import Dict, List, Optional

import torch

from ..models.layered import GU_BLOCK, round_up
from . import native as K
from .ragged import RaggedPlan, uniform_struct


def env_flag(name: str, default: bool) -> bool:
    v = os.environ.get(name)
    return default if v is None else v.strip().lower() in ("1", "true", "yes", "on")


class NativeLayered:
    """Subclasses implement ``_run(ids, positions, locs, T, work, single_rows, longest)``, which leaves the final rows in
    ``xa``, and ``set_context``."""
    ragged = True
    BLOCK = 64                            # tokens per block of the work list
    TC_MIN_TOKENS = 8                     # portions at least this long take the tensor-core form of the attention over heads
    attn_tc = False

    def __init__(self, model, kv, block_table: torch.Tensor, max_tokens: int, max_logit_rows: int, attn_splits: int,
                 status: torch.Tensor, pdl: bool, state=None):
        self.m, self.kv, self.bt, self.state = model, kv, block_table, state
        self.c = c = model.cfg
        self.T, self.status, self.pdl, self.attn_splits = max_tokens, status, pdl, attn_splits
        self.f32 = model.dtype == torch.float32
        if model.dtype not in (torch.float32, torch.bfloat16):
            raise ValueError(f"the {model.family} kernel chain runs in bfloat16 or float32")
        self.dt, self.dev = model.dtype, model.device
        self.d, self.d8 = c.hidden_size, round_up(c.hidden_size, 8)
        self.V = model.lm_head.shape[0]
        self.fused_lm_sample = not self.f32
        self.ctx_hint = 0
        self._lm_parts = None
        self._splits: Dict = {}
        self._side: Dict[int, tuple] = {}
        self.xa = torch.zeros(max_tokens, self.d8, dtype=self.dt, device=self.dev)
        # flat buffers, viewed per layer with that layer's own row width
        self._flat: Dict[str, torch.Tensor] = {}
        # the samplers read rows of float4
        self.logits = torch.empty(max_logit_rows, round_up(self.V, 4), dtype=torch.float32, device=self.dev)

    # ---- buffers ------------------------------------------------------------------------
    def _room(self, name: str, numel: int, dtype) -> None:
        self._flat[name] = torch.zeros(max(int(numel), 8), dtype=dtype, device=self.dev)

    def _rows(self, name: str, rows: int, width: int) -> torch.Tensor:
        return self._flat[name][:rows * width].view(rows, width)

    # ---- products -----------------------------------------------------------------------
    def _cluster(self, N: int, Kd: int, M: int) -> int:
        key = (N, Kd, M)
        if key not in self._splits:
            self._splits[key] = K.gemm_cluster_splits(N, Kd, M)
        return self._splits[key]

    def _gemm(self, W: torch.Tensor, X: torch.Tensor, out: torch.Tensor, M: int, ldx: Optional[int] = None) -> None:
        """out (fp32) = X W^T."""
        if self.f32:
            K.gemm_f32(W, X, out, N=W.shape[0], M=M, ldx=ldx, pdl=self.pdl)
        else:
            K.gemm_skinny(W, X, out, M=M, splits=self._cluster(W.shape[0], W.shape[1], M), epi=K.EPI_STORE_F32, ldx=ldx,
                          ldo=out.stride(0), status=self.status, pdl=self.pdl)

    def _relu2_gemm(self, W: torch.Tensor, X: torch.Tensor, act: torch.Tensor, M: int) -> None:
        """act = max(X W^T, 0)^2 in the activation type."""
        if self.f32:
            K.gemm_f32(W, X, act, N=W.shape[0], M=M, relu2=True, pdl=self.pdl)
        else:
            K.gemm_skinny(W, X, act, M=M, splits=self._cluster(W.shape[0], W.shape[1], M), epi=K.EPI_RELU2_BF16, ldo=act.stride(0),
                          status=self.status, pdl=self.pdl)

    def _gated_gemm(self, W: torch.Tensor, X: torch.Tensor, act: torch.Tensor, M: int, blk: int, link: "K.GroupLink",
                    shift: float) -> None:
        """act = gated unit of the interleaved gate / up product: the link's activation, ``shift`` added to the up value."""
        ff2 = W.shape[-2]
        if self.f32:
            gu = self._rows("gu", M, ff2)
            K.gemm_f32(W, X, gu, N=ff2, M=M, link=link, pdl=self.pdl)
            K.gated_unit_f32(gu, act, ff=ff2 // 2, blk=blk, limit=link.limit, slope=link.slope, shift=shift, M=M,
                             gelu=link.act == K.ACT_GELU, pdl=self.pdl)
            return
        splits = K.gemm_swiglu_splits(ff2, W.shape[-1], M) if link.mode == 0 else 1
        if link.mode == 0 and link.act == K.ACT_SILU:        # the plain build of the kernel has this unit
            K.gemm_skinny(W, X, act, M=M, splits=splits, epi=K.EPI_SWIGLU_BF16, ldo=act.stride(0), status=self.status, pdl=self.pdl)
            return
        K.gemm_grouped(W, X, act, N=ff2, M=M, splits=splits, epi=K.EPI_SWIGLU_BF16, link=link, status=self.status, pdl=self.pdl)

    def _per_head(self, W: torch.Tensor, X: torch.Tensor, out: torch.Tensor, M: int, H: int, x_cols: int, out_cols: int) -> None:
        """Head h: out[:, h * out_cols ..] = X[:, h * x_cols ..] W_h^T, in the activation type."""
        link = K.GroupLink(mode=K.GROUP_BATCHED, groups=H, w_rows=out_cols, x_cols=x_cols, out_cols=out_cols)
        if self.f32:
            K.gemm_f32(W, X, out, N=out_cols, M=M, link=link, pdl=self.pdl)
        else:
            K.gemm_grouped(W, X, out, N=out_cols, M=M, splits=1, epi=K.EPI_BF16, link=link, status=self.status, pdl=self.pdl)

    # ---- mixture of experts -------------------------------------------------------------
    def _room_experts(self, moe: List) -> None:
        """Buffers of the expert feed-forwards ``moe`` (specs)."""
        T, most = self.T, lambda it: max(it, default=0)
        pairs = T * most(f.router.top for f in moe)
        self._room("idx", pairs, torch.int32)
        self._room("wgt", pairs, torch.float32)
        self._room("slot", pairs, torch.int32)
        self._room("src", pairs, torch.int32)
        self._room("tiles", 4 * most(f.router.experts for f in moe) + 4 * (pairs // 16 + 1), torch.int32)
        self._room("xe", pairs * self.d8, self.dt)
        self._room("ea", pairs * most(round_up(f.expert.ff, GU_BLOCK) for f in moe), self.dt)
        self._room("ye", pairs * self.d, torch.float32)

    def _room_gate_up(self, dense: List[int], moe: List) -> None:
        """32-bit runs store gate / up rows: of gated units of these sizes and of the experts."""
        if self.f32:
            pairs = self.T * max((f.router.top for f in moe), default=0)
            units = list(dense) + [f.shared.ff for f in moe if f.shared]
            self._room("gu", max([pairs * 2 * round_up(f.expert.ff, GU_BLOCK) for f in moe] + [self.T * 2 * round_up(n, GU_BLOCK) for n in units],
                                 default=0), torch.float32)

    def _expert_rows(self, L, f, x: torch.Tensor, T: int, unit) -> None:
        """The chosen experts' outputs, one fp32 row per (token, choice) in "ye" at "slot", from the choices in "idx";
        ``unit(W, X, out, M, spec, link)`` runs the gated unit."""
        pdl, E, top, n = self.pdl, f.router.experts, f.router.top, T * f.router.top
        idx, slot, src, tiles = (self._flat[k] for k in ("idx", "slot", "src", "tiles"))
        avg = (n + E - 1) // E
        bn = 64 if self.f32 else 16 if avg <= 16 else 32 if avg <= 32 else 64 if avg <= 64 else 128
        max_tiles = n // bn + min(E, n)
        K.dispatch(idx, slot, src, tiles, n=n, top=top, experts=E, rows=bn, max_tiles=max_tiles, status=self.status, pdl=pdl)
        xe, ffp = self._rows("xe", n, self.d8), L.e_down.shape[-1]
        K.gather_rows(x, src, xe, n=n, n_src=T, status=self.status, pdl=pdl)
        ea, ye = self._rows("ea", n, ffp), self._rows("ye", n, self.d)
        unit(L.e_gu, xe, ea, n, f.expert, K.GroupLink(mode=K.GROUP_TILED, groups=E, w_rows=2 * ffp, tiles=K.ptr(tiles), max_tiles=max_tiles, bn=bn))
        link = K.GroupLink(mode=K.GROUP_TILED, groups=E, w_rows=self.d, tiles=K.ptr(tiles), max_tiles=max_tiles, bn=bn)
        if self.f32:
            K.gemm_f32(L.e_down, ea, ye, N=self.d, M=n, link=link, pdl=pdl)
            return
        units, slabs, kb, sp = min(E, n), (self.d + 127) // 128, (ffp + 63) // 64, 1
        while sp < 8 and units * slabs * sp * 2 <= 256 and kb // (sp * 2) >= 2:
            sp *= 2
        K.gemm_grouped(L.e_down, ea, ye, N=self.d, M=n, splits=sp, epi=K.EPI_STORE_F32, link=link, status=self.status, pdl=pdl)

    # ---- attention ----------------------------------------------------------------------
    def _capped(self, splits: int) -> int:
        cap = max(1, int(self.attn_splits))
        while splits > cap:
            splits //= 2
        return splits

    def _latent_splits(self, n_blk: int, tokens: int, H: int, Rp: int, window: int = 0) -> int:
        """Key ranges of a latent attention: ``n_blk`` blocks of at most ``tokens`` tokens."""
        if not self.attn_tc or Rp > K.latent_tc_max_width():
            return 1
        keys = min(self.ctx_hint, window + tokens) if window else self.ctx_hint
        return self._capped(K.latent_tc_splits(n_blk * ((tokens * H + 127) // 128), Rp, keys))

    def _latent_attention(self, lat: torch.Tensor, pool: torch.Tensor, ctx: torch.Tensor, H: int, scale: float, T: int, work: "K.Ragged",
                          longest: int, window: int = 0, sink: Optional[torch.Tensor] = None) -> None:
        Rp = pool.shape[1]
        a = K.LatentArgs(q=K.ptr(lat), pool=K.ptr(pool), out=K.ptr(ctx), block_table=K.ptr(self.bt), bt_stride=self.bt.stride(0),
                         bt_rows=self.bt.shape[0], n_pages=pool.shape[0] - 1, H=H, ldc=Rp, scale=scale, window=window, sink=K.ptr(sink),
                         r=work, status=K.ptr(self.status), pdl=int(self.pdl))
        if self.attn_tc and Rp <= K.latent_tc_max_width():
            tokens = min(longest, self.BLOCK)
            K.latent_attention_tc(a, tokens=T, blk_rows=tokens * H, splits=self._latent_splits(work.n_blk, tokens, H, Rp, window))
        else:
            K.latent_attention(a, self.f32)

    def _chunk_splits(self, tokens: int, m, chunk: int) -> int:
        """Key ranges of one layer's attention over heads for ``tokens`` tokens (``chunk``: length of a chunk or window, 0: all keys)."""
        keys = min(chunk, self.ctx_hint) if chunk else self.ctx_hint
        return self._capped(K.chunk_attention_splits(tokens, m.heads, m.kv_heads, round_up(max(m.dim, m.vdim), 8), keys))

    def _chunk_attention(self, a: "K.ChunkAttnArgs", m, chunk: int, T: int, longest: int) -> None:
        if self.attn_tc and longest >= self.TC_MIN_TOKENS and max(a.D, a.V) <= K.chunk_tc_max_width():
            K.chunk_attention_tc(a)
        else:
            K.chunk_attention(a, self.f32, self._chunk_splits(T, m, chunk))

    # ---- streams beside the main one ----------------------------------------------------
    @contextmanager
    def _full_order(self):
        """Launches that depend on work of two streams wait for all of it: no programmatic overlap with the kernel before."""
        kept, self.pdl = self.pdl, False
        try:
            yield
        finally:
            self.pdl = kept

    def _fork(self, which: int = 0) -> "torch.cuda.Stream":
        """A second (third, ..) stream, behind everything queued so far (in a capture it joins the same graph)."""
        if which not in self._side:
            self._side[which] = (torch.cuda.Stream(self.dev), torch.cuda.Event(), torch.cuda.Event())
        side, forked, _ = self._side[which]
        forked.record()
        side.wait_event(forked)
        return side

    def _join(self, which: int = 0) -> None:
        side, _, done = self._side[which]
        done.record(side)
        torch.cuda.current_stream().wait_event(done)

    @staticmethod
    def _walk(work: "K.Ragged", longest: int) -> "K.Ragged":
        """The work list with blocks of ``longest`` tokens where every sequence is one block anyway."""
        if longest < NativeLayered.BLOCK:
            work = K.Ragged.from_buffer_copy(work)
            work.B = longest
        return work

    # ---- forward ------------------------------------------------------------------------
    def _run(self, ids, positions, locs, T: int, work: "K.Ragged", single_rows: Optional[torch.Tensor], longest: int) -> torch.Tensor:
        raise NotImplementedError

    def forward(self, ids, positions, cache_locs, rows, prefix_lens, bs: int, E: int, two_pass: bool = False) -> torch.Tensor:
        """bs sequences of E new tokens each."""
        work = uniform_struct(rows, prefix_lens, bs, E, self.BLOCK)
        return self._run(ids, positions, cache_locs, bs * E, work, rows if E == 1 else None, E)

    def forward_plan(self, plan: RaggedPlan) -> torch.Tensor:
        self.ctx_hint = plan.max_keys
        return self._run(plan.ids, plan.positions, plan.locs, plan.T, plan.struct, plan.rows if plan.single else None,
                         plan.longest)

    # ---- head ---------------------------------------------------------------------------
    def final_hidden(self, rows_idx: torch.Tensor) -> torch.Tensor:
        return self.xa[rows_idx]

    def project(self, X: torch.Tensor, rows: int, ldx: Optional[int] = None) -> torch.Tensor:
        """fp32 logits of ``rows`` final rows X (pitch ``ldx``), left in the chain's logits buffer."""
        W, out = self.m.lm_head, self.logits
        if self.f32:
            K.gemm_f32(W, X, out, N=W.shape[0], M=rows, ldx=ldx, pdl=self.pdl)
        else:
            K.gemm_skinny(W, X, out, M=rows, splits=1, epi=K.EPI_STORE_F32, ldx=ldx, ldo=out.stride(0), status=self.status,
                          pdl=self.pdl)
        return out

    def lm_head(self, rows: int, row_offset: int = 0, row_step: int = 1) -> torch.Tensor:
        return self.project(self.xa[row_offset:], rows, self.d8 * row_step)

    def lm_head_sample(self, rows: int, row_offset: int, row_step: int, *, temperature: float, alpha: float, tokens_in, seed: int,
                       cycle_counter, call_id: int, tok_out, logp_out, logz_out) -> None:
        V = self.c.vocab_size
        if self._lm_parts is None or self._lm_parts.numel() < K.lm_parts_bytes(rows, V):
            self._lm_parts = torch.empty(K.lm_parts_bytes(max(rows, self.logits.shape[0]), V), dtype=torch.uint8, device=self.dev)
        K.lm_head_sample(self.m.lm_head, self.xa[row_offset:], M=rows, V=V, ldx=self.d8 * row_step, status=self.status,
                         temperature=temperature, alpha=alpha, softcap=float(self.c.logit_softcap), tokens_in=tokens_in, seed=seed,
                         cycle_counter=cycle_counter, call_id=call_id, parts=self._lm_parts, tok_out=tok_out, logp_out=logp_out,
                         logz_out=logz_out, pdl=self.pdl)
