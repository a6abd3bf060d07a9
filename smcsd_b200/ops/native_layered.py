"""What the kernel chains of the layer-by-layer families share: buffers viewed per layer with that layer's own widths, products
in bf16 (tensor cores) or in 32-bit, steps over sequences of unequal length (``ops/ragged.py``) or over a uniform batch that
can be captured in a graph, and the head."""
from __future__ import annotations

import os
from typing import Dict, Optional

import torch

from ..models.layered import round_up
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

    def _gated_gemm(self, W: torch.Tensor, X: torch.Tensor, act: torch.Tensor, M: int, blk: int, link: "K.GroupLink",
                    shift: float) -> None:
        """act = gated unit of the interleaved gate / up product: the link's activation, ``shift`` added to the up value."""
        ff2 = W.shape[-2]
        if self.f32:
            gu = self._rows("gu", M, ff2)
            K.gemm_f32(W, X, gu, N=ff2, M=M, link=link, pdl=self.pdl)
            K.gated_unit_f32(gu, act, ff=ff2 // 2, blk=blk, limit=link.limit, slope=link.slope, shift=shift, M=M, pdl=self.pdl)
            return
        splits = K.gemm_swiglu_splits(ff2, W.shape[-1], M) if link.mode == 0 else 1
        if link.mode == 0 and link.act == K.ACT_SILU:        # the plain build of the kernel has this unit
            K.gemm_skinny(W, X, act, M=M, splits=splits, epi=K.EPI_SWIGLU_BF16, ldo=act.stride(0), status=self.status, pdl=self.pdl)
            return
        K.gemm_grouped(W, X, act, N=ff2, M=M, splits=splits, epi=K.EPI_SWIGLU_BF16, link=link, status=self.status, pdl=self.pdl)

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
