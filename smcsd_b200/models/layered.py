"""What the layer-by-layer families (Pasizen, Makodra, Funevik, Padadra) have in common: padded weight layouts, checkpoints whose tensors are
named per layer and checked against the configuration, activations rounded and padded for the GEMMs."""
from __future__ import annotations

from typing import Iterator, List, Optional

import torch

from .config import ModelConfig
from .llama import interleave_gate_up
from .loader import Checkpoint

GU_BLOCK = 64


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def pad_to(w: torch.Tensor, *shape: int) -> torch.Tensor:
    """Zero-padded copy of ``w`` with the given (not smaller) shape."""
    out = torch.zeros(*shape, dtype=w.dtype, device=w.device)
    out[tuple(slice(0, n) for n in w.shape)] = w
    return out


def pad_heads(w: torch.Tensor, heads: int, to: int) -> torch.Tensor:
    """Rows [heads * size, d] -> [heads * to, d] with zero rows behind every head."""
    n, d = w.shape
    return pad_to(w.view(heads, n // heads, d), heads, to, d).view(heads * to, d)


class LayeredModel:
    """Subclasses fill the packed layout in ``_assemble(get)``, where ``get(name, *shape)`` returns a tensor by its
    checkpoint name (``None`` entries of a shape accept any size)."""
    has_state = True
    family = ""

    def __init__(self, cfg: ModelConfig, dtype=torch.bfloat16, device="cpu", tp_rank: int = 0, tp_size: int = 1,
                 max_positions: Optional[int] = None):
        if tp_size != 1:
            raise ValueError(f"{self.family} models run with tp_size=1")
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        self.tp_rank, self.tp_size, self.tp_group = 0, 1, None
        self.n_heads, self.n_kv_heads = cfg.n_heads, cfg.n_kv_heads
        self.layers: List = []
        self.embed = self.pos = self.lm_head = self.final_norm = None
        self.runs = cfg.layer_runs

    # ---- parameters --------------------------------------------------------------------
    def all_tensors(self) -> Iterator[torch.Tensor]:
        for t in (self.embed, self.pos, self.final_norm, self.lm_head if self.lm_head is not self.embed else None):
            if t is not None:
                yield t
        for L in self.layers:
            yield from L.tensors()

    def weight_bytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.all_tensors())

    def _assemble(self, get) -> "LayeredModel":
        raise NotImplementedError

    def load_hf(self, path: str) -> "LayeredModel":
        ck = Checkpoint(path)

        def get(name, *shape):
            t = ck.get(name)
            if len(t.shape) != len(shape) or any(w is not None and n != w for n, w in zip(t.shape, shape)):
                raise ValueError(f"{name}: shape {tuple(t.shape)} in the checkpoint, {tuple(shape)} by the configuration")
            return t
        try:
            return self._assemble(get)
        finally:
            ck.close()

    @staticmethod
    def _pack_glu(mat, p: str, ff: int, d: int):
        """Gate / up rows interleaved in blocks of GU_BLOCK channels, and the down matrix, of the gated unit named ``p``."""
        f, d8 = round_up(ff, GU_BLOCK), round_up(d, 8)
        gu = interleave_gate_up(pad_to(mat(p + "gate", ff, d), f, d8), pad_to(mat(p + "up", ff, d), f, d8), GU_BLOCK)
        return gu, pad_to(mat(p + "down", d, ff), d, f)

    def _pack_experts(self, mat, p: str, experts: int, ff: int, d: int):
        """The same of all experts, stacked."""
        packed = [self._pack_glu(mat, f"{p}e{e}.", ff, d) for e in range(experts)]
        return torch.stack([g for g, _ in packed]), torch.stack([w for _, w in packed])

    # ---- plain-PyTorch forward ----------------------------------------------------------
    @staticmethod
    def _mix_experts(x: torch.Tensor, idx: torch.Tensor, w: torch.Tensor, run) -> torch.Tensor:
        """fp32 sum over the chosen experts (ids and weights [T, top]); ``run(expert, rows of x)`` gives an expert's output."""
        out = None
        for e in idx.unique().tolist():
            t, j = (idx == e).nonzero(as_tuple=True)
            y = run(e, x[t])
            out = torch.zeros(x.shape[0], y.shape[1], device=x.device) if out is None else out
            out.index_add_(0, t, w[t, j].unsqueeze(1) * y)
        return out

    def _act(self, h: torch.Tensor) -> torch.Tensor:
        """fp32 rows in the activation dtype, padded to the GEMM operand width."""
        d8 = round_up(h.shape[1], 8)
        return pad_to(h.to(self.dtype), h.shape[0], d8) if d8 != h.shape[1] else h.to(self.dtype)

    def logits_torch(self, hidden: torch.Tensor) -> torch.Tensor:
        lg = (hidden @ self.lm_head.t()).float()
        cap = self.cfg.logit_softcap
        return torch.tanh(lg / cap) * cap if cap > 0 else lg
