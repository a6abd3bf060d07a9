"""What the layer-by-layer families (Pasizen, Makodra) have in common: padded weight layouts, checkpoints whose tensors are
named per layer and checked against the configuration, activations rounded and padded for the GEMMs."""
from __future__ import annotations

from typing import Iterator, List, Optional

import torch

from .config import ModelConfig
from .loader import Checkpoint

GU_BLOCK = 64


def round_up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def pad_to(w: torch.Tensor, *shape: int) -> torch.Tensor:
    """Zero-padded copy of ``w`` with the given (not smaller) shape."""
    out = torch.zeros(*shape, dtype=w.dtype, device=w.device)
    out[tuple(slice(0, n) for n in w.shape)] = w
    return out


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

    # ---- plain-PyTorch forward ----------------------------------------------------------
    def _act(self, h: torch.Tensor) -> torch.Tensor:
        """fp32 rows in the activation dtype, padded to the GEMM operand width."""
        d8 = round_up(h.shape[1], 8)
        return pad_to(h.to(self.dtype), h.shape[0], d8) if d8 != h.shape[1] else h.to(self.dtype)

    def logits_torch(self, hidden: torch.Tensor) -> torch.Tensor:
        lg = (hidden @ self.lm_head.t()).float()
        cap = self.cfg.logit_softcap
        return torch.tanh(lg / cap) * cap if cap > 0 else lg
