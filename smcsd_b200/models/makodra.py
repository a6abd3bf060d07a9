"""Makodra: a decoder whose layers mix tokens by a generalized delta rule, by a decaying memory over token-shifted inputs, or
by attention inside chunks, in any order.  Norms sit on the sublayers' outputs (x <- x + norm(f(x))), so sublayers read the
residual stream itself; a sinusoidal position vector enters at the embedding, the embedding also is the output matrix.

Weight layout (shared with the kernel chain; dim' and vdim' are rounded up to 8, with zero rows in between, as is every
reduction dimension):
  attention      win   [H dim' + G dim' + G vdim' + H vdim', d']   queries | keys | values | output gate
                 wo    [d, H vdim']
  general_delta  win   [5 H dim + rank', d']                       r | k | v | gate | removal rate | low-rank decay input
                 w2    [H dim, rank'], wo [d, (H dim)']
  wkv            win   [4 H dim, d']                               r | k | v | gate, each for its own shifted input
                 w1    [rank', d'], w2 [H dim, rank'], wo [d, (H dim)']
  swiglu         wgu   [2 ff', d']  gate / up rows interleaved in blocks of 64 channels, wdown [d, ff']
Norm weights, shift coefficients, decay offsets, bonuses and distance-bias numbers are kept in fp32.

The state of a sequence is its keys and values in the paged cache (attention layers, one row width each), the previous row
of the residual stream (wkv layers) and one matrix per head (both recurrent kinds), stored transposed [value, key] in fp32.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Iterator, List, Optional

import torch

from ..memory.pools import KVSpec, StateSpec
from .config import ChunkAttentionSpec, LayerSpec
from .layered import GU_BLOCK, LayeredModel, pad_heads, pad_to, round_up
from .layers import (ExtendBatch, bonus_memory, chunk_attention_reference, delta_memory, rms_unit, sinusoidal_positions, swiglu,
                     token_shift)
from .llama import split_gate_up

SHIFTED = "rkvgw"                            # order of the shifted inputs
DELTA_LOG_DECAY = math.exp(-0.5)             # largest -ln of a delta-rule decay


@dataclass
class MakodraLayerWeights:
    spec: LayerSpec
    index: int                                # among the layers with the same kind of memory (cache or matrices)
    win: torch.Tensor
    wo: torch.Tensor
    norm1: torch.Tensor
    # attention
    r1: Optional[torch.Tensor] = None
    r2: Optional[torch.Tensor] = None
    lam: float = 0.0                          # share of the first values; 0 in the layer that supplies them
    gives_values: bool = False
    # recurrent kinds
    shift_index: int = -1                     # among the layers with a token shift
    w1: Optional[torch.Tensor] = None
    w2: Optional[torch.Tensor] = None
    w0: Optional[torch.Tensor] = None
    a_bias: Optional[torch.Tensor] = None
    mu: Optional[torch.Tensor] = None
    bonus: Optional[torch.Tensor] = None
    onorm: Optional[torch.Tensor] = None
    # feed-forward
    norm2: Optional[torch.Tensor] = None
    wgu: Optional[torch.Tensor] = None
    wdown: Optional[torch.Tensor] = None

    @property
    def kind(self) -> str:
        return "attention" if isinstance(self.spec.mixer, ChunkAttentionSpec) else self.spec.mixer.kind

    def tensors(self) -> Iterator[torch.Tensor]:
        return (v for v in vars(self).values() if isinstance(v, torch.Tensor))


class MakodraModel(LayeredModel):
    family = "Makodra"

    @property
    def has_state(self) -> bool:
        return self.state_spec() is not None

    # ---- cache and state ---------------------------------------------------------------
    def kv_spec(self, dtype, fp8: bool = False) -> KVSpec:
        if fp8:
            raise ValueError("caches with a row width per layer have no fp8 layout")
        ms = [L.mixer for L in self.cfg.layers if isinstance(L.mixer, ChunkAttentionSpec)]
        widths = [(m.kv_heads * round_up(m.dim, 8), m.kv_heads * round_up(m.vdim, 8)) for m in ms]
        return KVSpec(len(widths), 1, max((w for w, _ in widths), default=0), dtype, row_widths=widths)

    def state_spec(self) -> Optional[StateSpec]:
        ms = [L.mixer for L in self.cfg.layers if not isinstance(L.mixer, ChunkAttentionSpec)]
        if not ms:
            return None
        return StateSpec(sum(m.kind == "wkv" for m in ms), round_up(self.cfg.hidden_size, 4), 2, 0, 0, 0, conv_dtype=torch.float32,
                         matrices=[(m.heads, m.dim, m.dim) for m in ms])

    # ---- parameters --------------------------------------------------------------------
    def _assemble(self, get) -> "MakodraModel":
        c, dt, dev = self.cfg, self.dtype, self.device
        d, d8 = c.hidden_size, round_up(c.hidden_size, 8)

        def mat(name, *shape):
            return get(name, *shape).to(device=dev, dtype=dt, copy=True)

        def vec(name, *shape):
            return get(name, *shape).to(device=dev, dtype=torch.float32, copy=True).contiguous()

        def rows(name, n):
            return pad_to(mat(name, n, d), n, d8)

        self.embed, self.final_norm = mat("embed", c.vocab_size, d), vec("final.norm", d)
        self.lm_head = self.embed if d8 == d else pad_to(self.embed, c.vocab_size, d8)
        n_attn = n_rec = n_shift = 0
        mixing = False                        # a layer before has supplied the first values
        for li, spec in enumerate(c.layers):
            p, m, f = f"l{li}.", spec.mixer, spec.mlp
            x = p + "mix."
            if isinstance(m, ChunkAttentionSpec):
                H, G, D8, V8 = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8)
                win = [pad_heads(rows(x + n, h * w), h, w8) for n, h, w, w8 in
                       (("q", H, m.dim, D8), ("k", G, m.dim, D8), ("v", G, m.vdim, V8), ("g", H, m.vdim, V8))]
                wo = pad_to(mat(x + "o", d, H * m.vdim).view(d, H, m.vdim), d, H, V8).view(d, H * V8)
                L = MakodraLayerWeights(spec, n_attn, torch.cat(win), wo, vec(p + "norm1", d), r1=vec(x + "r1", H), r2=vec(x + "r2", H),
                                        lam=float(get(x + "vmix")) if m.v_mix and mixing else 0.0, gives_values=m.v_mix and not mixing)
                mixing |= m.v_mix
                n_attn += 1
            else:
                HD, delta = m.heads * m.dim, m.kind == "general_delta"
                w1 = mat(x + "w1", None, d)
                rank = w1.shape[0]
                w1 = pad_to(w1, round_up(rank, 8), d8)
                win = [rows(x + n, HD) for n in ("r", "k", "v", "g") + (("a",) if delta else ())] + ([w1] if delta else [])
                L = MakodraLayerWeights(spec, n_rec, torch.cat(win), pad_to(mat(x + "o", d, HD), d, round_up(HD, 8)), vec(p + "norm1", d),
                                        w2=pad_to(mat(x + "w2", HD, rank), HD, w1.shape[0]), w0=vec(x + "w0", HD), onorm=vec(x + "norm", HD))
                if delta:
                    L.a_bias = vec(x + "a.b", HD)
                else:
                    L.shift_index, L.w1, L.bonus = n_shift, w1, vec(x + "u", m.heads, m.dim)
                    L.mu = torch.stack([vec(x + "mu." + s, d) for s in SHIFTED])
                    n_shift += 1
                n_rec += 1
            if f is not None:
                L.norm2 = vec(p + "norm2", d)
                L.wgu, L.wdown = self._pack_glu(mat, p + "mlp.", f.ff, d)
            self.layers.append(L)
        return self

    def init_random(self, seed: int = 0, std: float = 0.02) -> "MakodraModel":
        g = torch.Generator(device=self.device)
        g.manual_seed(seed)
        rank = 64 if self.cfg.hidden_size >= 1024 else 16

        def get(name, *shape):
            r = torch.randn([rank if n is None else n for n in shape], generator=g, device=self.device, dtype=torch.float32)
            leaf = name.rsplit(".", 1)[-1]
            if leaf.startswith("norm"):
                return 1.0 + 0.1 * r
            if ".mu." in name or leaf == "vmix":
                return 0.5 + 0.2 * r
            if leaf in ("r1", "r2"):
                return 0.5 * r.abs() + 0.1
            if leaf in ("w0", "b", "u"):
                return 0.5 * r
            return r * std
        return self._assemble(get)

    # ---- plain-PyTorch forward ----------------------------------------------------------
    def _attention(self, L: MakodraLayerWeights, x: torch.Tensor, batch: ExtendBatch, kv, block_table, v_first):
        m, T = L.spec.mixer, x.shape[0]
        H, G, D8, V8 = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8)
        q, k, v, g = (self._act(x) @ L.win.t()).float().split([H * D8, G * D8, G * V8, H * V8], dim=1)
        unit = lambda y, n: pad_to(rms_unit(y.view(T, n, D8)[..., :m.dim], self.cfg.rms_eps), T, n, D8)
        if L.gives_values:
            v_first = v
        elif m.v_mix:
            v = (1.0 - L.lam) * v + L.lam * v_first
        kv.write(L.index, batch.cache_locs, unit(k, G), v)
        o = chunk_attention_reference(unit(q, H).to(self.dtype), kv.k[L.index], kv.v[L.index], block_table, batch, G, m.scale, L.r1, L.r2,
                                      m.chunk)
        o = (o.reshape(T, -1) * torch.sigmoid(g)).to(self.dtype)
        return (o @ L.wo.t()).float(), v_first

    def _recurrent(self, L: MakodraLayerWeights, x: torch.Tensor, batch: ExtendBatch, state, rows) -> torch.Tensor:
        m, T = L.spec.mixer, x.shape[0]
        H, D, HD = m.heads, m.dim, m.heads * m.dim
        if m.kind == "general_delta":
            y = (self._act(x) @ L.win.t()).float()
            r, k, v, g, a = y[:, :5 * HD].split(HD, dim=1)
            low, a = torch.tanh(y[:, 5 * HD:]), torch.sigmoid(a + L.a_bias)
        else:
            sh = token_shift(x, L.mu, batch, state.conv[L.shift_index], rows)
            r, k, v, g = ((self._act(sh[:, i]) @ w.t()).float() for i, w in enumerate(L.win.split(HD)))
            low = torch.tanh((self._act(sh[:, 4]) @ L.w1.t()).float())
        z = (low.to(self.dtype) @ L.w2.t()).float() + L.w0
        if m.kind == "general_delta":
            w, gate = torch.exp(-DELTA_LOG_DECAY * torch.sigmoid(z)), torch.sigmoid(g)
        else:
            w, gate = torch.exp(-torch.exp(z)), g * torch.sigmoid(g)
        r, k, v, w = (t.reshape(T, H, D) for t in (r, k, v, w))
        o, S, t0 = torch.empty(T, H, D, device=x.device), state.matrix(L.index), 0
        for b, e in enumerate(batch.lens()):
            s, M = slice(t0, t0 + e), S[rows[b]]
            if m.kind == "general_delta":
                o[s] = delta_memory(M, r[s], w[s], k[s], v[s], a.view(T, H, D)[s])
            else:
                o[s] = bonus_memory(M, r[s], w[s], k[s], v[s], L.bonus)
            t0 += e
        o = rms_unit(o, self.cfg.rms_eps).reshape(T, HD) * L.onorm * gate
        return (self._act(o) @ L.wo.t()).float()

    def forward_torch(self, batch: ExtendBatch, kv, block_table: torch.Tensor, state=None, per_run: Optional[List] = None) -> torch.Tensor:
        """Post-norm hidden rows of the new tokens; ``per_run`` (a list) collects the residual stream after every layer."""
        if state is None and self.has_state:
            raise ValueError("Makodra models need a recurrent-state pool")
        c, v_first = self.cfg, None
        rows = (batch.state_rows if batch.state_rows is not None else batch.rows).long()
        x = self.embed[batch.input_ids.long()].float() + sinusoidal_positions(batch.positions, c.hidden_size)
        for L in self.layers:
            if L.kind == "attention":
                y, v_first = self._attention(L, x, batch, kv, block_table, v_first)
            else:
                y = self._recurrent(L, x, batch, state, rows)
            x = x + rms_unit(y, c.rms_eps) * L.norm1
            if L.spec.mlp is not None:
                gate, up = split_gate_up(self._act(x) @ L.wgu.t(), GU_BLOCK)
                x = x + rms_unit((swiglu(gate, up) @ L.wdown.t()).float(), c.rms_eps) * L.norm2
            if per_run is not None:
                per_run.append(x)
        return self._act(rms_unit(x, c.rms_eps) * self.final_norm)
