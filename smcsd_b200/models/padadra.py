"""Padadra: a decoder whose layers run a mixer and a feed-forward side by side on the same residual stream, each behind a norm
with a single weight: x <- x + m (mixer(norm1 x) + ff(norm2 x)).  Mixers, in any order: a delta rule with a decay per head and
channel behind a short convolution (queries and keys shared by groups of heads, decay and output gate through low-rank maps), and
a pair that reads the same input: attention inside a sliding window with learned sinks, whose values turn with their position and
back at the reader's, beside a memory whose forget gate also decides what is written (HGRN2); half the sum of both, each behind a
norm of its own.  The feed-forward is a squared relu between two matrices, or missing.  The embedding adds a row per pair of
neighbouring tokens.

Weight layout (shared with the kernel chain; sizes with a prime are rounded up to 8, with zero rows or columns in between):
  channel_delta  win    [(G dim + G dim + H vdim)' + H' + a_rank' + g_rank', d']   queries | keys | values | write strength |
                                                                                   decay input | gate input
                 conv   [2 G dim + H vdim, taps]                                   fp32
                 wa     [H dim, a_rank'], wg [H vdim, g_rank']                     low-rank maps of decay and gate
                 wo     [d, (H vdim)']
  parallel       win    [(H dim' + G dim' + G vdim' + 2 H2 dim2 + H2 vdim2)', d']  queries | keys | values of the attention, then
                                                                                   queries | forget gate | values of the memory
                 bias, conv, qk_norm                                               of the attention's columns, fp32
                 wo     [d, H vdim'], wo2 [d, (H2 vdim2)']
  feed-forward   wup    [ff', d'], wdown [d, ff']
Norm weights, biases, sinks, convolution taps, decay constants and bounds are kept in fp32.

The state of a sequence is its rows in the paged cache (rotated keys and values of the attention layers) and, all fp32, the
token before the next one, per memory its matrix, and per convolution the last taps - 1 projections.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Iterator, List, Optional

import torch
import torch.nn.functional as F

from ..memory.pools import KVSpec, StateSpec
from .config import GroupedAttentionSpec, LayerSpec, ParallelSpec, RecurrentSpec
from .layered import LayeredModel, pad_heads, pad_to, round_up
from .layers import (ExtendBatch, channel_delta_memory, chunk_attention_reference, forget_memory, pair_rows, rms_unit, rope_frequencies,
                     short_conv, turn_pairs)

UNIT_EPS = 1e-6                           # of the delta rule's unit queries and keys


@dataclass
class PadadraLayerWeights:
    spec: LayerSpec
    win: torch.Tensor
    wo: torch.Tensor
    norm1: torch.Tensor                       # [1]
    conv: torch.Tensor
    onorm: torch.Tensor                       # of the memory's read-out, repeated for every head
    state: int                                # first of the layer's entries in the state row: convolution, matrix
    cache: int = -1                           # among the layers with cached rows
    # channel_delta
    wa: Optional[torch.Tensor] = None
    wg: Optional[torch.Tensor] = None
    dt_bias: Optional[torch.Tensor] = None
    a_log: Optional[torch.Tensor] = None
    # parallel
    bias: Optional[torch.Tensor] = None
    qk_norm: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None
    f_bias: Optional[torch.Tensor] = None
    lower: Optional[torch.Tensor] = None
    wo2: Optional[torch.Tensor] = None
    out1: Optional[torch.Tensor] = None
    out2: Optional[torch.Tensor] = None
    # feed-forward
    norm2: Optional[torch.Tensor] = None
    wup: Optional[torch.Tensor] = None
    wdown: Optional[torch.Tensor] = None

    @property
    def parallel(self) -> bool:
        return isinstance(self.spec.mixer, ParallelSpec)

    def tensors(self) -> Iterator[torch.Tensor]:
        return (v for v in vars(self).values() if isinstance(v, torch.Tensor))


def attention_columns(m: GroupedAttentionSpec) -> int:
    return (m.heads + m.kv_heads) * round_up(m.dim, 8) + m.kv_heads * round_up(m.vdim, 8)


def delta_columns(m: RecurrentSpec) -> int:
    return 2 * m.kv_heads * m.dim + m.heads * m.values


def frequencies(rot) -> torch.Tensor:
    return rope_frequencies(rot.dims, rot.base, rot.scaling_dict())


class PadadraModel(LayeredModel):
    family = "Padadra"

    def __init__(self, *args, **kw):
        super().__init__(*args, **kw)
        self.bigram: Optional[torch.Tensor] = None

    # ---- cache and state ---------------------------------------------------------------
    def kv_spec(self, dtype, fp8: bool = False) -> KVSpec:
        if fp8:
            raise ValueError("caches with a row width per layer have no fp8 layout")
        widths = [(m.left.kv_heads * round_up(m.left.dim, 8), m.left.kv_heads * round_up(m.left.vdim, 8))
                  for m in (L.mixer for L in self.cfg.layers) if isinstance(m, ParallelSpec)]
        return KVSpec(len(widths), 1, max((w for w, _ in widths), default=0), dtype, row_widths=widths)

    def state_spec(self) -> StateSpec:
        parts = [(1, 1, 1)]                                   # the token before
        for m in (L.mixer for L in self.cfg.layers):
            if isinstance(m, ParallelSpec):
                parts += [(1, m.left.conv - 1, attention_columns(m.left)), (m.right.heads, m.right.values, m.right.dim)]
            else:
                parts += [(1, m.conv - 1, delta_columns(m)), (m.heads, m.values, m.dim)]
        return StateSpec(0, 1, 2, 0, 0, 0, conv_dtype=torch.float32, matrices=parts)

    # ---- parameters --------------------------------------------------------------------
    def all_tensors(self) -> Iterator[torch.Tensor]:
        yield from super().all_tensors()
        if self.bigram is not None:
            yield self.bigram

    def _assemble(self, get) -> "PadadraModel":
        c, dt, dev = self.cfg, self.dtype, self.device
        d, d8 = c.hidden_size, round_up(c.hidden_size, 8)
        if c.vocab_size > 1 << 24:
            raise ValueError("the state keeps token ids as fp32 numbers, exact up to 2^24")

        def mat(name, *shape):
            return get(name, *shape).to(device=dev, dtype=dt, copy=True)

        def vec(name, *shape):
            return get(name, *shape).to(device=dev, dtype=torch.float32, copy=True).contiguous()

        def one(name):
            return vec(name).reshape(1)

        def rows(name, n):
            return pad_to(mat(name, n, d), n, d8)

        def stack(*parts):
            w = torch.cat(parts)
            return pad_to(w, round_up(w.shape[0], 8), w.shape[1])

        self.embed, self.final_norm = mat("embed", c.vocab_size, d), one("final.norm")
        self.lm_head = pad_to(mat("head", c.vocab_size, d), c.vocab_size, d8)
        if c.bigram is not None:
            self.bigram = mat("bigram", c.bigram[0] + 1, d)
        n_cache, n_state = 0, 1
        for li, spec in enumerate(c.layers):
            p, m, f = f"l{li}.", spec.mixer, spec.mlp
            x, own = p + "mix.", dict(spec=spec, norm1=one(p + "norm1"), state=n_state)
            n_state += 2
            if isinstance(m, ParallelSpec):
                a, b, l, r = m.left, m.right, x + "left.", x + "right."
                H, G, D8, E8, HV = a.heads, a.kv_heads, round_up(a.dim, 8), round_up(a.vdim, 8), b.heads * b.values
                heads = (("q", H, a.dim, D8), ("k", G, a.dim, D8), ("v", G, a.vdim, E8))
                L = PadadraLayerWeights(
                    win=stack(*(pad_heads(rows(l + n, h * w), h, w8) for n, h, w, w8 in heads), rows(r + "q", b.heads * b.dim),
                              rows(r + "f", b.heads * b.dim), rows(r + "v", HV)), cache=n_cache,
                    bias=torch.cat([pad_heads(vec(f"{l}{n}.b", h * w).unsqueeze(1), h, w8) for n, h, w, w8 in heads]).squeeze(1).contiguous(),
                    conv=torch.cat([pad_heads(vec(f"{l}{n}.conv", h * w, a.conv), h, w8) for n, h, w, w8 in heads]),
                    qk_norm=torch.cat([pad_heads(vec(f"{l}{n}.norm", h * w).unsqueeze(1), h, w8) for n, h, w, w8 in heads[:2]]).squeeze(1).contiguous(),
                    sink=vec(l + "sink", H), wo=pad_to(mat(l + "o", d, H * a.vdim).view(d, H, a.vdim), d, H, E8).view(d, H * E8),
                    f_bias=vec(r + "f.b", b.heads * b.dim), lower=vec(r + "lower", b.heads * b.dim), onorm=vec(r + "norm", b.values).repeat(b.heads),
                    wo2=pad_to(mat(r + "o", d, HV), d, round_up(HV, 8)), out1=vec(l + "out", d), out2=vec(r + "out", d), **own)
                n_cache += 1
            else:
                H, G, D, E = m.heads, m.kv_heads, m.dim, m.values
                a1, g1 = mat(x + "a1", None, d), mat(x + "g1", None, d)
                wa, wg = mat(x + "a2", H * D, a1.shape[0]), mat(x + "g2", H * E, g1.shape[0])
                a1, g1 = (pad_to(w, round_up(w.shape[0], 8), d8) for w in (a1, g1))
                L = PadadraLayerWeights(
                    win=torch.cat([stack(rows(x + "q", G * D), rows(x + "k", G * D), rows(x + "v", H * E)), stack(rows(x + "b", H)), a1, g1]),
                    conv=torch.cat([vec(f"{x}{n}.conv", w, m.conv) for n, w in (("q", G * D), ("k", G * D), ("v", H * E))]),
                    wa=pad_to(wa, H * D, a1.shape[0]), wg=pad_to(wg, H * E, g1.shape[0]), dt_bias=vec(x + "dt_bias", H * D), a_log=vec(x + "A_log", H),
                    onorm=vec(x + "norm", E).repeat(H), wo=pad_to(mat(x + "o", d, H * E), d, round_up(H * E, 8)), **own)
            if f is not None:
                F8 = round_up(f.ff, 8)
                L.norm2 = one(p + "norm2")
                L.wup, L.wdown = pad_to(mat(p + "mlp.up", f.ff, d), F8, d8), pad_to(mat(p + "mlp.down", d, f.ff), d, F8)
            self.layers.append(L)
        return self

    def init_random(self, seed: int = 0, std: float = 0.02) -> "PadadraModel":
        g = torch.Generator(device=self.device)
        g.manual_seed(seed)
        rank = 64 if self.cfg.hidden_size >= 1024 else 16

        def get(name, *shape):
            r = torch.randn([rank if n is None else n for n in shape], generator=g, device=self.device, dtype=torch.float32)
            leaf = name.rsplit(".", 1)[-1]
            if leaf.startswith("norm") or leaf == "out":
                return 1.0 + 0.1 * r
            if leaf == "b" and len(shape) == 1:
                return (2.0 if ".f." in name else 0.0) + 0.5 * r
            if leaf == "lower":
                return 0.5 * torch.sigmoid(r)
            if leaf in ("sink", "A_log"):
                return r
            if leaf == "dt_bias":
                return r - 4.0
            if leaf == "conv":
                return 0.4 * r
            if leaf in ("a2", "g2"):
                return r * r.shape[1] ** -0.5
            return r * std
        return self._assemble(get)

    # ---- plain-PyTorch forward ----------------------------------------------------------
    @staticmethod
    def _conv(y: torch.Tensor, w: torch.Tensor, taps: int, batch: ExtendBatch, state, entry: int, rows) -> torch.Tensor:
        C = y.shape[1]
        hist = state.matrix(entry)[:, 0].transpose(1, 2) if taps > 1 else y.new_empty(int(rows.max()) + 1, C, 0)
        return short_conv(y, w, batch, hist, rows)

    def _delta(self, L: PadadraLayerWeights, x: torch.Tensor, batch: ExtendBatch, state, rows) -> torch.Tensor:
        m, T, C = L.spec.mixer, x.shape[0], delta_columns(L.spec.mixer)
        H, G, D, E, ra, rg = m.heads, m.kv_heads, m.dim, m.values, L.wa.shape[1], L.wg.shape[1]
        y = (x @ L.win.t()).float()
        C8 = round_up(C, 8)
        b, low_a, low_g = y[:, C8:C8 + H], y[:, -ra - rg:-rg], y[:, -rg:]
        u = F.silu(self._conv(y[:, :C], L.conv, m.conv, batch, state, L.state, rows))
        q, k, v = u.split([G * D, G * D, H * E], dim=1)
        unit = lambda z: z * torch.rsqrt((z * z).sum(-1, keepdim=True) + UNIT_EPS)
        q, k = (unit(z.reshape(T, G, D)).repeat_interleave(H // G, dim=1) for z in (q, k))
        z = ((low_a.to(x.dtype) @ L.wa.t()).float() + L.dt_bias).view(T, H, D)
        g = torch.exp(-torch.exp(L.a_log).view(1, H, 1) * F.softplus(z, threshold=100.0))
        o, M, t0 = torch.empty(T, H, E, device=x.device), state.matrix(L.state + 1), 0
        for s, e in enumerate(batch.lens()):
            t = slice(t0, t0 + e)
            o[t] = channel_delta_memory(M[rows[s]], q[t] * D ** -0.5, k[t], v[t].reshape(e, H, E), g[t], torch.sigmoid(b[t]))
            t0 += e
        gate = torch.sigmoid((low_g.to(x.dtype) @ L.wg.t()).float())
        return rms_unit(o, self.cfg.rms_eps).reshape(T, H * E) * L.onorm * gate

    def _attention(self, L: PadadraLayerWeights, y: torch.Tensor, batch: ExtendBatch, kv, block_table, state, rows) -> torch.Tensor:
        m, T, eps = L.spec.mixer.left, y.shape[0], self.cfg.rms_eps
        H, G, D8, E8 = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8)
        u = self._conv(y + L.bias, L.conv, m.conv, batch, state, L.state, rows)
        q, k, v = u.split([H * D8, G * D8, G * E8], dim=1)
        whole = lambda z, n: z * torch.rsqrt(z.pow(2).sum(-1, keepdim=True) / n + eps)
        q, k = whole(q, H * m.dim) * L.qk_norm[:H * D8], whole(k, G * m.dim) * L.qk_norm[H * D8:]
        freq, turn = frequencies(m.rot), frequencies(m.turn_values)
        q, k = (turn_pairs(z.reshape(T, n, D8), batch.positions, freq) for z, n in ((q, H), (k, G)))
        kv.write(L.cache, batch.cache_locs, k, turn_pairs(v.reshape(T, G, E8), batch.positions, turn))
        o = chunk_attention_reference(q.to(self.dtype), kv.k[L.cache], kv.v[L.cache], block_table, batch, G, m.scale, None, None, 0,
                                      window=m.window, sink=L.sink)
        return turn_pairs(o, batch.positions, turn, back=True).reshape(T, H * E8)

    def _memory(self, L: PadadraLayerWeights, y: torch.Tensor, batch: ExtendBatch, state, rows) -> torch.Tensor:
        m, T = L.spec.mixer.right, y.shape[0]
        H, D, E = m.heads, m.dim, m.values
        q, z, v = y[:, :H * (2 * D + E)].split([H * D, H * D, H * E], dim=1)
        z = z + L.f_bias
        f, write = ((L.lower + (1.0 - L.lower) * torch.sigmoid(z)).view(T, H, D), ((1.0 - L.lower) * torch.sigmoid(-z)).view(T, H, D))
        q, v = F.silu(q).reshape(T, H, D), v.reshape(T, H, E)
        o, M, t0 = torch.empty(T, H, E, device=y.device), state.matrix(L.state + 1), 0
        for s, e in enumerate(batch.lens()):
            t = slice(t0, t0 + e)
            o[t] = forget_memory(M[rows[s]], q[t], v[t], f[t], write[t])
            t0 += e
        return rms_unit(o, self.cfg.rms_eps).reshape(T, H * E) * L.onorm

    def forward_torch(self, batch: ExtendBatch, kv, block_table: torch.Tensor, state=None, per_run: Optional[List] = None) -> torch.Tensor:
        """Post-norm hidden rows of the new tokens; ``per_run`` (a list) collects the residual stream after every layer."""
        if state is None:
            raise ValueError("Padadra models need a recurrent-state pool")
        c, eps = self.cfg, self.cfg.rms_eps
        rows = (batch.state_rows if batch.state_rows is not None else batch.rows).long()
        x = self.embed[batch.input_ids.long()].float() * c.embed_scale
        if self.bigram is not None:
            x = x + self.bigram[pair_rows(batch.input_ids, batch, state.matrix(0)[:, 0, 0, 0], rows, *c.bigram)].float()
        for L in self.layers:
            unit = rms_unit(x, eps)
            h = self._act(unit * L.norm1)
            if L.parallel:
                y = (h @ L.win.t()).float()
                C = attention_columns(L.spec.mixer.left)
                left = (self._act(self._attention(L, y[:, :C], batch, kv, block_table, state, rows)) @ L.wo.t()).float()
                right = (self._act(self._memory(L, y[:, C:], batch, state, rows)) @ L.wo2.t()).float()
                o = 0.5 * (rms_unit(left, eps) * L.out1 + rms_unit(right, eps) * L.out2)
            else:
                o = (self._act(self._delta(L, h, batch, state, rows)) @ L.wo.t()).float()
            if L.spec.mlp is not None:
                act = torch.relu((self._act(unit * L.norm2) @ L.wup.t()).float()).square()
                o = o + (act.to(self.dtype) @ L.wdown.t()).float()
            x = x + c.residual_mult * o
            if per_run is not None:
                per_run.append(x)
        return self._act(rms_unit(x, eps) * self.final_norm)
