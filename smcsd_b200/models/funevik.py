"""Funevik: a decoder whose layers run a mixer and a feed-forward side by side on the same residual stream, each behind its own
norm and scaled per channel: x <- x + ls1 mixer(norm1 x) + ls2 ff(norm2 x).  Mixers, in any order: a matrix memory with
exponential gates (mLSTM), latent attention with a rotated part inside a sliding window and with learned sinks, and causal
attention behind a short convolution with soft-capped scores.  Feed-forwards: a gelu gated unit, or experts beside a gated
shared expert, or none.

Weight layout (shared with the kernel chain; sizes with a prime are rounded up to 8, with zero rows or columns in between):
  mlstm             win   [(H (2 dim + 2 vdim) + 2 H)', d']          q | k | v | output gate | input gate | forget gate
                    wo    [d, (H vdim)']
  attention         win   [(H dim' + G dim' + G vdim' + H)', d']     queries | keys | values | gate per head
                    conv  [H dim' + G dim' + G vdim', taps]          fp32
                    wo    [d, H vdim']
  latent_attention  win   [(q_rank' + kv_rank + rot)', d']           query latent | cached latent | rotated key
                    wuq   [H (dim + rot)', q_rank']                  per head the unrotated, then the rotated part
                    wuk_t [H R', (dim + rot)']                       per head: transposed key expansion, and an identity that
                                                                     passes the rotated part on to the columns behind it
                                                                     (R' = kv_rank + rot rounded up to 64, the cached row)
                    wuv   [H vdim, R'], wo [d, (H vdim)']
  geglu             wgu   [2 ff', d'], wdown [d, ff']                gate / up rows interleaved in blocks of 64 channels
  moe               e_gu, e_down, s_gu, s_down likewise; router [E + 1, d'] with the shared expert's gate as its last row
Norm weights, scales, gate and router biases, sinks and convolution taps are kept in fp32.

The state of a sequence is its rows in the paged cache (latent and rotated key, or keys and values, one width per layer) and
per memory layer the matrix with its normaliser (a value column of ones) and running maximum, per attention layer the last
taps - 1 projections in front of the convolution; all fp32.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Iterator, List, Optional

import torch
import torch.nn.functional as F

from ..memory.pools import KVSpec, StateSpec
from .config import GroupedAttentionSpec, LatentAttentionSpec, LayerSpec
from .layered import GU_BLOCK, LayeredModel, pad_heads, pad_to, round_up
from .layers import (ExtendBatch, chunk_attention_reference, gated_memory, latent_attention_reference, rms_unit, rotate_pairs, route_top,
                     short_conv, soft_cap, swiglu)
from .llama import split_gate_up


@dataclass
class FunevikLayerWeights:
    spec: LayerSpec
    win: torch.Tensor
    wo: torch.Tensor
    norm1: torch.Tensor
    ls1: torch.Tensor
    cache: int = -1                           # among the layers with cached rows
    state: int = -1                           # first of the layer's entries in the state row
    # mlstm
    gate_bias: Optional[torch.Tensor] = None  # [2 H]: input gates, forget gates
    onorm: Optional[torch.Tensor] = None
    # attention
    conv: Optional[torch.Tensor] = None
    # latent attention
    q_norm: Optional[torch.Tensor] = None
    c_norm: Optional[torch.Tensor] = None
    wuq: Optional[torch.Tensor] = None
    wuk_t: Optional[torch.Tensor] = None
    wuv: Optional[torch.Tensor] = None
    sink: Optional[torch.Tensor] = None
    # feed-forward
    norm2: Optional[torch.Tensor] = None
    ls2: Optional[torch.Tensor] = None
    wgu: Optional[torch.Tensor] = None
    wdown: Optional[torch.Tensor] = None
    router: Optional[torch.Tensor] = None
    router_bias: Optional[torch.Tensor] = None
    e_gu: Optional[torch.Tensor] = None
    e_down: Optional[torch.Tensor] = None
    s_gu: Optional[torch.Tensor] = None
    s_down: Optional[torch.Tensor] = None

    @property
    def kind(self) -> str:
        m = self.spec.mixer
        return "latent" if isinstance(m, LatentAttentionSpec) else "attention" if isinstance(m, GroupedAttentionSpec) else m.kind

    def tensors(self) -> Iterator[torch.Tensor]:
        return (v for v in vars(self).values() if isinstance(v, torch.Tensor))


def latent_row(m: LatentAttentionSpec) -> int:
    """Width of a cached row: latent, rotated key, zeros."""
    return round_up(m.kv_rank + m.rot.dims, 64)


def conv_channels(m: GroupedAttentionSpec) -> int:
    return (m.heads + m.kv_heads) * round_up(m.dim, 8) + m.kv_heads * round_up(m.vdim, 8)


class FunevikModel(LayeredModel):
    family = "Funevik"

    @property
    def has_state(self) -> bool:
        return self.state_spec() is not None

    # ---- cache and state ---------------------------------------------------------------
    def kv_spec(self, dtype, fp8: bool = False) -> KVSpec:
        if fp8:
            raise ValueError("caches with a row width per layer have no fp8 layout")
        widths = []
        for m in (L.mixer for L in self.cfg.layers):
            if isinstance(m, LatentAttentionSpec):
                widths.append((latent_row(m), 0))
            elif isinstance(m, GroupedAttentionSpec):
                widths.append((m.kv_heads * round_up(m.dim, 8), m.kv_heads * round_up(m.vdim, 8)))
        return KVSpec(len(widths), 1, max((w for w, _ in widths), default=0), dtype, row_widths=widths)

    def state_spec(self) -> Optional[StateSpec]:
        parts = []
        for m in (L.mixer for L in self.cfg.layers):
            if isinstance(m, GroupedAttentionSpec):
                parts.append((1, m.conv - 1, conv_channels(m)))
            elif not isinstance(m, LatentAttentionSpec):
                parts += [(m.heads, m.values + 1, m.dim), (m.heads, 1, 1)]
        if not any(h * r * c for h, r, c in parts):
            return None
        return StateSpec(0, 1, 2, 0, 0, 0, conv_dtype=torch.float32, matrices=parts)

    # ---- parameters --------------------------------------------------------------------
    def _assemble(self, get) -> "FunevikModel":
        c, dt, dev = self.cfg, self.dtype, self.device
        d, d8 = c.hidden_size, round_up(c.hidden_size, 8)

        def mat(name, *shape):
            return get(name, *shape).to(device=dev, dtype=dt, copy=True)

        def vec(name, *shape):
            return get(name, *shape).to(device=dev, dtype=torch.float32, copy=True).contiguous()

        def rows(name, n):
            return pad_to(mat(name, n, d), n, d8)

        def stack(*parts):
            w = torch.cat(parts)
            return pad_to(w, round_up(w.shape[0], 8), w.shape[1])

        self.embed, self.final_norm = mat("embed", c.vocab_size, d), vec("final.norm", d)
        self.lm_head = pad_to(mat("head", c.vocab_size, d), c.vocab_size, d8)
        n_cache = n_state = 0
        for li, spec in enumerate(c.layers):
            p, m, f = f"l{li}.", spec.mixer, spec.mlp
            x, H = p + "mix.", m.heads
            own = dict(spec=spec, norm1=vec(p + "norm1", d), ls1=vec(p + "ls1", d))
            if isinstance(m, LatentAttentionSpec):
                D, E, R, r, Q = m.dim, m.vdim, m.kv_rank, m.rot.dims, m.q_rank
                Q8, K8, Rp = round_up(Q, 8), round_up(D + r, 8), latent_row(m)
                up = torch.zeros(H, Rp, K8, dtype=dt, device=dev)
                up[:, :R, :D] = mat(x + "uk", H * D, R).view(H, D, R).transpose(1, 2)
                up[:, R:R + r, D:D + r] = torch.eye(r, dtype=dt, device=dev)
                L = FunevikLayerWeights(
                    win=stack(pad_to(mat(x + "dq", Q, d), Q8, d8), rows(x + "dkv", R + r)), cache=n_cache,
                    wo=pad_to(mat(x + "o", d, H * E), d, round_up(H * E, 8)), q_norm=vec(x + "dq.norm", Q), c_norm=vec(x + "dkv.norm", R),
                    wuq=pad_to(mat(x + "uq", H * (D + r), Q).view(H, D + r, Q), H, K8, Q8).view(H * K8, Q8), wuk_t=up.view(H * Rp, K8),
                    wuv=pad_to(mat(x + "uv", H * E, R), H * E, Rp), sink=vec(x + "sink", H), **own)
                n_cache += 1
            elif isinstance(m, GroupedAttentionSpec):
                G, D8, E8 = m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8)
                heads = (("q", H, m.dim, D8), ("k", G, m.dim, D8), ("v", G, m.vdim, E8))
                L = FunevikLayerWeights(
                    win=stack(*(pad_heads(rows(x + n, h * w), h, w8) for n, h, w, w8 in heads), rows(x + "g", H)), cache=n_cache, state=n_state,
                    wo=pad_to(mat(x + "o", d, H * m.vdim).view(d, H, m.vdim), d, H, E8).view(d, H * E8),
                    conv=torch.cat([pad_heads(vec(f"{x}{n}.conv", h * w, m.conv), h, w8) for n, h, w, w8 in heads]), **own)
                n_cache, n_state = n_cache + 1, n_state + 1
            else:
                D, E = m.dim, m.values
                L = FunevikLayerWeights(
                    win=stack(rows(x + "q", H * D), rows(x + "k", H * D), rows(x + "v", H * E), rows(x + "g", H * E), rows(x + "i", H),
                              rows(x + "f", H)), state=n_state, wo=pad_to(mat(x + "o", d, H * E), d, round_up(H * E, 8)),
                    gate_bias=torch.cat([vec(x + "i.b", H), vec(x + "f.b", H)]), onorm=vec(x + "norm", H * E), **own)
                n_state += 2
            if f is not None:
                L.norm2, L.ls2 = vec(p + "norm2", d), vec(p + "ls2", d)
                if f.kind == "moe":
                    E = f.router.experts
                    L.router, L.router_bias = rows(p + "mlp.router", E), vec(p + "mlp.router.b", E)
                    L.e_gu, L.e_down = self._pack_experts(mat, p + "mlp.", E, f.expert.ff, d)
                    if f.shared is not None:
                        L.s_gu, L.s_down = self._pack_glu(mat, p + "mlp.shared.", f.shared.ff, d)
                        L.router = torch.cat([L.router, rows(p + "mlp.shared.sg", 1)])
                else:
                    L.wgu, L.wdown = self._pack_glu(mat, p + "mlp.", f.ff, d)
            self.layers.append(L)
        return self

    def init_random(self, seed: int = 0, std: float = 0.02) -> "FunevikModel":
        g = torch.Generator(device=self.device)
        g.manual_seed(seed)

        def get(name, *shape):
            r = torch.randn(*shape, generator=g, device=self.device, dtype=torch.float32)
            leaf = name.rsplit(".", 1)[-1]
            if leaf.startswith("norm"):
                return 1.0 + 0.1 * r
            if leaf in ("ls1", "ls2"):
                return 0.5 + 0.1 * r
            if leaf == "b":
                return (4.0 if ".f." in name else 0.0) + 0.5 * r
            if leaf == "sink":
                return r
            if leaf == "conv":
                return 0.4 * r
            if leaf in ("uk", "uv", "uq"):
                return r * shape[1] ** -0.5
            return r * std
        return self._assemble(get)

    # ---- plain-PyTorch forward ----------------------------------------------------------
    def _memory(self, L: FunevikLayerWeights, x: torch.Tensor, batch: ExtendBatch, kv, block_table, state, rows) -> torch.Tensor:
        m, T = L.spec.mixer, x.shape[0]
        H, D, E = m.heads, m.dim, m.values
        y = (x @ L.win.t()).float()
        q, k, v, g, gates = y[:, :H * (2 * D + 2 * E + 2)].split([H * D, H * D, H * E, H * E, 2 * H], dim=1)
        i, f = soft_cap(gates + L.gate_bias, m.gate_cap).split(H, dim=1)
        f = F.logsigmoid(f)
        q, k, v = q.reshape(T, H, D) * D ** -0.5, k.reshape(T, H, D), v.reshape(T, H, E)
        o, M, top, t0 = torch.empty(T, H, E, device=x.device), state.matrix(L.state), state.matrix(L.state + 1), 0
        for b, e in enumerate(batch.lens()):
            s = slice(t0, t0 + e)
            o[s] = gated_memory(M[rows[b]], top[rows[b]], q[s], k[s], v[s], i[s], f[s])
            t0 += e
        return rms_unit(o, self.cfg.rms_eps).reshape(T, H * E) * L.onorm * torch.sigmoid(g)

    def _latent(self, L: FunevikLayerWeights, x: torch.Tensor, batch: ExtendBatch, kv, block_table, state, rows) -> torch.Tensor:
        m, T, eps = L.spec.mixer, x.shape[0], self.cfg.rms_eps
        H, D, E, R, r, Q, Q8 = m.heads, m.dim, m.vdim, m.kv_rank, m.rot.dims, m.q_rank, round_up(m.q_rank, 8)
        y = (x @ L.win.t()).float()
        c = rms_unit(y[:, Q8:Q8 + R], eps) * L.c_norm
        key = rotate_pairs(y[:, Q8 + R:Q8 + R + r], batch.positions, r, m.rot.base)
        kv.write_latent(L.cache, batch.cache_locs, torch.cat([c, key], dim=1).to(x.dtype))
        q = (self._act(rms_unit(y[:, :Q], eps) * L.q_norm) @ L.wuq.t()).float().view(T, H, -1)
        q = torch.cat([q[..., :D], rotate_pairs(q[..., D:D + r], batch.positions, r, m.rot.base), q[..., D + r:]], dim=-1).to(x.dtype)
        lat = torch.einsum("thd,hrd->thr", q, L.wuk_t.view(H, -1, q.shape[-1]))
        a = latent_attention_reference(lat, kv.k[L.cache], block_table, batch, m.scale, m.window, L.sink).to(x.dtype)
        return torch.einsum("thr,hvr->thv", a, L.wuv.view(H, E, -1)).reshape(T, H * E)

    def _attention(self, L: FunevikLayerWeights, x: torch.Tensor, batch: ExtendBatch, kv, block_table, state, rows) -> torch.Tensor:
        m, T = L.spec.mixer, x.shape[0]
        H, G, D8, E8, C = m.heads, m.kv_heads, round_up(m.dim, 8), round_up(m.vdim, 8), conv_channels(m)
        y = (x @ L.win.t()).float()
        hist = state.matrix(L.state)[:, 0].transpose(1, 2) if m.conv > 1 else y.new_empty(int(rows.max()) + 1, C, 0)
        u = short_conv(y[:, :C], L.conv, batch, hist, rows)
        q, k, v = u.split([H * D8, G * D8, G * E8], dim=1)
        q, k = (rotate_pairs(z.reshape(T, n, D8), batch.positions, m.rot.dims, m.rot.base) for z, n in ((q, H), (k, G)))
        kv.write(L.cache, batch.cache_locs, k, v)
        o = chunk_attention_reference(q.to(self.dtype), kv.k[L.cache], kv.v[L.cache], block_table, batch, G, m.scale, None, None, 0, m.softcap)
        return (o * torch.sigmoid(y[:, C:C + H]).unsqueeze(-1)).reshape(T, H * E8)

    @staticmethod
    def _unit(x, gu, down, act=swiglu):
        gate, up = split_gate_up(x @ gu.t(), GU_BLOCK)
        return (act(gate, up) @ down.t()).float()

    def _feed_forward(self, L: FunevikLayerWeights, h: torch.Tensor) -> torch.Tensor:
        """h: fp32 normalised rows."""
        f, x = L.spec.mlp, self._act(h)
        if f.kind == "geglu":
            return self._unit(x, L.wgu, L.wdown, lambda g, u: (F.gelu(g.float(), approximate="tanh") * u.float()).to(x.dtype))
        z = h @ L.router[:, :h.shape[1]].float().t()
        idx, w = route_top(z[:, :f.router.experts] + L.router_bias, f.router.top)
        out = self._mix_experts(x, idx, w, lambda e, rows: self._unit(rows, L.e_gu[e], L.e_down[e]))
        if f.shared is not None:
            out = out + self._unit(x, L.s_gu, L.s_down) * torch.sigmoid(z[:, f.router.experts:])
        return out

    def forward_torch(self, batch: ExtendBatch, kv, block_table: torch.Tensor, state=None, per_run: Optional[List] = None) -> torch.Tensor:
        """Post-norm hidden rows of the new tokens; ``per_run`` (a list) collects the residual stream after every layer."""
        if state is None and self.has_state:
            raise ValueError("Funevik models need a recurrent-state pool")
        c = self.cfg
        rows = (batch.state_rows if batch.state_rows is not None else batch.rows).long()
        x = self.embed[batch.input_ids.long()].float() * c.embed_scale
        for L in self.layers:
            unit = rms_unit(x, c.rms_eps)
            mixer = {"mlstm": self._memory, "latent": self._latent, "attention": self._attention}[L.kind]
            o = mixer(L, self._act(unit * L.norm1), batch, kv, block_table, state, rows)
            y = (self._act(o) @ L.wo.t()).float() * L.ls1
            if L.spec.mlp is not None:
                y = y + self._feed_forward(L, unit * L.norm2) * L.ls2
            x = x + y
            if per_run is not None:
                per_run.append(x)
        return self._act(rms_unit(x, c.rms_eps) * self.final_norm)
