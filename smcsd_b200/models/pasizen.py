"""Pasizen: a decoder whose residual is several hyper-connected streams, with a short causal convolution in front of every
mixer, latent attention without positions (a learned position vector enters at the embedding), PolyNorm or
mixture-of-experts feed-forwards, and a range of layers that may run several times in a row.

Weight layout (shared with the kernel chain; every reduction dimension is padded with zeros to a multiple of eight so that
the tensor-core GEMMs can fetch 16-byte aligned rows):
  wqc    [H * dim' + kv_rank, d']   query heads (dim' = dim rounded up to 8, zero rows in between), then the latent
  wuk_t  [H * R', dim']             per head the transposed key expansion: queries move into latent space (R' = kv_rank
                                    rounded up to 64, the row width of the latent cache)
  wuv    [H * vdim, R']             value expansion, applied to the attended latents
  wo     [d, (H * vdim)']
  wup    [ff', d'], wdown [d, ff']  dense feed-forward
  e_gu   [E, 2 * ff', d']           expert gate / up rows interleaved in blocks of 64 channels (ff' rounded up to 64)
  e_down [E, d, ff']                experts; s_gu / s_down likewise for the shared expert
Norm weights, convolution taps, hyper-connection coefficients and PolyNorm coefficients are kept in fp32.

The state of a sequence is its latent rows in the paged cache (one set per layer run) and, per layer run, the last
``taps - 1`` convolution inputs in the state pool.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Iterator, List, Optional

import torch

from ..memory.pools import KVSpec, StateSpec
from .config import LayerSpec
from .layered import GU_BLOCK, LayeredModel, pad_to, round_up
from .layers import (ExtendBatch, clamped_glu, hyper_read, hyper_write, latent_attention_reference, poly_norm, rms_unit,
                     route_grouped, short_conv)
from .llama import split_gate_up


@dataclass
class HyperWeights:
    w_in: torch.Tensor                     # [S] fp32
    w_out: torch.Tensor                    # [S] fp32
    w_mix: torch.Tensor                    # [S, S] fp32, indexed [from, to]


@dataclass
class PasizenLayerWeights:
    spec: LayerSpec
    norm1: torch.Tensor
    conv_w: torch.Tensor
    hc1: HyperWeights
    wqc: torch.Tensor
    c_norm: torch.Tensor
    wuk_t: torch.Tensor
    wuv: torch.Tensor
    wo: torch.Tensor
    norm2: Optional[torch.Tensor] = None
    hc2: Optional[HyperWeights] = None
    wup: Optional[torch.Tensor] = None
    wdown: Optional[torch.Tensor] = None
    poly: Optional[torch.Tensor] = None
    router: Optional[torch.Tensor] = None
    e_gu: Optional[torch.Tensor] = None
    e_down: Optional[torch.Tensor] = None
    s_gu: Optional[torch.Tensor] = None
    s_down: Optional[torch.Tensor] = None

    def tensors(self) -> Iterator[torch.Tensor]:
        for v in vars(self).values():
            if isinstance(v, torch.Tensor):
                yield v
            elif isinstance(v, HyperWeights):
                yield from vars(v).values()


class PasizenModel(LayeredModel):
    family = "Pasizen"

    # ---- cache and state ---------------------------------------------------------------
    def kv_spec(self, dtype, fp8: bool = False) -> KVSpec:
        if fp8:
            raise ValueError("the latent cache has no fp8 layout")
        widths = [round_up(self.cfg.layers[li].mixer.kv_rank, 64) for li in self.runs]
        return KVSpec(len(widths), 1, max(widths), dtype, latent_widths=widths)

    def state_spec(self) -> StateSpec:
        return StateSpec(len(self.runs), self.cfg.hidden_size, self.cfg.conv_taps, 0, 0, 0, conv_dtype=torch.float32)

    # ---- parameters --------------------------------------------------------------------
    def _assemble(self, get) -> "PasizenModel":
        """Fill the packed layout from ``get(name, *shape)``, which returns a tensor by its checkpoint name."""
        c, dt, dev = self.cfg, self.dtype, self.device
        d, d8, S = c.hidden_size, round_up(c.hidden_size, 8), c.streams

        def mat(name, *shape):
            return get(name, *shape).to(device=dev, dtype=dt, copy=True)

        def vec(name, *shape):
            return get(name, *shape).to(device=dev, dtype=torch.float32, copy=True).contiguous()

        def hyper(p):
            return HyperWeights(vec(p + "in", S), vec(p + "out", S), vec(p + "mix", S, S))

        self.embed, self.pos = mat("embed", c.vocab_size, d), mat("pos", c.max_position, d)
        self.final_norm = vec("final.norm", d)
        self.lm_head = pad_to(mat("head", c.vocab_size, d), c.vocab_size, d8)
        for li, spec in enumerate(c.layers):
            p, m = f"l{li}.", spec.mixer
            H, D, V, R = m.heads, m.dim, m.vdim, m.kv_rank
            D8, Rp = round_up(D, 8), round_up(R, 64)
            wq = pad_to(mat(p + "mix.q", H * D, d).view(H, D, d), H, D8, d8).view(H * D8, d8)
            wqc = torch.cat([wq, pad_to(mat(p + "mix.dkv", R, d), R, d8)], dim=0).contiguous()
            uk = mat(p + "mix.uk", H * D, R).view(H, D, R).transpose(1, 2)
            L = PasizenLayerWeights(
                spec, norm1=vec(p + "norm1", d), conv_w=vec(p + "canon1", d, c.conv_taps), hc1=hyper(p + "hc1."), wqc=wqc,
                c_norm=vec(p + "mix.dkv.norm", R), wuk_t=pad_to(uk, H, Rp, D8).view(H * Rp, D8),
                wuv=pad_to(mat(p + "mix.uv", H * V, R), H * V, Rp), wo=pad_to(mat(p + "mix.o", d, H * V), d, round_up(H * V, 8)))
            f = spec.mlp
            if f is not None:
                L.norm2, L.hc2 = vec(p + "norm2", d), hyper(p + "hc2.")
                if f.kind == "dense":
                    f8 = round_up(f.ff, 8)
                    L.wup, L.wdown = pad_to(mat(p + "mlp.up", f.ff, d), f8, d8), pad_to(mat(p + "mlp.down", d, f.ff), d, f8)
                    L.poly = vec(p + "mlp.act", 4)
                else:
                    L.router = pad_to(mat(p + "mlp.router", f.router.experts, d), f.router.experts, d8)
                    L.e_gu, L.e_down = self._pack_experts(mat, p + "mlp.", f.router.experts, f.expert.ff, d)
                    if f.shared is not None:
                        L.s_gu, L.s_down = self._pack_glu(mat, p + "mlp.shared.", f.shared.ff, d)
            self.layers.append(L)
        return self

    def init_random(self, seed: int = 0, std: float = 0.02) -> "PasizenModel":
        g = torch.Generator(device=self.device)
        g.manual_seed(seed)
        S = self.cfg.streams

        def get(name, *shape):
            r = torch.randn(*shape, generator=g, device=self.device, dtype=torch.float32)
            leaf = name.rsplit(".", 1)[-1]
            if "norm" in leaf or leaf.startswith("norm"):
                return 1.0 + 0.1 * r
            if leaf == "in":
                return 1.0 / S + 0.1 * r
            if leaf == "out":
                return 1.0 + 0.1 * r
            if leaf == "mix":
                return torch.eye(S, device=self.device) + 0.1 * r
            if leaf == "canon1":
                return 0.3 * r
            if leaf == "act":
                return torch.tensor([0.6, 0.3, 0.2, 0.05], device=self.device) + 0.05 * r
            if leaf in ("uk", "uv"):
                return r * shape[1] ** -0.5
            return r * std
        return self._assemble(get)

    # ---- plain-PyTorch forward ----------------------------------------------------------
    def _mixer(self, L: PasizenLayerWeights, x: torch.Tensor, batch: ExtendBatch, kv, block_table, run: int) -> torch.Tensor:
        m, eps = L.spec.mixer, self.cfg.rms_eps
        T, H, D8, R, Rp = x.shape[0], m.heads, round_up(m.dim, 8), m.kv_rank, round_up(m.kv_rank, 64)
        y = x @ L.wqc.t()
        c = (rms_unit(y[:, H * D8:].float(), eps) * L.c_norm).to(x.dtype)
        kv.write_latent(run, batch.cache_locs, c)
        q = torch.einsum("thd,hrd->thr", y[:, :H * D8].reshape(T, H, D8), L.wuk_t.view(H, Rp, D8)[:, :R])
        a = latent_attention_reference(q, kv.k[run], block_table, batch, m.scale).to(x.dtype)
        o = torch.einsum("thr,hvr->thv", a, L.wuv.view(H, m.vdim, Rp)[:, :, :R]).reshape(T, H * m.vdim)
        return (o @ L.wo[:, :H * m.vdim].t()).float()

    @staticmethod
    def _glu(x, gu, down, limit):
        gate, up = split_gate_up(x @ gu.t(), GU_BLOCK)
        return (clamped_glu(gate, up, limit).to(x.dtype) @ down.t()).float()

    def _feed_forward(self, L: PasizenLayerWeights, h: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
        """h: fp32 normalised input (router), x: the same rows padded in the activation dtype."""
        f = L.spec.mlp
        if f.kind == "dense":
            z = (x @ L.wup.t()).float()[:, :f.ff]
            a = poly_norm(z, L.poly, self.cfg.rms_eps).to(x.dtype)
            return (a @ L.wdown[:, :f.ff].t()).float()
        r = f.router
        idx, w = route_grouped(h @ L.router[:, :h.shape[1]].float().t(), r.top, r.groups, r.keep)
        out = self._mix_experts(x, idx, w, lambda e, rows: self._glu(rows, L.e_gu[e], L.e_down[e], f.expert.limit))
        if f.shared is not None:
            out = out + self._glu(x, L.s_gu, L.s_down, f.shared.limit)
        return out

    def forward_torch(self, batch: ExtendBatch, kv, block_table: torch.Tensor, state=None, per_run=None) -> torch.Tensor:
        """Post-norm hidden rows of the new tokens; ``per_run`` (a list) collects the summed streams after every layer run."""
        if state is None:
            raise ValueError("Pasizen models need a recurrent-state pool")
        c = self.cfg
        rows = (batch.state_rows if batch.state_rows is not None else batch.rows).long()
        e = self.embed[batch.input_ids.long()].float() + self.pos[batch.positions.long()].float()
        x = e.unsqueeze(1).repeat(1, c.streams, 1)
        for run, li in enumerate(self.runs):
            L = self.layers[li]
            h = rms_unit(hyper_read(x, L.hc1.w_in), c.rms_eps) * L.norm1
            h = h + short_conv(h, L.conv_w, batch, state.conv[run], rows)
            x = hyper_write(x, self._mixer(L, self._act(h), batch, kv, block_table, run), L.hc1.w_mix, L.hc1.w_out)
            if L.spec.mlp is not None:
                h = rms_unit(hyper_read(x, L.hc2.w_in), c.rms_eps) * L.norm2
                x = hyper_write(x, self._feed_forward(L, h, self._act(h)), L.hc2.w_mix, L.hc2.w_out)
            if per_run is not None:
                per_run.append(x.sum(1))
        return self._act(rms_unit(x.sum(1), c.rms_eps) * self.final_norm)
