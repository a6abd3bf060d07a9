"""Plain-PyTorch layer math: the fp32 oracle for the sm_100a kernels, the CPU path and
the cuBLAS baseline.  Also the batch descriptor shared by every forward mode.

One descriptor covers prefill, single-token decode, the two-token draft head and the
(gamma+1)-token verify pass: each sequence row has ``prefix_len`` tokens already in the
paged cache and ``extend_len`` new tokens, attended causally (the reference expresses
the same thing as EXTEND / TARGET_VERIFY forward modes, smcsd/core/info.py:206-365).
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import List, Optional

import torch
import torch.nn.functional as F


@dataclass
class ExtendBatch:
    input_ids: torch.Tensor        # [T]
    positions: torch.Tensor        # [T]
    cache_locs: torch.Tensor       # [T] page id each new token's K/V is written to
    rows: torch.Tensor             # [bs] block-table row of each sequence
    prefix_lens: torch.Tensor      # [bs] tokens already cached per row
    extend_len: int = 1            # uniform new tokens per row (0 => use extend_lens)
    extend_lens: Optional[List[int]] = None   # varlen (prefill) new tokens per row
    prefix_lens_host: Optional[List[int]] = None
    state_rows: Optional[torch.Tensor] = None  # [bs] recurrent-state rows (hybrids); defaults to rows
    save_steps: bool = False       # hybrids: keep per-position intermediate recurrent states
    logits_rows: Optional[torch.Tensor] = None  # token indices whose logits are wanted (None = all)

    @property
    def bs(self) -> int:
        return int(self.rows.shape[0])

    @property
    def uniform(self) -> bool:
        return self.extend_lens is None

    def lens(self) -> List[int]:
        return [self.extend_len] * self.bs if self.extend_lens is None else list(self.extend_lens)


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, plus_one: bool = False) -> torch.Tensor:
    xf = x.float()
    y = xf * torch.rsqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    wf = w.float() + 1.0 if plus_one else w.float()
    return (y * wf).to(x.dtype)


def rope_frequencies(head_dim: int, theta: float, scaling: Optional[dict] = None) -> torch.Tensor:
    """fp64 angle per position of every pair of a rotation over ``head_dim`` entries."""
    inv = 1.0 / (theta ** (torch.arange(0, head_dim, 2, dtype=torch.float64) / head_dim))
    if scaling:
        kind = scaling.get("rope_type", scaling.get("type", "default"))
        if kind == "llama3":
            factor = scaling["factor"]
            lo, hi = scaling["low_freq_factor"], scaling["high_freq_factor"]
            old = scaling["original_max_position_embeddings"]
            wavelen = 2 * math.pi / inv
            smooth = ((old / wavelen) - lo) / (hi - lo)
            scaled = torch.where(wavelen > old / lo, inv / factor, inv)
            mid = (wavelen <= old / lo) & (wavelen >= old / hi)
            inv = torch.where(mid, (1 - smooth) * inv / factor + smooth * inv, scaled)
        elif kind == "linear":
            inv = inv / scaling["factor"]
    return inv


def rope_inv_freq(head_dim: int, theta: float, scaling: Optional[dict]) -> torch.Tensor:
    return rope_frequencies(head_dim, theta, scaling).float()


def rope_table(rotary_dim: int, theta: float, scaling: Optional[dict], max_pos: int, device) -> torch.Tensor:
    """[max_pos, rotary_dim] fp32: cos in the first half of each row, sin in the second."""
    inv = rope_inv_freq(rotary_dim, theta, scaling).to(device)
    ang = torch.arange(max_pos, device=device, dtype=torch.float32).unsqueeze(1) * inv.unsqueeze(0)
    return torch.cat([ang.cos(), ang.sin()], dim=-1).contiguous()


def apply_rope(x: torch.Tensor, positions: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """x [T, H, D]; rotates the first ``table.shape[1]`` dims (HF half-split convention)."""
    rd = table.shape[1]
    half = rd // 2
    cs = table[positions.long()]
    cos, sin = cs[:, :half].unsqueeze(1), cs[:, half:].unsqueeze(1)
    xf = x.float()
    x1, x2 = xf[..., :half], xf[..., half:rd]
    out = torch.cat([x1 * cos - x2 * sin, x2 * cos + x1 * sin, xf[..., rd:]], dim=-1)
    return out.to(x.dtype)


def kv_rows_to_float(rows: torch.Tensor, n_kv_heads: int, head_dim: int) -> torch.Tensor:
    from ..memory.pools import kv_rows_to_float as f       # e4m3 page rows carry their scales (memory/pools.py)
    return f(rows, n_kv_heads, head_dim)


def paged_attention_reference(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor,
                              block_table: torch.Tensor, batch: ExtendBatch, n_kv_heads: int,
                              scale: Optional[float] = None) -> torch.Tensor:
    """Causal attention of the new tokens over [cached prefix + new tokens], all read through
    the block table (the new tokens' K/V must already be written).  q [T, Hq, D] -> [T, Hq, D]."""
    T, Hq, D = q.shape
    G = Hq // n_kv_heads
    scale = scale if scale is not None else D ** -0.5
    out = torch.empty_like(q)
    lens = batch.lens()
    pref = batch.prefix_lens_host if batch.prefix_lens_host is not None else batch.prefix_lens.tolist()
    t0 = 0
    for b, (p, e) in enumerate(zip(pref, lens)):
        if e == 0:
            continue
        L = p + e
        pages = block_table[batch.rows[b].long(), :L].long()
        k = kv_rows_to_float(k_pool[pages], n_kv_heads, D)
        v = kv_rows_to_float(v_pool[pages], n_kv_heads, D)
        qb = q[t0:t0 + e].float().view(e, n_kv_heads, G, D)
        s = torch.einsum("ehgd,lhd->hgel", qb, k) * scale
        causal = torch.arange(L, device=q.device).unsqueeze(0) <= (p + torch.arange(e, device=q.device)).unsqueeze(1)
        s = s.masked_fill(~causal.view(1, 1, e, L), float("-inf"))
        o = torch.einsum("hgel,lhd->ehgd", torch.softmax(s, dim=-1), v)
        out[t0:t0 + e] = o.reshape(e, Hq, D).to(q.dtype)
        t0 += e
    return out


def swiglu(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    return F.silu(gate.float()).mul(up.float()).to(gate.dtype)


# ----------------------------------------------------------------------------- mechanisms of layered architectures
def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """fp32 ``x`` divided by its root mean square over the last dimension."""
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def short_conv(h: torch.Tensor, w: torch.Tensor, batch: ExtendBatch, history: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
    """Causal depthwise convolution of the new tokens of every sequence.  h [T, C] fp32, w [C, taps]; ``history``
    [rows, C, taps - 1] holds the inputs before the first new token (oldest first) and is advanced in place."""
    taps = w.shape[1]
    out = torch.empty_like(h)
    t0 = 0
    for b, e in enumerate(batch.lens()):
        if e == 0:
            continue
        r = rows[b]
        seq = torch.cat([history[r].to(h.dtype), h[t0:t0 + e].t()], dim=1)          # [C, taps - 1 + e]
        out[t0:t0 + e] = (seq.unfold(1, taps, 1) * w.to(h.dtype).unsqueeze(1)).sum(-1).t()
        if taps > 1:
            history[r] = seq[:, -(taps - 1):].to(history.dtype)
        t0 += e
    return out


def latent_attention_reference(q: torch.Tensor, pool: torch.Tensor, block_table: torch.Tensor, batch: ExtendBatch,
                               scale: float, window: int = 0, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention in latent space: q [T, H, R] (queries already multiplied by the key expansion), cached latents
    ``pool`` [pages, >= R] read through the block table as keys and as values; with a ``window`` a token sees itself and the
    window - 1 tokens before it, ``sink`` [H] are logits in the softmax sum without a value.  Returns fp32 [T, H, R]."""
    T, H, R = q.shape
    out = torch.empty(T, H, R, dtype=torch.float32, device=q.device)
    pref = batch.prefix_lens_host if batch.prefix_lens_host is not None else batch.prefix_lens.tolist()
    t0 = 0
    for b, (p, e) in enumerate(zip(pref, batch.lens())):
        if e == 0:
            continue
        L = p + e
        c = pool[block_table[batch.rows[b].long(), :L].long()][:, :R].float()
        s = torch.einsum("ehr,lr->hel", q[t0:t0 + e].float(), c) * scale
        i, j = torch.arange(p, L, device=q.device).unsqueeze(1), torch.arange(L, device=q.device).unsqueeze(0)
        hidden = (j > i) | (i - j >= window) if window else j > i
        s = s.masked_fill(hidden, float("-inf"))
        if sink is not None:
            s = torch.cat([s, sink.view(H, 1, 1).expand(H, e, 1)], dim=-1)
        out[t0:t0 + e] = torch.einsum("hel,lr->ehr", torch.softmax(s, dim=-1)[..., :L], c)
        t0 += e
    return out


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """coef[0] N(z) + coef[1] N(z^2) + coef[2] N(z^3) + coef[3], N dividing a row by its root mean square (fp32)."""
    z = z.float()
    return coef[0] * rms_unit(z, eps) + coef[1] * rms_unit(z * z, eps) + coef[2] * rms_unit(z * z * z, eps) + coef[3]


GLU_SIGMOID_SLOPE = 1.702


def clamped_glu(gate: torch.Tensor, up: torch.Tensor, limit: float) -> torch.Tensor:
    g = gate.float().clamp(max=limit)
    u = up.float().clamp(-limit, limit)
    return g * torch.sigmoid(GLU_SIGMOID_SLOPE * g) * (u + 1.0)


def route_grouped(z: torch.Tensor, top: int, groups: int, keep: int):
    """Router logits [T, E] -> (expert ids [T, top], weights [T, top]): softmax over all experts, the ``top`` best among
    the experts of the ``keep`` groups with the largest single score, weights renormalised to one."""
    s = torch.softmax(z.float(), dim=-1)
    T, E = s.shape
    if keep < groups:
        g = s.view(T, groups, E // groups).amax(dim=-1)
        drop = torch.ones(T, groups, dtype=torch.bool, device=z.device)
        drop.scatter_(1, g.topk(keep, dim=-1).indices, False)
        cand = s.masked_fill(drop.repeat_interleave(E // groups, dim=1), -1.0)
    else:
        cand = s
    idx = cand.topk(top, dim=-1).indices
    w = s.gather(1, idx)
    return idx, w / (w.sum(-1, keepdim=True) + 1e-20)


def hyper_read(x: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    """Sublayer input of the hyper-connected streams x [T, S, d]: sum_s w_in[s] x_s."""
    return torch.einsum("tsd,s->td", x, w_in)


def hyper_write(x: torch.Tensor, y: torch.Tensor, w_mix: torch.Tensor, w_out: torch.Tensor) -> torch.Tensor:
    """New streams x_t' = sum_s w_mix[s, t] x_s + w_out[t] y."""
    return torch.einsum("tsd,su->tud", x, w_mix) + w_out.view(1, -1, 1) * y.unsqueeze(1)


def route_top(z: torch.Tensor, top: int):
    """Router logits [T, E] -> (expert ids [T, top], weights [T, top]): the largest logits, softmax over the chosen ones."""
    best = z.float().topk(top, dim=-1)
    return best.indices, torch.softmax(best.values, dim=-1)


# ---- positions, token shift and memory matrices
def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """fp32 x [T, ..., n]: the first ``dims`` entries rotated by position, entries 2i and 2i + 1 paired."""
    return turn_pairs(x, positions, rope_frequencies(dims, base))


def turn_pairs(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, back: bool = False) -> torch.Tensor:
    """fp32 x [T, ..., n]: entries 2i and 2i + 1 turn by position * freq[i] (fp64), or back by as much; entries behind the pairs
    pass."""
    dims = 2 * freq.numel()
    ang = positions.double().unsqueeze(1) * freq.to(x.device) * (-1.0 if back else 1.0)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    c, s = ang.cos().float().view(shape), ang.sin().float().view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    return torch.cat([torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2), x[..., dims:]], dim=-1)


def sinusoidal_positions(positions: torch.Tensor, d: int, base: float = 10000.0) -> torch.Tensor:
    """fp32 [T, d]: entry 2i is sin(p base^(-2i/d)), entry 2i + 1 the cosine of the same angle."""
    c = torch.arange(d, device=positions.device)
    freq = base ** (-(c - c % 2).double() / d)
    ang = positions.double().unsqueeze(1) * freq.unsqueeze(0)
    return torch.where(c % 2 == 0, ang.sin(), ang.cos()).float()


def token_shift(h: torch.Tensor, mu: torch.Tensor, batch: ExtendBatch, history: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
    """h [T, d] fp32, mu [n, d] -> [T, n, d]: h + (h' - h) mu with h' the row of the token before.  ``history`` [rows, >= d, 1]
    holds the row before the first new token and is advanced in place."""
    d, t0 = h.shape[1], 0
    prev = torch.empty_like(h)
    for b, e in enumerate(batch.lens()):
        if e == 0:
            continue
        r = rows[b]
        prev[t0] = history[r, :d, 0].to(h.dtype)
        prev[t0 + 1:t0 + e] = h[t0:t0 + e - 1]
        history[r, :d, 0] = h[t0 + e - 1].to(history.dtype)
        t0 += e
    return h.unsqueeze(1) + (prev - h).unsqueeze(1) * mu


DELTA_UNIT_EPS = 1e-6


def delta_memory(state: torch.Tensor, r, w, k, v, a) -> torch.Tensor:
    """Generalized delta rule of one sequence, token by token: with u = k / |k| and M the matrix before the token,
    M <- diag(w) M - (a u) (u^T M) + k v^T, read out with r.  r, w, k, a [T, H, dk], v [T, H, dv]; ``state`` [H, dv, dk] fp32
    holds M transposed and is advanced in place.  Returns [T, H, dv]."""
    u = k * torch.rsqrt((k * k).sum(-1, keepdim=True) + DELTA_UNIT_EPS)
    M, out = state.clone(), torch.empty_like(v)
    for t in range(r.shape[0]):
        gone = (M * u[t].unsqueeze(1)).sum(-1, keepdim=True)                  # [H, dv, 1]
        M = M * w[t].unsqueeze(1) - gone * (a[t] * u[t]).unsqueeze(1) + v[t].unsqueeze(-1) * k[t].unsqueeze(1)
        out[t] = (M * r[t].unsqueeze(1)).sum(-1)
    state.copy_(M)
    return out


def bonus_memory(state: torch.Tensor, r, w, k, v, bonus) -> torch.Tensor:
    """Decaying memory of one sequence: out = (M + diag(bonus) k v^T)^T r, then M <- diag(w) M + k v^T; layouts as in
    ``delta_memory``, bonus [H, dk]."""
    M, out = state.clone(), torch.empty_like(v)
    for t in range(r.shape[0]):
        kv = v[t].unsqueeze(-1) * k[t].unsqueeze(1)
        out[t] = ((M + kv * bonus.unsqueeze(1)) * r[t].unsqueeze(1)).sum(-1)
        M = M * w[t].unsqueeze(1) + kv
    state.copy_(M)
    return out


def channel_delta_memory(state: torch.Tensor, q, k, v, g, beta) -> torch.Tensor:
    """Delta rule with a decay per channel, one sequence, token by token: M <- diag(g) M, u = beta (v - M^T k), M <- M + k u^T, read
    out with q.  q, k, g [T, H, dk], v [T, H, dv], beta [T, H]; ``state`` [H, dv, dk] fp32 holds M transposed and is advanced in
    place.  Returns [T, H, dv]."""
    M, out = state.clone(), torch.empty_like(v)
    for t in range(q.shape[0]):
        M = M * g[t].unsqueeze(1)
        u = beta[t].unsqueeze(1) * (v[t] - (M * k[t].unsqueeze(1)).sum(-1))
        M = M + u.unsqueeze(-1) * k[t].unsqueeze(1)
        out[t] = (M * q[t].unsqueeze(1)).sum(-1)
    state.copy_(M)
    return out


def forget_memory(state: torch.Tensor, q, v, f, write) -> torch.Tensor:
    """Forget-gated memory of one sequence: M <- diag(f) M + write v^T with write = 1 - f, read out with q afterwards.  q, f and
    write [T, H, dk], v [T, H, dv]; layouts as in ``channel_delta_memory``."""
    M, out = state.clone(), torch.empty_like(v)
    for t in range(q.shape[0]):
        M = M * f[t].unsqueeze(1) + v[t].unsqueeze(-1) * write[t].unsqueeze(1)
        out[t] = (M * q[t].unsqueeze(1)).sum(-1)
    state.copy_(M)
    return out


def pair_rows(ids: torch.Tensor, batch: ExtendBatch, history: torch.Tensor, rows: torch.Tensor, buckets: int, mul_prev: int,
              mul_cur: int) -> torch.Tensor:
    """Rows of an embedding of token pairs: (token before * mul_prev + token * mul_cur) mod buckets, and row ``buckets`` for a
    sequence's first token.  ``history`` [rows] holds the token before the first new one and is advanced in place."""
    ids = ids.long()
    out, t0 = torch.empty_like(ids), 0
    pref = batch.prefix_lens_host if batch.prefix_lens_host is not None else batch.prefix_lens.tolist()
    for b, (p, e) in enumerate(zip(pref, batch.lens())):
        if e == 0:
            continue
        mine = ids[t0:t0 + e]
        prev = torch.cat([history[rows[b]].long().view(1), mine[:-1]])
        out[t0:t0 + e] = (prev * mul_prev + mine * mul_cur) % buckets
        if p == 0:
            out[t0] = buckets
        history[rows[b]] = mine[-1].to(history.dtype)
        t0 += e
    return out


def soft_cap(z: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(z / cap)


NORMALISER_EPS = 1e-6


def gated_memory(state: torch.Tensor, top: torch.Tensor, q, k, v, i, f) -> torch.Tensor:
    """Matrix memory of one sequence with log input gates i and log forget gates f [T, H]: with the running maximum
    m <- max(f + m, i), M and the normaliser n decay by exp(f + m_old - m) and gain exp(i - m) times k v^T and k; the read-out
    M^T q is divided by max(|n q|, exp(-m)) + NORMALISER_EPS.  q, k [T, H, dk], v [T, H, dv]; ``state`` [H, dv + 1, dk] fp32 holds M transposed
    and n as its last row, ``top`` [H, 1, 1] the maximum; both are advanced in place.  Returns [T, H, dv]."""
    M, m, out = state.clone(), top[:, 0, 0].clone(), torch.empty_like(v)
    v1 = torch.cat([v, torch.ones_like(v[..., :1])], dim=-1)
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m_new), torch.exp(i[t] - m_new)
        m = m_new
        M = M * keep.view(-1, 1, 1) + (v1[t] * add.unsqueeze(1)).unsqueeze(-1) * k[t].unsqueeze(1)
        o = (M * q[t].unsqueeze(1)).sum(-1)
        out[t] = o[:, :-1] / (torch.maximum(o[:, -1].abs(), torch.exp(-m)) + NORMALISER_EPS).unsqueeze(1)
    state.copy_(M)
    top[:, 0, 0] = m
    return out


def chunk_attention_reference(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, block_table: torch.Tensor,
                              batch: ExtendBatch, kv_heads: int, scale: float, r1: Optional[torch.Tensor],
                              r2: Optional[torch.Tensor], chunk: int, softcap: float = 0.0, window: int = 0,
                              sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention inside chunks of ``chunk`` positions (0: no chunks) or inside a ``window`` with scores
    scale q.k - r1 ln(1 + r2 distance), or soft-capped ones, and a sink of score 0 or of the logits ``sink`` [H].  q [T, H, D];
    pools [pages, kv_heads * width]; returns fp32 [T, H, value width]."""
    T, H, D = q.shape
    rep, V = H // kv_heads, v_pool.shape[1] // kv_heads
    out = torch.empty(T, H, V, dtype=torch.float32, device=q.device)
    pref = batch.prefix_lens_host if batch.prefix_lens_host is not None else batch.prefix_lens.tolist()
    chunk, t0 = chunk or 1 << 30, 0
    for b, (p, e) in enumerate(zip(pref, batch.lens())):
        if e == 0:
            continue
        lo, L = max(0, p - window + 1) if window else p // chunk * chunk, p + e
        pages = block_table[batch.rows[b].long(), lo:L].long()
        kk = k_pool[pages].view(L - lo, kv_heads, -1)[:, :, :D].float().repeat_interleave(rep, dim=1)
        vv = v_pool[pages].view(L - lo, kv_heads, V).float().repeat_interleave(rep, dim=1)
        i = torch.arange(p, L, device=q.device).unsqueeze(1)
        j = torch.arange(lo, L, device=q.device).unsqueeze(0)
        dist = (i - j).clamp(min=0).float()
        s = torch.einsum("ehd,lhd->hel", q[t0:t0 + e].float(), kk) * scale
        if softcap:
            s = soft_cap(s, softcap)
        if r1 is not None:
            s = s - r1.view(H, 1, 1) * torch.log1p(r2.view(H, 1, 1) * dist)
        s = s.masked_fill((j > i) | ((i - j >= window) if window else (i // chunk != j // chunk)), float("-inf"))
        extra = torch.zeros(H, 1, 1, device=q.device) if sink is None else sink.view(H, 1, 1)
        top = torch.maximum(s.amax(-1, keepdim=True), extra)
        ex = torch.exp(s - top)
        out[t0:t0 + e] = torch.einsum("hel,lhv->ehv", ex / (torch.exp(extra - top) + ex.sum(-1, keepdim=True)), vv)
        t0 += e
    return out
