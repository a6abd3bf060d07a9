"""The kernels of layered architectures one by one against plain fp32 PyTorch (needs a B200)."""
import pytest
import torch

import pasizen_oracle as O

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _k():
    from smcsd_b200.ops import native as K
    K.layered_lib()
    return K


def _status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def _rnd(*shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed + sum(shape))
    return (torch.randn(*shape, generator=g) * scale).to(DEV)


def _ints(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def _close(a, b, tol):
    a, b = a.double(), b.double()
    err = (a - b).abs().max().item()
    assert err <= tol * max(1.0, b.abs().max().item()), err


@pytest.mark.parametrize("M", [1, 63, 64, 150, 300])
@pytest.mark.parametrize("N,Kd", [(40, 24), (400, 328), (130, 136)])
def test_gemm_f32(M, N, Kd):
    K = _k()
    W, X = _rnd(N, Kd), _rnd(M, Kd, seed=1)
    out = torch.empty(M, N, device=DEV)
    K.gemm_f32(W, X, out, N=N, M=M)
    _close(out, X.double() @ W.double().t(), 2e-6)


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("H,N,Kd,M", [(3, 64, 40, 5), (7, 64, 72, 150), (5, 24, 72, 33), (4, 256, 128, 300)])
def test_per_head_products(f32, H, N, Kd, M):
    K = _k()
    dt = torch.float32 if f32 else torch.bfloat16
    W, X = _rnd(H * N, Kd).to(dt), _rnd(M, H * Kd, seed=1).to(dt)
    out = torch.zeros(M, H * N, device=DEV, dtype=dt)
    link = K.GroupLink(mode=K.GROUP_BATCHED, groups=H, w_rows=N, x_cols=Kd, out_cols=N)
    st = _status()
    if f32:
        K.gemm_f32(W, X, out, N=N, M=M, link=link)
    else:
        K.gemm_grouped(W, X, out, N=N, M=M, splits=1, epi=K.EPI_BF16, link=link, status=st)
    ref = torch.einsum("mhk,hnk->mhn", X.view(M, H, Kd).double(), W.view(H, N, Kd).double()).reshape(M, H * N)
    _close(out, ref, 2e-6 if f32 else 8e-3)
    assert int(st) == 0


def _dispatch(K, idx, E, rows):
    T, top = idx.shape
    n = T * top
    slot, src = _ints([-1] * n), _ints([-1] * n)
    max_tiles = n // rows + min(E, n)
    tiles = torch.full((max_tiles, 4), -1, dtype=torch.int32, device=DEV)
    st = _status()
    K.dispatch(idx.reshape(-1).contiguous(), slot, src, tiles, n=n, top=top, experts=E, rows=rows, max_tiles=max_tiles, status=st)
    assert int(st) == 0
    return slot, src, tiles, max_tiles


@pytest.mark.parametrize("T,top,E,rows", [(1, 2, 8, 16), (7, 3, 5, 16), (150, 3, 10, 64), (700, 2, 33, 32), (90, 1, 3, 128)])
def test_dispatch_sorts_pairs_by_expert(T, top, E, rows):
    K = _k()
    g = torch.Generator().manual_seed(T)
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32).to(DEV)
    idx[: T // 2, 0] = idx[0, 0] if top == 1 else idx[: T // 2, 0]       # a crowded expert spans several tiles
    slot, src, tiles, _ = _dispatch(K, idx, E, rows)
    n = T * top
    assert sorted(slot.tolist()) == list(range(n))
    assert torch.equal(src[slot.long()].cpu(), torch.arange(n, dtype=torch.int32) // top)
    expert_of_slot = torch.empty(n, dtype=torch.int32)
    expert_of_slot[slot.cpu().long()] = idx.reshape(-1).cpu()
    seen = torch.zeros(n, dtype=torch.int32)
    for e, a, b, _ in tiles.tolist():
        assert 0 <= b - a <= rows
        seen[a:b] += 1
        assert (expert_of_slot[a:b] == e).all()
    assert (seen == 1).all()


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("T,top,E,d,ff", [(1, 2, 8, 136, 64), (20, 3, 10, 328, 128), (150, 3, 10, 328, 128), (300, 2, 4, 136, 192)])
def test_expert_products_and_weighted_sum(f32, T, top, E, d, ff):
    """dispatch, gather, tiled gate / up with the gated unit, tiled down, weighted rows added by the stream step."""
    from smcsd_b200.models.layers import GLU_SIGMOID_SLOPE
    from smcsd_b200.models.llama import interleave_gate_up
    K = _k()
    dt = torch.float32 if f32 else torch.bfloat16
    g = torch.Generator().manual_seed(1)
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32).to(DEV)
    wgt = torch.rand(T, top, generator=g).to(DEV)
    gate, up = _rnd(E, ff, d, scale=d ** -0.5).to(dt), _rnd(E, ff, d, seed=5, scale=d ** -0.5).to(dt)
    down = _rnd(E, d, ff, seed=6, scale=ff ** -0.5).to(dt)
    gu = torch.stack([interleave_gate_up(gate[e], up[e], 64) for e in range(E)])
    x = _rnd(T, d, seed=7).to(dt)
    rows = 64 if f32 else 16
    slot, src, tiles, max_tiles = _dispatch(K, idx, E, rows)
    n, st = T * top, _status()
    xe, ea, ye = (torch.zeros(n, w, device=DEV, dtype=t) for w, t in ((d, dt), (ff, dt), (d, torch.float32)))
    K.gather_rows(x, src, xe, n=n, n_src=T, status=st)
    assert torch.equal(xe, x[src.long()])
    link = K.GroupLink(mode=K.GROUP_TILED, groups=E, w_rows=2 * ff, tiles=K.ptr(tiles), max_tiles=max_tiles, bn=rows,
                       act=K.ACT_CLAMPED, limit=0.8, slope=GLU_SIGMOID_SLOPE)
    link2 = K.GroupLink(mode=K.GROUP_TILED, groups=E, w_rows=d, tiles=K.ptr(tiles), max_tiles=max_tiles, bn=rows)
    if f32:
        g32 = torch.zeros(n, 2 * ff, device=DEV)
        K.gemm_f32(gu, xe, g32, N=2 * ff, M=n, link=link)
        K.gated_unit_f32(g32, ea, ff=ff, blk=64, limit=0.8, slope=GLU_SIGMOID_SLOPE, shift=1.0, M=n)
        K.gemm_f32(down, ea, ye, N=d, M=n, link=link2)
    else:
        K.gemm_grouped(gu, xe, ea, N=2 * ff, M=n, splits=1, epi=K.EPI_SWIGLU_BF16, link=link, status=st)
        K.gemm_grouped(down, ea, ye, N=d, M=n, splits=2, epi=K.EPI_STORE_F32, link=link2, status=st)
    per = torch.zeros(T, top, d, dtype=torch.float64, device=DEV)
    xd = x.double()
    for e in range(E):
        t, j = (idx == e).nonzero(as_tuple=True)
        act = O.clamped_glu(xd[t] @ gate[e].double().t(), xd[t] @ up[e].double().t(), 0.8)
        per[t, j] = act @ down[e].double().t()
    _close(ye[slot.long()].view(T, top, d), per, 1e-5 if f32 else 1e-2)
    # the stream step adds sum_k w_k * row_k
    S = 2
    xs, y = _rnd(T, S, d, seed=9), _rnd(T, d, seed=10)
    mix, wout, win, nw = _rnd(S, S), _rnd(S), _rnd(S, seed=2), _rnd(d)
    ref = torch.einsum("tsd,su->tud", xs.double(), mix.double()) + \
        wout.double().view(1, S, 1) * (y.double() + (wgt.double().unsqueeze(-1) * per).sum(1)).unsqueeze(1)
    n_out = torch.zeros(T, d, device=DEV)
    a = K.HyperArgs(x=K.ptr(xs), S=S, d=d, y=K.ptr(y), ldy=d, ye=K.ptr(ye), ldye=d, top=top, route_slot=K.ptr(slot),
                    route_w=K.ptr(wgt), w_mix=K.ptr(mix), w_out=K.ptr(wout), w_in=K.ptr(win), norm_w=K.ptr(nw), eps=1e-5,
                    n_out=K.ptr(n_out), ldxa=d, status=K.ptr(st))
    K.hyper_step(a, T, f32)
    _close(xs, ref, 1e-5 if f32 else 1e-2)
    u = torch.einsum("tsd,s->td", xs.double(), win.double())
    _close(n_out, O.rms_normalise(u, 1e-5) * nw.double(), 1e-5)
    assert int(st) == 0


@pytest.mark.parametrize("T", [1, 9, 301])
@pytest.mark.parametrize("d,E,top,groups,keep", [(328, 10, 3, 5, 3), (136, 8, 2, 4, 2), (72, 64, 8, 8, 8), (64, 6, 1, 1, 1), (250, 40, 6, 5, 2)])
def test_router(T, d, E, top, groups, keep):
    K = _k()
    h, w = _rnd(T, d, seed=3), _rnd(E, d, seed=4, scale=d ** -0.5)
    idx, wgt = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV)
    K.route(h, w, idx, wgt, d=d, top=top, groups=groups, keep=keep, T=T, f32=True)
    ri, rw = O.route(h.double().cpu() @ w.double().cpu().t(), {"top": top, "groups": {"count": groups, "keep": keep}})
    same = (idx.cpu().long() == ri).all(-1)
    assert same.float().mean() > 0.99                          # a tie of two fp32 scores may fall either way
    _close(wgt.cpu()[same], rw[same], 1e-5)


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("ff", [400, 200, 77])
def test_poly_norm(f32, ff):
    K = _k()
    z, coef = _rnd(13, ff, scale=1.7), _rnd(4)
    out = torch.zeros(13, ff, device=DEV, dtype=torch.float32 if f32 else torch.bfloat16)
    K.poly_norm(z, coef, out, ff=ff, M=13, eps=1e-3, f32=f32)
    _close(out, O.poly_norm(z.double(), coef.double(), 1e-3), 1e-5 if f32 else 1e-2)


def _work(K, seqs, block=64):
    """Ragged work list of (row, prefix, length) sequences."""
    rows, pref, lens = zip(*seqs)
    off = [sum(lens[:i]) for i in range(len(lens))]
    cells = [(s, b) for s, n in enumerate(lens) for b in range(0, n, block)]
    t = [_ints(list(v)) for v in (rows, pref, off, lens, [c[0] for c in cells], [c[1] for c in cells])]
    return K.Ragged(seq_row=K.ptr(t[0]), seq_prefix=K.ptr(t[1]), seq_off=K.ptr(t[2]), seq_len=K.ptr(t[3]), blk_seq=K.ptr(t[4]),
                    blk_start=K.ptr(t[5]), n_seq=len(seqs), n_blk=len(cells), E=0, B=block), t


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
@pytest.mark.parametrize("d", [72, 328, 250])
def test_short_conv_over_portions(taps, d):
    """Any cut of a sequence into portions (shorter than the window, across blocks) gives the whole convolution."""
    K = _k()
    w, h = _rnd(d, taps), _rnd(75, d, seed=2)
    ref = h.double() + O.causal_short_conv(h.double().cpu(), w.double().cpu()).to(DEV)
    for cuts in ([75], [1, 1, 2, 33, 38], [40, 2, 1, 32], [1] * 75):
        hist = torch.zeros(3, d, taps - 1, device=DEV)
        other = _rnd(5, d, seed=8)
        got, at, st = [], 0, _status()
        for n in cuts:
            inp = torch.cat([other, h[at:at + n]])
            xa = torch.zeros(inp.shape[0], d, device=DEV)
            work, keep = _work(K, [(2, 0, 5), (1, at, n)])
            K.short_conv(inp.contiguous(), xa, w, hist, work, status=st, f32=True)
            got.append(xa[5:])
            at += n
        _close(torch.cat(got), ref, 1e-5)
        assert int(st) == 0 and hist[0].abs().sum() == 0


@pytest.mark.parametrize("S,d,taps", [(1, 64, 4), (3, 328, 5), (5, 250, 2), (8, 136, 1), (11, 68, 4), (4, 2048, 3)])
def test_stream_step_with_folded_convolution(S, d, taps):
    """Embedding start, update, single-token convolution and the final sum."""
    K = _k()
    T, V, P, eps = 6, 50, 40, 1e-4
    emb, pos, nw = _rnd(V, d), _rnd(P, d, seed=1), _rnd(d, seed=2)
    mix, wout, win, cw = _rnd(S, S, seed=3), _rnd(S, seed=4), _rnd(S, seed=5), _rnd(d, taps, seed=6)
    ids, positions, rows = _ints([3, 49, 0, 7, 7, 20]), _ints([0, 39, 5, 5, 1, 2]), _ints([4, 0, 6, 1, 2, 5])
    x, y, st = torch.zeros(T, S, d, device=DEV), _rnd(T, d, seed=7), _status()
    hist = _rnd(7, d, max(taps - 1, 1), seed=8)[..., :taps - 1].contiguous()
    xa, n = torch.zeros(T, d, device=DEV), torch.zeros(T, d, device=DEV)
    common = dict(x=K.ptr(x), S=S, d=d, vocab=V, max_pos=P, norm_w=K.ptr(nw), eps=eps, ldy=d, ldye=d, ldxa=d, status=K.ptr(st))
    K.hyper_step(K.HyperArgs(**common, ids=K.ptr(ids), positions=K.ptr(positions), embed=K.ptr(emb), pos=K.ptr(pos), w_in=K.ptr(win),
                             n_out=K.ptr(n), xa=K.ptr(xa)), T, True)
    e = (emb[ids.long()] + pos[positions.long()]).double()
    _close(x, e.unsqueeze(1).expand(T, S, d), 1e-6)
    _close(n, O.rms_normalise(e * win.double().sum(), eps) * nw.double(), 1e-5)
    assert torch.equal(n, xa)
    h0 = hist.clone()
    K.hyper_step(K.HyperArgs(**common, y=K.ptr(y), w_mix=K.ptr(mix), w_out=K.ptr(wout), w_in=K.ptr(win), xa=K.ptr(xa),
                             conv_w=K.ptr(cw), hist=K.ptr(hist), rows=K.ptr(rows), taps=taps, n_rows=7), T, True)
    x2 = O.hyper_step([e] * S, win.double(), mix.double(), wout.double(), lambda u: y.double())
    _close(x, torch.stack(x2, 1), 1e-5)
    u = sum(win[s].double() * x2[s] for s in range(S))
    nn = O.rms_normalise(u, eps) * nw.double()
    seq = torch.cat([h0[rows.long()].double(), nn.unsqueeze(-1)], -1)
    _close(xa, nn + (seq * cw.double()).sum(-1), 1e-5)
    _close(hist[rows.long()], seq[..., 1:], 1e-5) if taps > 1 else None
    before = x.clone()
    K.hyper_step(K.HyperArgs(**common, y=K.ptr(y), w_mix=K.ptr(mix), w_out=K.ptr(wout), xa=K.ptr(xa)), T, True)
    x3 = O.hyper_step([before[:, s].double() for s in range(S)], win.double(), mix.double(), wout.double(), lambda u: y.double())
    _close(xa, O.rms_normalise(sum(x3), eps) * nw.double(), 1e-5)
    assert torch.equal(x, before) and int(st) == 0


def _latent_case(K, dt, H, R, seqs, seed=0, far=()):
    """Cached latents of sequences on scattered pages; ``far``: (sequence, token, key) whose score is made to stand out."""
    Rp = (R + 63) // 64 * 64
    T = sum(n for _, _, n in seqs)
    n_pages = sum(p + n for _, p, n in seqs) + 7
    g = torch.Generator().manual_seed(seed)
    perm = (torch.randperm(n_pages, generator=g) + 1).tolist()
    bt = torch.zeros(8, 1200, dtype=torch.int32)
    pool = torch.zeros(n_pages + 1, Rp)
    pool[:, :R] = torch.randn(n_pages + 1, R, generator=g)
    q = torch.zeros(T, H, Rp)
    q[..., :R] = torch.randn(T, H, R, generator=g)
    at = 0
    for row, p, n in seqs:
        bt[row, :p + n] = torch.tensor(perm[at:at + p + n])
        at += p + n
    off = 0
    for s, (row, p, n) in enumerate(seqs):
        for fs, tok, key in far:
            if fs == s:
                q[off + tok, :, :R] = pool[bt[row, key].item(), :R] * 3.0
        off += n
    return bt.to(DEV), pool.to(dt).to(DEV), q.view(T, H * Rp).to(dt).to(DEV), Rp


def _latent_ref(bt, pool, q, H, Rp, seqs, scale):
    out = torch.zeros(q.shape[0], H, Rp, dtype=torch.float64, device=DEV)
    off = 0
    for row, p, n in seqs:
        c = pool[bt[row, :p + n].long()].double()
        s = torch.einsum("thr,lr->htl", q[off:off + n].view(n, H, Rp).double(), c) * scale
        mask = torch.arange(p + n, device=DEV).unsqueeze(0) <= (p + torch.arange(n, device=DEV)).unsqueeze(1)
        out[off:off + n] = torch.einsum("htl,lr->thr", torch.softmax(s.masked_fill(~mask, float("-inf")), -1), c)
        off += n
    return out.view(q.shape[0], H * Rp)


SEQS = [[(1, 0, 1)], [(2, 0, 37)], [(0, 63, 1), (5, 64, 1), (3, 500, 1)], [(4, 130, 2), (1, 0, 70), (6, 1000, 17)]]


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("H,R", [(7, 64), (3, 48), (5, 200), (16, 256)])
@pytest.mark.parametrize("seqs", SEQS)
def test_latent_attention(f32, H, R, seqs):
    K = _k()
    dt = torch.float32 if f32 else torch.bfloat16
    last = seqs[-1]
    far = [(len(seqs) - 1, last[2] - 1, 0), (len(seqs) - 1, 0, last[1])]
    bt, pool, q, Rp = _latent_case(K, dt, H, R, seqs, far=far)
    out, st = torch.zeros_like(q), _status()
    work, keep = _work(K, seqs)
    a = K.LatentArgs(q=K.ptr(q), pool=K.ptr(pool), out=K.ptr(out), block_table=K.ptr(bt), bt_stride=bt.stride(0), bt_rows=bt.shape[0],
                     n_pages=pool.shape[0] - 1, H=H, ldc=Rp, scale=R ** -0.5, r=work, status=K.ptr(st))
    K.latent_attention(a, f32)
    _close(out, _latent_ref(bt, pool, q, H, Rp, seqs, R ** -0.5), 1e-5 if f32 else 1e-2)
    assert int(st) == 0


def _page_order(bt, seqs, kind):
    """Pages of every sequence renumbered: consecutive ascending, consecutive descending, or left scattered."""
    if kind == "scattered":
        return bt
    out, at = torch.zeros_like(bt), 1
    for row, p, n in seqs:
        ids = torch.arange(at, at + p + n, dtype=torch.int32, device=bt.device)
        out[row, :p + n] = ids if kind == "up" else ids.flip(0)
        at += p + n
    return out


TC_SEQS = SEQS + [[(0, 0, 200)], [(2, 63, 2), (3, 64, 65), (1, 127, 1), (5, 128, 3)], [(4, 900, 130), (6, 1, 1)]]


@pytest.mark.parametrize("splits", [1, 2, 8])
@pytest.mark.parametrize("pages", ["scattered", "up", "down"])
@pytest.mark.parametrize("H,R", [(7, 64), (3, 48), (5, 180), (16, 256), (7, 320), (20, 384), (2, 448), (16, 512)])
@pytest.mark.parametrize("seqs", TC_SEQS)
def test_latent_attention_on_tensor_cores(seqs, H, R, pages, splits):
    """Row tiles that straddle tokens, key tiles at every causal edge, prompts beside single tokens, merged key splits;
    a query that singles out the first key, the last cached key, its own key and the next (invisible) one."""
    K = _k()
    s, (row, p, n) = len(seqs) - 1, seqs[-1]
    far = [(s, n - 1, 0), (s, 0, p)] + ([(s, n // 2, p + n // 2 + 1)] if n > 2 else []) + ([(0, 0, seqs[0][1] - 1)] if seqs[0][1] else [])
    bt, pool, q, Rp = _latent_case(K, torch.bfloat16, H, R, seqs, far=far)
    bt = _page_order(bt, seqs, pages)
    T = q.shape[0]
    out, st = torch.zeros_like(q), _status()
    work, keep = _work(K, seqs)
    a = K.LatentArgs(q=K.ptr(q), pool=K.ptr(pool), out=K.ptr(out), block_table=K.ptr(bt), bt_stride=bt.stride(0), bt_rows=bt.shape[0],
                     n_pages=pool.shape[0] - 1, H=H, ldc=Rp, scale=R ** -0.5, r=work, status=K.ptr(st))
    K.latent_attention_tc(a, tokens=T, blk_rows=min(64, max(x[2] for x in seqs)) * H, splits=splits)
    assert int(st) == 0
    _close(out, _latent_ref(bt, pool, q, H, Rp, seqs, R ** -0.5), 1.5e-2)


@pytest.mark.parametrize("f32", [False, True])
def test_new_latents_reach_their_pages(f32):
    K = _k()
    dt = torch.float32 if f32 else torch.bfloat16
    M, nq, R, ldc = 9, 3 * 40, 48, 64
    proj, nw, pool = _rnd(M, nq + R), _rnd(R, seed=1), torch.zeros(31, ldc, dtype=dt, device=DEV)
    q, locs, st = torch.zeros(M, nq, dtype=dt, device=DEV), _ints([5, 1, 30, 2, 17, 9, 8, 3, 4]), _status()
    K.latent_new(K.LatentNewArgs(proj=K.ptr(proj), ldp=proj.stride(0), nq=nq, c_off=nq, R=R, c_norm=K.ptr(nw), eps=1e-4, q=K.ptr(q),
                                 ldq=q.stride(0), pool=K.ptr(pool), ldc=pool.stride(0), n_pages=pool.shape[0] - 1, locs=K.ptr(locs),
                                 status=K.ptr(st)), M, f32)
    ref = O.rms_normalise(proj[:, nq:].double(), 1e-4) * nw.double()
    _close(pool[locs.long(), :R], ref, 1e-5 if f32 else 8e-3)
    assert pool[:, R:].abs().sum() == 0 and (q == proj[:, :nq].to(dt)).all() and int(st) == 0
