"""Every kernel of the Makodra chain alone against the float64 oracle's functions (needs a B200)."""
import math

import pytest
import torch

import makodra_oracle as O

pytestmark = pytest.mark.gpu
DEV = "cuda"


def K():
    from smcsd_b200.ops import native
    return native


def rnd(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


def work(lens, prefix, rows, block=64):
    """Ragged work list with its tensors kept alive."""
    k = K()
    off, blk_seq, blk_start = [0], [], []
    for s, n in enumerate(lens):
        off.append(off[-1] + n)
        blk_seq += [s] * len(range(0, n, block))
        blk_start += list(range(0, n, block))
    t = [torch.tensor(v, dtype=torch.int32, device=DEV) for v in (rows, prefix, off[:-1], lens, blk_seq, blk_start)]
    r = k.Ragged(seq_row=k.ptr(t[0]), seq_prefix=k.ptr(t[1]), seq_off=k.ptr(t[2]), seq_len=k.ptr(t[3]), blk_seq=k.ptr(t[4]),
                 blk_start=k.ptr(t[5]), n_seq=len(lens), n_blk=len(blk_seq), E=0, B=block)
    return r, t


def close(got, ref, tol):
    ref = ref.double()
    e = (got.double().cpu() - ref).abs().max() / ref.abs().max()
    assert e < tol, e.item()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("d", [64, 100, 2048, 8192, 77])
def test_post_norm_step(d, f32):
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    T, d8, n = 5, (d + 7) // 8 * 8, 5
    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    embed, y, w, wf, mu = rnd(11, d).to(dt), rnd(T, d, seed=1), rnd(d, seed=2), rnd(d, seed=3), rnd(n, d, seed=4)
    ids, pos = torch.tensor([3, 0, 10, 7, 7], dtype=torch.int32), torch.tensor([0, 1, 77, 5000, 900_000], dtype=torch.int32)
    x = torch.zeros(T, d, device=DEV)
    xa = torch.zeros(T, d8, dtype=dt, device=DEV)
    freq = (10000.0 ** (-2.0 * torch.arange((d + 1) // 2, dtype=torch.float64) / d)).to(DEV)
    gd = [t.to(DEV) for t in (embed, ids, pos, y, w, wf, mu)]
    base = dict(x=k.ptr(x), d=d, vocab=11, eps=1e-3, xa=k.ptr(xa), ldxa=d8, ldy=d, status=k.ptr(st))
    k.post_norm_step(k.PostNormArgs(ids=k.ptr(gd[1]), positions=k.ptr(gd[2]), embed=k.ptr(gd[0]), freq=k.ptr(freq), **base), T, f32)
    c = torch.arange(d)
    ang = pos.double().unsqueeze(1) * 10000.0 ** (-(c - c % 2).double() / d)
    x0 = embed[ids.long()].double() + torch.where(c % 2 == 0, ang.sin(), ang.cos())
    close(x, x0, 2e-6)
    close(xa[:, :d], x0, 1e-6 if f32 else 8e-3)
    ldh = (d + 3) // 4 * 4
    hist = rnd(4, ldh, seed=5).to(DEV)
    old = hist.clone()
    rows = torch.tensor([2, 0, 3, 1, 9], dtype=torch.int32, device=DEV)       # the last row does not exist
    mix = torch.zeros(T, n, d8, dtype=dt, device=DEV)
    k.post_norm_step(k.PostNormArgs(y=k.ptr(gd[3]), w=k.ptr(gd[4]), mu=k.ptr(gd[6]), mix=k.ptr(mix), hist=k.ptr(hist), rows=k.ptr(rows),
                                    n_mix=n, ldh=ldh, n_rows=4, **base), T, f32)
    x1 = x0 + O.over_rms(y.double(), 1e-3) * w.double()
    close(x, x1, 2e-6)
    want = x1[:4].unsqueeze(1) + (old.cpu()[[2, 0, 3, 1], :d].double() - x1[:4]).unsqueeze(1) * mu.double()
    close(mix[:4, :, :d], want, 2e-6 if f32 else 8e-3)
    close(hist[[2, 0, 3, 1], :d], x1[:4], 2e-6)
    assert int(st) == k.ERR_BOUNDS and not mix[4].any()
    st.zero_()
    kept = x.clone()
    k.post_norm_step(k.PostNormArgs(y=k.ptr(gd[3]), w=k.ptr(gd[4]), w_final=k.ptr(gd[5]), **base), T, f32)
    close(xa[:, :d], O.over_rms(x1 + O.over_rms(y.double(), 1e-3) * w.double(), 1e-3) * wf.double(), 3e-6 if f32 else 8e-3)
    assert torch.equal(x, kept) and int(st) == 0


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("d,n", [(64, 5), (50, 2), (520, 3)])
def test_token_shift(d, n, f32):
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    lens, rows = [1, 130, 2, 17, 64], [4, 0, 2, 1, 5]
    T, ldm, ldh = sum(lens), (d + 7) // 8 * 8, (d + 3) // 4 * 4
    x, mu, hist = rnd(T, d).to(DEV), rnd(n, d, seed=1).to(DEV), rnd(6, ldh, seed=2).to(DEV)
    old, st = hist.cpu().clone(), torch.zeros(1, dtype=torch.int32, device=DEV)
    mix = torch.zeros(T, n, ldm, dtype=dt, device=DEV)
    r, keep = work(lens, [0] * 5, rows)
    k.token_shift(x, mu, mix, hist, r, ldm=ldm, status=st, f32=f32)
    at = 0
    for row, m in zip(rows, lens):
        h = x[at:at + m].cpu().double()
        back = torch.cat([old[row:row + 1, :d].double(), h[:-1]])
        close(mix[at:at + m, :, :d], h.unsqueeze(1) + (back - h).unsqueeze(1) * mu.cpu().double(), 2e-6 if f32 else 8e-3)
        assert torch.equal(hist[row, :d], x[at + m - 1])
        at += m
    assert torch.equal(hist[3].cpu(), old[3]) and int(st) == 0


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("H,G,dim,vdim", [(4, 2, 20, 12), (8, 8, 64, 128), (6, 1, 130, 36)])
def test_new_heads(H, G, dim, vdim, f32):
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    r8 = lambda n: (n + 7) // 8 * 8
    T, D, V = 7, r8(dim), r8(vdim)
    heads = lambda n, w, w8, s: torch.nn.functional.pad(rnd(T, n, w, seed=s), (0, w8 - w)).reshape(T, n * w8)
    q, kk, v = heads(H, dim, D, 0), heads(G, dim, D, 1), heads(G, vdim, V, 2)
    proj = torch.cat([q, kk, v, rnd(T, 8, seed=3)], 1).to(DEV)
    first = heads(G, vdim, V, 4).to(DEV)
    q_out = torch.zeros(T, H * D, dtype=dt, device=DEV)
    kp, vp = torch.zeros(10, G * D, dtype=dt, device=DEV), torch.zeros(10, G * V, dtype=dt, device=DEV)
    locs, st = torch.tensor([9, 1, 4, 2, 7, 3, 5], dtype=torch.int32, device=DEV), torch.zeros(1, dtype=torch.int32, device=DEV)
    args = dict(proj=k.ptr(proj), ldp=proj.shape[1], H=H, G=G, D=D, V=V, dim=dim, eps=1e-2, q=k.ptr(q_out), kpool=k.ptr(kp),
                vpool=k.ptr(vp), n_pages=9, locs=k.ptr(locs), status=k.ptr(st))
    tol = 2e-6 if f32 else 8e-3
    unit = lambda t, n: O.over_rms(t.view(T, n, D)[..., :dim].double(), 1e-2)
    at = locs.long().cpu()
    for lam, gives, vf in ((0.3, 0, first), (0.0, 1, first), (0.0, 0, None)):
        k.heads_new(k.HeadsNewArgs(lam=lam, gives=gives, v_first=k.ptr(vf), **args), T, f32)
        want = v.double()
        if lam:
            want = 0.7 * want + 0.3 * first.cpu().double()
        close(vp.cpu()[at], want, tol)
        if gives:
            assert torch.equal(first.cpu(), v)
    close(q_out.view(T, H, D)[..., :dim], unit(q, H), tol)
    close(kp.cpu()[at].view(T, G, D)[..., :dim], unit(kk, G), tol)
    assert not kp[0].any() and int(st) == 0


SHAPES = [(4, 2, 24, 40, 48), (2, 2, 64, 64, 64), (8, 2, 128, 128, 100), (3, 1, 16, 96, 1000), (2, 2, 200, 256, 33), (6, 2, 80, 8, 1), (2, 1, 40, 360, 90)]


@pytest.mark.parametrize("form,splits", [("f32", 1), ("f32", 4), ("bf16", 1), ("bf16", 2), ("bf16", 8), ("bf16_tc", 1)])
@pytest.mark.parametrize("H,G,D,V,chunk", SHAPES)
def test_chunk_attention(H, G, D, V, chunk, form, splits):
    """Portions inside, at and across chunk edges; equal tokens far apart stand out; scattered pages."""
    k, f32 = K(), form == "f32"
    if form == "bf16_tc" and max(D, V) > k.chunk_tc_max_width():
        pytest.skip("beyond the tensor-core form")
    dt = torch.float32 if f32 else torch.bfloat16
    prefix, lens = [0, 63, 130, 47, 95], [150, 2, 65, 1, 9]
    total = [p + n for p, n in zip(prefix, lens)]
    gen = torch.Generator().manual_seed(3)
    bt = torch.zeros(7, 300, dtype=torch.int32)
    perm, at = torch.randperm(600, generator=gen) + 1, 0
    rows = [5, 0, 3, 6, 2]
    qs, ks, vs = [], [], []
    kp, vp = torch.zeros(601, G * D), torch.zeros(601, G * V)
    for s, n in enumerate(total):
        kk, v = O.over_rms(rnd(n, G, D, seed=s), 1e-5), rnd(n, G, V, seed=50 + s)
        q = O.over_rms(rnd(n, H, D, seed=90 + s), 1e-5)
        q[-1] = kk[max(0, (n - 1) // chunk * chunk)].repeat_interleave(H // G, 0)      # asks for the chunk's first key
        pages = perm[at:at + n]
        at += n
        bt[rows[s], :n] = pages.to(torch.int32)
        kp[pages], vp[pages] = kk.reshape(n, -1), v.reshape(n, -1)
        qs.append(q), ks.append(kk), vs.append(v)
    kp, vp = kp.to(dt).to(DEV), vp.to(dt).to(DEV)
    q = torch.cat([x[p:] for x, p in zip(qs, prefix)]).to(dt)
    T = q.shape[0]
    gate, r1, r2 = rnd(T, H * V + 4, seed=7), torch.rand(H, generator=gen) + 0.1, 3 * torch.rand(H, generator=gen)
    qd, gd, r1d, r2d, btd = q.to(DEV).contiguous(), gate.to(DEV), r1.to(DEV), r2.to(DEV), bt.to(DEV)
    out = torch.zeros(T, H * V, dtype=dt, device=DEV)
    st = torch.zeros(1, dtype=torch.int32, device=DEV)
    r, keep = work(lens, prefix, rows)
    scale = 6.0 / D
    args = dict(q=k.ptr(qd), kpool=k.ptr(kp), vpool=k.ptr(vp), out=k.ptr(out), block_table=k.ptr(btd), bt_stride=300, bt_rows=7,
                n_pages=600, H=H, G=G, D=D, V=V, chunk=chunk, scale=scale, r=r, status=k.ptr(st))
    run = (lambda a: k.chunk_attention_tc(a)) if form == "bf16_tc" else (lambda a: k.chunk_attention(a, f32, splits))
    run(k.ChunkAttnArgs(gate=k.ptr(gd), ldg=H * V + 4, r1=k.ptr(r1d), r2=k.ptr(r2d), sink=1, **args))
    near = dt if not f32 else torch.float64
    ref = torch.cat([O.chunk_attention(x.to(near).double(), y.to(near).double(), z.to(near).double(), scale, r1.double(), r2.double(), chunk)[p:]
                     for x, y, z, p in zip(qs, ks, vs, prefix)])
    gated = ref.reshape(T, -1) * torch.sigmoid(gate[:, :H * V].double())
    close(out, gated, 3e-6 if f32 else 1.2e-2)
    # no gate, no bias, no sink: the plain softmax of the first sequence's first rows
    run(k.ChunkAttnArgs(sink=0, **args))
    n = min(chunk, 20)
    s = torch.einsum("ihd,jhd->hij", qs[0][:n].to(near).double(), ks[0][:n].to(near).double().repeat_interleave(H // G, 1)) * scale
    p = torch.softmax(s.masked_fill(~torch.ones(n, n, dtype=torch.bool).tril(), float("-inf")), -1)
    plain = torch.einsum("hij,jhv->ihv", p, vs[0][:n].to(near).double().repeat_interleave(H // G, 1)).reshape(n, -1)
    close(out[:n], plain, 3e-6 if f32 else 1.2e-2)
    assert int(st) == 0


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("N,rank,M", [(2048, 64, 8), (75, 16, 3), (100, 24, 32), (64, 600, 1)])
def test_decay_logits(N, rank, M, f32):
    """One launch for few tokens, and the activation of the GEMM form."""
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    x, W = rnd(M, rank + 4), (rnd(N, rank, seed=1) * rank ** -0.5).to(dt)
    xd, z, low = x.to(DEV), torch.zeros(M, N + 3, device=DEV), torch.zeros(M, rank, dtype=dt, device=DEV)
    k.low_rank(xd, W.to(DEV).contiguous(), z, M=M, f32=f32)
    k.tanh_rows(xd, low, n=rank, M=M, f32=f32)
    want = torch.tanh(x[:, :rank].double())
    close(low, want, 1e-6 if f32 else 4e-3)
    close(z[:, :N], want @ W.double().T, 2e-6 if f32 else 6e-3)
    assert not z[:, N:].any()


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("rule", ["delta", "wkv"])
@pytest.mark.parametrize("H,D", [(3, 16), (2, 20), (5, 50), (4, 64), (48, 32), (1, 100), (2, 128), (1, 160), (1, 200), (1, 256), (80, 8)])
def test_memory_scan(H, D, rule, f32):
    """Ragged portions with states carried on between two launches; other rows stay untouched."""
    k, is_delta = K(), rule == "delta"
    HD, rows, n_rows, eps = H * D, [3, 0, 5], 6, 1e-3
    parts = [[1, 17, 40], [33, 2, 1]]
    total = [sum(p[s] for p in parts) for s in range(3)]
    n = 5 if is_delta else 4
    gain = torch.tensor([1.0, D ** -0.5, 1.0, 1.0, 1.0][:n]).repeat_interleave(HD)
    proj = [rnd(t, n * HD + 3, seed=s) * torch.cat([gain, torch.ones(3)]) for s, t in enumerate(total)]
    z = [rnd(t, HD, seed=20 + s) for s, t in enumerate(total)]
    slow = torch.where(torch.rand(HD, generator=torch.Generator().manual_seed(1)) < 0.5, -8.0, -0.5)
    w0, bias, onorm = slow, rnd(HD, seed=30), rnd(HD, seed=31)
    sig, D64 = torch.sigmoid, torch.float64
    heads = lambda t: t.to(D64).reshape(t.shape[0], H, D)
    ref = []
    for s in range(3):
        r, kk, v, g = (heads(proj[s][:, i * HD:(i + 1) * HD]) for i in range(4))
        zz = heads(z[s] + w0)
        if is_delta:
            a = sig(heads(proj[s][:, 4 * HD:5 * HD] + bias))
            w = torch.exp(-math.exp(-0.5) * sig(zz))
            o = torch.stack([O.delta_rule(r[:, h], w[:, h], kk[:, h], v[:, h], a[:, h]) for h in range(H)], 1)
            gate = sig(g)
        else:
            w = torch.exp(-torch.exp(zz))
            o = torch.stack([O.bonus_memory(r[:, h], w[:, h], kk[:, h], v[:, h], bias.to(D64).view(H, D)[h]) for h in range(H)], 1)
            gate = g * sig(g)
        ref.append((O.over_rms(o, eps) * gate).reshape(-1, HD) * onorm.to(D64))
    stride = (HD * D + 31) // 32 * 32 + 32
    state = torch.zeros(n_rows, stride, device=DEV)
    state[1] = 7.0
    w0d, bd, od = w0.to(DEV), bias.to(DEV), onorm.to(DEV)
    st, at = torch.zeros(1, dtype=torch.int32, device=DEV), [0, 0, 0]
    ldo = (HD + 7) // 8 * 8
    for lens in parts:
        p = torch.cat([proj[s][at[s]:at[s] + m] for s, m in enumerate(lens)]).to(DEV)
        zd = torch.cat([z[s][at[s]:at[s] + m] for s, m in enumerate(lens)]).to(DEV)
        out = torch.zeros(p.shape[0], ldo, dtype=torch.float32 if f32 else torch.bfloat16, device=DEV)
        r, keep = work(lens, at, rows)
        k.memory_scan(k.ScanArgs(proj=k.ptr(p), ldp=p.shape[1], r_off=0, k_off=HD, v_off=2 * HD, g_off=3 * HD, a_off=4 * HD, z=k.ptr(zd),
                                 ldz=HD, w0=k.ptr(w0d), a_bias=k.ptr(bd), bonus=k.ptr(bd), onorm=k.ptr(od), state=k.ptr(state),
                                 row_stride=stride, n_rows=n_rows, out=k.ptr(out), ldo=ldo, H=H, D=D, V=D, eps=eps, unit_eps=1e-6,
                                 log_decay=math.exp(-0.5), r=r, status=k.ptr(st)), k.SCAN_DELTA if is_delta else k.SCAN_BONUS, f32)
        want = torch.cat([ref[s][at[s]:at[s] + m] for s, m in enumerate(lens)])
        close(out[:, :HD], want, 3e-5 if f32 else 8e-3)
        at = [a + m for a, m in zip(at, lens)]
    assert (state[1] == 7).all() and not state[2].any() and not state[:, HD * D:][[0, 3, 5]].any() and int(st) == 0
