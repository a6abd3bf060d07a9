"""Every kernel of the Padadra chain alone against the float64 oracle's functions (needs a B200)."""
import pytest
import torch

import padadra_oracle as O
from test_funevik_kernels_gpu import BOTH, dev, ints, status
from test_makodra_kernels_gpu import DEV, K, close, rnd, work

pytestmark = pytest.mark.gpu


def table(positions, freq):
    """{sine, cosine} [T, n, 2] of the step's positions, as the stream step leaves them."""
    ang = torch.tensor(positions, dtype=torch.float64).unsqueeze(1) * torch.tensor(freq, dtype=torch.float64)
    return torch.stack([ang.sin(), ang.cos()], -1).float().to(DEV).contiguous()


def turned(x, positions, freq, sign=1.0):
    """Rows of x [T, ..., n] at their own positions, by way of the oracle's rotation."""
    full = torch.zeros((max(positions) + 1,) + tuple(x.shape[1:]), dtype=torch.float64)
    out = torch.empty(x.shape, dtype=torch.float64)
    for i, p in enumerate(positions):
        full[p] = x[i].double()
        out[i] = O.rotate(full[:p + 1], freq, sign)[p]
    return out


@BOTH
@pytest.mark.parametrize("d", [64, 100, 77, 2048, 8192])
def test_stream_step_of_a_pair(d, f32):
    """One scale for both outputs, norms with single weights, half the sum of two normed mixers."""
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    T, d8 = 5, (d + 7) // 8 * 8
    st, eps, tol, mult = status(), 1e-3, 3e-6 if f32 else 8e-3, 0.37
    x0, y1, yb, y2, o1, o2 = (rnd(*s, seed=i) for i, s in enumerate([(T, d)] * 4 + [(d,)] * 2))
    yb[3] = 0.0                                                # a silent mixer stays silent
    w1, w2 = torch.tensor([1.7]), torch.tensor([-0.6])
    xa, xb = (torch.zeros(T, d8, dtype=dt, device=DEV) for _ in range(2))
    x, *g = dev(x0, y1, yb, y2, o1, o2, w1, w2)
    base = dict(x=k.ptr(x), d=d, vocab=11, eps=eps, ldy=d, ldye=d, xa=k.ptr(xa), xb=k.ptr(xb), ldxa=d8, mult=mult, one_weight=1, status=k.ptr(st))
    ref = x0.double()
    normed = 0.5 * (O.over_rms(y1.double(), eps) * o1.double() + O.over_rms(yb.double(), eps) * o2.double())
    for args, mixer, f in ((dict(yb=k.ptr(g[1]), o1=k.ptr(g[3]), o2=k.ptr(g[4])), normed, False),
                           (dict(yb=k.ptr(g[1]), o1=k.ptr(g[3]), o2=k.ptr(g[4])), normed, True), ({}, y1.double(), True), ({}, y1.double(), False)):
        if f:
            args["y2"] = k.ptr(g[2])
        k.side_step(k.SideArgs(y1=k.ptr(g[0]), w1=k.ptr(g[5]), w2=k.ptr(g[6]), **args, **base), T, f32)
        ref = ref + mult * (mixer + (y2.double() if f else 0.0))
        close(x, ref, 3e-6)
        close(xa[:, :d], O.over_rms(ref, eps) * 1.7, tol)
        close(xb[:, :d], O.over_rms(ref, eps) * -0.6, tol)
    kept, b = x.clone(), xb.clone()
    k.side_step(k.SideArgs(y1=k.ptr(g[0]), w1=k.ptr(g[6]), final=1, **base), T, f32)
    close(xa[:, :d], O.over_rms(ref + mult * y1.double(), eps) * -0.6, tol)
    assert torch.equal(x, kept) and torch.equal(xb, b) and int(st) == 0 and not xa[:, d:].any()


@BOTH
@pytest.mark.parametrize("d", [64, 77, 2048])
def test_embedding_of_pairs(d, f32):
    """Ragged portions in three launches: the token before the first new one comes from the state; angles of far positions."""
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    d8, V, n, a, c, rows = (d + 7) // 8 * 8, 50, 31, 2 ** 33 + 5, 77, [4, 0, 2]
    embed, pairs, w = rnd(V, d).to(dt), rnd(n + 1, d, seed=1).to(dt), torch.tensor([1.2])
    parts, at = [[1, 70, 2], [66, 1, 1], [1, 1, 1]], [0, 0, 0]
    ids = [torch.randint(0, V, (sum(p[s] for p in parts),), generator=torch.Generator().manual_seed(s)).tolist() for s in range(3)]
    freq = [1.0, 0.37, 1e-4]
    state, st, gf = torch.zeros(6, 40, device=DEV), status(), torch.tensor(freq, dtype=torch.float64, device=DEV)
    state[1] = 7.0
    ge, gp, gw = dev(embed, pairs, w)
    far = 900_000                                              # the positions the angles see are shifted
    for lens in parts:
        T = sum(lens)
        flat = ints([t for s, m in enumerate(lens) for t in ids[s][at[s]:at[s] + m]])
        pos = [at[s] + i + far for s, m in enumerate(lens) for i in range(m)]
        gpos, ang = ints(pos), torch.zeros(T, 3, 2, device=DEV)
        x, xa = torch.zeros(T, d, device=DEV), torch.zeros(T, d8, dtype=dt, device=DEV)
        r, keep = work(lens, at, rows)
        k.side_step(k.SideArgs(x=k.ptr(x), d=d, vocab=V, eps=1e-5, ldy=d, ldye=d, xa=k.ptr(xa), ldxa=d8, one_weight=1, w1=k.ptr(gw), ids=k.ptr(flat),
                               embed=k.ptr(ge), embed_scale=0.3, pairs=k.ptr(gp), buckets=n, mul_prev=a, mul_cur=c, before=k.ptr(state),
                               before_stride=40, n_rows=6, r=r, positions=k.ptr(gpos), freq=k.ptr(gf), n_freq=3, angles=k.ptr(ang),
                               status=k.ptr(st)), T, f32)
        full = [O.embed(i, {"embed": embed.double(), "bigram": pairs.double()}, {"scale": 0.3, "bigram": {"buckets": n, "mul_prev": a, "mul_cur": c}})
                for i in ids]
        ref = torch.cat([full[s][at[s]:at[s] + m] for s, m in enumerate(lens)])
        close(x, ref, 2e-6)
        close(xa[:, :d], O.over_rms(ref, 1e-5) * 1.2, 3e-6 if f32 else 8e-3)
        close(ang, table(pos, freq).cpu(), 1e-6)
        at = [p + m for p, m in zip(at, lens)]
        assert state[rows, 0].tolist() == [float(ids[s][at[s] - 1]) for s in range(3)]
    assert int(st) == 0 and (state[1] == 7).all() and not state[:, 1:][rows].any()


@BOTH
@pytest.mark.parametrize("H,G,dim,vdim,rot,taps", [(4, 2, 24, 40, 12, 3), (6, 3, 64, 64, 64, 4), (2, 2, 5, 14, 2, 1), (3, 1, 126, 72, 6, 8),
                                                   (1, 1, 40, 8, 40, 2), (34, 17, 128, 4, 128, 5), (40, 2, 128, 256, 32, 4)])
def test_normed_heads(H, G, dim, vdim, rot, taps, f32):
    """Ragged portions in two launches: the second continues from the kept projections; other rows stay untouched."""
    k, dt, tol, eps = K(), torch.float32 if f32 else torch.bfloat16, 6e-6 if f32 else 8e-3, 1e-3
    D, V = (dim + 7) // 8 * 8, (vdim + 7) // 8 * 8
    nq, nk, nv = H * D, G * D, G * V
    C, rows, base = nq + nk + nv, [4, 0, 2, 5], 800.0
    parts = [[1, 70, 2, 17], [66, 1, 30, 2]]
    total = [sum(p[s] for p in parts) for s in range(4)]
    real = torch.cat([torch.arange(n * w) % w < o for n, w, o in ((H, D, dim), (G, D, dim), (G, V, vdim))])
    u, w = [rnd(n, C + 4, seed=s) for s, n in enumerate(total)], rnd(C, taps, seed=8) * real.unsqueeze(1)
    for x in u:
        x[:, :C] *= real
    bias, gain = rnd(C, seed=9) * real, rnd(nq + nk, seed=10) * real[:nq + nk]
    freq, turn = O.frequencies(rot, base, {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 60}), O.frequencies(vdim, base)
    want = []
    for x in u:
        y = O.causal_conv(x[:, :C].double() + bias.double(), w.double())
        q, kk, v = y.split([nq, nk, nv], 1)
        whole = lambda z, n: z / torch.sqrt((z * z).sum(1, keepdim=True) / n + eps)
        q, kk = whole(q, H * dim) * gain[:nq].double(), whole(kk, G * dim) * gain[nq:].double()
        rows_of = lambda z, n, f: O.rotate(z.reshape(z.shape[0], n, -1), f).reshape(z.shape[0], -1)
        want.append(torch.cat([rows_of(q, H, freq), rows_of(kk, G, freq), rows_of(v, G, turn)], 1))
    stride = ((taps - 1) * C + 63) // 32 * 32
    hist, st = torch.zeros(6, stride, device=DEV), status()
    hist[1] = 7.0
    wt, gb, gg = dev(w.t(), bias, gain)
    kp, vp = torch.zeros(301, nk, dtype=dt, device=DEV), torch.zeros(301, nv, dtype=dt, device=DEV)
    at, page = [0] * 4, 1
    for lens in parts:
        proj = dev(torch.cat([u[s][at[s]:at[s] + n] for s, n in enumerate(lens)]))[0]
        pos = [at[s] + i for s, n in enumerate(lens) for i in range(n)]
        T = len(pos)
        q, locs, ang = torch.zeros(T, nq, dtype=dt, device=DEV), ints(range(page, page + T)), table(pos, [9.0] + turn + freq)
        r, keep = work(lens, at, rows)
        k.normed_heads(k.ConvHeadsArgs(proj=k.ptr(proj), ldp=C + 4, H=H, G=G, D=D, V=V, rot=rot, conv=k.ptr(wt), taps=taps, hist=k.ptr(hist),
                                       row_stride=stride, n_rows=6, q=k.ptr(q), kpool=k.ptr(kp), vpool=k.ptr(vp), n_pages=300, locs=k.ptr(locs),
                                       bias=k.ptr(gb), qk_norm=k.ptr(gg), dim=dim, eps=eps, angles=k.ptr(ang), ld_angles=ang.shape[1],
                                       qk_first=1 + len(turn), v_first=1, turn=vdim, r=r, status=k.ptr(st)), f32)
        ref = torch.cat([want[s][at[s]:at[s] + n] for s, n in enumerate(lens)])
        close(q, ref[:, :nq], tol)
        close(kp[page:page + T], ref[:, nq:nq + nk], tol)
        close(vp[page:page + T], ref[:, nq + nk:], tol)
        at, page = [a + n for a, n in zip(at, lens)], page + T
    for s, row in enumerate(rows):
        assert torch.equal(hist[row, :(taps - 1) * C].cpu(), (u[s][total[s] - taps + 1:, :C] + bias).reshape(-1))
    assert (hist[1] == 7).all() and not hist[3].any() and not kp[page:].any() and not kp[0].any() and int(st) == 0


@pytest.mark.parametrize("form,splits", [("f32", 1), ("f32", 4), ("bf16", 1), ("bf16", 8), ("bf16_tc", 1)])
@pytest.mark.parametrize("H,G,D,vdim,window", [(4, 2, 24, 40, 1), (8, 2, 128, 128, 64), (3, 1, 16, 92, 63), (2, 2, 200, 256, 100), (16, 2, 64, 32, 1000),
                                               (5, 5, 128, 64, 65)])
def test_windowed_attention_with_sinks_and_turned_heads(H, G, D, vdim, window, form, splits):
    """Portions inside and across the window; every row's oldest visible key stands out, the one before it even more."""
    k, f32, V = K(), form == "f32", (vdim + 7) // 8 * 8
    dt = torch.float32 if f32 else torch.bfloat16
    prefix, lens, rows = [0, 63, 200, 47, 130], [150, 2, 65, 1, 9], [5, 0, 3, 6, 2]
    gen = torch.Generator().manual_seed(3)
    bt, perm, at = torch.zeros(7, 300, dtype=torch.int32), torch.randperm(900, generator=gen) + 1, 0
    kp, vp, sink, scale = torch.zeros(901, G * D), torch.zeros(901, G * V), 2.0 * rnd(H, seed=5), 3.0 / D
    turn, qs, ks, vs = O.frequencies(vdim, 500.0), [], [], []
    for s, (p, n) in enumerate(zip(prefix, lens)):
        kk, v, q = O.over_rms(rnd(p + n, G, D, seed=s), 1e-5), rnd(p + n, G, V, seed=50 + s), 0.4 * rnd(p + n, H, D, seed=90 + s)
        v[..., vdim:] = 0.0
        i, wide = torch.arange(p + n), kk.repeat_interleave(H // G, 1)
        q += wide[(i - window + 1).clamp(min=0)] + 2.0 * wide[(i - window).clamp(min=0)] * (i >= window).view(-1, 1, 1)
        pages = perm[at:at + p + n]
        at += p + n
        bt[rows[s], :p + n] = pages.to(torch.int32)
        kp[pages], vp[pages] = kk.reshape(p + n, -1), v.reshape(p + n, -1)
        qs.append(q), ks.append(kk), vs.append(v)
    q = torch.cat([x[p:] for x, p in zip(qs, prefix)]).to(dt)
    T, pos = q.shape[0], [p + i for p, n in zip(prefix, lens) for i in range(n)]
    gq, gk, gv, gb, gs = dev(q, kp.to(dt), vp.to(dt), bt, sink)
    out, st, ang = torch.zeros(T, H * V, dtype=dt, device=DEV), status(), table(pos, [0.3, 0.2] + turn)
    r, keep = work(lens, prefix, rows)
    a = k.ChunkAttnArgs(q=k.ptr(gq), kpool=k.ptr(gk), vpool=k.ptr(gv), out=k.ptr(out), block_table=k.ptr(gb), bt_stride=300, bt_rows=7, n_pages=900,
                        H=H, G=G, D=D, V=V, scale=scale, sink=1, sink_logit=k.ptr(gs), window=window, angles=k.ptr(ang), ld_angles=ang.shape[1],
                        angle_first=2, turn=vdim, r=r, status=k.ptr(st))
    if form == "bf16_tc":
        k.chunk_attention_tc(a)
    else:
        k.chunk_attention(a, f32, splits)
    near = torch.float64 if f32 else dt
    ref = []
    for qq, kk, v, p in zip(qs, ks, vs, prefix):
        qq, kk, v = (t.to(near).double() for t in (qq, kk, v))
        o = torch.stack([O.window_softmax(qq[:, h] @ kk[:, h // (H // G)].T * scale, v[:, h // (H // G)], window, sink[h]) for h in range(H)], 1)
        ref.append(O.rotate(o, turn, -1.0)[p:])
    close(out, torch.cat(ref).reshape(T, -1), 4e-6 if f32 else 1.2e-2)
    assert int(st) == 0


@BOTH
@pytest.mark.parametrize("few", [True, False])
@pytest.mark.parametrize("C,taps,k1,k2,n1,n2", [(100, 3, 8, 24, 50, 33), (1028, 4, 64, 64, 300, 200), (77, 1, 16, 8, 5, 260), (64, 8, 128, 72, 128, 128)])
def test_convolution_and_low_rank_maps(C, taps, k1, k2, n1, n2, few, f32):
    k, dt, rows = K(), torch.float32 if f32 else torch.bfloat16, [4, 0, 2, 5]
    parts = [[1, 5, 2, 3], [1, 1, 1, 1], [3, 1, 19, 2]] if few else [[1, 70, 2, 17], [66, 1, 30, 2]]
    total, low_off = [sum(p[s] for p in parts) for s in range(4)], (C + 7) // 8 * 8 + 8
    ldp = low_off + k1 + k2
    u, w = [rnd(n, ldp, seed=s) for s, n in enumerate(total)], rnd(C, taps, seed=8)
    w1, w2 = rnd(n1, k1, seed=20).to(dt), rnd(n2, k2, seed=21).to(dt)
    conv = [O.silu(O.causal_conv(x[:, :C].double(), w.double())) for x in u]
    stride = ((taps - 1) * C + 63) // 32 * 32
    hist, st = torch.zeros(6, stride, device=DEV), status()
    hist[1] = 7.0
    wt, g1, g2 = dev(w.t(), w1, w2)
    at = [0] * 4
    for lens in parts:
        p = torch.cat([u[s][at[s]:at[s] + n] for s, n in enumerate(lens)])
        T, gp = p.shape[0], dev(p)[0]
        out, low = torch.zeros(T, C, device=DEV), torch.zeros(T, k1 + k2, dtype=dt, device=DEV)
        z1, z2 = torch.zeros(T, n1, device=DEV), torch.zeros(T, n2, device=DEV)
        r, keep = work(lens, at, rows)
        k.conv_act(k.ConvActArgs(proj=k.ptr(gp), ldp=ldp, C=C, conv=k.ptr(wt), taps=taps, hist=k.ptr(hist), row_stride=stride, n_rows=6, out=k.ptr(out),
                                 ldo=C, low_off=low_off, k1=k1, k2=k2, low=None if few else k.ptr(low), w1=k.ptr(g1), w2=k.ptr(g2), z1=k.ptr(z1),
                                 z2=k.ptr(z2), n1=n1, n2=n2, r=r, status=k.ptr(st)), f32)
        close(out, torch.cat([conv[s][at[s]:at[s] + n] for s, n in enumerate(lens)]), 4e-6)
        x = p[:, low_off:].to(dt)
        if few:
            close(z1, x[:, :k1].double() @ w1.double().T, 3e-6)
            close(z2, x[:, k1:].double() @ w2.double().T, 3e-6)
        else:
            assert torch.equal(low.cpu(), x) and not z1.any() and not z2.any()
        at = [a + n for a, n in zip(at, lens)]
    for s, row in enumerate(rows):
        kept = torch.cat([torch.zeros(taps, C), u[s][:, :C]])[-taps + 1:] if taps > 1 else torch.zeros(0)
        assert torch.equal(hist[row, :(taps - 1) * C].cpu(), kept.reshape(-1))
    assert (hist[1] == 7).all() and not hist[3].any() and int(st) == 0


PARTS = [[1, 17, 40], [1, 1, 1], [33, 2, 1], [1, 1, 1]]        # steps of single tokens take the kernel of their own
SIZES = [(3, 16, 16), (2, 20, 33), (6, 50, 24), (4, 64, 130), (48, 32, 48), (1, 100, 300), (2, 128, 256), (1, 160, 64), (1, 256, 500), (80, 8, 1),
         (1, 3, 7), (2, 36, 100), (16, 128, 128)]


def run_memory(kind, args_of, columns, ref, H, D, V, f32):
    """Ragged portions with the state carried on between launches; other rows stay untouched."""
    k, rows, n_rows = K(), [3, 0, 5], 6
    total = [sum(p[s] for p in PARTS) for s in range(3)]
    data = [columns(t, s) for s, t in enumerate(total)]
    want = [ref(*x) for x in data]
    stride = (H * V * D + 31) // 32 * 32
    state, st, at, ldo = torch.zeros(n_rows, stride, device=DEV), status(), [0, 0, 0], (H * V + 7) // 8 * 8
    state[1] = 7.0
    for lens in PARTS:
        g = dev(*(torch.cat([data[s][i][at[s]:at[s] + m] for s, m in enumerate(lens)]) for i in range(len(data[0]))))
        out = torch.zeros(g[0].shape[0], ldo, dtype=torch.float32 if f32 else torch.bfloat16, device=DEV)
        r, keep = work(lens, at, rows)
        args = k.ScanArgs(state=k.ptr(state), row_stride=stride, n_rows=n_rows, out=k.ptr(out), ldo=ldo, H=H, D=D, V=V, r=r, status=k.ptr(st),
                          **args_of(k, *g))
        if max(lens) == 1 and k.memory_step_takes(D, V):
            k.memory_step(args, kind, f32)
        else:
            k.memory_scan(args, kind, f32, sum(lens))
        close(out[:, :H * V], torch.cat([want[s][at[s]:at[s] + m] for s, m in enumerate(lens)]), 5e-5 if f32 else 8e-3)
        at = [a + m for a, m in zip(at, lens)]
    assert (state[1] == 7).all() and not state[2].any() and not state[:, H * V * D:][[0, 3, 5]].any() and int(st) == 0


@BOTH
@pytest.mark.parametrize("H,D,V", SIZES)
def test_channel_delta_memory(H, D, V, f32):
    rep, eps = 3 if H % 3 == 0 else 2 if H % 2 == 0 else 1, 1e-3
    G = H // rep
    w0 = (torch.where(torch.arange(H) % 2 == 0, -8.0, 0.0).view(H, 1) + rnd(H, D, seed=30)).reshape(-1)      # half of the heads keep what they hold
    a_log, onorm = 0.5 * rnd(H, seed=31), rnd(H * V, seed=32)
    gw, ga, go = (t.to(DEV) for t in (w0, a_log, onorm))

    def columns(T, seed):
        return rnd(T, 2 * G * D + H * V + 3, seed=seed), rnd(T, H * D, seed=40 + seed), rnd(T, H + 5, seed=50 + seed), rnd(T, H * V, seed=60 + seed)

    def ref(x, z, b, gate):
        T = x.shape[0]
        x, z, b, gate = (t.double() for t in (x, z, b, gate))
        q, kk, v = x[:, :2 * G * D + H * V].split([G * D, G * D, H * V], 1)
        unit = lambda y: y / torch.sqrt((y * y).sum(-1, keepdim=True) + 1e-6)
        q, kk, v = unit(q.reshape(T, G, D)) * D ** -0.5, unit(kk.reshape(T, G, D)), v.reshape(T, H, V)
        g = torch.exp(-torch.exp(a_log.double()).view(1, H, 1) * O.softplus((z + w0.double()).view(T, H, D)))
        o = torch.stack([O.channel_delta_rule(q[:, h // rep], kk[:, h // rep], v[:, h], g[:, h], torch.sigmoid(b[:, h])) for h in range(H)], 1)
        return O.over_rms(o, eps).reshape(T, H * V) * onorm.double() * torch.sigmoid(gate)

    def args_of(k, x, z, b, gate):
        return dict(proj=k.ptr(x), ldp=x.shape[1], r_off=0, k_off=G * D, v_off=2 * G * D, z=k.ptr(z), ldz=H * D, w0=k.ptr(gw), r_scale=D ** -0.5,
                    beta=k.ptr(b), ldb=H + 5, gate=k.ptr(gate), ldg=H * V, a_log=k.ptr(ga), rep=rep, onorm=k.ptr(go), eps=eps, unit_eps=1e-6)
    run_memory(K().SCAN_CHANNEL, args_of, columns, ref, H, D, V, f32)


@BOTH
@pytest.mark.parametrize("H,D,V", SIZES)
def test_forget_memory(H, D, V, f32):
    eps, n = 1e-3, 2 * H * D + H * V
    bias = (torch.where(torch.arange(H) % 2 == 0, 7.0, 0.0).view(H, 1) + rnd(H, D, seed=30)).reshape(-1)
    lower, onorm = 0.5 * torch.rand(H * D, generator=torch.Generator().manual_seed(4)), rnd(H * V, seed=31)
    gb, gl, go = (t.to(DEV) for t in (bias, lower, onorm))

    def ref(x):
        T = x.shape[0]
        q, z, v = x[:, 4:4 + n].double().split([H * D, H * D, H * V], 1)
        f = (lower.double() + (1.0 - lower.double()) * torch.sigmoid(z + bias.double())).view(T, H, D)
        q, v = O.silu(q).reshape(T, H, D), v.reshape(T, H, V)
        o = torch.stack([O.forget_write(q[:, h], v[:, h], f[:, h]) for h in range(H)], 1)
        return O.over_rms(o, eps).reshape(T, H * V) * onorm.double()

    def args_of(k, x):
        return dict(proj=k.ptr(x), ldp=x.shape[1], r_off=4, a_off=4 + H * D, v_off=4 + 2 * H * D, a_bias=k.ptr(gb), lower=k.ptr(gl), onorm=k.ptr(go),
                    eps=eps)
    run_memory(K().SCAN_FORGET, args_of, lambda T, seed: (rnd(T, n + 7, seed=seed),), ref, H, D, V, f32)


@BOTH
@pytest.mark.parametrize("M,N,Kd", [(1, 72, 64), (8, 1000, 640), (20, 128, 72), (130, 400, 128), (300, 1544, 256)])
def test_squared_relu_product(M, N, Kd, f32):
    k, dt, st = K(), torch.float32 if f32 else torch.bfloat16, status()
    x, w = rnd(M, Kd).to(dt), (rnd(N, Kd, seed=1) * Kd ** -0.5).to(dt)
    gx, gw = dev(x, w)
    out = torch.full((M, N + 8), 5.0, dtype=dt, device=DEV)
    if f32:
        k.gemm_f32(gw, gx, out, N=N, M=M, relu2=True)
    else:
        for splits in {1, k.gemm_cluster_splits(N, Kd, M)}:
            k.gemm_skinny(gw, gx, out, M=M, splits=splits, epi=k.EPI_RELU2_BF16, ldo=N + 8, status=st)
    close(out[:, :N], (x.double() @ w.double().T).clamp(min=0.0) ** 2, 6e-6 if f32 else 8e-3)
    assert (out[:, N:] == 5).all() and int(st) == 0
