"""Every kernel of the Funevik chain alone against the float64 oracle's functions (needs a B200)."""
import math

import pytest
import torch

import funevik_oracle as O
from test_makodra_kernels_gpu import DEV, K, close, rnd, work

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])


def dev(*ts):
    return [t.to(DEV).contiguous() for t in ts]


def ints(v):
    return torch.tensor(v, dtype=torch.int32, device=DEV)


def status():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def frequencies(base, dims):
    return (base ** (-torch.arange(0, dims, 2, dtype=torch.float64) / dims)).to(DEV)


def rotated(x, positions, base, dims):
    """Rows of x [T, ..., n] at their own positions, by way of the oracle's rotation."""
    T = int(max(positions)) + 1
    full = torch.zeros((T,) + tuple(x.shape[1:]), dtype=torch.float64)
    out = []
    for i, p in enumerate(positions):
        full[p] = x[i].double()
        out.append(O.rotate(full, base, dims)[p])
    return torch.stack(out)


@BOTH
@pytest.mark.parametrize("d", [64, 100, 77, 2048, 8192])
def test_side_step(d, f32):
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    T, d8, top = 5, (d + 7) // 8 * 8, 3
    st, eps, tol = status(), 1e-3, 3e-6 if f32 else 8e-3
    embed, y1, y2, ye = rnd(11, d).to(dt), rnd(T, d, seed=1), rnd(T, d, seed=2), rnd(T * top, d, seed=3)
    s1, s2, w1, w2, gate, rw = (rnd(*s, seed=9 + i) for i, s in enumerate([(d,), (d,), (d,), (d,), (T,), (T, top)]))
    slot = torch.randperm(T * top, generator=torch.Generator().manual_seed(0)).view(T, top)
    ids = [3, 0, 10, 7, 12]                                    # the last token does not exist
    x, n2 = torch.zeros(T, d, device=DEV), torch.zeros(T, d, device=DEV)
    xa, xb = (torch.zeros(T, d8, dtype=dt, device=DEV) for _ in range(2))
    g = dev(embed, y1, y2, ye, s1, s2, w1, w2, gate, rw)
    gi, gs = ints(ids), slot.to(torch.int32).to(DEV)
    base = dict(x=k.ptr(x), d=d, vocab=11, eps=eps, ldy=d, ldye=d, xa=k.ptr(xa), xb=k.ptr(xb), ldxa=d8, status=k.ptr(st))
    k.side_step(k.SideArgs(ids=k.ptr(gi), embed=k.ptr(g[0]), embed_scale=2.5, w1=k.ptr(g[6]), w2=k.ptr(g[7]), n2=k.ptr(n2), **base), T, f32)
    x0 = embed[[3, 0, 10, 7, 0]].double() * 2.5
    assert int(st) == k.ERR_BOUNDS
    st.zero_()

    def both(xs):
        close(x, xs, 2e-6)
        u = O.over_rms(xs, eps)
        close(xa[:, :d], u * w1.double(), tol)
        close(xb[:, :d], u * w2.double(), tol)
    both(x0)
    close(n2, O.over_rms(x0, eps) * w2.double(), 3e-6)
    # a plain feed-forward, a gated one beside experts, experts alone, none
    mixed = (rw.double().unsqueeze(-1) * ye.double()[slot]).sum(1)
    ye_args = dict(ye=k.ptr(g[3]), top=top, route_slot=k.ptr(gs), route_w=k.ptr(g[9]))
    for args, f in ((dict(y2=k.ptr(g[2])), y2.double()), (dict(y2=k.ptr(g[2]), gate=k.ptr(g[8]), **ye_args), gate.double().unsqueeze(1) * y2.double() + mixed),
                    (ye_args, mixed), ({}, None)):
        if f is not None:
            args["s2"] = k.ptr(g[5])
        k.side_step(k.SideArgs(y1=k.ptr(g[1]), s1=k.ptr(g[4]), w1=k.ptr(g[6]), w2=k.ptr(g[7]), **args, **base), T, f32)
        x0 = x0 + s1.double() * y1.double() + (0.0 if f is None else s2.double() * f)
        both(x0)
    kept, b = x.clone(), xb.clone()
    k.side_step(k.SideArgs(y1=k.ptr(g[1]), s1=k.ptr(g[4]), w1=k.ptr(g[7]), final=1, **base), T, f32)
    close(xa[:, :d], O.over_rms(x0 + s1.double() * y1.double(), eps) * w2.double(), tol)
    assert torch.equal(x, kept) and torch.equal(xb, b) and int(st) == 0 and not xa[:, d:].any()


@BOTH
@pytest.mark.parametrize("H,G,D,V,rot,taps", [(4, 2, 24, 40, 12, 3), (6, 3, 64, 64, 64, 4), (2, 2, 8, 16, 2, 1), (3, 1, 128, 72, 6, 8), (1, 1, 40, 8, 40, 2)])
def test_conv_heads(H, G, D, V, rot, taps, f32):
    """Ragged portions in two launches: the second continues from the kept projections; other rows stay untouched."""
    k, dt, tol = K(), torch.float32 if f32 else torch.bfloat16, 4e-6 if f32 else 8e-3
    nq, nk, nv = H * D, G * D, G * V
    C, rows, base = nq + nk + nv, [4, 0, 2, 5], 800.0
    parts = [[1, 70, 2, 17], [66, 1, 30, 2]]
    total = [sum(p[s] for p in parts) for s in range(4)]
    u, w = [rnd(n, C + 4, seed=s) for s, n in enumerate(total)], rnd(C, taps, seed=8)
    want = [O.causal_conv(x[:, :C].double(), w.double()) for x in u]
    turn = lambda x, heads: O.rotate(x.reshape(x.shape[0], heads, D), base, rot).reshape(x.shape[0], -1)
    want = [torch.cat([turn(x[:, :nq], H), turn(x[:, nq:nq + nk], G), x[:, nq + nk:]], 1) for x in want]
    stride = (taps - 1) * C + 40
    hist, st, freq = torch.zeros(6, stride, device=DEV), status(), frequencies(base, rot)
    hist[1] = 7.0
    wt = dev(w.t())[0]
    kp, vp = torch.zeros(301, nk, dtype=dt, device=DEV), torch.zeros(301, nv, dtype=dt, device=DEV)
    at, page = [0] * 4, 1
    for lens in parts:
        proj = dev(torch.cat([u[s][at[s]:at[s] + n] for s, n in enumerate(lens)]))[0]
        pos = [at[s] + i for s, n in enumerate(lens) for i in range(n)]
        T = len(pos)
        q, locs, gp = torch.zeros(T, nq, dtype=dt, device=DEV), ints(range(page, page + T)), ints(pos)
        r, keep = work(lens, at, rows)
        k.conv_heads(k.ConvHeadsArgs(proj=k.ptr(proj), ldp=C + 4, H=H, G=G, D=D, V=V, rot=rot, conv=k.ptr(wt), taps=taps, hist=k.ptr(hist),
                                     row_stride=stride, n_rows=6, freq=k.ptr(freq), positions=k.ptr(gp), q=k.ptr(q), kpool=k.ptr(kp),
                                     vpool=k.ptr(vp), n_pages=300, locs=k.ptr(locs), r=r, status=k.ptr(st)), f32)
        ref = torch.cat([want[s][at[s]:at[s] + n] for s, n in enumerate(lens)])
        close(q, ref[:, :nq], tol)
        close(kp[page:page + T], ref[:, nq:nq + nk], tol)
        close(vp[page:page + T], ref[:, nq + nk:], tol)
        at, page = [a + n for a, n in zip(at, lens)], page + T
    for s, row in enumerate(rows):
        assert torch.equal(hist[row, :(taps - 1) * C].cpu(), u[s][total[s] - taps + 1:, :C].reshape(-1))
    assert (hist[1] == 7).all() and not hist[3].any() and not kp[page:].any() and not kp[0].any() and int(st) == 0


@BOTH
@pytest.mark.parametrize("heads,width,first,rot", [(3, 32, 24, 8), (5, 24, 7, 16), (16, 192, 128, 64), (2, 40, 0, 40)])
def test_rotate_heads(heads, width, first, rot, f32):
    k, dt = K(), torch.float32 if f32 else torch.bfloat16
    pos = [0, 1, 5, 77, 300]
    x, freq = rnd(5, heads * width + 4), frequencies(500.0, rot)
    out, xd = torch.zeros(5, heads * width, dtype=dt, device=DEV), x.to(DEV)
    k.rotate_heads(xd, out, freq, ints(pos), heads=heads, width=width, first=first, rot=rot, M=5, f32=f32)
    h = x[:, :heads * width].double().view(5, heads, width)
    want = torch.cat([h[..., :first], rotated(h[..., first:first + rot], pos, 500.0, rot), h[..., first + rot:]], -1)
    close(out, want.reshape(5, -1), 3e-6 if f32 else 8e-3)


@BOTH
def test_new_latents_with_a_query_latent_and_a_rotated_key(f32):
    k, dt, tol = K(), torch.float32 if f32 else torch.bfloat16, 4e-6 if f32 else 8e-3
    T, Q, Q8, R, rot, ldc, eps = 6, 21, 24, 40, 10, 64, 1e-3
    pos = [3, 0, 60, 7, 8, 250]
    proj, qn, cn = rnd(T, Q8 + R + rot + 2), rnd(Q, seed=1), rnd(R, seed=2)
    q, pool = torch.full((T, Q8), 3.0, dtype=dt, device=DEV), torch.zeros(31, ldc, dtype=dt, device=DEV)
    locs, st, freq = [5, 1, 30, 2, 17, 9], status(), frequencies(600.0, rot)
    g, gp, gl = dev(proj, qn, cn), ints(pos), ints(locs)
    k.latent_new(k.LatentNewArgs(proj=k.ptr(g[0]), ldp=proj.shape[1], nq=Q8, c_off=Q8, R=R, rot=rot, q_norm=k.ptr(g[1]), nq_real=Q, c_norm=k.ptr(g[2]),
                                 eps=eps, freq=k.ptr(freq), positions=k.ptr(gp), q=k.ptr(q), ldq=Q8, pool=k.ptr(pool), ldc=ldc, n_pages=30,
                                 locs=k.ptr(gl), status=k.ptr(st)), T, f32)
    close(q[:, :Q], O.over_rms(proj[:, :Q].double(), eps) * qn.double(), tol)
    close(pool[locs, :R], O.over_rms(proj[:, Q8:Q8 + R].double(), eps) * cn.double(), tol)
    close(pool[locs, R:R + rot], rotated(proj[:, Q8 + R:Q8 + R + rot], pos, 600.0, rot), tol)
    assert not q[:, Q:].any() and not pool[:, R + rot:].any() and not pool[0].any() and int(st) == 0


@pytest.mark.parametrize("form,splits", [("f32", 1), ("bf16", 1), ("bf16_tc", 1), ("bf16_tc", 2), ("bf16_tc", 8)])
@pytest.mark.parametrize("H,R,window", [(3, 64, 1), (6, 128, 64), (5, 192, 100), (16, 320, 63), (2, 512, 1000), (7, 64, 0)])
def test_windowed_latent_attention_with_sinks(H, R, window, form, splits):
    """Portions inside and across the window; every row's oldest visible key stands out, the one before it even more."""
    k, f32 = K(), form == "f32"
    dt = torch.float32 if f32 else torch.bfloat16
    prefix, lens, rows = [0, 63, 200, 47, 130], [150, 2, 65, 1, 9], [5, 0, 3, 6, 2]
    gen = torch.Generator().manual_seed(3)
    bt, perm, at = torch.zeros(7, 300, dtype=torch.int32), torch.randperm(700, generator=gen) + 1, 0
    pool, sink, scale = torch.zeros(901, R), 2.0 * rnd(H, seed=5), 3.0 / R
    qs, cs = [], []
    for s, (p, n) in enumerate(zip(prefix, lens)):
        c = O.over_rms(rnd(p + n, R, seed=s), 1e-5)
        pages = perm[at:at + p + n] if s else torch.arange(701, 701 + p + n)       # one sequence with pages in a row
        at += p + n
        bt[rows[s], :p + n] = pages.to(torch.int32)
        pool[pages] = c
        i = torch.arange(p, p + n)
        q = 0.4 * rnd(n, H, R, seed=90 + s)
        if window:
            q += c[(i - window + 1).clamp(min=0)].unsqueeze(1) + 2.0 * (c[(i - window).clamp(min=0)] * (i >= window).unsqueeze(1)).unsqueeze(1)
        qs.append(q), cs.append(c)
    q = torch.cat(qs).to(dt)
    T = q.shape[0]
    gq, gp, gb, gs = dev(q, pool.to(dt), bt, sink)
    out, st = torch.zeros(T, H, R, dtype=dt, device=DEV), status()
    r, keep = work(lens, prefix, rows)
    a = k.LatentArgs(q=k.ptr(gq), pool=k.ptr(gp), out=k.ptr(out), block_table=k.ptr(gb), bt_stride=300, bt_rows=7, n_pages=900, H=H, ldc=R,
                     scale=scale, window=window, sink=k.ptr(gs), r=r, status=k.ptr(st))
    if form == "bf16_tc":
        k.latent_attention_tc(a, tokens=T, blk_rows=64 * H, splits=splits)
    else:
        k.latent_attention(a, f32)
    near = torch.float64 if f32 else dt
    ref = []
    for qq, c, p in zip(qs, cs, prefix):
        c, qq = c.to(near).double(), qq.to(near).double()
        full = torch.zeros(c.shape[0], H, R, dtype=torch.float64)
        full[p:] = qq
        ref.append(torch.stack([O.window_softmax(full[:, h] @ c.T * scale, c, lambda i: i - window + 1 if window else 0, sink[h]) for h in range(H)], 1)[p:])
    close(out, torch.cat(ref), 4e-6 if f32 else 1.2e-2)
    assert int(st) == 0


@pytest.mark.parametrize("form,splits", [("f32", 1), ("f32", 4), ("bf16", 1), ("bf16", 8), ("bf16_tc", 1)])
@pytest.mark.parametrize("H,G,D,V,cap", [(4, 2, 24, 40, 3.0), (8, 2, 128, 128, 20.0), (3, 1, 16, 96, 50.0), (2, 2, 200, 256, 5.0)])
def test_soft_capped_attention_with_head_gates(H, G, D, V, cap, form, splits):
    k, f32 = K(), form == "f32"
    dt = torch.float32 if f32 else torch.bfloat16
    prefix, lens, rows = [0, 63, 130, 200], [150, 2, 65, 1], [5, 0, 3, 6]
    gen = torch.Generator().manual_seed(3)
    bt, perm, at = torch.zeros(7, 300, dtype=torch.int32), torch.randperm(900, generator=gen) + 1, 0
    kp, vp, scale = torch.zeros(901, G * D), torch.zeros(901, G * V), 6.0 / D
    qs, ks, vs = [], [], []
    for s, (p, n) in enumerate(zip(prefix, lens)):
        kk, v, q = rnd(p + n, G, D, seed=s), rnd(p + n, G, V, seed=50 + s), 0.5 * rnd(p + n, H, D, seed=90 + s)
        q[-1] += kk[0].repeat_interleave(H // G, 0)            # the last token asks for the first key
        pages = perm[at:at + p + n]
        at += p + n
        bt[rows[s], :p + n] = pages.to(torch.int32)
        kp[pages], vp[pages] = kk.reshape(p + n, -1), v.reshape(p + n, -1)
        qs.append(q), ks.append(kk), vs.append(v)
    q = torch.cat([x[p:] for x, p in zip(qs, prefix)]).to(dt)
    T = q.shape[0]
    gate = rnd(T, H + 4, seed=7)
    gq, gk, gv, gg, gb = dev(q, kp.to(dt), vp.to(dt), gate, bt)
    out, st = torch.zeros(T, H * V, dtype=dt, device=DEV), status()
    r, keep = work(lens, prefix, rows)
    a = k.ChunkAttnArgs(q=k.ptr(gq), kpool=k.ptr(gk), vpool=k.ptr(gv), out=k.ptr(out), gate=k.ptr(gg), ldg=H + 4, gate_heads=1, block_table=k.ptr(gb),
                        bt_stride=300, bt_rows=7, n_pages=900, H=H, G=G, D=D, V=V, chunk=1 << 30, scale=scale, softcap=cap, sink=1, r=r,
                        status=k.ptr(st))
    if form == "bf16_tc":
        k.chunk_attention_tc(a)
    else:
        k.chunk_attention(a, f32, splits)
    near = torch.float64 if f32 else dt
    ref = []
    for qq, kk, v, p in zip(qs, ks, vs, prefix):
        qq, kk, v = (t.to(near).double() for t in (qq, kk, v))
        s = lambda h: cap * torch.tanh(qq[:, h] @ kk[:, h // (H // G)].T * scale / cap)
        ref.append(torch.stack([O.window_softmax(s(h), v[:, h // (H // G)], lambda i: 0, 0.0) for h in range(H)], 1)[p:])
    close(out, (torch.cat(ref) * torch.sigmoid(gate[:, :H].double()).unsqueeze(-1)).reshape(T, -1), 4e-6 if f32 else 1.2e-2)
    assert int(st) == 0


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16_chunks"])
@pytest.mark.parametrize("H,D,V", [(3, 16, 16), (2, 20, 33), (5, 50, 24), (4, 64, 130), (48, 32, 48), (1, 100, 300), (2, 128, 256), (1, 160, 64),
                                   (1, 256, 500), (80, 8, 1), (1, 3, 7),
                                   (2, 36, 100), (1, 64, 512), (2, 100, 196)])
def test_gated_memory(H, D, V, form):
    """Ragged portions with state, normaliser and maximum carried on between launches; other rows stay untouched."""
    k, rows, n_rows, eps, cap, f32 = K(), [3, 0, 5], 6, 1e-3, 6.0, form == "f32"
    parts = [[1, 17, 40], [1, 1, 1], [33, 2, 1], [1, 1, 1]]     # steps of single tokens take the kernel of their own
    if form == "bf16_chunks":
        parts = [[65, 130, 64], [1, 1, 1], [190, 2, 63]]
        if not k.gated_chunk_takes(D, V):
            pytest.skip("beyond the chunked form")
    total = [sum(p[s] for p in parts) for s in range(3)]
    cols, ldp = H * (2 * D + 2 * V) + 2 * H, (H * (2 * D + 2 * V) + 2 * H + 7) // 8 * 8
    proj = [rnd(t, ldp, seed=s) for s, t in enumerate(total)]
    for x in proj:
        x[:, cols - 2 * H:cols] *= 4.0
    bias = torch.cat([rnd(H, seed=30), torch.where(torch.arange(H) % 2 == 0, 20.0, 1.0)])        # half of the heads keep what they hold
    onorm, ref, tops = rnd(H * V, seed=31), [], []
    for x in (p[:, :cols].double() for p in proj):
        T = x.shape[0]
        q, kk, v, g, i, f = x.split([H * D, H * D, H * V, H * V, H, H], 1)
        q, kk, v = q.reshape(T, H, D) * D ** -0.5, kk.reshape(T, H, D), v.reshape(T, H, V)
        i = cap * torch.tanh((i + bias[:H]) / cap)
        f = O.log_sigmoid(cap * torch.tanh((f + bias[H:]) / cap))
        o = torch.stack([O.matrix_memory(q[:, h], kk[:, h], v[:, h], i[:, h], f[:, h]) for h in range(H)], 1)
        ref.append(O.over_rms(o, eps).reshape(T, H * V) * onorm.double() * torch.sigmoid(g))
        m = torch.zeros(H, dtype=torch.float64)
        for t in range(T):
            m = torch.maximum(f[t] + m, i[t])
        tops.append(m)
    at_top = (H * (V + 1) * D + 31) // 32 * 32
    stride = at_top + (H + 31) // 32 * 32
    state, st, at, ldo = torch.zeros(n_rows, stride, device=DEV), status(), [0, 0, 0], (H * V + 7) // 8 * 8
    state[1] = 7.0
    gb, go = dev(bias, onorm)
    for lens in parts:
        p = dev(torch.cat([proj[s][at[s]:at[s] + m] for s, m in enumerate(lens)]))[0]
        out = torch.zeros(p.shape[0], ldo, dtype=torch.float32 if f32 else torch.bfloat16, device=DEV)
        r, keep = work(lens, at, rows)
        args = k.ScanArgs(proj=k.ptr(p), ldp=p.shape[1], r_off=0, k_off=H * D, v_off=2 * H * D, g_off=H * (2 * D + V), a_off=2 * H * (D + V),
                          a_bias=k.ptr(gb), onorm=k.ptr(go), state=k.ptr(state), row_stride=stride, n_rows=n_rows, out=k.ptr(out), ldo=ldo,
                          H=H, D=D, V=V, eps=eps, unit_eps=1e-6, top=k.ptr(state[:, at_top:]), gate_cap=cap, r_scale=D ** -0.5, r=r,
                          status=k.ptr(st))
        if max(lens) == 1 and k.gated_step_takes(D, V):
            k.gated_step(args, f32)
        elif form == "bf16_chunks":
            k.gated_chunk(args)
        else:
            k.memory_scan(args, k.SCAN_GATED, f32)
        close(out[:, :H * V], torch.cat([ref[s][at[s]:at[s] + m] for s, m in enumerate(lens)]), 5e-5 if f32 else 1e-2 if form == "bf16_chunks" else 8e-3)
        at = [a + m for a, m in zip(at, lens)]
    for row, m in zip(rows, tops):
        assert (state[row, at_top:at_top + H].cpu().double() - m).abs().max() < 1e-4
    assert (state[1] == 7).all() and not state[2].any() and not state[:, H * (V + 1) * D:at_top][[0, 3, 5]].any() and int(st) == 0


@BOTH
@pytest.mark.parametrize("T", [3, 301])
def test_router_bias_and_shared_gate(T, f32):
    k, dt, d, E, top = K(), torch.float32 if f32 else torch.bfloat16, 100, 6, 3
    h, w, b = rnd(T, d), rnd(E + 1, 104, seed=1).to(dt), 3.0 * rnd(E, seed=2)
    w[:, d:] = 0
    idx, wgt, gate = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV), torch.zeros(T, device=DEV)
    g = dev(h, w, b)
    k.route(g[0], g[1], idx, wgt, d=d, top=top, groups=1, keep=1, T=T, f32=f32, bias=g[2], gate=gate)
    z = h.double() @ w[:, :d].double().T
    best = (z[:, :E] + b.double()).topk(top, dim=1)
    assert torch.equal(idx.cpu().long(), best.indices)
    close(wgt, torch.softmax(best.values, 1), 1e-5)
    close(gate, torch.sigmoid(z[:, E]), 1e-5)


@BOTH
def test_gelu_unit(f32):
    k, M, ff, d = K(), 20, 128, 72
    dt = torch.float32 if f32 else torch.bfloat16
    x, wg, wu = rnd(M, d).to(dt), (2 * rnd(ff, d, seed=1) * d ** -0.5).to(dt), rnd(ff, d, seed=2).to(dt)
    from smcsd_b200.models.llama import interleave_gate_up
    W, st = interleave_gate_up(wg, wu, 64), status()
    act, g = torch.zeros(M, ff, dtype=dt, device=DEV), dev(W, x)
    if f32:
        gu = torch.zeros(M, 2 * ff, device=DEV)
        k.gemm_f32(g[0], g[1], gu, N=2 * ff, M=M)
        k.gated_unit_f32(gu, act, ff=ff, blk=64, limit=math.inf, slope=1.0, shift=0.0, M=M, gelu=True)
    else:
        k.gemm_grouped(g[0], g[1], act, N=2 * ff, M=M, splits=1, epi=k.EPI_SWIGLU_BF16, link=k.GroupLink(act=k.ACT_GELU, limit=math.inf, slope=1.0), status=st)
    gate, up = x.double() @ wg.double().T, x.double() @ wu.double().T
    close(act, O.gelu_tanh(gate) * up, 3e-6 if f32 else 8e-3)
    assert int(st) == 0
