"""Checks of a layer-by-layer family's engine against its float64 oracle, shared by the CPU and the GPU tests of all such
families.  ``ctx`` supplies the family (its oracle and its test models), the device, the dtype, the tolerance and the share of
rows that may exceed it (bf16 expert choices can fall the other way)."""
from dataclasses import dataclass
from typing import Any

import torch

import pasizen_models
import pasizen_oracle
from pasizen_models import far_effect, row_error


@dataclass
class Ctx:
    device: str
    dtype: str
    tol: float
    slack: float = 0.0                    # share of rows allowed beyond tol
    models: Any = pasizen_models
    oracle: Any = pasizen_oracle


def engine(ctx, folder, max_tokens=2000, **kw):
    from smcsd_b200 import SMCEngine
    from smcsd_b200.models import resolve_config
    base = dict(n_particles=1, gamma=1, dtype=ctx.dtype, device=ctx.device, max_running_requests=4, max_total_tokens=max_tokens,
                context_length=min(resolve_config(folder).max_position, 4096), skip_tokenizer_init=True, in_process=True)
    base.update(kw)
    return SMCEngine(folder, base.pop("draft", folder), **base)


def check(ctx, got, ref, what=""):
    e = row_error(got, ref)
    bad = (e > ctx.tol).float().mean().item()
    assert bad <= ctx.slack, (what, e.max().item(), (e > ctx.tol).nonzero().flatten().tolist()[:20])


def idle(eng):
    s = eng._sched
    assert not s.feeder.live and s.feeder.held_pages == 0
    s.check_idle_invariants()
    s.alloc.check_conservation()


def feed_in_cuts(eng, rid, ids, cuts):
    out, at = [], 0
    for n in cuts:
        out.append(eng.feed([(rid, ids[at:at + n], list(range(n)))]).cpu())
        at += n
    assert at == len(ids)
    eng.feed([], [rid])
    return torch.cat(out)


def whole_portions_and_decoding(ctx, tmp_path, name):
    """One sequence whole, in portions of several sizes (two tokens at the least), and token by token."""
    folder, cfg, W = ctx.models.save_model(tmp_path / name, name)
    ids = ctx.models.tokens(cfg, 150)
    ref = ctx.oracle.forward(cfg, W, ids)
    eng = engine(ctx, folder)
    effect = far_effect(lambda x: ctx.oracle.forward(cfg, W, x), cfg, ids, ref)
    assert effect > 0.05
    for cuts in ([150], [2, 3, 64, 65, 16], [63, 2, 64, 21], [1] * 20 + [2] * 20 + [90], [118] + [1] * 32):
        got = feed_in_cuts(eng, "a", ids, cuts)
        check(ctx, got, ref, (name, cuts[:6]))
        # the far key matters: another first token would move the last row by much more than it is off
        if ctx.slack < 0.1:
            assert row_error(got[-1:], ref[-1:]).item() < 0.4 * effect, (name, cuts[:6], effect)
    idle(eng)


def mixed_batches(ctx, tmp_path, name):
    """Unequal requests in one batch, each as if alone; sequences pause; rows and pages are freed and used again in a pool
    that holds one generation of requests only."""
    folder, cfg, W = ctx.models.save_model(tmp_path / name, name, seed=3)
    lens = {"a": 130, "b": 40, "c": 70, "d": 5}
    eng = engine(ctx, folder, max_tokens=sum(lens.values()) + 3)
    for gen in range(3):
        ids = {k: ctx.models.tokens(cfg, n, seed=10 * gen + i) for i, (k, n) in enumerate(lens.items())}
        ref = {k: ctx.oracle.forward(cfg, W, v) for k, v in ids.items()}
        at, got = {k: 0 for k in ids}, {k: [] for k in ids}
        plan = [{"a": 64, "b": 1}, {"b": 2, "c": 66}, {"a": 1, "b": 30, "c": 1, "d": 3}, {"a": 62, "d": 1}, {"a": 1, "b": 5, "c": 1, "d": 1},
                {"a": 2, "b": 2, "c": 2}]
        for st in plan:
            entries = [(k + str(gen), ids[k][at[k]:at[k] + n], list(range(n))) for k, n in (st.items() if gen % 2 else reversed(st.items()))]
            out, o = eng.feed(entries).cpu(), 0
            for rid, toks, _ in entries:
                got[rid[0]].append(out[o:o + len(toks)])
                at[rid[0]] += len(toks)
                o += len(toks)
        for k in ids:
            assert at[k] == lens[k]
            check(ctx, torch.cat(got[k]), ref[k], (name, gen, k))
        eng.feed([], [k + str(gen) for k in ids])
        idle(eng)


def long_decoding(ctx, tmp_path, name, n=330):
    """Hundreds of single-token steps behind a short prompt, three sequences at once at different lengths."""
    folder, cfg, W = ctx.models.save_model(tmp_path / name, name, seed=5)
    seqs = {k: ctx.models.tokens(cfg, n + i, seed=20 + i) for i, k in enumerate("xyz")}
    eng = engine(ctx, folder)
    got = {k: [] for k in seqs}
    out = eng.feed([(k, seqs[k][:2 + i], [1 + i]) for i, k in enumerate(seqs)])
    for i, k in enumerate(seqs):
        got[k].append(out[i:i + 1].cpu())
    for t in range(n - 2):
        out = eng.feed([(k, [seqs[k][2 + i + t]], [0]) for i, k in enumerate(seqs)]).cpu()
        for i, k in enumerate(seqs):
            got[k].append(out[i:i + 1])
    for i, k in enumerate(seqs):
        check(ctx, torch.cat(got[k]), ctx.oracle.forward(cfg, W, seqs[k])[1 + i:], (name, k))
    eng.feed([], list(seqs))
    idle(eng)


def greedy_generation(ctx, tmp_path, name, gammas=(1, 3), **kw):
    """Greedy output of ``generate``: every token is the oracle's argmax given the tokens before it, or within the tolerance
    of it.  The proposal is the model itself at temperature 0, so the text is the target's own greedy text."""
    folder, cfg, W = ctx.models.save_model(tmp_path / name, name, seed=7)
    prompts = [ctx.models.tokens(cfg, n, seed=40 + n) for n in (1, 9, 70)]
    outs = {}
    for gamma in gammas:
        for defer in (True, False):
            eng = engine(ctx, folder, gamma=gamma, draft_temperature=0.0, target_temperature=0.0, defer_bonus=defer, **kw)
            res = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 21, "ignore_eos": True})
            for p, r in zip(prompts, res):
                ids = r["output_ids"]
                assert len(ids) == 21
                lg = ctx.oracle.forward(cfg, W, p + ids[:-1])[len(p) - 1:]
                gap = (lg.max(-1).values - lg.gather(1, torch.tensor(ids).unsqueeze(1))[:, 0]) / lg.std()
                assert (gap <= 4 * ctx.tol).float().mean() >= 1 - ctx.slack, (name, gamma, defer, gap.max().item())
            outs[gamma, defer] = [r["output_ids"] for r in res]
            idle(eng)
    return outs


def chunk_edges(ctx, tmp_path, cfg, size, n):
    """One attention layer alone: a changed token moves exactly the rows of its own chunk behind it, and the first rows of every
    chunk (few keys beside the sink) are right."""
    seen_by(ctx, tmp_path, cfg, n, (0, size - 2, size - 1, size, 2 * size - 1, 2 * size), lambda j: (j // size + 1) * size)


def seen_by(ctx, tmp_path, cfg, n, changed, end, weights_seed=4):
    """One layer alone: changing the token at j (each of ``changed``) moves rows j up to end(j) and no others, whether they come
    with the prompt or are decoded."""
    folder, cfg, W = ctx.models.save_model(tmp_path / "edges", cfg, seed=weights_seed)
    eng = engine(ctx, folder)
    ids = ctx.models.tokens(cfg, n, seed=6)
    ref = ctx.oracle.forward(cfg, W, ids)
    base = feed_in_cuts(eng, "a", ids, [n])
    check(ctx, base, ref)
    for j in changed:
        other = list(ids)
        other[j] = (ids[j] + 1) % cfg["vocab"]
        lo, hi = j, min(n, end(j))
        for cuts in ([n], [j + 1] + [1] * (n - j - 1), [max(j - 1, 1), n - max(j - 1, 1)]):
            got = feed_in_cuts(eng, "b", other, cuts)
            e = row_error(got, base)
            out = torch.cat([e[:lo], e[hi:]])
            assert out.numel() == 0 or out.max() <= ctx.tol, (j, cuts[:3], out.max().item())
            assert e[lo:hi].min() > 0 and e[lo] > 0.05
            check(ctx, got, ctx.oracle.forward(cfg, W, other), (j, cuts[:3]))
    idle(eng)


def window_ends(ctx, tmp_path, cfg, size):
    """One layer with a window alone: the seeking token stands just inside and just outside the window of the token it seeks, in
    the prompt and decoded; inside, it hears it loudly, outside not at all."""
    folder, cfg, W = ctx.models.save_model(tmp_path / "window", cfg, seed=9)
    sought, seeker = ctx.models.pair(cfg)
    eng = engine(ctx, folder)
    ids = ctx.models.tokens(cfg, 2 * size + 40, seed=8)
    ids[0] = 1
    for j in (0, 1, 15, size - 1, size + 3):
        for inside in (True, False):
            at = j + size - inside
            a = list(ids[:at + 3])
            a[j], a[at] = sought, seeker
            b = list(a)
            b[j] = 2
            ref, other = ctx.oracle.forward(cfg, W, a), ctx.oracle.forward(cfg, W, b)
            moved = row_error(other[at:at + 1], ref[at:at + 1]).item()
            assert moved > 0.3 if inside else moved == 0.0
            for cuts in ([at + 3], [at] + [1] * 3, [j + 1, 2] + [1] * (at - j), [at - 1, 2, 2]):
                got = feed_in_cuts(eng, "a", a, cuts)
                check(ctx, got, ref, (j, inside, cuts[:3]))
                assert row_error(got[at:at + 1], ref[at:at + 1]).item() < 0.1
    idle(eng)
