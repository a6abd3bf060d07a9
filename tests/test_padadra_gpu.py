"""Padadra on the kernel chain, in 32-bit and in bf16, against the float64 oracle (needs a B200)."""
import pytest
import torch

import layered_suite as S
import padadra_models as M
import padadra_oracle as O
from padadra_models import CONFIGS, attn, both, config, delta, dense, save_model, tokens
from pasizen_models import far_effect, row_error
from test_padadra_cpu import alone

pytestmark = pytest.mark.gpu

F32 = S.Ctx("cuda", "float32", 3e-5, models=M, oracle=O)
BF16 = S.Ctx("cuda", "bfloat16", 0.06, slack=0.01, models=M, oracle=O)
BOTH = pytest.mark.parametrize("ctx", [F32, BF16], ids=["f32", "bf16"])


@BOTH
@pytest.mark.parametrize("name", ["all_kinds", "odd_sizes", "delta_only"])
def test_whole_portions_and_decoding(ctx, tmp_path, name):
    S.whole_portions_and_decoding(ctx, tmp_path, name)


@BOTH
@pytest.mark.parametrize("name", list(CONFIGS))
def test_mixed_batches_and_reuse(ctx, tmp_path, name):
    S.mixed_batches(ctx, tmp_path, name)


@BOTH
@pytest.mark.parametrize("size", [1, 21, 64, 80])
def test_window_holds_exactly_its_tokens(ctx, tmp_path, size):
    S.seen_by(ctx, tmp_path, alone(size, pairs=None), 2 * size + 20, (0, 1, 15, 16, size), lambda j: j + size)


@BOTH
def test_window_behind_convolution_and_pairs(ctx, tmp_path):
    S.seen_by(ctx, tmp_path, alone(64, conv=4), 150, (0, 1, 62, 63, 64), lambda j: j + 64 + 3 + 1)


@BOTH
@pytest.mark.parametrize("size", [16, 64, 100])
def test_window_ends(ctx, tmp_path, size):
    S.window_ends(ctx, tmp_path, alone(size, pairs=None), size)


@BOTH
@pytest.mark.parametrize("layer", [delta(4, 2, 16, 24), both(attn(4, 2, 16, 24, 8, 7), 2, 16, 24)], ids=["delta", "hgrn2"])
def test_memories_see_every_token_before(ctx, tmp_path, layer):
    S.seen_by(ctx, tmp_path, config(64, [(layer, None)], mult=3.0), 90, (0, 1, 63, 64, 70), lambda j: 90)


@BOTH
def test_long_decoding(ctx, tmp_path):
    S.long_decoding(ctx, tmp_path, "all_kinds")


@BOTH
@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation(ctx, tmp_path, graph):
    S.greedy_generation(ctx, tmp_path, "all_kinds", cycle_graph=graph)


def test_greedy_generation_without_cache(tmp_path):
    S.greedy_generation(F32, tmp_path, "delta_only", cycle_graph=True)


def test_rows_do_not_depend_on_cuts_or_company(tmp_path):
    """bf16 rows of one sequence fed in different cuts, pages and company agree far below the rounding of the model."""
    folder, cfg, W = save_model(tmp_path / "m", config(64, [(delta(4, 2, 16, 24), dense(48)), (both(attn(2, 1, 16, 24, 8, 50), 2, 40, 40), None),
                                                            (delta(2, 2, 40, 40), None)]))
    eng = S.engine(BF16, folder)
    ids, other = tokens(cfg, 260), tokens(cfg, 200, seed=4)
    whole = S.feed_in_cuts(eng, "a", ids, [260])
    eng.feed([("o", other, [])])                               # other pages in between
    cut = S.feed_in_cuts(eng, "a", ids, [1, 2, 61, 66, 2, 64, 63, 1])
    assert row_error(cut, whole).max() < 0.02
    eng.feed([], ["o"])
    S.idle(eng)


def test_wide_heads(tmp_path):
    """Heads beyond the tensor-core attention, memories whose columns are split over a cluster of eight and of sixteen CTAs,
    thousands of query columns under one norm."""
    cfg = config(128, [(both(attn(2, 1, 300, 40, 32, 90), 1, 256, 500), None), (delta(1, 1, 256, 500), dense(64)), (delta(2, 1, 128, 200), None),
                       (both(attn(34, 17, 128, 72, 64, 70, conv=8), 2, 128, 130), None)])
    folder, cfg, W = save_model(tmp_path / "wide", cfg)
    ids = tokens(cfg, 130)
    ref = O.forward(cfg, W, ids)
    for ctx in (F32, BF16):
        eng = S.engine(ctx, folder)
        for cuts in ([130], [70, 59, 1]):
            S.check(ctx, S.feed_in_cuts(eng, "a", ids, cuts), ref, cuts)


def test_many_heads_take_one_cta_each(tmp_path):
    """Enough (sequence, head) pairs that no memory is split; the chain's cap on tokens cuts a prompt into passes."""
    cfg = config(64, [(delta(48, 24, 16, 24), None), (both(attn(4, 4, 16, 16, 4, 300), 40, 24, 8), dense(40))])
    folder, cfg, W = save_model(tmp_path / "many", cfg, seed=2)
    eng = S.engine(F32, folder)
    nm = eng._sched.native_runner._prefill_chain("target")
    nm.T = 90                                                  # the buffers hold more; cut earlier
    ids = tokens(cfg, 201)
    ref = O.forward(cfg, W, ids)
    S.check(F32, S.feed_in_cuts(eng, "a", ids, [201]), ref)
    got = eng.feed([("a", ids[:80], [79]), ("b", ids[:41], [40]), ("c", ids, [89, 90, 200]), ("d", ids[:33], [])], ["a", "b", "c", "d"])
    S.check(F32, got, ref[[79, 40, 89, 90, 200]])
    S.idle(eng)


@pytest.mark.parametrize("layer,quiet", [(delta(2, 2, 128, 32), False), (both(attn(4, 2, 32, 32, 8, 2060), 2, 32, 24), True),
                                         (both(attn(4, 2, 32, 32, 8, 20), 2, 32, 24), False)], ids=["delta", "attention", "hgrn2"])
def test_first_token_from_far_away(tmp_path, layer, quiet):
    """The first token still decides the last row two thousand tokens on, with the prompt and decoded."""
    cfg = config(96, [(layer, None)], mult=4.0, quiet=quiet)
    folder, cfg, W = save_model(tmp_path / "long", cfg, seed=2)
    ids = tokens(cfg, 2060)
    ref = O.forward(cfg, W, ids)
    effect = far_effect(lambda x: O.forward(cfg, W, x), cfg, ids, ref)
    assert effect > 0.1
    for ctx in (F32, BF16):
        eng = S.engine(ctx, folder, max_tokens=2200)
        for cuts in ([2060], [2050] + [1] * 10):
            got = S.feed_in_cuts(eng, "a", ids, cuts)
            S.check(ctx, got, ref)
            assert row_error(got[-1:], ref[-1:]).item() < 0.4 * effect


@pytest.mark.parametrize("pair", [("all_kinds", "all_kinds"), ("all_kinds", "dense"), ("dense", "all_kinds")])
def test_particles_graph_against_eager(tmp_path, pair):
    """SMC decoding with resampling after every cycle (states and pages follow their ancestors): the captured cycle and the
    same launches one by one give the same tokens."""
    from smcsd_b200 import SMCEngine
    from smcsd_b200.models.config import ModelConfig
    llama = ModelConfig(arch="llama", vocab_size=211, hidden_size=256, n_layers=2, n_heads=4, n_kv_heads=2, head_dim=64, ffn_size=512,
                        max_position=700, name="dense")
    pick = lambda n: llama if n == "dense" else save_model(tmp_path / n, n)[0]
    prompts = [tokens(CONFIGS["all_kinds"], n, seed=n) for n in (3, 40, 90)]
    outs = []
    for graph in (True, False):
        eng = SMCEngine(pick(pair[0]), pick(pair[1]), n_particles=4, gamma=3, draft_temperature=0.9, target_temperature=0.8,
                        resample_threshold=1.0, max_running_requests=4, max_total_tokens=6000, context_length=700, device="cuda",
                        cycle_graph=graph, random_seed=5, skip_tokenizer_init=True)
        res = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 30, "ignore_eos": True})
        assert all(r["completion_tokens"] == 30 for r in res)
        assert eng._sched.stats["resampled_groups"] > 0 and eng._sched.native_runner.check_status() == 0
        outs.append([r["output_ids"] for r in res])
        S.idle(eng)
    assert outs[0] == outs[1]


def test_one_stream_gives_the_same_rows(tmp_path, monkeypatch):
    """Feed-forward and memory beside the mixer on streams of their own, or everything on one: the same launches, the same rows."""
    folder, cfg, W = save_model(tmp_path / "m", "all_kinds")
    ids, rows = tokens(cfg, 140), []
    for beside in ("1", "0"):
        monkeypatch.setenv("SMC_BESIDE", beside)
        eng = S.engine(BF16, folder)
        rows.append(S.feed_in_cuts(eng, "a", ids, [90, 40] + [1] * 10))
    assert torch.equal(*rows)
