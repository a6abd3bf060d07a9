"""Pasizen on the kernel chain, in 32-bit and in bf16, against the float64 oracle (needs a B200)."""
import pytest
import torch

import layered_suite as S
import pasizen_oracle as O
from pasizen_models import CONFIGS, config, dense, far_effect, mixer, moe, row_error, save_model, tokens

pytestmark = pytest.mark.gpu

F32 = S.Ctx("cuda", "float32", 3e-5)
# bf16: rounding noise of a few percent; an expert choice that falls the other way moves single rows further
BF16 = S.Ctx("cuda", "bfloat16", 0.06, slack=0.02)
# one expert per token, three passes: the plain PyTorch forward in bf16 is off in every tenth row of this model as well
BF16_TOP1 = S.Ctx("cuda", "bfloat16", 0.06, slack=0.25)
pick_ctx = lambda ctx, name: BF16_TOP1 if ctx is BF16 and name == "looped_all" else ctx
BOTH = pytest.mark.parametrize("ctx", [F32, BF16], ids=["f32", "bf16"])


@BOTH
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_portions_and_decoding(ctx, tmp_path, name):
    S.whole_portions_and_decoding(pick_ctx(ctx, name), tmp_path, name)


@BOTH
@pytest.mark.parametrize("name", ["looped_mix", "odd_sizes", "looped_all"])
def test_mixed_batches_and_reuse(ctx, tmp_path, name):
    S.mixed_batches(pick_ctx(ctx, name), tmp_path, name)


@BOTH
@pytest.mark.parametrize("name", ["looped_mix", "one_layer"])
def test_long_decoding(ctx, tmp_path, name):
    S.long_decoding(ctx, tmp_path, name)


@BOTH
@pytest.mark.parametrize("graph", [True, False])
def test_greedy_generation(ctx, tmp_path, graph):
    S.greedy_generation(ctx, tmp_path, "looped_mix", cycle_graph=graph)


def test_rows_do_not_depend_on_cuts_or_company(tmp_path):
    """bf16 rows of one sequence fed in different cuts, pages and company agree far below the rounding of the model."""
    folder, cfg, W = save_model(tmp_path / "m", "one_layer")
    eng = S.engine(BF16, folder)
    ids, other = tokens(cfg, 260), tokens(cfg, 200, seed=4)
    whole = S.feed_in_cuts(eng, "a", ids, [260])
    eng.feed([("o", other, [])])                               # other pages in between
    cut = S.feed_in_cuts(eng, "a", ids, [1, 2, 61, 66, 2, 64, 63, 1])
    assert row_error(cut, whole).max() < 0.02
    eng.feed([], ["o"])
    S.idle(eng)


def test_wide_latents_take_both_attention_kernels(tmp_path):
    """512-wide latents (split output columns) and wider ones (beyond the tensor-core kernel)."""
    cfg = config(128, [(mixer(4, 64, 32, 500), dense(160)), (mixer(2, 32, 64, 600), None)], streams=2, taps=4)
    folder, cfg, W = save_model(tmp_path / "wide", cfg)
    ids = tokens(cfg, 300)
    ref = O.forward(cfg, W, ids)
    for ctx in (F32, BF16):
        eng = S.engine(ctx, folder)
        for cuts in ([300], [200, 99, 1]):
            S.check(ctx, S.feed_in_cuts(eng, "a", ids, cuts), ref, cuts)


def test_key_splits_in_decoding(tmp_path):
    """A long context and one sequence: the attention splits its keys over CTAs; the first key still decides the last row."""
    cfg = config(96, [(mixer(3, 32, 32, 128), dense(128))], streams=2, taps=4, positions=3000)
    folder, cfg, W = save_model(tmp_path / "long", cfg, seed=2)
    ids = tokens(cfg, 2100)
    ref = O.forward(cfg, W, ids)
    eng = S.engine(BF16, folder, max_tokens=2200)
    nm = eng._sched.native_runner._prefill_chain("target")
    got = S.feed_in_cuts(eng, "a", ids, [2090] + [1] * 10)
    nm.ctx_hint = 2100
    assert nm._latent_splits(1, 1, 3, 128) > 1
    S.check(BF16, got, ref)
    effect = far_effect(lambda x: O.forward(cfg, W, x), cfg, ids, ref)
    assert effect > 0.05 and row_error(got[-1:], ref[-1:]).item() < 0.4 * effect


def test_prompts_longer_than_one_pass(tmp_path):
    """A prompt beyond the chain's token capacity continues from the cache and the state of the pass before."""
    cfg = config(64, [(mixer(2, 16, 16, 32), moe(4, 2, 2, 1, 24, 0.8)), (mixer(2, 16, 16, 32), dense(64))], streams=2, taps=4, positions=5000)
    folder, cfg, W = save_model(tmp_path / "m", cfg, seed=2)
    eng = S.engine(F32, folder, max_tokens=5000)
    nm = eng._sched.native_runner._prefill_chain("target")
    nm.T = 500                                                 # the buffers hold more; cut earlier
    ids = tokens(cfg, 1201)
    S.check(F32, S.feed_in_cuts(eng, "a", ids, [1201]), O.forward(cfg, W, ids))
    got = eng.feed([("a", ids[:300], [299]), ("b", ids[:301], [300]), ("c", ids, [499, 500, 1200])], ["a", "b", "c"])
    S.check(F32, got, O.forward(cfg, W, ids)[[299, 300, 499, 500, 1200]])
    S.idle(eng)


@pytest.mark.parametrize("pair", [("looped_mix", "looped_mix"), ("looped_mix", "dense"), ("dense", "looped_mix")])
def test_particles_graph_against_eager(tmp_path, pair):
    """SMC decoding with resampling after every cycle (states and latent pages follow their ancestors): the captured cycle
    and the same launches one by one give the same tokens."""
    from smcsd_b200.models.config import ModelConfig
    llama = ModelConfig(arch="llama", vocab_size=211, hidden_size=256, n_layers=2, n_heads=4, n_kv_heads=2, head_dim=64, ffn_size=512,
                        max_position=700, name="dense")
    pick = lambda n: llama if n == "dense" else save_model(tmp_path / n, n)[0]
    prompts = [tokens(CONFIGS["looped_mix"], n, seed=n) for n in (3, 40, 90)]
    outs = []
    for graph in (True, False):
        from smcsd_b200 import SMCEngine
        eng = SMCEngine(pick(pair[0]), pick(pair[1]), n_particles=4, gamma=3, draft_temperature=0.9, target_temperature=0.8,
                        resample_threshold=1.0, max_running_requests=4, max_total_tokens=6000, context_length=700, device="cuda",
                        cycle_graph=graph, random_seed=5, skip_tokenizer_init=True)
        res = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 30, "ignore_eos": True})
        assert all(r["completion_tokens"] == 30 for r in res)
        assert eng._sched.stats["resampled_groups"] > 0 and eng._sched.native_runner.check_status() == 0
        outs.append([r["output_ids"] for r in res])
        S.idle(eng)
    assert outs[0] == outs[1]


def test_fed_tokens_through_the_dense_and_hybrid_chains():
    """The step of given tokens serves the other families as well: portions agree with the whole prompt."""
    from smcsd_b200 import SMCEngine
    for preset in ("tiny-target", "tiny-hybrid"):
        kw = dict(n_particles=1, gamma=1, max_running_requests=4, max_total_tokens=800, context_length=512, device="cuda")
        eng = SMCEngine(f"preset:{preset}", f"preset:{preset}", backend="native", **kw)
        ref = SMCEngine(f"preset:{preset}", f"preset:{preset}", backend="torch", **kw)
        ids = torch.randint(0, 4096, (120,), generator=torch.Generator().manual_seed(1)).tolist()
        want = list(range(120))
        r = ref.feed([("a", ids, want)], ["a"]).cpu()
        for cuts in ([120], [17, 2, 64, 36, 1]):
            assert row_error(S.feed_in_cuts(eng, "a", ids, cuts), r).max() < 0.08, (preset, cuts)
        both = eng.feed([("a", ids[:50], [49]), ("b", ids[:33], [32])], ["a", "b"]).cpu()
        assert row_error(both, r[[49, 32]]).max() < 0.08
        S.idle(eng)
