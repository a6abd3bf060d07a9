"""Pasizen on the CPU path: configuration, loading, mechanisms and the engine around it against the float64 oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layered_suite as S
import pasizen_oracle as O
from pasizen_models import CONFIGS, config, dense, make_weights, mixer, moe, row_error, save_model, tokens

CTX = S.Ctx("cpu", "float32", 2e-5)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_portions_and_decoding(tmp_path, name):
    S.whole_portions_and_decoding(CTX, tmp_path, name)


@pytest.mark.parametrize("name", ["looped_mix", "odd_sizes"])
def test_mixed_batches_and_reuse(tmp_path, name):
    S.mixed_batches(CTX, tmp_path, name)


@pytest.mark.parametrize("name", ["looped_mix", "one_layer"])
def test_greedy_generation(tmp_path, name):
    outs = S.greedy_generation(CTX, tmp_path, name)
    assert len({json.dumps(v) for v in outs.values()}) == 1      # whatever the cycle length and the schedule


def test_stream_after_every_layer_run(tmp_path):
    folder, cfg, W = save_model(tmp_path / "m", "looped_mix")
    from smcsd_b200.memory.pools import KVPool, StatePool
    from smcsd_b200.models import build_model
    from smcsd_b200.models.layers import ExtendBatch
    m = build_model(folder, torch.float32)
    ids, ref, got = tokens(cfg, 12), [], []
    O.forward(cfg, W, ids, ref)
    kv, st = KVPool(m.kv_spec(torch.float32), 20, "cpu"), StatePool(m.state_spec(), 1, "cpu")
    bt = torch.arange(1, 21, dtype=torch.int32).unsqueeze(0)
    b = ExtendBatch(torch.tensor(ids), torch.arange(12), bt[0, :12], torch.tensor([0]), torch.tensor([0]), extend_len=0,
                    extend_lens=[12], prefix_lens_host=[0])
    m.forward_torch(b, kv, bt, st, per_run=got)
    assert len(ref) == len(got) == len(m.cfg.layer_runs) == 5
    for a, r in zip(got, ref):
        assert (a - r).abs().max() < 1e-4 * r.abs().max()


# ---------------------------------------------------------------------------------- mechanisms alone
def test_poly_norm_glu_and_router_match_the_equations():
    from smcsd_b200.models import layers as ly
    g = torch.Generator().manual_seed(0)
    z = torch.randn(9, 40, generator=g) * 2
    coef = torch.tensor([0.7, -0.4, 0.3, 0.15])
    assert torch.allclose(ly.poly_norm(z, coef, 1e-3).double(), O.poly_norm(z.double(), coef.double(), 1e-3), atol=1e-5)
    u = torch.randn(9, 40, generator=g) * 2
    got = ly.clamped_glu(z, u, 1.1)
    assert torch.allclose(got.double(), O.clamped_glu(z.double(), u.double(), 1.1), atol=1e-5)
    # by hand: gate beyond the limit on one side only, up on both
    a = ly.clamped_glu(torch.tensor([5.0, -5.0]), torch.tensor([9.0, -9.0]), 2.0)
    sig = lambda v: 1 / (1 + np.exp(-1.702 * v))
    assert np.allclose(a.numpy(), [2 * sig(2.0) * 3, -5 * sig(-5.0) * -1], atol=1e-6)
    zz = torch.randn(50, 12, generator=g)
    idx, w = ly.route_grouped(zz, 4, 4, 3)
    ri, rw = O.route(zz.double(), {"top": 4, "groups": {"count": 4, "keep": 3}})
    assert torch.equal(idx, ri) and torch.allclose(w.double(), rw, atol=1e-6)
    # a group's score is its best expert: the second-best expert overall is out when its group is not kept
    s = torch.tensor([[4.0, 3.9, 0.0, 0.1, 3.8, -9.0]])
    idx, w = ly.route_grouped(s, 2, 3, 1)
    assert idx.tolist() == [[0, 1]] and abs(w.sum().item() - 1) < 1e-6
    idx, _ = ly.route_grouped(s[:, [0, 5, 1, 3, 4, 2]], 2, 3, 2)
    assert idx.tolist() == [[0, 2]]


def test_short_convolution_history_and_first_tokens():
    from smcsd_b200.models import layers as ly
    w, h = torch.randn(6, 4), torch.randn(9, 6)
    ref = O.causal_short_conv(h.double(), w.double())
    assert torch.allclose(ref[0], (w[:, 3] * h[0]).double(), atol=1e-6)         # nothing before the first token
    hist = torch.zeros(2, 6, 3)
    rows, got, at = torch.tensor([1]), [], 0
    for n in (1, 2, 6):
        b = ly.ExtendBatch(None, None, None, rows, torch.tensor([at]), extend_len=0, extend_lens=[n])
        got.append(ly.short_conv(h[at:at + n], w, b, hist, rows))
        at += n
    assert torch.allclose(torch.cat(got).double(), ref, atol=1e-5)
    assert torch.equal(hist[1], h[-3:].t()) and hist[0].abs().sum() == 0


def test_hyper_connections_index_from_to():
    from smcsd_b200.models import layers as ly
    x, y = torch.randn(5, 3, 8), torch.randn(5, 8)
    wi, wo, wm = torch.randn(3), torch.randn(3), torch.randn(3, 3)
    ref = O.hyper_step(list(x.double().unbind(1)), wi.double(), wm.double(), wo.double(), lambda u: y.double())
    assert torch.allclose(ly.hyper_write(x, y, wm, wo).double(), torch.stack(ref, 1), atol=1e-5)
    wm2 = torch.zeros(3, 3)
    wm2[0, 2] = 1.0                                                             # stream 0 goes to stream 2 only
    out = ly.hyper_write(x, y, wm2, torch.zeros(3))
    assert torch.equal(out[:, 2], x[:, 0]) and out[:, :2].abs().sum() == 0


def test_latent_attention_edges():
    """A key that stands out is found far back, is not seen one position too early, and a first token sees itself only."""
    from smcsd_b200.models import layers as ly
    R, L = 16, 90
    c = torch.randn(L + 1, R) * 0.1
    bt = torch.randperm(L)[:L].to(torch.int32).unsqueeze(0) + 1
    pool = torch.zeros(L + 2, R)
    pool[bt[0].long()] = c[:L]
    for key in (0, 63, 64, 88):
        q = (c[key] * 2000).view(1, 1, R).expand(L, 2, R).contiguous()
        b = ly.ExtendBatch(None, None, None, torch.tensor([0]), torch.tensor([0]), extend_len=0, extend_lens=[L], prefix_lens_host=[0])
        out = ly.latent_attention_reference(q, pool, bt, b, 1.0)
        assert torch.allclose(out[key:, 0], c[key].expand(L - key, R), atol=1e-3)
        if key:
            assert (out[:key, 0] - c[key]).abs().amax(-1).min() > 1e-2
        assert torch.allclose(out[0, 1], c[0], atol=1e-6)


# ---------------------------------------------------------------------------------- configuration and loading
def test_configuration_is_read_in_full():
    from smcsd_b200.models.config import ModelConfig, preset
    c = ModelConfig.from_hf_dict(CONFIGS["looped_mix"])
    assert (c.arch, c.n_layers, c.layer_runs, c.streams, c.conv_taps) == ("pasizen", 3, [0, 1, 2, 1, 2], 2, 3)
    assert c.layers[2].mlp is None and c.layers[1].mlp.shared.limit == 1.3 and c.layers[1].mlp.router.keep == 2
    n = sum(v.numel() for v in make_weights(CONFIGS["looped_mix"]).values())
    assert c.param_count() == n
    assert preset("tiny-pasizen").layer_runs == [0, 1, 2, 1, 2] and preset("pasizen-2048").param_count() > 5e8
    with pytest.raises(ValueError, match="router"):
        ModelConfig.from_hf_dict(config(64, [(mixer(1, 8, 8, 8), moe(8, 5, 4, 2, 8, 1.0))], 1, 1))
    with pytest.raises(ValueError, match="mixer type"):
        bad = json.loads(json.dumps(CONFIGS["one_layer"]))
        bad["layers"][0]["type"] = "other"
        ModelConfig.from_hf_dict(bad)
    with pytest.raises(ValueError, match="loop"):
        ModelConfig.from_hf_dict(dict(CONFIGS["one_layer"], loop={"start": 0, "stop": 2, "times": 2}))


def test_checkpoint_shapes_are_checked(tmp_path):
    from smcsd_b200.models import build_model
    folder, cfg, W = save_model(tmp_path / "m", "one_layer")
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(dict(cfg, width=72), f)
    with pytest.raises(ValueError, match="shape"):
        build_model(folder, torch.float32)


def test_state_and_cache_budget():
    from smcsd_b200.memory.pools import KVPool, StatePool
    from smcsd_b200.models import build_model
    m = build_model("preset:tiny-pasizen", torch.bfloat16)
    spec = m.kv_spec(torch.bfloat16)
    assert spec.latent_widths == [64, 128, 64, 128, 64] and spec.cell_bytes == 2 * sum(spec.latent_widths)
    kv, st = KVPool(spec, 9, "cpu"), StatePool(m.state_spec(), 3, "cpu")
    assert [t.shape for t in kv.k] == [(10, w) for w in spec.latent_widths] and kv.v == []
    assert st.conv.shape == (5, 3, 136, 2) and st.temporal.numel() == 0
    assert m.state_spec().row_bytes == 5 * 136 * 2 * 4
    with pytest.raises(ValueError):
        m.kv_spec(torch.bfloat16, True)


def test_refused_layouts(tmp_path):
    from smcsd_b200.models import build_model
    folder, cfg, _ = save_model(tmp_path / "m", "one_layer")
    with pytest.raises(ValueError, match="tp_size"):
        build_model(folder, torch.float32, tp_size=2)
    with pytest.raises(ValueError, match="learned positions"):
        S.engine(CTX, folder, context_length=cfg["max_positions"] + 1)
    with pytest.raises(ValueError, match="dense models"):
        S.engine(CTX, folder, kv_cache_dtype="fp8_e4m3")


# ---------------------------------------------------------------------------------- feeding and replay
def test_feeder_refuses_what_does_not_fit(tmp_path):
    folder, cfg, _ = save_model(tmp_path / "m", "one_layer")
    eng = S.engine(CTX, folder, max_tokens=64)
    with pytest.raises(RuntimeError, match="do not fit"):
        eng.feed([("a", [1] * 65, [])])
    with pytest.raises(ValueError, match="vocabulary"):
        eng.feed([("a", [cfg["vocab"]], [])])
    with pytest.raises(ValueError, match="wanted"):
        eng.feed([("a", [1], [1])])
    with pytest.raises(ValueError, match="once per step"):
        eng.feed([("a", [1], []), ("a", [2], [])])
    S.idle(eng)
    for k in "abcd":
        eng.feed([(k, [1, 2], [])])
    with pytest.raises(RuntimeError, match="row"):
        eng.feed([("e", [1], [])])
    assert eng.feed([("a", [], []), ("b", [3], [0])], ["a", "b", "c", "d"]).shape == (1, cfg["vocab"])
    S.idle(eng)


def test_fed_sequences_live_beside_generation(tmp_path):
    """Generated requests and fed sequences share pages and rows without touching one another."""
    folder, cfg, W = save_model(tmp_path / "m", "looped_mix")
    eng = S.engine(CTX, folder, draft_temperature=0.0, target_temperature=0.0)
    ids = tokens(cfg, 30)
    a = eng.feed([("a", ids[:11], list(range(11)))])
    o1 = eng.generate(input_ids=ids[:9], sampling_params={"max_new_tokens": 8, "ignore_eos": True})["output_ids"]
    b = eng.feed([("a", ids[11:], list(range(19)))], ["a"])
    S.check(CTX, torch.cat([a, b]), O.forward(cfg, W, ids))
    o2 = eng.generate(input_ids=ids[:9], sampling_params={"max_new_tokens": 8, "ignore_eos": True})["output_ids"]
    assert o1 == o2
    S.idle(eng)


def test_particles_with_another_family_as_draft(tmp_path):
    """SMC decoding with resampling: Pasizen as target, proposal and both, next to a dense model of the same vocabulary."""
    from smcsd_b200 import SMCEngine
    kw = dict(n_particles=4, gamma=3, draft_temperature=0.9, target_temperature=0.7, dtype="float32", device="cpu",
              max_running_requests=2, resample_threshold=1.0)
    prompts = [list(range(5, 25)), list(range(40, 49))]
    for t, d in (("tiny-pasizen", "tiny-draft"), ("tiny-target", "tiny-pasizen"), ("tiny-pasizen", "tiny-pasizen")):
        eng = SMCEngine(f"preset:{t}", f"preset:{d}", **kw)
        outs = eng.generate(input_ids=prompts, sampling_params={"max_new_tokens": 14, "ignore_eos": True})
        assert all(o["completion_tokens"] == 14 for o in outs) and eng._sched.stats["resampled_groups"] > 0
        S.idle(eng)


def test_replay_program(tmp_path):
    folder, cfg, W = save_model(tmp_path / "m", "looped_mix")
    ids, other = tokens(cfg, 20), tokens(cfg, 6, seed=1)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ids[:13], "want": [2, 12]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": other, "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": ids[13:], "want": [6]}, {"id": "b", "tokens": other[:2], "want": [1]}],
              "end": ["a", "b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "64", "--device", "cpu"], input="\n".join(json.dumps(s) for s in steps) + "\n", text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    ra, rb = O.forward(cfg, W, ids), O.forward(cfg, W, other)
    load = lambda k: torch.from_numpy(np.fromfile(out / f"{k}.f32", dtype="<f4")).view(-1, cfg["vocab"])
    assert row_error(load(0), ra[[2, 12]]).max() < 2e-5
    assert row_error(load(2), torch.stack([ra[19], rb[1]])).max() < 2e-5
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32"]


def test_command_line_takes_the_model():
    import argparse

    from smcsd_b200.config import EngineArgs
    p = argparse.ArgumentParser()
    EngineArgs.add_cli_args(p)
    a = EngineArgs.from_cli_args(p.parse_args(["--model", "preset:tiny-pasizen", "--draft-model", "preset:tiny-pasizen", "--dtype",
                                               "float32", "--device", "cpu", "-N", "2", "-g", "2"])).finalize()
    from smcsd_b200.runtime.scheduler import SMCScheduler
    s = SMCScheduler(a)
    assert s.target.cfg.arch == "pasizen" and s.target is s.draft and s.server_info()["target"] == "tiny-pasizen"
