"""Padadra on the CPU path: configuration, loading, mechanisms and the engine around it against the float64 oracle."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layered_suite as S
import padadra_models as M
import padadra_oracle as O
from padadra_models import CONFIGS, attn, both, config, delta, dense, make_weights, save_model, tokens
from pasizen_models import row_error
from test_makodra_cpu import batch

CTX = S.Ctx("cpu", "float32", 2e-5, models=M, oracle=O)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", ["all_kinds", "odd_sizes"])
def test_whole_portions_and_decoding(tmp_path, name):
    S.whole_portions_and_decoding(CTX, tmp_path, name)


@pytest.mark.parametrize("name", ["all_kinds", "delta_only"])
def test_mixed_batches_and_reuse(tmp_path, name):
    S.mixed_batches(CTX, tmp_path, name)


def alone(size, conv=1, **kw):
    """One layer whose memory is silent: what is left are window, convolution and pairs."""
    return config(64, [(both(attn(4, 2, 16, 24, 8, size, conv=conv), 2, 16, 8), None)], quiet=True, mult=2.0, **kw)


@pytest.mark.parametrize("size", [1, 16, 21])
def test_window_holds_exactly_its_tokens(tmp_path, size):
    S.seen_by(CTX, tmp_path, alone(size, pairs=None), 2 * size + 19, (0, 1, 15, 16, size), lambda j: j + size)


def test_window_behind_convolution_and_pairs(tmp_path):
    """A token reaches the keys of the next ``taps - 1`` tokens through the convolution and of one more through the pair embedding."""
    S.seen_by(CTX, tmp_path, alone(12, conv=4), 40, (0, 1, 11, 13), lambda j: j + 12 + 3 + 1)


@pytest.mark.parametrize("size", [16, 21])
def test_window_ends(tmp_path, size):
    S.window_ends(CTX, tmp_path, alone(size, pairs=None), size)


@pytest.mark.parametrize("name", ["all_kinds", "parallel_only", "delta_only"])
def test_greedy_generation(tmp_path, name):
    outs = S.greedy_generation(CTX, tmp_path, name)
    assert len({json.dumps(v) for v in outs.values()}) == 1      # whatever the cycle length and the schedule


def test_stream_after_every_layer(tmp_path):
    folder, cfg, W = save_model(tmp_path / "m", "all_kinds")
    from smcsd_b200.memory.pools import KVPool, StatePool
    from smcsd_b200.models import build_model
    from smcsd_b200.models.layers import ExtendBatch
    m = build_model(folder, torch.float32)
    ids, ref, got = tokens(cfg, 60), [], []
    O.forward(cfg, W, ids, ref)
    kv, st = KVPool(m.kv_spec(torch.float32), 70, "cpu"), StatePool(m.state_spec(), 1, "cpu")
    bt = torch.arange(1, 71, dtype=torch.int32).unsqueeze(0)
    b = ExtendBatch(torch.tensor(ids), torch.arange(60), bt[0, :60], torch.tensor([0]), torch.tensor([0]), extend_len=0,
                    extend_lens=[60], prefix_lens_host=[0])
    m.forward_torch(b, kv, bt, st, per_run=got)
    assert len(ref) == len(got) == 4
    for a, r in zip(got, ref):
        assert (a - r).abs().max() < 1e-4 * r.abs().max()


# ---------------------------------------------------------------------------------- mechanisms alone
def test_pair_rows_carry_the_token_before():
    from smcsd_b200.models.layers import pair_rows
    ids, n, a, c = [5, 5, 9, 0, 2 ** 20, 7], 89, 2 ** 31 + 11, 65537
    want = [n] + [(p * a + t * c) % n for p, t in zip(ids, ids[1:])]
    for cuts in ([6], [1] * 6, [2, 3, 1]):
        hist, got, t = torch.zeros(3), [], 0
        for e in cuts:
            got += pair_rows(torch.tensor(ids[t:t + e]), batch([e], [t]), hist, torch.tensor([1]), n, a, c).tolist()
            t += e
        assert got == want and hist.tolist() == [0.0, 7.0, 0.0]


def test_scaled_frequencies_by_hand():
    from smcsd_b200.models.config import RotarySpec
    from smcsd_b200.models.padadra import frequencies
    got = frequencies(RotarySpec(8, 10000.0, (4.0, 1.0, 2.0, 400.0))).tolist()
    # wave lengths 6.28, 62.8, 628, 6283 against 200 (kept below) and 400 (divided above)
    assert np.allclose(got, [1.0, 0.1, 0.01 / 4, 0.001 / 4], rtol=1e-12)
    s = (400.0 / (2 * math.pi / 0.0225) - 1.0) / 1.0           # base such that the second wave (279) lies between
    assert np.allclose(frequencies(RotarySpec(4, 0.0225 ** -2, (4.0, 1.0, 2.0, 400.0))).tolist(), [1.0, (1 - s) * 0.0225 / 4 + s * 0.0225])
    for dims, base, sc in ((12, 900.0, M.SLOWED), (40, 3000.0, None)):
        spec = RotarySpec(dims, base, tuple(sc[k] for k in ("factor", "low", "high", "original")) if sc else None)
        assert np.allclose(frequencies(spec).tolist(), O.frequencies(dims, base, sc), rtol=1e-12)


def test_values_turn_back_to_relative_positions():
    """A value read at its own position comes out as it was; read further on, turned by the distance alone."""
    from smcsd_b200.models.layers import turn_pairs
    v, freq = torch.randn(1, 10, generator=torch.Generator().manual_seed(0)), torch.tensor([1.0, 0.3, 0.01, 0.2, 0.5], dtype=torch.float64)
    at = lambda x, p, back=False: turn_pairs(x, torch.tensor([p]), freq, back)
    assert torch.allclose(at(at(v, 900_001), 900_001, True), v, atol=1e-6)
    assert torch.allclose(at(at(v, 700_000), 700_003, True), at(v, 3, True), atol=1e-6)
    x = torch.randn(40, 3, 12, generator=torch.Generator().manual_seed(1))
    got = turn_pairs(x, torch.arange(40), freq)
    assert torch.allclose(got.double(), O.rotate(x.double(), freq.tolist()), atol=1e-5) and torch.equal(got[..., 10:], x[..., 10:])


def test_delta_memory_carries_its_state():
    from smcsd_b200.models.layers import channel_delta_memory
    g = torch.Generator().manual_seed(1)
    T, H, D, E = 30, 2, 6, 4
    q, k, v = torch.randn(T, H, D, generator=g), torch.randn(T, H, D, generator=g), torch.randn(T, H, E, generator=g)
    k = k / k.norm(dim=-1, keepdim=True)
    w, b = torch.rand(T, H, D, generator=g), torch.rand(T, H, generator=g)
    want = torch.stack([O.channel_delta_rule(*(t[:, h].double() for t in (q, k, v, w, b))) for h in range(H)], 1)
    for cuts in ([30], [1, 2, 27], [1] * 30):
        state, got, t = torch.zeros(H, E, D), [], 0
        for n in cuts:
            s = slice(t, t + n)
            got.append(channel_delta_memory(state, q[s], k[s], v[s], w[s], b[s]))
            t += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5)


def test_delta_memory_by_hand():
    """A full write at a unit key is read back exactly and replaces what stood there after the decay."""
    from smcsd_b200.models.layers import channel_delta_memory
    state = torch.zeros(1, 1, 2)
    k = torch.tensor([[[1.0, 0.0]], [[0.6, 0.8]], [[1.0, 0.0]]])
    v, g, b = torch.tensor([[[2.0]], [[3.0]], [[5.0]]]), torch.tensor([[[1.0, 1.0]], [[0.5, 1.0]], [[1.0, 0.25]]]), torch.tensor([[1.0], [0.5], [1.0]])
    out = channel_delta_memory(state, k, k, v, g, b)[:, 0, 0]
    m = torch.tensor([1.0, 0.0]) + 0.5 * (3.0 - 0.6) * k[1, 0]            # decayed to (1, 0), then half of what was missing
    assert torch.allclose(out, torch.tensor([2.0, 0.6 + 0.5 * 2.4, 5.0]))
    assert torch.allclose(state[0, 0], torch.tensor([5.0, m[1] * 0.25]))


def test_forget_memory_by_hand_and_carried():
    from smcsd_b200.models.layers import forget_memory
    state, f = torch.zeros(1, 1, 2), torch.tensor([[[0.25, 1.0]], [[0.5, 0.0]]])
    out = forget_memory(state, torch.ones(2, 1, 2), torch.tensor([[[4.0]], [[8.0]]]), f, 1.0 - f)
    assert out[:, 0, 0].tolist() == [3.0, 1.5 + 4.0 + 8.0] and state[0, 0].tolist() == [5.5, 8.0]
    g = torch.Generator().manual_seed(2)
    q, v, f = torch.randn(20, 3, 5, generator=g), torch.randn(20, 3, 7, generator=g), torch.rand(20, 3, 5, generator=g)
    want = torch.stack([O.forget_write(*(t[:, h].double() for t in (q, v, f))) for h in range(3)], 1)
    for cuts in ([20], [1, 2, 17], [1] * 20):
        state, got, t = torch.zeros(3, 7, 5), [], 0
        for n in cuts:
            s = slice(t, t + n)
            got.append(forget_memory(state, q[s], v[s], f[s], 1.0 - f[s]))
            t += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5)


def test_window_and_learned_sink_by_hand():
    from smcsd_b200.models.layers import chunk_attention_reference
    q, k, v = torch.zeros(3, 2, 2), torch.zeros(9, 2), torch.zeros(9, 1)
    k[3], k[5], v[3], v[5], v[2] = torch.tensor([1.0, 0.0]), torch.tensor([0.0, 1.0]), 4.0, 6.0, 1.0
    q[2, 0, 0], q[2, 1, 1] = 3.0, 2.0
    bt, sink = torch.tensor([[3, 5, 2]]), torch.tensor([0.7, -1.0])
    run = lambda window, sink: chunk_attention_reference(q, k, v, bt, batch([3]), 1, 0.5, None, None, 0, window=window, sink=sink)
    out, e = run(3, sink), [math.exp(1.5), 1.0, 1.0]
    assert abs(out[2, 0, 0] - (4 * e[0] + 6 + 1) / (sum(e) + math.exp(0.7))) < 1e-5
    assert abs(out[2, 1, 0] - (4 + 6 * math.e + 1) / (2 + math.e + math.exp(-1.0))) < 1e-5
    assert abs(run(2, sink)[2, 0, 0] - (6 + 1) / (2 + math.exp(0.7))) < 1e-5
    assert abs(run(1, None)[2, 0, 0] - 1 / 2) < 1e-6           # without learned ones the sink has score 0


# ---------------------------------------------------------------------------------- configuration and loading
def test_configuration_errors_and_counts(tmp_path):
    from smcsd_b200.models import build_model, preset
    from smcsd_b200.models.config import ModelConfig
    from smcsd_b200.models.loader import save_safetensors
    c = config(64, [(both(attn(4, 2, 16, 24, 8, 9), 3, 16, 20), None), (delta(4, 2, 16, 24), dense(40))])
    for li, path, bad in ((0, ("type",), "mamba"), (0, ("mixer", "left", "kv_heads"), 3), (0, ("mixer", "left", "rot", "dims"), 18),
                          (0, ("mixer", "left", "rot", "dims"), 7), (0, ("mixer", "left", "vdim"), 23), (0, ("mixer", "left", "mask", "size"), 0),
                          (1, ("mixer", "kv_heads"), 3), (1, ("mixer", "conv"), 0), (1, ("mlp", "kind"), "soft")):
        broken = json.loads(json.dumps(c))
        at = broken["layers"][li]
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = bad
        with pytest.raises(ValueError, match=f"layer {li}"):
            ModelConfig.from_hf_dict(broken)
    W = make_weights(c)
    low = sum(W[f"l1.mix.{n}"].numel() for n in ("a1", "a2", "g1", "g2"))
    assert ModelConfig.from_hf_dict(c).param_count() + low == sum(t.numel() for t in W.values())
    plain = dict(c, embedding={"scale": 1.0, "bigram": None})
    assert ModelConfig.from_hf_dict(plain).bigram is None
    with open(tmp_path / "config.json", "w") as f:
        json.dump(c, f)
    for name, bad in (("l1.mix.a2", W["l1.mix.a2"][:, :-3]), ("l0.mix.left.q.norm", W["l0.mix.left.q.norm"][:-1]), ("bigram", W["bigram"][:-1])):
        save_safetensors({**W, name: bad.contiguous()}, str(tmp_path / "model.safetensors"))
        with pytest.raises(ValueError, match=name):
            build_model(str(tmp_path), torch.float32)
    assert preset("padadra-2048").param_count() > 5e8
    assert build_model("preset:tiny-padadra", torch.float32).weight_bytes() > 0


def test_pool_layout():
    from smcsd_b200.memory.pools import StatePool
    from smcsd_b200.models.config import ModelConfig
    from smcsd_b200.models.padadra import PadadraModel
    m = PadadraModel(ModelConfig.from_hf_dict(CONFIGS["all_kinds"]), torch.float32)
    kv, st = m.kv_spec(torch.bfloat16), m.state_spec()
    assert kv.row_widths == [(3 * 24, 3 * 40), (40, 24)] and kv.cell_bytes == 2 * (72 + 120 + 64)
    pool = StatePool(st, 3, "cpu")
    assert [tuple(pool.matrix(i).shape[1:]) for i in range(9)] == [
        (1, 1, 1), (1, 2, 9 * 24 + 3 * 40), (3, 24, 40), (1, 3, 2 * 2 * 40 + 4 * 24), (4, 24, 40), (1, 0, 5 * 40 + 24), (5, 56, 24),
        (1, 1, 10 * 24 + 5 * 56), (5, 56, 24)]
    pool.matrix(4)[2] = 1.0
    pool.matrix(0)[2] = 77.0
    pool.copy_rows(torch.tensor([0]), torch.tensor([2]))
    assert (pool.matrix(4)[0] == 1).all() and pool.matrix(0).flatten().tolist() == [77.0, 0.0, 77.0] and not pool.matrix(2).any()
    pool.clear_rows(torch.tensor([0, 2]))
    assert not pool.temporal.any()


def test_trace_replay_in_a_process_of_its_own(tmp_path):
    folder, cfg, W = save_model(tmp_path / "m", "all_kinds")
    ids = tokens(cfg, 40)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": ids[30:39], "want": []}, {"id": "y", "tokens": ids[:2], "want": [1]}], "end": ["y"]},
             {"step": 2, "entries": [{"id": "x", "tokens": ids[39:], "want": [0]}], "end": ["x"]}]
    os.makedirs(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(tmp_path / "out"),
                        "--max-tokens", "128", "--device", "cpu"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, env=dict(os.environ, PATH=os.path.dirname(sys.executable) + ":" + os.environ["PATH"]))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == ["done 0", "done 1", "done 2"]
    ref = O.forward(cfg, W, ids)
    for n, rows in ((0, [0, 29]), (1, [1]), (2, [39])):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4")).view(len(rows), -1)
        assert row_error(got, ref[rows]).max() < 2e-5
