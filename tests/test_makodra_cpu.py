"""Makodra on the CPU path: configuration, loading, mechanisms and the engine around it against the float64 oracle."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import layered_suite as S
import makodra_models as M
import makodra_oracle as O
from makodra_models import CONFIGS, attn, config, delta, make_weights, save_model, tokens, wkv
from pasizen_models import row_error

CTX = S.Ctx("cpu", "float32", 2e-5, models=M, oracle=O)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", ["all_kinds", "odd_sizes", "memory_only"])
def test_whole_portions_and_decoding(tmp_path, name):
    S.whole_portions_and_decoding(CTX, tmp_path, name)


@pytest.mark.parametrize("name", ["all_kinds", "attention_only"])
def test_mixed_batches_and_reuse(tmp_path, name):
    S.mixed_batches(CTX, tmp_path, name)


@pytest.mark.parametrize("size", [16, 21])
def test_chunk_edges(tmp_path, size):
    S.chunk_edges(CTX, tmp_path, config(64, [(attn(4, 2, 16, 24, size), None)]), size, 3 * size + 2)


@pytest.mark.parametrize("name", ["all_kinds", "attention_only", "memory_only"])
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
def batch(lens, prefix=None):
    from smcsd_b200.models.layers import ExtendBatch
    n = len(lens)
    prefix = prefix or [0] * n
    T = sum(lens)
    return ExtendBatch(torch.zeros(T), torch.zeros(T), torch.zeros(T), torch.arange(n), torch.tensor(prefix), extend_len=0,
                       extend_lens=lens, prefix_lens_host=prefix)


def test_positions_far_away_and_odd_widths():
    from smcsd_b200.models.layers import sinusoidal_positions
    for d in (10, 13):
        assert torch.allclose(sinusoidal_positions(torch.arange(50), d).double(), O.sinusoid(50, d), atol=1e-6)
    p = sinusoidal_positions(torch.tensor([900_001]), 8)[0].double()
    want = [f(900_001 / 10000.0 ** (2 * (c // 2) / 8)) for c, f in enumerate([np.sin, np.cos] * 4)]
    assert np.allclose(p.numpy(), want, atol=1e-6)


def test_token_shift_history():
    from smcsd_b200.models.layers import token_shift
    g = torch.Generator().manual_seed(0)
    h, mu = torch.randn(7, 6, generator=g), torch.randn(2, 6, generator=g)
    back = O.shifted(h.double())
    want = h.double().unsqueeze(1) + (back - h.double()).unsqueeze(1) * mu.double()
    hist = torch.zeros(3, 8, 1)
    hist[0] = 9.0                                            # another sequence's row
    got = [token_shift(h[:1], mu, batch([1]), hist, torch.tensor([2])), token_shift(h[1:3], mu, batch([2]), hist, torch.tensor([2]))]
    both = torch.cat([torch.randn(1, 6, generator=g), h[3:]])
    got.append(token_shift(both, mu, batch([1, 4]), hist, torch.tensor([1, 2]))[1:])
    assert torch.allclose(torch.cat(got).double(), want, atol=1e-6)
    assert torch.equal(hist[2, :6, 0], h[6]) and (hist[0] == 9.0).all()


def test_memories_carry_their_state():
    from smcsd_b200.models.layers import bonus_memory, delta_memory
    g = torch.Generator().manual_seed(1)
    T, H, D = 30, 2, 6
    r, k, v = (torch.randn(T, H, D, generator=g) for _ in range(3))
    w, a, u = torch.rand(T, H, D, generator=g), torch.rand(T, H, D, generator=g), torch.randn(H, D, generator=g)
    dd = lambda *xs: [x.double() for x in xs]
    want_d = torch.stack([O.delta_rule(*dd(r[:, h], w[:, h], k[:, h], v[:, h], a[:, h])) for h in range(H)], 1)
    want_b = torch.stack([O.bonus_memory(*dd(r[:, h], w[:, h], k[:, h], v[:, h], u[h])) for h in range(H)], 1)
    for cuts in ([30], [1, 2, 27], [1] * 30):
        S1, S2, got_d, got_b, t = torch.zeros(H, D, D), torch.zeros(H, D, D), [], [], 0
        for n in cuts:
            s = slice(t, t + n)
            got_d.append(delta_memory(S1, r[s], w[s], k[s], v[s], a[s]))
            got_b.append(bonus_memory(S2, r[s], w[s], k[s], v[s], u))
            t += n
        assert torch.allclose(torch.cat(got_d).double(), want_d, atol=1e-4) and torch.allclose(torch.cat(got_b).double(), want_b, atol=1e-4)


def test_delta_rule_removes_what_a_key_held():
    """No decay and full removal: writing a unit key again replaces its value; the bonus form adds and delays."""
    one = torch.ones(1, 1, 3)
    from smcsd_b200.models.layers import bonus_memory, delta_memory
    k = torch.tensor([[[0.0, 1.0, 0.0]]])
    S1, S2 = torch.zeros(1, 3, 3), torch.zeros(1, 3, 3)
    v1, v2 = torch.tensor([[[1.0, 2.0, 3.0]]]), torch.tensor([[[5.0, 6.0, 7.0]]])
    delta_memory(S1, k, one, k, v1, one)
    assert torch.allclose(delta_memory(S1, k, one, k, v2, one), v2, atol=1e-4)
    bonus_memory(S2, k, one, k, v1, torch.zeros(1, 3))
    assert torch.allclose(bonus_memory(S2, k, one, k, v2, torch.zeros(1, 3)), v1)
    assert torch.allclose(bonus_memory(S2, k, one, k, v2, 2 * torch.ones(1, 3)), v1 + 3 * v2)


def test_chunk_attention_sink_and_bias_by_hand():
    from smcsd_b200.models.layers import chunk_attention_reference
    q, k = torch.full((2, 1, 2), 0.0), torch.zeros(9, 2)
    k[3], k[5] = torch.tensor([1.0, 0.0]), torch.tensor([0.0, 1.0])
    v = torch.zeros(9, 1)
    v[3], v[5] = 2.0, 10.0
    q[1, 0, 0] = 3.0
    bt = torch.tensor([[3, 5]])
    r1, r2 = torch.tensor([0.7]), torch.tensor([4.0])
    out = chunk_attention_reference(q, k, v, bt, batch([2]), 1, 0.5, r1, r2, 2)
    assert abs(out[0, 0, 0] - 2.0 / 2) < 1e-6                                       # one key of score 0 beside the sink
    e0, e1 = np.exp(1.5 - 0.7 * np.log(5.0)), 1.0
    assert abs(out[1, 0, 0] - (2 * e0 + 10 * e1) / (1 + e0 + e1)) < 1e-5
    alone = chunk_attention_reference(q, k, v, bt, batch([2]), 1, 0.5, r1, r2, 1)   # the second token starts a chunk
    assert abs(alone[1, 0, 0] - 10.0 / 2) < 1e-6


# ---------------------------------------------------------------------------------- configuration and loading
def test_configuration_errors_and_counts(tmp_path):
    from smcsd_b200.models import build_model, preset
    from smcsd_b200.models.config import ModelConfig
    c = config(64, [attn(4, 2, 16, 24, 16)])
    for key, bad in (("type", "mamba"), ("mlp", {"kind": "moe", "ff": 3})):
        broken = json.loads(json.dumps(c))
        broken["layers"][0][key] = bad
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(broken)
    with pytest.raises(ValueError, match="one shape"):
        ModelConfig.from_hf_dict(config(64, [attn(4, 2, 16, 24, 16), attn(4, 4, 16, 24, 16)]))
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(config(64, [attn(4, 3, 16, 24, 16)]))
    W = make_weights(c)
    W["l0.mix.v"] = W["l0.mix.v"][:-1]
    from smcsd_b200.models.loader import save_safetensors
    with open(tmp_path / "config.json", "w") as f:
        json.dump(c, f)
    save_safetensors(W, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l0.mix.v"):
        build_model(str(tmp_path), torch.float32)
    assert preset("makodra-2048").param_count() > 5e8
    assert build_model("preset:tiny-makodra", torch.float32).weight_bytes() > 0


def test_pool_layout():
    from smcsd_b200.memory.pools import KVPool, StatePool
    from smcsd_b200.models.makodra import MakodraModel
    from smcsd_b200.models.config import ModelConfig
    m = MakodraModel(ModelConfig.from_hf_dict(CONFIGS["all_kinds"]), torch.float32)
    kv, st = m.kv_spec(torch.bfloat16), m.state_spec()
    assert kv.row_widths == [(2 * 24, 2 * 40), (2 * 72, 2 * 40)] and kv.cell_bytes == 2 * (48 + 80 + 144 + 80)
    pool = StatePool(st, 3, "cpu")
    assert pool.matrix(0).shape == (3, 3, 40, 40) and pool.matrix(1).shape == (3, 5, 24, 24) and pool.conv.shape == (1, 3, 136, 1)
    assert st.row_bytes * 3 == pool.conv.numel() * 4 + pool.temporal.numel() * 4
    pool.matrix(1)[2] = 1.0
    pool.copy_rows(torch.tensor([0]), torch.tensor([2]))
    assert (pool.matrix(1)[0] == 1).all() and (pool.matrix(0) == 0).all()
    pool.clear_rows(torch.tensor([0, 2]))
    assert not pool.temporal.any()
    assert [t.shape[1] for t in KVPool(kv, 4, "cpu").v] == [80, 80]


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
