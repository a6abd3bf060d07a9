"""Funevik on the CPU path: configuration, loading, mechanisms and the engine around it against the float64 oracle."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import funevik_models as M
import funevik_oracle as O
import layered_suite as S
from funevik_models import CONFIGS, attn, config, dense, latent, make_weights, mem, moe, save_model, tokens
from pasizen_models import row_error
from test_makodra_cpu import batch

CTX = S.Ctx("cpu", "float32", 2e-5, models=M, oracle=O)
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("name", ["all_kinds", "odd_sizes", "memory_only"])
def test_whole_portions_and_decoding(tmp_path, name):
    S.whole_portions_and_decoding(CTX, tmp_path, name)


@pytest.mark.parametrize("name", ["all_kinds", "latent_only"])
def test_mixed_batches_and_reuse(tmp_path, name):
    S.mixed_batches(CTX, tmp_path, name)


@pytest.mark.parametrize("size", [1, 16, 21])
def test_window_holds_exactly_its_tokens(tmp_path, size):
    S.seen_by(CTX, tmp_path, config(64, [(latent(4, 16, 24, 40, 32, 8, size), None)]), 2 * size + 19, (0, 1, 15, 16, size), lambda j: j + size)


@pytest.mark.parametrize("size", [16, 21])
def test_window_ends(tmp_path, size):
    S.window_ends(CTX, tmp_path, config(64, [(latent(4, 16, 24, 40, 32, 8, size), None)]), size)


@pytest.mark.parametrize("name", ["all_kinds", "latent_only", "memory_only"])
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
def test_rotation_near_and_far():
    from smcsd_b200.models.layers import rotate_pairs
    x = torch.randn(40, 3, 10, generator=torch.Generator().manual_seed(0))
    got = rotate_pairs(x, torch.arange(40), 6, 700.0)
    assert torch.allclose(got.double(), O.rotate(x.double(), 700.0, 6), atol=1e-5) and torch.equal(got[..., 6:], x[..., 6:])
    p = 900_001
    far = rotate_pairs(torch.tensor([[1.0, 0.0, 0.0, 1.0]]), torch.tensor([p]), 4, 700.0)[0].double()
    a = [p, p * 700.0 ** -0.5]
    assert np.allclose(far.numpy(), [math.cos(a[0]), math.sin(a[0]), -math.sin(a[1]), math.cos(a[1])], atol=1e-6)


def test_gated_memory_carries_its_state():
    from smcsd_b200.models.layers import gated_memory
    g = torch.Generator().manual_seed(1)
    T, H, D, E = 30, 2, 6, 4
    q, k, v = torch.randn(T, H, D, generator=g), torch.randn(T, H, D, generator=g), torch.randn(T, H, E, generator=g)
    i, f = 4 * torch.randn(T, H, generator=g), -torch.rand(T, H, generator=g)
    want = torch.stack([O.matrix_memory(*(t[:, h].double() for t in (q, k, v, i, f))) for h in range(H)], 1)
    for cuts in ([30], [1, 2, 27], [1] * 30):
        state, top, got, t = torch.zeros(H, E + 1, D), torch.zeros(H, 1, 1), [], 0
        for n in cuts:
            s = slice(t, t + n)
            got.append(gated_memory(state, top, q[s], k[s], v[s], i[s], f[s]))
            t += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-4)


def test_gated_memory_by_hand():
    """The maximum starts at zero: a weak first input is divided by one, not by itself; a strong one by its own read-out."""
    from smcsd_b200.models.layers import gated_memory
    k = torch.tensor([[[0.5, 0.0]]])
    v = torch.tensor([[[2.0]]])
    zero = torch.zeros(1, 1)
    for i, want in ((-3.0, 2.0 * 0.25 * math.exp(-3.0) / (1.0 + 1e-6)), (7.0, 2.0 * 0.25 / (0.25 + 1e-6))):
        top = torch.zeros(1, 1, 1)
        got = gated_memory(torch.zeros(1, 2, 2), top, k, k, v, torch.full((1, 1), i), zero)
        assert abs(got.item() - want) < 1e-5 * want and top.item() == max(i, 0.0)


def test_latent_window_and_sink_by_hand():
    from smcsd_b200.models.layers import latent_attention_reference
    pool = torch.zeros(9, 3)
    pool[3], pool[5], pool[2] = torch.tensor([1.0, 0.0, 4.0]), torch.tensor([0.0, 1.0, 6.0]), torch.tensor([0.0, 0.0, 1.0])
    q = torch.zeros(3, 2, 3)
    q[2, 0, 0], q[2, 1, 1] = 3.0, 2.0
    bt, sink = torch.tensor([[3, 5, 2]]), torch.tensor([0.7, -1.0])
    out = latent_attention_reference(q, pool, bt, batch([3]), 0.5, window=3, sink=sink)
    e = [math.exp(1.5), 1.0, 1.0]
    assert abs(out[2, 0, 2] - (4 * e[0] + 6 + 1) / (sum(e) + math.exp(0.7))) < 1e-5
    e = [1.0, math.exp(1.0), 1.0]
    assert abs(out[2, 1, 2] - (4 + 6 * e[1] + 1) / (sum(e) + math.exp(-1.0))) < 1e-5
    near = latent_attention_reference(q, pool, bt, batch([3]), 0.5, window=2, sink=sink)
    assert abs(near[2, 0, 2] - (6 + 1) / (2 + math.exp(0.7))) < 1e-5
    plain = latent_attention_reference(q, pool, bt, batch([3]), 0.5)
    assert abs(plain[1, 0, 2] - 5.0) < 1e-6


def test_soft_capped_scores_and_sink_by_hand():
    from smcsd_b200.models.layers import chunk_attention_reference
    q, k, v = torch.zeros(2, 1, 2), torch.zeros(9, 2), torch.zeros(9, 1)
    k[3], k[5], v[3], v[5] = torch.tensor([1.0, 0.0]), torch.tensor([0.0, 1.0]), 2.0, 10.0
    q[1, 0, 0] = 30.0
    out = chunk_attention_reference(q, k, v, torch.tensor([[3, 5]]), batch([2]), 1, 0.5, None, None, 0, softcap=4.0)
    e = math.exp(4.0 * math.tanh(15.0 / 4.0))
    assert abs(out[0, 0, 0] - 1.0) < 1e-6 and abs(out[1, 0, 0] - (2 * e + 10) / (1 + e + 1)) < 1e-5


def test_chosen_experts_and_their_weights():
    from smcsd_b200.models.layers import route_top
    idx, w = route_top(torch.tensor([[0.0, 3.0, -1.0, 2.0], [5.0, 5.5, 9.0, -7.0]]), 2)
    assert idx.tolist() == [[1, 3], [2, 1]]
    for row, gap in zip(w, (1.0, 3.5)):
        assert torch.allclose(row, torch.tensor([1.0, math.exp(-gap)]) / (1 + math.exp(-gap)))


def test_convolution_history():
    from smcsd_b200.models.layers import short_conv
    g = torch.Generator().manual_seed(2)
    u, w = torch.randn(9, 4, generator=g), torch.randn(4, 4, generator=g)
    want = O.causal_conv(u.double(), w.double())
    for cuts in ([9], [1] * 9, [2, 1, 6]):
        hist, got, t = torch.zeros(2, 4, 3), [], 0
        for n in cuts:
            got.append(short_conv(u[t:t + n], w, batch([n]), hist, torch.tensor([1])))
            t += n
        assert torch.allclose(torch.cat(got).double(), want, atol=1e-5) and torch.equal(hist[1], u[-3:].t()) and not hist[0].any()


# ---------------------------------------------------------------------------------- configuration and loading
def test_configuration_errors_and_counts(tmp_path):
    from smcsd_b200.models import build_model, preset
    from smcsd_b200.models.config import ModelConfig
    from smcsd_b200.models.loader import save_safetensors
    c = config(64, [(attn(4, 2, 16, 24, 8), None), (latent(2, 16, 16, 24, 24, 8, 9), moe(4, 2, 16, 8)), (mem(2, 16, 24), dense(40))])
    for li, path, bad in ((0, ("type",), "mamba"), (0, ("mixer", "kv_heads"), 3), (0, ("mixer", "rot", "dims"), 18), (0, ("mixer", "rot", "dims"), 7),
                          (1, ("mixer", "rot", "dims"), 6), (1, ("mixer", "mask", "size"), 0), (1, ("mlp", "kind"), "soft"),
                          (1, ("mlp", "router", "top"), 5)):
        broken = json.loads(json.dumps(c))
        at = broken["layers"][li]
        for key in path[:-1]:
            at = at[key]
        at[path[-1]] = bad
        with pytest.raises(ValueError, match=f"layer {li}"):
            ModelConfig.from_hf_dict(broken)
    W = make_weights(c)
    assert ModelConfig.from_hf_dict(c).param_count() == sum(t.numel() for t in W.values())
    W["l1.mix.uq"] = W["l1.mix.uq"][:-1]
    with open(tmp_path / "config.json", "w") as f:
        json.dump(c, f)
    save_safetensors(W, str(tmp_path / "model.safetensors"))
    with pytest.raises(ValueError, match="l1.mix.uq"):
        build_model(str(tmp_path), torch.float32)
    assert preset("funevik-2048").param_count() > 5e8
    assert build_model("preset:tiny-funevik", torch.float32).weight_bytes() > 0


def test_pool_layout():
    from smcsd_b200.memory.pools import KVPool, StatePool
    from smcsd_b200.models.config import ModelConfig
    from smcsd_b200.models.funevik import FunevikModel
    m = FunevikModel(ModelConfig.from_hf_dict(CONFIGS["all_kinds"]), torch.float32)
    kv, st = m.kv_spec(torch.bfloat16), m.state_spec()
    assert kv.row_widths == [(64, 0), (2 * 40, 2 * 24)] and kv.cell_bytes == 2 * (64 + 80 + 48)
    pool = StatePool(st, 3, "cpu")
    assert [tuple(pool.matrix(i).shape[1:]) for i in range(5)] == [(3, 25, 40), (3, 1, 1), (1, 2, 6 * 40 + 2 * 24), (5, 57, 24), (5, 1, 1)]
    pool.matrix(3)[2] = 1.0
    pool.copy_rows(torch.tensor([0]), torch.tensor([2]))
    assert (pool.matrix(3)[0] == 1).all() and not pool.matrix(2).any()
    pool.clear_rows(torch.tensor([0, 2]))
    assert not pool.temporal.any()
    assert [t.shape[1] for t in KVPool(kv, 4, "cpu").v] == [0, 48]
    assert FunevikModel(ModelConfig.from_hf_dict(CONFIGS["latent_only"]), torch.float32).state_spec() is None


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
