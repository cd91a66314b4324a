"""The plain restatement of the Bonolorn design against hand-made cases, and the checkpoint writer's layout. No GPU."""
import json
import math

import numpy as np
import torch

from tests import bonolorn_plain as P
from uzu_b200 import safetensors_io as st
from uzu_b200 import synth

F64 = torch.float64


def small_config():
    return P.make_config(40, 53, [
        P.layer(4, 2, 8, 6, 7, 3, 5, 4, [0.5, 0.9, 1.0], P.moe_mlp(12, 6, 2, (3, 2), 1.5, 0.8, shared=18, shared_limit=1.1), left_scale=0.6, right_scale=1.2),
        P.layer(2, 1, 4, 10, 3, 2, 6, 8, [0.99, 0.3], None),
        P.layer(3, 3, 6, 6, 20, 1, 8, 8, [0.7], P.dense_mlp(24)),
    ])


def test_position_vectors_interleave_sine_and_cosine():
    v = P.position_vectors([0, 3], 6)
    assert v[0].tolist() == [0.0, 1.0, 0.0, 1.0, 0.0, 1.0]
    f = 10000.0 ** (-2.0 / 6.0)
    assert torch.allclose(v[1, :4], torch.tensor([math.sin(3.0), math.cos(3.0), math.sin(3 * f), math.cos(3 * f)], dtype=F64))
    assert P.position_vectors([2], 5).shape == (1, 5)


def test_layer_norm_takes_the_mean_off_and_eps_sits_in_the_root():
    y = P.layer_norm(torch.tensor([[1.0, 2.0, 3.0, 6.0]]), torch.tensor([1.0, 1.0, 2.0, 1.0]), 0.5)
    assert torch.allclose(y, torch.tensor([[-2.0, -1.0, 0.0, 3.0]], dtype=F64) / 2.0)        # variance 3.5, plus 0.5


def test_slopes_of_eight_and_of_three_heads():
    assert [P.slope(h, 8) for h in range(8)] == [2.0 ** -(h + 1) for h in range(8)]
    assert abs(P.slope(1, 3) - 2.0 ** (-16.0 / 3.0)) < 1e-15


def test_window_holds_the_position_itself_and_the_ones_before():
    T, size = 8, 3
    k = torch.zeros(T, 1, 2)
    v = torch.eye(T).reshape(T, 1, T)
    o = P.biased_window_attention(torch.zeros(T, 1, 2), k, v, list(range(T)), list(range(T)), 1.0, size)
    for i in range(T):
        assert o[i, 0].nonzero().flatten().tolist() == list(range(max(0, i - size + 1), i + 1))
    s = 2.0 ** -8
    w = [math.exp(-2 * s), math.exp(-s), 1.0]
    assert torch.allclose(o[5, 0, 3:6], torch.tensor(w, dtype=F64) / sum(w))
    assert P.biased_window_attention(torch.zeros(T, 1, 2), k, v, list(range(T)), list(range(T)), 1.0, 0)[7, 0].count_nonzero() == 8


def test_head_gate_is_one_number_per_head_of_the_same_input():
    W = {"q": torch.zeros(2, 1), "k": torch.zeros(1, 1), "v": torch.zeros(1, 1), "q.norm": torch.ones(1), "k.norm": torch.ones(1),
         "g": torch.tensor([[0.0], [1000.0]]), "o": torch.eye(2)}
    mc = {"heads": 2, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 1.0, "mask": {"size": 4}}
    o = P.attention_mixer(torch.ones(1, 1, dtype=F64), W, "", mc, 1e-6, [0], torch.zeros(1, 1, 1), torch.full((1, 1, 1), 6.0))
    assert torch.allclose(o, torch.tensor([[3.0, 6.0]], dtype=F64))


def test_memory_reads_its_own_write_and_decays():
    q, k, v = torch.ones(3, 1, 1), torch.tensor([[[1.0]], [[0.0]], [[2.0]]]), torch.tensor([[[4.0]], [[9.0]], [[1.0]]])
    o, S = P.memory_scan(q, k, v, [0.5], torch.zeros(1, 1, 1))
    assert o[:, 0, 0].tolist() == [4.0, 2.0, 3.0] and float(S) == 3.0
    a, s = P.memory_scan(q[:1], k[:1], v[:1], [0.5], torch.zeros(1, 1, 1))
    b, _ = P.memory_scan(q[1:], k[1:], v[1:], [0.5], s)
    assert torch.equal(torch.cat([a, b]), o)


def test_memory_heads_are_normed_together():
    W = {n: torch.eye(2) for n in "qkv"} | {"g": torch.zeros(2, 2), "o": torch.eye(2), "norm": torch.tensor([1.0, 3.0])}
    x = torch.tensor([[1.0, 2.0]], dtype=F64)
    y, _ = P.memory_mixer(x, W, "", {"heads": 2, "dim": 1, "vdim": 1, "decay": [0.5, 0.5]}, 0.0, torch.zeros(2, 1, 1))
    o = P.silu(x) ** 3                                            # S^T q of a fresh state: q k v, one channel each
    want = o / torch.sqrt((o ** 2).mean()) * torch.tensor([1.0, 3.0]) * 0.5
    assert torch.allclose(y, want)


def test_gelu_and_expert_values():
    assert abs(float(P.gelu_tanh(torch.tensor(1.0, dtype=F64))) - 0.8411919906082768) < 1e-12
    W = {"gate": torch.tensor([[1.0]]), "up": torch.tensor([[-1.0]]), "down": torch.tensor([[2.0]])}
    sig = lambda a: 1 / (1 + math.exp(-a))
    y = P.clamped_expert(torch.tensor([[9.0], [-9.0], [1.0]], dtype=F64), W, "", 2.0)
    want = [2 * sig(3.404) * -1 * 2, -9 * sig(-9 * 1.702) * 3 * 2, sig(1.702) * 0 * 2]       # the gate has no lower bound; u + 1 follows the clamp
    assert torch.allclose(y[:, 0], torch.tensor(want, dtype=F64), atol=1e-12)


def test_choice_goes_by_corrected_scores_in_the_best_groups_and_weights_do_not():
    logit = lambda s: math.log(s / (1 - s))
    z = [logit(s) for s in (0.9, 0.01, 0.6, 0.5, 0.55, 0.5)]
    ro = {"groups": {"count": 3, "keep": 2}, "top": 2, "scale": 2.0}
    got = P.choose_experts(z, [0.0] * 6, ro)
    assert [e for e, _ in got] == [2, 4] and np.allclose([w for _, w in got], [2 * 0.6 / 1.15, 2 * 0.55 / 1.15])
    got = P.choose_experts(z, [-3.0] * 5 + [-2.9], ro)                           # all choice scores negative: group 0 stays out
    assert [e for e, _ in got] == [2, 5] and np.allclose([w for _, w in got], [2 * 0.6 / 1.1, 2 * 0.5 / 1.1])
    assert [e for e, _ in P.choose_experts(z, [0.0] * 6, {"top": 3, "scale": 1.0})] == [0, 2, 4]


def test_portions_equal_the_whole_prompt():
    cfg = small_config()
    w = P.random_weights(cfg, 1)
    toks = [int(x) for x in np.random.default_rng(0).integers(0, 53, 40)]
    whole, runs = P.forward(cfg, w, toks)
    assert runs.shape == (3, 40, 40) and torch.isfinite(whole).all()
    m = P.Model(cfg, w)
    parts = [m.feed(toks[lo:hi]) for lo, hi in ((0, 2), (2, 9), (9, 10), (10, 31), (31, 33), (33, 40))]
    assert (torch.cat(parts) - whole).abs().max() < 1e-10


def test_checkpoint_writer_matches_the_design(tmp_path):
    cfg = synth.bonolorn_config(40, 53, [
        synth.bonolorn_layer(4, 2, 8, 6, 7, 3, 5, 4, synth.bonolorn_moe_mlp(12, 6, 2, (3, 2), 1.5, 0.8, shared=18, shared_limit=1.1), left_scale=0.6, right_scale=1.2),
        synth.bonolorn_layer(2, 1, 4, 10, 3, 2, 6, 8, None),
        synth.bonolorn_layer(3, 3, 6, 6, 20, 1, 8, 8, synth.bonolorn_dense_mlp(24)),
    ])
    path = synth.write_bonolorn_model(cfg, tmp_path / "m", seed=3)
    assert json.loads((path / "config.json").read_text())["architecture"] == "Bonolorn"
    tensors, dtypes, _ = st.load(path / "model.safetensors")
    ref = P.random_weights(small_config(), 0)
    assert set(tensors) == set(ref)
    for name, v in tensors.items():
        assert tuple(v.shape) == tuple(ref[name].shape) and dtypes[name] == "BF16", name
    w = {k: torch.from_numpy(np.asarray(synth.st_bits_to_f32(np.asarray(v))).reshape(v.shape).copy()) for k, v in tensors.items()}
    logits, runs = P.forward(cfg, w, [1, 2, 3, 4, 5])
    assert torch.isfinite(logits).all() and runs.shape == (3, 5, 40)
    preset = synth.bonolorn_preset(256, 100, layers=4)
    assert [L["mlp"]["kind"] for L in preset["layers"]] == ["dense", "moe", "dense", "moe"]
    beside = synth.vugipel_side_by_side_preset(256, 100, layers=4)
    active = lambda ml: ml["ff"] if ml["kind"] == "dense" else ml["router"]["top"] * ml["expert"]["ff"] + ml.get("shared", {"ff": 0})["ff"]
    assert [active(L["mlp"]) for L in preset["layers"]] == [active(L["mlp"]) for L in beside["layers"]]
