"""The plain restatement of the Relidra design against hand-made cases, and the checkpoint writer's layout. No GPU."""
import math

import numpy as np
import torch

from tests import relidra_plain as P
from uzu_b200 import safetensors_io as st
from uzu_b200 import synth

F64 = torch.float64


def small_config():
    return P.make_config(40, 53, [
        P.delta_layer(4, 2, 6, 5, 4),
        P.attention_layer(4, 2, 8, 7, 24, rot_dims=6),
        P.delta_layer(2, 2, 5, 9, 2, 20),
    ], streams=3, loop=(1, 3, 2))


def test_layer_norm_takes_the_mean_off_and_eps_sits_in_the_root():
    y = P.layer_norm(torch.tensor([[1.0, 2.0, 3.0, 6.0]]), torch.tensor([1.0, 1.0, 2.0, 1.0]), 0.5)
    assert torch.allclose(y, torch.tensor([[-2.0, -1.0, 0.0, 3.0]], dtype=F64) / 2.0)        # variance 3.5, plus 0.5
    assert torch.allclose(P.layer_norm(torch.tensor([[5.0, 5.0]]), torch.ones(2), 1e-3), torch.zeros(1, 2, dtype=F64))


def test_exact_gelu_values():
    z = torch.tensor([0.0, 1.0, -1.0, 2.0], dtype=F64)
    assert torch.allclose(P.gelu_exact(z), torch.tensor([0.0, 0.8413447460685429, -0.15865525393145707, 1.9544997361036416], dtype=F64), atol=1e-12)


def test_streams_are_mixed_from_the_old_copies_with_from_to_indices():
    X = torch.tensor([[[1.0]], [[10.0]]])
    mix = torch.tensor([[1.0, 2.0], [3.0, 4.0]])            # mix[from, to]
    out = P.streams_write(X, torch.tensor([[100.0]]), mix, torch.tensor([0.5, -1.0]))
    assert out[:, 0, 0].tolist() == [1 * 1 + 3 * 10 + 50, 2 * 1 + 4 * 10 - 100]
    assert float(P.streams_read(X, torch.tensor([0.5, 0.25]))) == 3.0


def test_rotation_frequencies_are_divided_by_the_factor_and_pairs_are_halves():
    rot = {"base": 100.0, "dims": 4, "scaling": {"factor": 3.0}}
    assert np.allclose(P.rot_frequencies(rot), [1.0 / 3.0, 0.1 / 3.0])
    x = torch.zeros(2, 1, 6, dtype=F64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 7.0
    y = P.rotate_halves(x, [0, 3], rot)
    assert torch.allclose(y[0], x[0])
    assert abs(float(y[1, 0, 0]) - math.cos(1.0)) < 1e-12 and abs(float(y[1, 0, 2]) - math.sin(1.0)) < 1e-12
    assert float(y[1, 0, 1]) == 0.0 and float(y[1, 0, 5]) == 7.0


def test_chunks_count_from_position_zero():
    seen = P.chunk_mask([4, 5, 9], list(range(10)), 5)
    assert seen[0].nonzero().flatten().tolist() == [0, 1, 2, 3, 4]
    assert seen[1].nonzero().flatten().tolist() == [5]
    assert seen[2].nonzero().flatten().tolist() == [5, 6, 7, 8, 9]
    assert bool(P.chunk_mask([9], [0], 0)[0, 0])


def test_sink_takes_weight_but_has_no_value():
    q, k, v = torch.ones(1, 1, 2), torch.zeros(1, 1, 2), torch.tensor([[[4.0, 8.0]]])
    seen = torch.ones(1, 1, dtype=torch.bool)
    o = P.sink_attention(q, k, v, seen, 10.0, torch.tensor([math.log(3.0)]))
    assert torch.allclose(o, torch.tensor([[[1.0, 2.0]]], dtype=F64), atol=1e-6)                  # weight 1 / (1 + 3); not scaled by 10
    assert torch.allclose(P.sink_attention(q, k, v, seen, 10.0, None), v.to(F64))


def test_values_are_the_biased_keys_before_norm_and_rotation():
    W = {"m.mix.q": torch.eye(4), "m.mix.k": torch.eye(4), "m.mix.q.b": torch.zeros(4), "m.mix.k.b": torch.tensor([0.0, 0.0, 0.0, 2.0]),
         "m.mix.sink": torch.tensor([-50.0]), "m.mix.o": torch.eye(4)}
    mc = {"heads": 1, "kv_heads": 1, "dim": 4, "vdim": 4, "scale": 1.0, "mask": {"size": 9}, "rot": {"base": 10.0, "dims": 4, "scaling": {"factor": 1.0}}}
    o, _ = P.attention_mixer(torch.tensor([[3.0, 0.0, 0.0, 1.0]]), W, "m.", mc, 1e-6, [5])
    assert torch.allclose(o, torch.tensor([[3.0, 0.0, 0.0, 3.0]], dtype=F64), atol=1e-9)


def test_short_convolution_last_tap_is_the_current_token():
    x = torch.tensor([[1.0], [2.0], [4.0]])
    y, tail = P.short_conv(x, torch.tensor([[100.0, 10.0, 1.0]]), torch.tensor([[0.0], [7.0]]))
    assert y[:, 0].tolist() == [71.0, 712.0, 124.0]
    assert tail[:, 0].tolist() == [2.0, 4.0]
    y, tail = P.short_conv(x, torch.tensor([[3.0]]), torch.zeros(0, 1))
    assert y[:, 0].tolist() == [3.0, 6.0, 12.0] and tail.shape == (0, 1)


def test_delta_rule_replaces_what_a_key_holds_and_reads_its_own_write():
    k = torch.tensor([[[1.0, 0.0]], [[1.0, 0.0]], [[0.0, 1.0]]], dtype=F64)
    v = torch.tensor([[[5.0]], [[3.0]], [[2.0]]], dtype=F64)
    one = torch.ones(3, 1, dtype=F64)
    o, S = P.delta_scan(k, k, v, one, one, torch.zeros(1, 2, 1))
    assert o[:, 0, 0].tolist() == [5.0, 3.0, 2.0]                 # the second write replaced the first, each read sees its own write
    assert S[0, :, 0].tolist() == [3.0, 2.0]
    half = 0.5 * one
    o, S = P.delta_scan(k, k, v, half, half, torch.zeros(1, 2, 1))
    # S = 2.5; decayed to 1.25, + 0.5 (3 - 1.25) = 2.125; decayed to 1.0625, the other key takes 0.5 * 2
    assert o[:, 0, 0].tolist() == [2.5, 2.125, 1.0] and S[0, :, 0].tolist() == [1.0625, 1.0]


def test_decay_and_unit_vectors():
    g = P.delta_decay(torch.tensor([0.0, math.log(2.0)]), torch.tensor([1.0, 0.0]), torch.tensor([[-1.0, 0.0]]))
    assert torch.allclose(g, torch.tensor([[0.5, 0.25]], dtype=F64), atol=1e-7)
    assert torch.allclose(P.unit_l2(torch.tensor([3.0, 4.0])), torch.tensor([0.6, 0.8], dtype=F64), atol=1e-6)
    assert P.unit_l2(torch.zeros(4)).abs().max() == 0


def test_looped_layers_run_as_a_block_with_states_of_their_own():
    cfg = small_config()
    assert P.run_order(cfg) == [0, 1, 2, 1, 2]
    cfg["loop"] = {"start": 0, "stop": 1, "times": 3}
    assert P.run_order(cfg) == [0, 0, 0, 1, 2]
    cfg["loop"] = None
    assert P.run_order(cfg) == [0, 1, 2]


def test_portions_equal_the_whole_prompt():
    cfg = small_config()
    w = P.random_weights(cfg, 1)
    toks = [int(x) for x in np.random.default_rng(0).integers(0, 53, 40)]
    whole, runs = P.forward(cfg, w, toks)
    assert runs.shape == (5, 40, 40) and torch.isfinite(whole).all()
    m = P.Model(cfg, w)
    parts = [m.feed(toks[lo:hi]) for lo, hi in ((0, 2), (2, 9), (9, 10), (10, 31), (31, 33), (33, 40))]
    assert (torch.cat(parts) - whole).abs().max() < 1e-11


def test_checkpoint_writer_matches_the_design(tmp_path):
    cfg = synth.relidra_config(40, 53, [
        synth.relidra_delta_layer(4, 2, 6, 5, 4, None),
        synth.relidra_attention_layer(4, 2, 8, 7, synth.relidra_dense_mlp(24), rot_dims=6),
        synth.relidra_delta_layer(2, 2, 5, 9, 2, synth.relidra_dense_mlp(20)),
    ], streams=3, loop={"start": 1, "stop": 3, "times": 2})
    path = synth.write_relidra_model(cfg, tmp_path / "m", seed=3)
    tensors, dtypes, _ = st.load(path / "model.safetensors")
    ref = P.random_weights(small_config(), 0)
    assert set(tensors) == set(ref)
    for name, v in tensors.items():
        assert tuple(v.shape) == tuple(ref[name].shape) and dtypes[name] == "BF16", name
    w = {k: torch.from_numpy(np.asarray(synth.st_bits_to_f32(np.asarray(v))).reshape(v.shape).copy()) for k, v in tensors.items()}
    logits, runs = P.forward(cfg, w, [1, 2, 3, 4, 5])
    assert torch.isfinite(logits).all() and runs.shape == (5, 5, 40)
