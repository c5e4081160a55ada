"""Sipelorn without a GPU: reading config.json, the plan it turns into, which tensors each layer declares, the caches its
mixers ask for, and the plain implementation against its own reading token by token and by hand."""

import copy
import json
import math
import os

import numpy as np
import pytest
import torch

import plain_sipelorn as plain
from sipelorn_configs import S_A, S_B, S_C, SIPELORN

from dynalm_b200.errors import InvalidArgument, NotFound, Unsupported
from dynalm_b200.parts import CONNECTIONS, FEED_FORWARDS, MIXERS
from dynalm_b200.registry import find_architecture
from dynalm_b200.weights import write_model_folder
from dynalm_b200.weights.loader import WeightMismatch, expected_tensors, open_model_folder


def _plan(cfg, present=None):
    arch = find_architecture(cfg)
    return arch.read_config(cfg), arch.plan(arch.read_config(cfg), present)


def test_config_reads_every_size_per_layer():
    cfg, plan = _plan(S_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale, cfg.side_dim) == (310, 96, 1e-5, 3.0, 16)
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (83, 1009, 31)
    assert [l.type for l in cfg.layers] == ["attention", "attention", "latent_attention", "attention", "latent_attention"]
    a = cfg.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.taps, a.window, a.kv_from) == (8, 2, 32, 16, 1.3, 4, 21, None)
    assert cfg.layers[1].mixer.kv_from == 0 and cfg.layers[1].mlp.ff == 72
    l = cfg.layers[2].mixer
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.kv_rank, l.scale, l.rot_dims, l.rot_base) == (3, 16, 16, 24, 40, 0.8, 16, 900.0)
    assert (l.stretch.factor, l.stretch.original, l.stretch.fast, l.stretch.slow) == (6.0, 128, 16.0, 1.0)
    f = cfg.layers[0].mlp
    assert (f.ff, f.experts, f.top, f.groups, f.keep_groups, f.shared_ff) == (40, 6, 2, 3, 2, 56)
    assert cfg.layers[3].mlp is None
    m = plan.layers[0].mixer
    assert (m.kind, m.conv, m.window, m.distance_bias, m.own_kv, m.gated, m.position) == ("gated_attention", 4, 21, "log", True, True, None)
    assert set(m.tensors) == {"q", "k", "v", "o", "q_bias", "k_bias", "v_bias", "q_conv", "k_conv", "v_conv", "gate",
                              "distance_rate", "distance_step"}
    r = plan.layers[1].mixer
    assert not r.own_kv and set(r.tensors) == {"q", "o", "q_bias", "q_conv", "gate", "distance_rate", "distance_step"}
    assert [(run.layer, run.cache_of) for run in plan.order] == [(0, None), (1, 0), (2, None), (3, None), (4, None)]
    e = plan.layers[0].ffn
    assert (e.scores, e.group_score, e.renormalize, e.corrected, e.activation, e.shared_inner) == ("sigmoid", "top2", False, True, "swiglu", 56)
    assert plan.layers[1].ffn.kind == "mlp" and plan.layers[1].ffn.activation == "xielu"
    assert "ffn" not in plan.layers[3].parts and "ffn_gate" not in plan.layers[3].parts and {"l3.norm2", "l3.rg2.b"} <= set(plan.ignorable)
    assert [b.side.index for b in plan.layers] == [0, 1, 2, 3, 4]
    assert plan.layers[0].mixer_gate.tensors == {"weight": "l0.rg1", "bias": "l0.rg1.b"}
    assert not plan.head.tied and plan.embedding.pair_rows == 83


def test_a_cache_reaches_as_far_back_as_its_widest_reader():
    _, plan = _plan(S_A)
    assert (plan.layers[0].mixer.window, plan.layers[0].mixer.cache_window) == (21, 37)
    assert (plan.layers[3].mixer.window, plan.layers[3].mixer.cache_window) == (16, 16)
    _, plan = _plan(S_C)
    assert (plan.layers[1].mixer.window, plan.layers[1].mixer.cache_window) == (160, 0), "one reader sees every key"
    _, plan = _plan(S_B)
    assert (plan.layers[2].mixer.window, plan.layers[2].mixer.cache_window) == (0, 0)


def test_keys_left_out_switch_a_mechanism_off():
    cfg, plan = _plan(S_B)
    assert (cfg.embedding_scale, cfg.bigram, cfg.side_dim) == (1.0, None, 0)
    assert plan.embedding.pair_rows == 0 and "side" not in plan.layers[0].parts
    assert plan.layers[0].mixer.conv == 0 and "q_conv" not in plan.layers[0].mixer.tensors
    assert plan.layers[0].ffn.groups == 1 and plan.layers[0].ffn.shared_inner == 0
    assert plan.layers[3].mixer.position is None


def test_the_stretch_keeps_divides_and_ramps():
    cfg, plan = _plan(S_A)
    pos = plan.layers[2].mixer.position
    f, mag = plain.yarn(900.0, 16, {"factor": 6.0, "original": 128, "fast": 16.0, "slow": 1.0})
    base, one = plain.yarn(900.0, 16, None)
    assert np.allclose(base / np.array(pos.factors), f, rtol=1e-12) and one == 1.0
    assert pos.magnitude == mag == 0.1 * math.log(6.0) + 1.0
    assert pos.factors[0] == 1.0 and np.isclose(pos.factors[-1], 6.0) and any(1.01 < x < 5.9 for x in pos.factors)
    assert plan.layers[4].mixer.position.factors is None and plan.layers[4].mixer.position.magnitude == 1.0
    # a range that lies wholly in front of the first pair: every frequency is divided
    f, _ = plain.yarn(10000.0, 8, {"factor": 2.0, "original": 4, "fast": 32.0, "slow": 1.0})
    assert np.allclose(f, plain.yarn(10000.0, 8, None)[0] / np.array([1.0, 2.0, 2.0, 2.0]))


def test_refusals():
    def broken(change):
        cfg = copy.deepcopy(S_A)
        change(cfg)
        return cfg
    with pytest.raises(Unsupported):
        _plan(broken(lambda c: c["layers"][0].update(type="conv")))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3)))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][1]["mixer"].update(kv_from=2)))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][1]["mixer"].update(kv_from=1)))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][1]["mixer"].update(vdim=20)))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=15)))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][0]["mlp"]["router"].update(experts=7)))
    with pytest.raises(InvalidArgument):
        _plan(broken(lambda c: c["layers"][2]["mlp"]["router"].update(top=5)))
    with pytest.raises(Unsupported):
        _plan(broken(lambda c: c["layers"][0]["mlp"].update(kind="gated")))
    with pytest.raises(NotFound):
        _plan(broken(lambda c: c["layers"][0]["mlp"].pop("router")))
    with pytest.raises(NotFound):
        _plan(broken(lambda c: c.pop("layers")))


def test_declared_tensors_and_the_loaders_one_error(tmp_path):
    _, plan = _plan(S_A)
    want = expected_tensors(plan)
    assert want["bigram"].shape == (84, 96) and want["side.embed"].shape == (310, 80) and want["head"].shape == (310, 96)
    assert want["l0.mix.k"].shape == (64, 96) and want["l0.mix.v.conv"].shape == (32, 4) and want["l0.mix.q.b"].shape == (256,)
    assert want["l0.mix.g"].shape == (128, 96) and want["l0.mix.r1"].shape == (8,)
    assert "l1.mix.k" not in want and "l1.mix.v.conv" not in want and want["l1.mix.q.conv"].shape == (128, 4)
    assert want["l2.mix.q"].shape == (96, 96) and want["l2.mix.dkv"].shape == (56, 96) and want["l2.mix.uv"].shape == (72, 40)
    assert want["l1.mlp.act"].shape == (2,) and want["l0.mlp.correction"].shape == (6,) and want["l0.mlp.shared.sg"].shape == (1, 96)
    assert want["l0.mlp.e5.gate"].shape == (40, 96) and want["l0.rg2"].shape == (96, 96) and "l3.rg2" not in want
    assert want["l4.side.proj"].shape == (96, 16)
    write_model_folder(str(tmp_path), S_A, 1, dtype=torch.float32)
    bad = copy.deepcopy(S_A)
    bad["layers"][0]["mixer"]["conv"] = 3
    bad["layers"][2]["mlp"]["router"].update(experts=10)
    with open(os.path.join(str(tmp_path), "config.json"), "w") as f:
        json.dump(bad, f)
    with pytest.raises(WeightMismatch) as e:
        open_model_folder(str(tmp_path))
    assert "l2.mlp.e9.gate" in e.value.missing and any(n == "l0.mix.k.conv" for n, _, _ in e.value.wrong_shape)


def test_layers_of_one_structure_compare_equal_whatever_their_piece_of_a_shared_table():
    cfg = copy.deepcopy(S_A)
    cfg["layers"] = [copy.deepcopy(cfg["layers"][0]) for _ in range(3)]
    _, plan = _plan(cfg)
    assert plan.layers[0] == plan.layers[1] == plan.layers[2] and plan.layers[2].side.index == 2


def test_registries_hold_the_new_kinds():
    assert "gated_attention" in MIXERS.kinds() and {"routed_mlp", "token_side"} <= set(FEED_FORWARDS.kinds())
    assert "sigmoid_gate" in CONNECTIONS.kinds()


@pytest.mark.parametrize("name", sorted(SIPELORN))
def test_plain_whole_equals_plain_token_by_token(name, tmp_path):
    cfg, seed = SIPELORN[name]
    write_model_folder(str(tmp_path), cfg, seed, dtype=torch.float32)
    model = plain.PlainSipelorn(str(tmp_path))
    toks = [int(t) for t in np.random.RandomState(3).randint(0, cfg["vocab"], 75)]
    whole = model.logits(toks)
    assert np.abs(model.logits_stepwise(toks) - whole).max() < 1e-10
    assert np.abs(model.logits(toks, cuts=[2, 31, 3, 20]) - whole).max() < 1e-10


def test_plain_mechanisms_by_hand():
    # the mask: a window of 3
    assert [[j for j in range(6) if plain.visible(i, j, 3)] for i in (0, 2, 5)] == [[0], [0, 1, 2], [3, 4, 5]]
    # the distance bias: two keys of equal score, one three tokens back: weights 1 : (1 + 2 * 3)^-1.5
    q, k = np.zeros((1, 1, 4)), np.ones((4, 1, 4))
    v = np.array([1.0, 0.0, 0.0, 0.0]).reshape(4, 1, 1)
    w = (1 + 2.0 * np.arange(3, -1, -1)) ** -1.5
    assert np.allclose(plain.attend(q, k, v, [3], range(4), 1.0, 0, [1.5], [2.0]), w[0] / w.sum())
    # convolution: the last tap is the current token's, zeros in front of the start, the last inputs are kept
    y, kept = plain.convolve(np.array([[1.0], [2.0], [3.0]]), np.array([[10.0, 1.0, 0.5]]), np.zeros((2, 1)))
    assert np.allclose(y.ravel(), [0.5, 2.0, 13.5]) and np.allclose(kept.ravel(), [2.0, 3.0])
    # pairs of tokens: the last row for a first token, then (prev * 5 + cur * 2) mod 7
    table = {"buckets": 7, "mul_prev": 5, "mul_cur": 2}
    assert plain.bigram_rows([3, 4, 1], None, table) == [7, (15 + 8) % 7, (20 + 2) % 7]
    assert plain.bigram_rows([4], 3, table) == [(15 + 8) % 7]
    # xIELU: continuous at zero, and by its definition on both sides
    assert plain.xielu(0.0, 1.0, 2.0) == 0.0
    assert np.isclose(plain.xielu(2.0, 0.3, 9.0), math.log(1 + math.exp(0.3)) * 4.0 + 1.0)
    assert np.isclose(plain.xielu(-2.0, 9.0, 0.3), (0.5 + math.log(1 + math.exp(0.3))) * (math.exp(-2.0) + 1.0) - 1.0)
    # routing: a group wins by the sum of its two best; the weights are the scores without the correction, as they are
    z = np.array([9.0, -9.0, 1.0, 1.0])
    chosen, w = plain.route(z, np.zeros(4), 1, 2, 1)
    assert chosen == [2] and np.isclose(w[0], plain.sigmoid(1.0)), "the best expert's group loses"
    chosen, w = plain.route(np.zeros(4), np.array([-3.0, -2.0, -4.0, -0.5]), 2, 2, 1)
    assert chosen == [3, 2] and np.allclose(w, 0.5), "negative choice scores of a kept group beat none of the others"
    # rotation with a factor: a quarter turn of (1, 0), twice as long
    assert np.allclose(plain.rotate_pairs(np.array([[1.0, 0.0, 5.0]]), [1], np.array([np.pi / 2]), 2.0), [[0.0, 2.0, 5.0]])
