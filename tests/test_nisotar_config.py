"""Nisotar without a GPU: reading config.json, the plan it turns into, which tensors each layer declares, and the plain
implementation against its own reading token by token and by hand."""

import copy
import json
import math
import os

import numpy as np
import pytest
import torch

import plain_nisotar as plain
from nisotar_configs import N_A, N_B, N_C, NISOTAR

from dynalm_b200.errors import InvalidArgument, NotFound, Unsupported
from dynalm_b200.parts import FEED_FORWARDS, MIXERS, POSITIONS
from dynalm_b200.registry import find_architecture
from dynalm_b200.weights import write_model_folder
from dynalm_b200.weights.loader import WeightMismatch, expected_tensors, open_model_folder


def _plan(cfg, present=None):
    arch = find_architecture(cfg)
    return arch.read_config(cfg), arch.plan(arch.read_config(cfg), present)


def test_config_reads_every_size_per_layer():
    cfg, plan = _plan(N_A)
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.embedding_scale) == (301, 104, 1e-5, 2.5)
    assert [l.type for l in cfg.layers] == ["parallel", "attention", "latent_attention", "parallel", "attention"]
    left, right = cfg.layers[0].mixer.left, cfg.layers[0].mixer.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale, left.size) == (4, 2, 32, 32, 0.7, 37)
    assert (left.rot.dims, left.rot.base, left.rot.stretch) == (32, 3000.0, None)
    assert (right.heads, right.kv_heads, right.dim, right.vdim, right.taps, right.decay_rank, right.gate_rank) == (4, 1, 24, 16, 3, 16, 8)
    assert (cfg.layers[0].mlp.ff, cfg.layers[0].mlp.limit) == (88, 0.9)
    a = cfg.layers[1].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.size, a.rot.dims) == (6, 3, 48, 32, 0.6, 21, 24)
    assert (a.rot.stretch.factor, a.rot.stretch.original, a.rot.stretch.fast, a.rot.stretch.slow) == (6.0, 128, 16.0, 1.0)
    l = cfg.layers[2].mixer
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.kv_rank, l.scale, l.window, l.rot.dims) == (3, 16, 16, 24, 40, 1.2, 29, 16)
    assert (cfg.layers[1].mlp.ff, cfg.layers[1].mlp.experts, cfg.layers[1].mlp.top) == (40, 6, 3) and cfg.layers[3].mlp is None


def test_the_plan_of_every_mixer():
    _, plan = _plan(N_A)
    p = plan.layers[0].mixer
    assert p.kind == "side_by_side" and (p.left_scale, p.right_scale, p.normed, p.eps) == (0.5, 0.5, True, 1e-5)
    assert (p.left.kind, p.left.window, p.left.chunk, p.left.values, p.left.sink, p.left.qk_norm) == \
        ("gated_attention", 0, 37, "keys", "zero", "head_first")
    assert (p.right.kind, p.right.decay, p.right.gate, p.right.decay_rank, p.right.gate_rank) == ("gated_delta", "channel", "sigmoid", 16, 8)
    assert "left.v" not in p.tensors and p.tensors["right.decay_out"] == "l0.mix.right.a2" and p.tensors["left_norm"] == "l0.mix.left.out"
    a = plan.layers[1].mixer
    assert (a.window, a.chunk, a.values, a.sink, a.position.kind) == (21, 0, "own", "zero", "rotary_halves")
    l = plan.layers[2].mixer
    assert (l.kind, l.q_rank, l.window, l.position.kind, l.position.factors) == ("latent_attention", 0, 29, "rotary_halves", None)
    f, e = plan.layers[0].ffn, plan.layers[1].ffn
    assert (f.kind, f.activation, f.limit, f.gate_scale) == ("gated_mlp", "clamped_swiglu", 0.9, 1.702)
    assert (e.kind, e.scores, e.renormalize, e.biased, e.activation, e.groups) == ("routed_mlp", "softmax", True, True, "swiglu", 1)
    assert "ffn" not in plan.layers[3].parts and "l3.norm2" in plan.ignorable
    assert plan.layers[0].mixer_norm.kind == "layer" and set(plan.layers[0].mixer_norm.tensors) == {"weight"}
    assert not plan.head.tied and [b.kind for b in plan.layers] == ["pre_norm"] * 5


def test_keys_left_out_switch_a_mechanism_off():
    cfg, plan = _plan(N_B)
    assert cfg.embedding_scale == 1.0
    assert plan.layers[0].mixer.window == 0 and plan.layers[3].mixer.left.chunk == 0 and plan.layers[3].mixer.left.position is None
    assert plan.layers[4].mixer.position is None and plan.layers[4].mixer.window == 0


def test_the_inner_sizes_come_from_the_tensors_shapes():
    cfg = copy.deepcopy(N_A)
    for i in (0, 3):
        del cfg["layers"][i]["mixer"]["right"]["decay_rank"], cfg["layers"][i]["mixer"]["right"]["gate_rank"]
    shapes = {f"l{i}.mix.right.{n}": (r, 104) for i, a, g in ((0, 11, 3), (3, 2, 9)) for n, r in (("a1", a), ("g1", g))}
    _, plan = _plan(cfg, shapes)
    assert [(plan.layers[i].mixer.right.decay_rank, plan.layers[i].mixer.right.gate_rank) for i in (0, 3)] == [(11, 3), (2, 9)]
    with pytest.raises(NotFound):
        _plan(cfg)


def test_the_stretch_keeps_divides_and_ramps():
    _, plan = _plan(N_A)
    pos = plan.layers[1].mixer.position
    f, mag = plain.yarn(900.0, 24, {"factor": 6.0, "original": 128, "fast": 16.0, "slow": 1.0})
    base, one = plain.yarn(900.0, 24, None)
    assert np.allclose(base / np.array(pos.factors), f, rtol=1e-12) and one == 1.0
    assert pos.magnitude == mag == 0.1 * math.log(6.0) + 1.0
    assert pos.factors[0] == 1.0 and np.isclose(pos.factors[-1], 6.0) and any(1.01 < x < 5.9 for x in pos.factors)
    part = POSITIONS.get("rotary_halves")(pos, type("R", (), {"device": "cpu"}))
    assert np.allclose(part.frequencies.numpy(), f, rtol=1e-12)


def test_an_order_of_neighbours_turns_halves_into_pairs():
    """Rows reordered by `neighbours`, pairs (2i, 2i + 1) turned: the same vector as halves turned, reordered."""
    _, plan = _plan(N_A)
    part = POSITIONS.get("rotary_halves")(plan.layers[2].mixer.position, type("R", (), {"device": "cpu"}))
    order = part.neighbours(20).numpy()
    assert sorted(order) == list(range(20)) and list(order[:4]) == [0, 8, 1, 9] and list(order[16:]) == [16, 17, 18, 19]
    x, freq = np.random.RandomState(0).randn(3, 20), part.frequencies.numpy()
    want = plain.rotate_halves(x, [0, 5, 900], freq)[:, order]
    y = x[:, order].copy()
    for t, p in enumerate([0, 5, 900]):
        for i, f in enumerate(freq):
            u, v = y[t, 2 * i], y[t, 2 * i + 1]
            y[t, 2 * i], y[t, 2 * i + 1] = u * np.cos(p * f) - v * np.sin(p * f), v * np.cos(p * f) + u * np.sin(p * f)
    assert np.allclose(y, want, atol=1e-12)


def test_refusals():
    def broken(change):
        cfg = copy.deepcopy(N_A)
        change(cfg["layers"])
        return cfg
    for error, change in (
            (Unsupported, lambda ls: ls[0].update(type="conv")),
            (InvalidArgument, lambda ls: ls[1]["mixer"].update(kv_heads=4)),
            (InvalidArgument, lambda ls: ls[0]["mixer"]["right"].update(kv_heads=3)),
            (InvalidArgument, lambda ls: ls[0]["mixer"]["left"].update(vdim=16)),
            (InvalidArgument, lambda ls: ls[1]["mixer"]["rot"].update(dims=23)),
            (InvalidArgument, lambda ls: ls[2]["mixer"]["rot"].update(dims=18)),
            (InvalidArgument, lambda ls: ls[1]["mixer"]["mask"].update(size=0)),
            (InvalidArgument, lambda ls: ls[1]["mlp"]["router"].update(top=7)),
            (InvalidArgument, lambda ls: ls[0]["mlp"].pop("limit")),
            (Unsupported, lambda ls: ls[0]["mlp"].update(kind="gated")),
            (NotFound, lambda ls: ls[1]["mlp"].pop("router")),
            (NotFound, lambda ls: ls[0]["mixer"].pop("right")),
            (NotFound, lambda ls: ls[1].pop("mixer"))):
        with pytest.raises(error):
            _plan(broken(change))


def test_declared_tensors_and_the_loaders_one_error(tmp_path):
    _, plan = _plan(N_A)
    want = {n: d.shape for n, d in expected_tensors(plan).items()}
    assert want["l0.mix.left.q"] == (128, 104) and want["l0.mix.left.k"] == (64, 104) and "l0.mix.left.v" not in want
    assert want["l0.mix.left.q.norm"] == want["l0.mix.left.k.norm"] == (32,) and want["l0.mix.left.out"] == (104,)
    assert want["l0.mix.right.q"] == (24, 104) and want["l0.mix.right.v.conv"] == (64, 3) and want["l0.mix.right.A_log"] == (4,)
    assert want["l0.mix.right.a1"] == (16, 104) and want["l0.mix.right.a2"] == (96, 16) and want["l0.mix.right.dt_bias"] == (96,)
    assert want["l0.mix.right.g1"] == (8, 104) and want["l0.mix.right.g2"] == (64, 8) and want["l0.mix.right.norm"] == (16,)
    assert want["l0.mlp.gate.b"] == (88,) and want["l0.mlp.down.b"] == (104,) and want["l1.mlp.router.b"] == (6,)
    assert want["l1.mix.v"] == (96, 104) and want["l1.mix.o"] == (104, 192) and want["l2.mix.dkv"] == (56, 104)
    assert "l0.norm1.b" not in want and "l3.norm2" not in want and want["head"] == (301, 104)
    write_model_folder(str(tmp_path), N_A, 1, dtype=torch.float32)
    bad = copy.deepcopy(N_A)
    bad["layers"][0]["mixer"]["right"]["conv"] = 4
    bad["layers"][2]["mlp"]["router"].update(experts=9)
    with open(os.path.join(str(tmp_path), "config.json"), "w") as f:
        json.dump(bad, f)
    with pytest.raises(WeightMismatch) as e:
        open_model_folder(str(tmp_path))
    assert "l2.mlp.e8.gate" in e.value.missing and any(n == "l0.mix.right.k.conv" for n, _, _ in e.value.wrong_shape)


def test_layers_of_one_structure_compare_equal():
    cfg = copy.deepcopy(N_C)
    cfg["layers"] = [copy.deepcopy(cfg["layers"][i]) for i in (1, 1, 3)]
    _, plan = _plan(cfg)
    assert plan.layers[0] == plan.layers[1] != plan.layers[2]


def test_registries_hold_the_new_kinds():
    assert {"gated_attention", "gated_delta", "side_by_side"} <= set(MIXERS.kinds())
    assert {"routed_mlp", "gated_mlp"} <= set(FEED_FORWARDS.kinds()) and "rotary_halves" in POSITIONS.kinds()


@pytest.mark.parametrize("name", sorted(NISOTAR))
def test_plain_whole_equals_plain_token_by_token(name, tmp_path):
    cfg, seed = NISOTAR[name]
    write_model_folder(str(tmp_path), cfg, seed, dtype=torch.float32)
    model = plain.PlainNisotar(str(tmp_path))
    toks = [int(t) for t in np.random.RandomState(3).randint(0, cfg["vocab"], 75)]
    whole = model.logits(toks)
    assert np.abs(model.logits_stepwise(toks) - whole).max() < 1e-10
    assert np.abs(model.logits(toks, cuts=[2, 31, 3, 20]) - whole).max() < 1e-10


def test_plain_mechanisms_by_hand():
    # masks: a window of 3, chunks of 3
    assert [[j for j in range(6) if plain.visible(i, j, window=3)] for i in (0, 2, 5)] == [[0], [0, 1, 2], [3, 4, 5]]
    assert [[j for j in range(8) if plain.visible(i, j, chunk=3)] for i in (0, 2, 3, 7)] == [[0], [0, 1, 2], [3], [6, 7]]
    # the sink: two keys of score 0 share the denominator with it; one key of a score far below zero almost vanishes
    q, k, v = np.zeros((1, 1, 4)), np.ones((2, 1, 4)), np.array([3.0, 6.0]).reshape(2, 1, 1)
    assert np.isclose(plain.attend(q, k, v, [1], [0, 1], 1.0, sink=True)[0, 0, 0], 3.0)
    assert np.isclose(plain.attend(q, k, v, [1], [0, 1], 1.0)[0, 0, 0], 4.5)
    low = plain.attend(np.full((1, 1, 4), -2.0), k[:1], v[:1], [0], [0], 1.0, sink=True)[0, 0, 0]
    assert np.isclose(low, 3.0 * math.exp(-8) / (1 + math.exp(-8)))
    # halves: numbers 0 and 2 turn by a quarter, the fifth passes
    assert np.allclose(plain.rotate_halves(np.array([[1.0, 2.0, 0.0, 0.0, 5.0]]), [1], np.array([np.pi / 2, 0.0]), 2.0),
                       [[0.0, 4.0, 2.0, 0.0, 5.0]])
    # delta rule: rows forget by themselves, then v is written along k and read along q, all within the token
    S, o = plain.delta_step(np.array([[2.0], [10.0]]), np.array([1.0, 1.0]), np.array([1.0, 0.0]), np.array([7.0]), np.array([0.5, 0.1]), 0.5)
    assert np.allclose(S, [[4.0], [1.0]]) and np.allclose(o, [5.0])
    # the pair's sum, clamped halves, the router
    assert np.allclose(plain.half_sum(np.array([3.0, 3.0]), np.array([0.0, 8.0]), 1.0, np.array([1.0, 2.0]), 0.0), [0.5, 0.5 + math.sqrt(2.0)])
    assert np.isclose(plain.clamped_gate(9.0, -9.0, 2.0), 2.0 / (1 + math.exp(-3.404)) * -1.0)
    assert np.isclose(plain.clamped_gate(-9.0, 0.5, 2.0), -9.0 / (1 + math.exp(1.702 * 9)) * 1.5)
    chosen, w = plain.route(np.array([0.0, 3.0, -1.0, 2.0]), 2)
    assert chosen == [1, 3] and np.allclose(w, [1 / (1 + math.exp(-1)), 1 / (1 + math.exp(1))])
