"""The Felovik configuration: what it reads, what it refuses, the parts it builds and what they
ask of the cache, and the plain model's own mechanisms on hand-made inputs. No GPU."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_felovik as plain
from semantic_aware_adaptive_kv_cache_precision_b200.cache import KVNeed, MultiNeed, SequenceCache, StateNeed
from semantic_aware_adaptive_kv_cache_precision_b200.config import (ConfigError, QueryTemperature,
                                                                   config_from_dict,
                                                                   known_architectures)
from semantic_aware_adaptive_kv_cache_precision_b200.engine.model import DecoderModel
from semantic_aware_adaptive_kv_cache_precision_b200.parts import build_part
from felovik_configs import CONFIGS, MIXED, ODD, WIDE


def spec_of(config):
    return config_from_dict(copy.deepcopy(config)).model_spec()


def test_registered_and_round_trips():
    assert "Felovik" in known_architectures()
    for config, _ in CONFIGS.values():
        typed = config_from_dict(copy.deepcopy(config))
        assert config_from_dict(typed.to_dict()) == typed


def test_the_parts_descriptions_carry_the_configuration_and_the_design_s_constants():
    spec = spec_of(MIXED)
    assert spec.position_name == "pos" and spec.max_positions == 640 and spec.embed_scale == 2.5
    assert not spec.tie_head and spec.head_name == "head" and spec.final_norm.eps == 1e-5
    assert [c.block for c in spec.run_order] == [c.cache for c in spec.run_order] == [0, 1, 2, 3]
    block = spec.blocks[0]
    assert block.kind == "post_norm_block" and block.alpha == 2.0 and block.prefix == "l0."
    mixer = block.mixer
    assert mixer.scale == 0.5 and mixer.branch_norm == block.norm and mixer.norm_name == "out"
    a, b = mixer.left, mixer.right
    assert a.qk_norm == "head" and a.gate and not a.bias and not a.sink and a.window is None
    assert a.position is None and a.q_temp == QueryTemperature(0.4, 37) and a.scale == 0.25
    assert spec.blocks[2].mixer.left.q_temp is None and spec.blocks[2].ffn is None
    assert (b.heads, b.value_dim, b.state, b.groups, b.taps, b.norm_groups) == (4, 16, 24, 2, 4, 2)
    dense = block.ffn
    assert dense.activation == "clamped" and (dense.limit, dense.alpha, dense.plus) == (0.6, 1.702, 1.0)
    routed = spec.blocks[1].ffn
    assert routed.score == "softmax" and routed.renormalize and not routed.weight_input
    assert (routed.experts, routed.top, routed.groups, routed.keep_groups) == (8, 3, 4, 2)
    assert math.isinf(routed.expert.limit) and (routed.expert.alpha, routed.expert.plus) == (1.0, 0.0)
    assert routed.shared is None and not routed.correction and routed.identity == 0
    assert (spec.blocks[3].ffn.groups, spec.blocks[3].ffn.keep_groups) == (1, 1)


def test_declared_tensors_carry_the_configuration_s_sizes():
    spec = spec_of(MIXED)
    shapes = {d.name: tuple(d.shape) for d in DecoderModel.tensor_decls_of(spec)}
    assert shapes["embed"] == shapes["head"] == (211, 96) and shapes["pos"] == (640, 96)
    assert shapes["final.norm"] == shapes["l0.norm1"] == shapes["l0.norm2"] == (96,)
    assert shapes["l0.mix.left.q"] == (128, 96) and shapes["l0.mix.left.k"] == (64, 96)
    assert shapes["l0.mix.left.v"] == (48, 96) and shapes["l0.mix.left.g"] == (96, 96)
    assert shapes["l0.mix.left.o"] == (96, 96) and shapes["l0.mix.left.out"] == (96,)
    assert "l0.mix.left.q.norm" not in shapes and "l0.mix.left.q.b" not in shapes
    assert shapes["l0.mix.right.in"] == (2 * 64 + 2 * 2 * 24 + 4, 96)
    assert shapes["l0.mix.right.conv"] == (64 + 96, 4) and shapes["l0.mix.right.conv.b"] == (160,)
    for n in ("dt_bias", "A_log", "D"):
        assert shapes[f"l0.mix.right.{n}"] == (4,)
    assert shapes["l0.mix.right.norm"] == (64,) and shapes["l0.mix.right.o"] == (96, 64)
    assert shapes["l0.mlp.gate"] == (80, 96) and shapes["l0.mlp.down"] == (96, 80)
    assert shapes["l1.mlp.router"] == (8, 96) and shapes["l1.mlp.e7.up"] == (48, 96)
    assert "l1.mlp.e8.up" not in shapes and "l2.norm2" not in shapes and "l2.mlp.gate" not in shapes
    assert spec.ignore_tensors == ("l2.norm2",)


def test_what_the_layers_ask_of_the_cache_and_needs_inside_needs():
    needs = DecoderModel(spec_of(MIXED), "float32", "cpu").cache_needs()
    assert needs[0] == MultiNeed((KVNeed(2, 32, None, value_dim=24),
                                  MultiNeed((StateNeed((3, 160), "float32"),
                                             StateNeed((4, 16, 24), "float32")))))
    cache = SequenceCache(needs, 512, 640, torch.float32, "cpu", max_slots=3)
    assert cache.max_seq_len == 512
    (slot,) = cache.open(1)
    cache.reserve([slot], [70])
    tables = [torch.from_numpy(t) for t in cache.tables_for([slot])]
    keys, state = cache.entry_view(0, tables).parts
    assert keys.keys.shape[1:] == (2, 64, 32) and keys.values.shape[1:] == (2, 64, 24)
    assert state.parts[0].state.shape == (3, 3, 160) and state.parts[1].state.shape == (3, 4, 16, 24)
    state.parts[1].state[slot] = 5.0            # a slot that is taken again starts from zero
    cache.close([slot])
    (again,) = cache.open(1)
    assert again == slot and not cache.entry_view(0, tables).parts[1].parts[1].state[slot].any()
    cache.close([again])
    cache.check()


def test_every_problem_is_named_at_once():
    bad = copy.deepcopy(MIXED)
    bad["width"] = 0
    del bad["postln_alpha"]
    bad["layers"][0]["mixer"]["left"]["kv_heads"] = 3
    bad["layers"][0]["mlp"]["limit"] = None
    bad["layers"][1]["mixer"]["right"]["norm_groups"] = 5
    bad["layers"][1]["mlp"]["router"]["groups"] = {"count": 3, "keep": 1}
    bad["layers"][2]["mixer"]["right"]["groups"] = 4
    bad["layers"][2]["mixer"]["left"]["scale"] = "0.3"
    bad["layers"][3]["type"] = "mamba2"
    with pytest.raises(ConfigError) as err:
        config_from_dict(bad)
    text = str(err.value)
    for piece in ("width", "postln_alpha", "kv_heads", "mlp.limit", "norm_groups", "router.groups",
                  "4 groups", "left.scale", "'mamba2'"):
        assert piece in text, piece
    for groups, top in (({"count": 2, "keep": 3}, 3), ({"count": 4, "keep": 1}, 3)):
        bad = copy.deepcopy(MIXED)
        bad["layers"][1]["mlp"]["router"].update(groups=groups, top=top)
        with pytest.raises(ConfigError):
            config_from_dict(bad)


def test_the_number_of_positions_may_come_from_the_table():
    raw = copy.deepcopy(WIDE)
    del raw["max_positions"]
    assert config_from_dict(raw, {"pos": (333, 128)}).max_positions == 333
    with pytest.raises(ConfigError):
        config_from_dict(raw)


def test_query_temperature_by_hand_and_in_the_part_s_table():
    temp = {"coef": 0.4, "every": 37}
    f = plain.query_temperature(120, temp)
    assert f[0] == f[35] == 1.0
    assert math.isclose(f[36], 1 + 0.4 * math.log(2)) and f[36] == f[72]
    assert math.isclose(f[73], 1 + 0.4 * math.log(3)) and math.isclose(f[119], 1 + 0.4 * math.log(4))
    assert (plain.query_temperature(9, None) == 1).all()
    part = build_part(spec_of(MIXED).blocks[0].mixer.left, "x.", "float32")
    part.prepare("cpu", 120)
    assert np.array_equal(part.temperature.numpy(), f.astype(np.float32))
    one = plain.query_temperature(4, {"coef": 1.0, "every": 1})
    assert np.allclose(one, 1 + np.log(np.arange(1, 5) + 1.0))


def test_the_scan_by_hand():
    """Two heads that share B and C, one number each: S after token 1 is fade S0 + dt1 B1 x1."""
    x = np.array([[[2.0], [1.0]], [[3.0], [-1.0]]])
    B, C = np.array([[[0.5]], [[1.5]]]), np.array([[[2.0]], [[-1.0]]])
    dt = np.array([[0.1, 0.2], [0.3, 0.4]])
    a_log, d = np.log([1.0, 3.0]), np.array([0.5, 0.0])
    y, S = plain.dual_scan(x, B, C, dt, a_log, d)
    s0 = np.array([0.1 * 0.5 * 2.0, 0.2 * 0.5 * 1.0])
    s1 = np.exp(-np.array([1.0, 3.0]) * dt[1]) * s0 + dt[1] * 1.5 * x[1, :, 0]
    assert np.allclose(y[0, :, 0], 2.0 * s0 + d * x[0, :, 0])
    assert np.allclose(y[1, :, 0], -1.0 * s1 + d * x[1, :, 0]) and np.allclose(S[:, 0, 0], s1)
    # four heads over two groups: heads 0, 1 read the first
    rng = np.random.default_rng(0)
    x, B, C = rng.standard_normal((3, 4, 2)), rng.standard_normal((3, 2, 5)), rng.standard_normal((3, 2, 5))
    dt = rng.uniform(0.1, 1.0, (3, 4))
    whole, _ = plain.dual_scan(x, B, C, dt, np.zeros(4), np.ones(4))
    for h in range(4):
        alone, _ = plain.dual_scan(x[:, h:h + 1], B[:, h // 2:h // 2 + 1], C[:, h // 2:h // 2 + 1],
                                   dt[:, h:h + 1], np.zeros(1), np.ones(1))
        assert np.allclose(alone[:, 0], whole[:, h])


def test_convolution_gate_and_norm_by_hand():
    w, b = np.array([[3.0, 2.0, 1.0]]), np.array([0.5])
    out = plain.causal_conv(np.array([[1.0], [10.0], [100.0]]), w, b)[:, 0]
    assert np.allclose(out, plain.silu(np.array([1.5, 12.5, 123.5])))     # 100 + 2*10 + 3*1 + 0.5
    y, z = np.array([[1.0, 2.0, 3.0, 4.0]]), np.array([[1.0, -1.0, 0.0, 2.0]])
    g = y * plain.silu(z)
    got = plain.gate_then_norm(y, z, np.array([1.0, 2.0, 3.0, 4.0]), 2, 1e-3)
    want = np.concatenate([g[0, :2] / math.sqrt((g[0, :2] ** 2).mean() + 1e-3),
                           g[0, 2:] / math.sqrt((g[0, 2:] ** 2).mean() + 1e-3)])
    assert np.allclose(got[0], want * [1, 2, 3, 4])


def test_routing_by_hand():
    """Six experts in three groups of two, two groups open: expert 2 is the second best of all
    and closed when the groups of experts 0 and 5 are better."""
    t = {"router": np.array([[3.0], [0.5], [2.0], [1.9], [1.0], [2.5]])}
    h = np.array([[1.0]])
    chosen, w = plain.route(h, t, "", {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}})
    assert chosen.tolist() == [[0, 5, 4]]
    s = np.exp([3.0, 2.5, 1.0])
    assert np.allclose(w, s / s.sum())
    assert plain.route(h, t, "", {"experts": 6, "top": 3})[0].tolist() == [[0, 5, 2]]
    for e in range(6):
        t[f"e{e}.gate"], t[f"e{e}.up"] = np.array([[2.0]]), np.array([[-3.0]])
        t[f"e{e}.down"] = np.array([[float(e + 1)]])
    mlp = {"router": {"experts": 6, "top": 3, "groups": {"count": 3, "keep": 2}}}
    y = plain.silu(2.0) * -3.0
    assert np.allclose(plain.experts(h, t, "", mlp), (w[0] * [1.0, 6.0, 5.0]).sum() * y)


def test_the_dense_feed_forward_clamps_one_side_of_the_gate_and_both_of_the_rest():
    t = {"gate": np.array([[5.0], [-5.0], [1.0]]), "up": np.array([[4.0], [-4.0], [0.5]]),
         "down": np.eye(3)}
    got = plain.clamped_mlp(np.array([[1.0]]), t, "", 1.5)[0]
    s = plain.sigmoid
    assert np.allclose(got, [1.5 * s(1.702 * 1.5) * 2.5, -5.0 * s(-1.702 * 5.0) * -0.5,
                             1.0 * s(1.702) * 1.5])


def test_the_layer_norms_the_weighted_sum():
    config = copy.deepcopy(ODD)
    rng = np.random.default_rng(1)
    shapes = {d.name: tuple(d.shape) for d in DecoderModel.tensor_decls_of(spec_of(config))}
    t = {k: rng.standard_normal(s) * 0.2 for k, s in shapes.items()}
    x = rng.standard_normal((3, 100))
    got = plain.layer(x, t, config, 2)                 # (no feed-forward)
    m = plain.parallel(x, t, "l2.mix.", config["layers"][2]["mixer"], 3e-6)
    v = 0.7 * x + m
    assert np.allclose(got, v / np.sqrt((v * v).mean(-1, keepdims=True) + 3e-6) * t["l2.norm1"])
    assert np.array_equal(plain.embed(t, [4, 4, 9], 2.0)[1], 2.0 * t["embed"][4] + t["pos"][1])
