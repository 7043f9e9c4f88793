"""The Gozolix configuration: what it reads, what it refuses, the parts it builds and what they
ask of the cache, and the plain model's own mechanisms on hand-made inputs. No GPU."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_gozolix as plain
from semantic_aware_adaptive_kv_cache_precision_b200.cache import KVNeed, MultiNeed, SequenceCache, StateNeed
from semantic_aware_adaptive_kv_cache_precision_b200.config import (BigramSpec, ConfigError,
                                                                   config_from_dict,
                                                                   known_architectures)
from semantic_aware_adaptive_kv_cache_precision_b200.engine.model import DecoderModel
from semantic_aware_adaptive_kv_cache_precision_b200.parts import build_part
from gozolix_configs import CONFIGS, MIXED, ODD, WIDE


def spec_of(config):
    return config_from_dict(copy.deepcopy(config)).model_spec()


def test_registered_and_round_trips():
    assert "Gozolix" in known_architectures()
    for config, _ in CONFIGS.values():
        typed = config_from_dict(copy.deepcopy(config))
        assert config_from_dict(typed.to_dict()) == typed


def test_the_parts_descriptions_carry_the_configuration_and_the_design_s_constants():
    spec = spec_of(MIXED)
    assert spec.embed_scale == 2.5 and spec.bigram == BigramSpec("bigram", 101, 13, 5)
    assert not spec.tie_head and spec.head_name == "head" and spec.final_norm.eps == 1e-5
    assert [c.block for c in spec.run_order] == list(range(7))
    assert [c.cache for c in spec.run_order] == [0, 1, 0, 2, 3, 3, 0]
    block = spec.blocks[0]
    assert block.kind == "parallel_block" and block.prefix == "l0." and block.norm_name == "norm1"
    a = block.mixer
    assert a.bias and a.own_kv and not a.sink and a.window is None and a.qk_norm is None
    assert not a.gate and a.position is None and (a.scale, a.softcap) == (0.25, 4.0)
    assert (a.q_temp.coef, a.q_temp.every) == (0.4, 37)
    assert a.slopes == (2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8)
    b = spec.blocks[2].mixer
    assert not b.own_kv and b.softcap is None and b.q_temp is None and b.scale == 0.4
    assert spec.blocks[4].mixer.slopes[0] == 2.0 ** (-8 / 6)
    d = spec.blocks[1].mixer
    assert (d.heads, d.kv_heads, d.head_dim, d.value_dim, d.taps) == (6, 3, 24, 16, 4)
    assert d.q_scale == 24 ** -0.5 and d.unit_eps == 1e-6 and d.eps == 1e-5
    assert block.ffn.activation == "relu_squared" and spec.blocks[3].ffn is None
    routed = spec.blocks[1].ffn
    assert routed.score == "sigmoid" and routed.renormalize and not routed.weight_input
    assert (routed.experts, routed.top, routed.groups, routed.keep_groups) == (8, 3, 4, 2)
    assert routed.group_top == 2 and routed.scale == 2.0 and not routed.shared_gate
    assert math.isinf(routed.expert.limit) and (routed.expert.alpha, routed.expert.plus) == (1.0, 0.0)
    assert routed.shared.intermediate == 56 and spec.blocks[2].ffn.shared is None
    assert spec_of(WIDE).bigram is None and spec_of(ODD).blocks[2].ffn.scale == 1.0


def test_declared_tensors_carry_the_configuration_s_sizes():
    spec = spec_of(MIXED)
    shapes = {d.name: tuple(d.shape) for d in DecoderModel.tensor_decls_of(spec)}
    assert shapes["embed"] == shapes["head"] == (211, 96) and shapes["bigram"] == (102, 96)
    assert shapes["final.norm"] == shapes["l0.norm1"] == (96,) and "l0.norm2" not in shapes
    assert shapes["l0.mix.q"] == (128, 96) and shapes["l0.mix.k.b"] == (64,)
    assert shapes["l0.mix.v"] == (48, 96) and shapes["l0.mix.o"] == (96, 96)
    assert shapes["l2.mix.q.b"] == (128,) and "l2.mix.k" not in shapes and "l2.mix.v.b" not in shapes
    assert "l0.mix.o.b" not in shapes
    assert shapes["l1.mix.q"] == shapes["l1.mix.k"] == (72, 96) and shapes["l1.mix.v"] == (96, 96)
    assert shapes["l1.mix.g"] == (96, 96) and shapes["l1.mix.a"] == shapes["l1.mix.b"] == (6, 96)
    assert shapes["l1.mix.k.conv"] == (72, 4) and shapes["l1.mix.v.conv"] == (96, 4)
    assert shapes["l1.mix.A_log"] == shapes["l1.mix.dt_bias"] == (6,)
    assert shapes["l1.mix.norm"] == (16,) and shapes["l1.mix.o"] == (96, 96)
    assert "l1.mix.q.b" not in shapes and "l3.mlp.up" not in shapes
    assert shapes["l0.mlp.up"] == (80, 96) and "l0.mlp.gate" not in shapes
    assert shapes["l1.mlp.router"] == (8, 96) and shapes["l1.mlp.e7.up"] == (48, 96)
    assert shapes["l1.mlp.shared.down"] == (96, 56) and "l2.mlp.shared.up" not in shapes
    assert "bigram" not in {d.name for d in DecoderModel.tensor_decls_of(spec_of(WIDE))}


def test_what_the_layers_ask_of_the_cache_and_a_slot_taken_again():
    model = DecoderModel(spec_of(MIXED), "float32", "cpu")
    needs = model.cache_needs()
    assert needs == [KVNeed(2, 32, None, value_dim=24),
                     MultiNeed((StateNeed((3, 240), "float32"), StateNeed((6, 16, 24), "float32"))),
                     MultiNeed((StateNeed((2, 288), "float32"), StateNeed((4, 40, 16), "float32"))),
                     KVNeed(1, 48, None, value_dim=16), StateNeed((1,), "int32")]
    assert len(DecoderModel(spec_of(WIDE), "float32", "cpu").cache_needs()) == 5
    cache = SequenceCache(needs, 512, 640, torch.float32, "cpu", max_slots=3)
    (slot,) = cache.open(1)
    cache.reserve([slot], [70])
    tables = [torch.from_numpy(t) for t in cache.tables_for([slot])]
    conv, state = cache.entry_view(1, tables).parts
    last = cache.entry_view(4, tables).state
    assert conv.state.shape == (3, 3, 240) and state.state.shape == (3, 6, 16, 24)
    assert last.shape == (3, 1) and last.dtype == torch.int32
    state.state[slot], last[slot] = 5.0, 7
    cache.close([slot])
    (again,) = cache.open(1)
    assert again == slot and not state.state[slot].any() and not last[slot].any()
    cache.close([again])
    cache.check()


def test_every_problem_is_named_at_once():
    bad = copy.deepcopy(MIXED)
    bad["width"] = 0
    bad["norm"] = {}
    bad["embedding"]["bigram"]["buckets"] = 0
    bad["layers"][0]["mixer"]["scale"] = "0.3"
    bad["layers"][0]["mixer"]["softcap"] = 0.0
    bad["layers"][1]["mixer"]["kv_heads"] = 4
    bad["layers"][1]["mlp"]["router"]["groups"] = {"count": 3, "keep": 1}
    bad["layers"][2]["mixer"]["kv_from"] = 1                 # (not attention)
    bad["layers"][3]["mixer"]["conv"] = 0
    bad["layers"][4]["type"] = "mamba2"
    bad["layers"][6]["mlp"]["kind"] = "gated"
    with pytest.raises(ConfigError) as err:
        config_from_dict(bad)
    text = str(err.value)
    for piece in ("width", "norm.eps", "bigram.buckets", "mixer.scale", "softcap", "4 kv_heads",
                  "router.groups", "kv_from: 1", "mixer.conv", "'mamba2'", "'gated'"):
        assert piece in text, piece


@pytest.mark.parametrize("layer,change", [
    (2, {"kv_from": 2}), (2, {"kv_from": 4}), (2, {"kv_from": -1}), (2, {"kv_from": True}),
    (6, {"kv_from": 2}), (2, {"kv_heads": 4}), (2, {"dim": 16}), (2, {"vdim": 32})])
def test_a_layer_reads_only_an_earlier_attention_layer_of_equal_sizes(layer, change):
    bad = copy.deepcopy(MIXED)
    bad["layers"][layer]["mixer"].update(change)
    with pytest.raises(ConfigError, match="kv_from"):
        config_from_dict(bad)


def test_absent_keys_are_absent():
    raw = copy.deepcopy(WIDE)
    del raw["embedding"]
    del raw["layers"][2]["mlp"]["router"]["scale"]
    del raw["layers"][2]["mlp"]["router"]["groups"]
    del raw["layers"][4]["mixer"]["kv_heads"]
    config = config_from_dict(raw)
    spec = config.model_spec()
    assert spec.embed_scale == 1.0 and spec.bigram is None
    assert (spec.blocks[2].ffn.scale, spec.blocks[2].ffn.groups) == (1.0, 1)
    assert spec.blocks[4].mixer.kv_heads == 2


def test_the_parts_tables():
    part = build_part(spec_of(MIXED).blocks[0].mixer, "x.", "float32")
    part.prepare("cpu", 120)
    f = plain.query_temperature(120, {"coef": 0.4, "every": 37})
    assert np.array_equal(part.temperature.numpy(), f.astype(np.float32))
    assert f[35] == 1.0 and math.isclose(f[36], 1 + 0.4 * math.log(2))
    assert np.array_equal(part.slopes.numpy(), plain.head_slopes(4).astype(np.float32))
    assert np.allclose(plain.head_slopes(6), [2 ** (-8 * (h + 1) / 6) for h in range(6)])
    reader = build_part(spec_of(MIXED).blocks[2].mixer, "x.", "float32")
    assert reader.input_rows == 128 and [d.name for d in reader.input_decls(None)] == ["x.q"]


def test_a_table_of_pairs_beside_learned_positions_is_refused():
    spec = spec_of(ODD)
    from dataclasses import replace
    with pytest.raises(ValueError):
        DecoderModel(replace(spec, position_name="pos"), "float32", "cpu")


def test_pairs_by_hand():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 4}
    assert plain.bigram_rows([2, 5, 5, 1], b) == [10, (6 + 20) % 10, (15 + 20) % 10, (15 + 4) % 10]
    rng = np.random.default_rng(0)
    t = {"embed": rng.standard_normal((6, 3)), "bigram": rng.standard_normal((11, 3))}
    x = plain.embed(t, [2, 5], {"scale": 2.0, "bigram": b})
    assert np.allclose(x, [2 * t["embed"][2] + t["bigram"][10], 2 * t["embed"][5] + t["bigram"][6]])
    assert np.allclose(plain.embed(t, [2, 5], {}), t["embed"][[2, 5]])


def test_the_delta_rule_by_hand():
    """Two heads that share q and k, keys of two numbers, values of one."""
    q = np.array([[[1.0, 0.0]], [[0.6, 0.8]]])
    k = np.array([[[0.8, 0.6]], [[0.0, 1.0]]])
    v = np.array([[[2.0], [1.0]], [[3.0], [-1.0]]])
    g, beta = np.array([[0.5, 0.9], [0.25, 1.0]]), np.array([[1.0, 0.5], [0.5, 0.2]])
    o, S = plain.delta_scan(q, k, v, g, beta)
    for h, (b0, b1, fade, v0, v1) in enumerate([(1.0, 0.5, 0.25, 2.0, 3.0), (0.5, 0.2, 1.0, 1.0, -1.0)]):
        s = np.array([0.8, 0.6]) * b0 * v0               # the state starts at zero
        assert np.allclose(o[0, h, 0], s[0])
        s = fade * s
        s = s + np.array([0.0, 1.0]) * b1 * (v1 - s[1])   # what lies along the key is corrected
        assert np.allclose(o[1, h, 0], 0.6 * s[0] + 0.8 * s[1]) and np.allclose(S[h, :, 0], s)
    # a unit key with beta 1 replaces what the state says of it
    S1 = plain.delta_scan(k[1:], k[1:], v[1:], np.ones((1, 2)), np.ones((1, 2)), S)[1]
    assert np.allclose(S1[:, 1, 0], v[1, :, 0])
    # four heads over two q/k heads: heads 0, 1 read the first
    rng = np.random.default_rng(0)
    q, k = (plain.unit(rng.standard_normal((3, 2, 5))) for _ in range(2))
    v, g, beta = rng.standard_normal((3, 4, 2)), rng.uniform(0, 1, (3, 4)), rng.uniform(0, 1, (3, 4))
    whole, _ = plain.delta_scan(q, k, v, g, beta)
    for h in range(4):
        alone, _ = plain.delta_scan(q[:, h // 2:h // 2 + 1], k[:, h // 2:h // 2 + 1], v[:, h:h + 1],
                                    g[:, h:h + 1], beta[:, h:h + 1])
        assert np.allclose(alone[:, 0], whole[:, h])


def test_four_tokens_unrolled_say_the_same_as_one_by_one():
    """The identity the prompt's kernel rests on: sums from the state at a group's start, products
    of keys and queries inside the group, and the decays between its tokens."""
    rng = np.random.default_rng(1)
    D, Dv, n = 6, 3, 4
    q, k = plain.unit(rng.standard_normal((n, D))), plain.unit(rng.standard_normal((n, D)))
    v, g, beta = rng.standard_normal((n, Dv)), rng.uniform(0.2, 1, n), rng.uniform(0, 1, n)
    S0 = rng.standard_normal((D, Dv))
    want, last = plain.delta_scan(q[:, None], k[:, None], v[:, None], g[:, None], beta[:, None],
                                  S0[None])
    c = np.cumprod(g)
    u = np.zeros((n, Dv))
    for i in range(n):
        u[i] = beta[i] * (v[i] - c[i] * S0.T @ k[i]
                          - sum(c[i] / c[j] * (k[j] @ k[i]) * u[j] for j in range(i)))
        o = c[i] * S0.T @ q[i] + sum(c[i] / c[j] * (k[j] @ q[i]) * u[j] for j in range(i + 1))
        assert np.allclose(o, want[i, 0])
    assert np.allclose(c[-1] * S0 + sum(c[-1] / c[j] * np.outer(k[j], u[j]) for j in range(n)), last[0])


def test_convolution_unit_vectors_decays_and_the_gated_norm_by_hand():
    out = plain.causal_conv(np.array([[1.0], [10.0], [100.0]]), np.array([[3.0, 2.0, 1.0]]))[:, 0]
    assert np.allclose(out, plain.silu(np.array([1.0, 12.0, 123.0])))     # 100 + 2*10 + 3*1
    assert np.allclose(plain.unit(np.array([3e-3, 4e-3])), np.array([3e-3, 4e-3]) / math.sqrt(2.6e-5))
    assert np.allclose(plain.decay(np.array([0.3]), np.log([2.0]), np.array([0.2])),
                       math.exp(-2.0 * math.log1p(math.exp(0.5))))
    o, z = np.array([[[1.0, 2.0], [3.0, 4.0]]]), np.array([[1.0, -1.0, 0.0, 2.0]])
    got = plain.norm_then_gate(o, z, np.array([1.0, 2.0]), 1e-3)
    want = np.concatenate([o[0, h] / math.sqrt((o[0, h] ** 2).mean() + 1e-3) * [1, 2] for h in (0, 1)])
    assert np.allclose(got[0], want * plain.silu(z[0]))


def test_scores_are_capped_before_the_distance_is_taken_off():
    t = {"q": np.array([[3.0]]), "k": np.array([[2.0]]), "v": np.array([[1.0]]), "o": np.array([[1.0]]),
         "q.b": np.array([0.5]), "k.b": np.array([-1.0]), "v.b": np.array([2.0])}
    h = np.array([[1.0], [2.0]])
    m = {"heads": 1, "kv_heads": 1, "dim": 1, "vdim": 1, "scale": 0.5, "softcap": 2.0}
    y, (k, v) = plain.attention(h, t, "", m)
    s = [2 * math.tanh(6.5 * kk * 0.5 / 2) for kk in (1.0, 3.0)]
    w = np.exp([s[0] - 2.0 ** -8, s[1]])
    assert np.allclose(y[1, 0], (w * [3.0, 4.0]).sum() / w.sum()) and np.allclose(y[0, 0], 3.0)
    # another layer's keys and values, this layer's queries
    other = plain.attention(h, dict(t, q=np.array([[-1.0]])), "", m, (k, v))[0]
    s = [2 * math.tanh(-1.5 * kk * 0.5 / 2) for kk in (1.0, 3.0)]
    w = np.exp([s[0] - 2.0 ** -8, s[1]])
    assert np.allclose(other[1, 0], (w * [3.0, 4.0]).sum() / w.sum())


def test_routing_by_hand():
    """Six experts in two groups of three: the group with the best expert loses to the one whose
    two best sum to more."""
    t = {"router": np.array([[3.0], [-3.0], [-4.0], [2.0], [1.5], [-1.0]])}
    h = np.array([[1.0]])
    router = {"experts": 6, "top": 2, "groups": {"count": 2, "keep": 1}, "scale": 2.5}
    chosen, w = plain.route(h, t, "", router)
    s = plain.sigmoid(np.array([2.0, 1.5]))
    assert chosen.tolist() == [[3, 4]] and np.allclose(w, 2.5 * s / s.sum())
    assert plain.route(h, t, "", {"experts": 6, "top": 2})[0].tolist() == [[0, 3]]
    one = {"experts": 6, "top": 2, "groups": {"count": 6, "keep": 2}}
    assert plain.route(h, t, "", one)[0].tolist() == [[0, 3]]            # groups of one expert
    for e in ["shared"] + [f"e{i}" for i in range(6)]:
        t[f"{e}.gate"], t[f"{e}.up"] = np.array([[2.0]]), np.array([[-3.0]])
        t[f"{e}.down"] = np.array([[10.0 if e == "shared" else float(e[1:])]])
    y = plain.silu(2.0) * -3.0
    got = plain.experts(h, t, "", {"router": router, "shared": {"ff": 1}})
    assert np.allclose(got, (10.0 + w[0] @ [3.0, 4.0]) * y)
    assert np.allclose(plain.experts(h, t, "", {"router": router}), (w[0] @ [3.0, 4.0]) * y)


def test_the_layer_adds_both_sublayers_of_one_norm():
    config = copy.deepcopy(ODD)
    rng = np.random.default_rng(1)
    shapes = {d.name: tuple(d.shape) for d in DecoderModel.tensor_decls_of(spec_of(config))}
    t = {k: rng.standard_normal(s) * 0.2 for k, s in shapes.items()}
    x = rng.standard_normal((3, 100))
    h = x / np.sqrt((x * x).mean(-1, keepdims=True) + 3e-6) * t["l1.norm1"]
    m = plain.delta_mixer(h, t, "l1.mix.", config["layers"][1]["mixer"], 3e-6)
    f = np.maximum(h @ t["l1.mlp.up"].T, 0) ** 2 @ t["l1.mlp.down"].T
    assert np.allclose(plain.layer(x, t, config, 1, {}), x + m + f)
    h4 = x / np.sqrt((x * x).mean(-1, keepdims=True) + 3e-6) * t["l4.norm1"]
    assert np.allclose(plain.layer(x, t, config, 4, {}),               # (no feed-forward)
                       x + plain.delta_mixer(h4, t, "l4.mix.", config["layers"][4]["mixer"], 3e-6))
