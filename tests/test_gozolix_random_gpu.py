"""Gozolix configurations drawn at random over what config.json allows (widths, head counts, key and
value sizes of both mixers, taps, caps, temperatures, layers that read another's cache, dense and
routed feed-forwards and none, groups of experts, shared experts, tables of pairs), each through the
engine against the plain model: whole prompts, the last tokens one by one, and an unequal batch."""

import copy

import numpy as np
import pytest

import plain_gozolix as plain
import semantic_aware_adaptive_kv_cache_precision_b200 as sakv
from helpers import assert_same_logits
from gozolix_configs import attention, bigram, delta, dense, moe

pytestmark = pytest.mark.gpu


def divisors(n):
    return [d for d in range(1, n + 1) if n % d == 0]


def draw(seed, all_chosen=False):
    rng = np.random.default_rng(5000 + seed)
    pick = lambda options: options[int(rng.integers(len(options)))]
    width = pick([40, 48, 64, 72, 100, 128, 160, 200, 320])

    def mlp():
        kind = rng.random()
        if kind < 0.2:
            return None
        if kind < 0.5:
            return dense(pick([16, 30, 64, 128, 256]))
        experts = pick([1, 2, 3, 4, 6, 8, 12, 24])
        count = pick(divisors(experts))
        keep = int(rng.integers(1, count + 1))
        most = experts // count * keep
        groups = None if rng.random() < 0.2 else (count, keep)
        top = int(rng.integers(1, min(most, 5) + 1))
        if all_chosen:
            groups, top = (groups and (count, count)), experts
        return moe(experts, top, pick([16, 22, 50, 64, 130]), groups,
                   None if rng.random() < 0.3 else pick([16, 40, 128]), float(pick([0.5, 1.0, 2.5])))

    layers, own = [], []
    for i in range(int(rng.integers(1, 7))):
        if rng.random() < 0.5:
            kv_heads = pick([1, 2, 3, 4])
            layers.append(delta(kv_heads * pick([1, 2, 3]), kv_heads, pick([4, 8, 12, 24, 40, 64, 100, 128, 200]),
                                pick([4, 5, 8, 16, 20, 64, 128]), pick([1, 2, 3, 4, 7]), mlp()))
            continue
        cap = None if rng.random() < 0.2 else float(pick([1.0, 5.0, 30.0]))
        temp = None if rng.random() < 0.25 else (float(rng.uniform(0.05, 1.0)),
                                                 pick([1, 2, 7, 32, 64, 100, 4096]))
        source = pick(own) if own and rng.random() < 0.5 else None
        if source is None:
            kv_heads, dim = pick([1, 2, 3, 4]), pick([4, 8, 12, 16, 24, 48, 64, 96, 128])
            heads, vdim = kv_heads * pick([1, 2, 3, 4]), pick([4, 8, 12, 32, 80, 96])
            own.append(i)
        else:
            m = layers[source]["mixer"]
            heads, kv_heads, dim, vdim = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        layers.append(attention(heads, kv_heads, dim, vdim, float(dim ** -0.5 * rng.uniform(0.5, 2)), cap,
                                temp, mlp(), source))
    embedding = {"scale": float(pick([1.0, 2.0, 5.0]))}
    if rng.random() < 0.8:
        embedding["bigram"] = bigram(pick([1, 7, 97, 1000]), pick([1, 29, 1009]), pick([1, 11, 65537]))
    return {"architecture": "Gozolix", "vocab": int(rng.integers(50, 700)), "width": width,
            "norm": {"eps": float(pick([1e-6, 1e-5]))}, "embedding": embedding,
            "initializer_range": 0.1, "layers": layers}


def row_errors(got, want):
    """Each row's largest difference over its spread."""
    return np.abs(np.asarray(got, dtype=np.float64) - want).max(axis=-1) / want.std(axis=-1)


def conditioning(cfg, tensors, p, want):
    """How a drawn model answers rounding, from the plain model alone: the median row's
    difference when every weight moves by up to 2^-8 of itself, over 0.05 (what it is for most
    draws or less), 1 at least. (Some draws answer ten times as strongly.)"""
    rng = np.random.default_rng(1)
    moved = {k: np.asarray(v, dtype=np.float64) * (1 + rng.uniform(-1, 1, np.shape(v)) * 2.0 ** -8)
             for k, v in tensors.items()}
    return max(1.0, np.median(row_errors(plain.forward(cfg, moved, p), want)) / 0.05)


@pytest.mark.parametrize("seed", range(24))
def test_a_drawn_configuration_in_32_bits(seed, tmp_path):
    config = draw(seed)
    folder = sakv.write_random_model(tmp_path / "m", copy.deepcopy(config), seed, dtype="float32")
    cfg, tensors = plain.read_model_folder(folder)
    engine = sakv.Engine(folder, dtype="float32", max_tokens=1024, poison_freed=True).load_weights()
    rng = np.random.default_rng(seed)
    prompts = [rng.integers(0, config["vocab"], n).astype(np.int64) for n in (170, 37, 2)]
    whole = [engine.forward(p) for p in prompts]
    for got, p in zip(whole, prompts):
        want = plain.forward(cfg, tensors, p)
        err, answer = row_errors(got, want), conditioning(cfg, tensors, p, want)
        assert np.quantile(err, 0.97) <= 5e-5 * answer and err.max() <= 2e-3 * answer, \
            f"seed {seed}: worst row {err.max():.2e}, 97 of 100 within {np.quantile(err, 0.97):.2e}"
    # the longest prompt again: most of it in one step, its last 40 tokens one by one
    p = prompts[0]
    (slot,) = engine.open(1)
    rows = [engine.step([slot], [p[:130]], [list(range(130))]).cpu().numpy()]
    for t in range(130, len(p)):
        rows.append(engine.step([slot], [p[t:t + 1]]).cpu().numpy())
    engine.close([slot])
    assert_same_logits(np.concatenate(rows), whole[0], "float32", f"seed {seed}: decoded")
    # the three together, then decoded together until each ends
    slots = engine.open(3)
    heads = [len(q) - k for q, k in zip(prompts, (5, 3, 1))]
    out = engine.step(slots, [q[:h] for q, h in zip(prompts, heads)],
                      [list(range(h)) for h in heads]).cpu().numpy()
    got = [[out[sum(heads[:i]):sum(heads[:i + 1])]] for i in range(3)]
    fed = list(heads)
    live = [0, 1, 2]
    while live:
        out = engine.step([slots[i] for i in live], [prompts[i][fed[i]:fed[i] + 1] for i in live])
        for k, i in enumerate(live):
            got[i].append(out[k:k + 1].cpu().numpy())
            fed[i] += 1
        done = [i for i in live if fed[i] == len(prompts[i])]
        if done:
            engine.close([slots[i] for i in done])
        live = [i for i in live if fed[i] < len(prompts[i])]
    for i in range(3):
        assert_same_logits(np.concatenate(got[i]), whole[i], "float32",
                           f"seed {seed}: request {i} of the batch")
    engine.cache.check()
    assert engine.graph_failure is None


@pytest.mark.parametrize("seed", range(24))
def test_a_drawn_configuration_in_16_bits(seed, tmp_path):
    """A prompt long enough for the recurrence to cross many groups of four, then tokens one by one; every
    expert chosen for every token (a choice that rounding turns is no fault); judged by the
    median row, within a tenth of its spread where the model is well conditioned."""
    config = draw(seed, all_chosen=True)
    folder = sakv.write_random_model(tmp_path / "m", copy.deepcopy(config), seed, dtype="bfloat16")
    cfg, tensors = plain.read_model_folder(folder)
    engine = sakv.Engine(folder, dtype="bfloat16", max_tokens=1024, poison_freed=True).load_weights()
    p = np.random.default_rng(seed).integers(0, config["vocab"], 330).astype(np.int64)
    want = plain.forward(cfg, tensors, p)
    (slot,) = engine.open(1)
    rows = [engine.step([slot], [p[:290]], [list(range(290))]).cpu().numpy()]
    for t in range(290, len(p)):
        rows.append(engine.step([slot], [p[t:t + 1]]).cpu().numpy())
    engine.close([slot])
    got = np.concatenate(rows)
    assert np.isfinite(got).all()
    err, answer = row_errors(got, want), conditioning(cfg, tensors, p, want)
    for what, rows in (("prompt", err[:290]), ("decoded tokens", err[290:])):
        assert np.median(rows) <= 0.1 * answer, f"seed {seed}: the {what}'s median row {np.median(rows):.3f}"
    assert engine.graph_failure is None
