"""Gozolix models with random weights through the engine, against the plain model: whole
prompts and the stream after every layer, pieces of prompts down to two tokens, the last tokens
one by one, unequal batches whose slots, cache blocks and states are used again, layers that read
another layer's cache, long decoding past block borders and temperature steps, a far token that an
asker recalls, greedy generation through `Engine.generate`, the trace-replay program and the command
line."""

import copy

import numpy as np
import pytest

import plain_gozolix as plain
import semantic_aware_adaptive_kv_cache_precision_b200 as sakv
from helpers import assert_same_logits
from gozolix_configs import CONFIGS
from gesuvik_configs import rows_agree

pytestmark = pytest.mark.gpu


def config_for(name, dtype):
    """The configuration as it is for float32. In bfloat16 a token's router scores are off by
    rounding, which now and then turns a choice between two experts (or two groups) of nearly
    equal score; such a row then differs by much, and no margin taken from the exact model says
    which rows those are. So the bfloat16 runs choose every expert for every token (the weights
    still are the scores'); choosing is tested in float32 here and in both types at the
    kernels."""
    config = copy.deepcopy(CONFIGS[name][0])
    if dtype == "bfloat16":
        for layer in config["layers"]:
            if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe":
                r = layer["mlp"]["router"]
                r["top"] = r["experts"]
                if "groups" in r:
                    r["groups"]["keep"] = r["groups"]["count"]
    return config


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("gozolix")
    made = {}

    def get(name, dtype):
        if (name, dtype) not in made:
            made[name, dtype] = sakv.write_random_model(
                root / f"{name}_{dtype}", config_for(name, dtype), CONFIGS[name][1], dtype=dtype)
        return made[name, dtype]

    return get


def prompts_of(name, lengths, seed=0):
    rng = np.random.default_rng(seed)
    return [rng.integers(0, CONFIGS[name][0]["vocab"], n).astype(np.int64) for n in lengths]


def compare(got, want, dtype, what, same=False):
    """`got` against `want`: the plain model's logits, or with `same` another run of the
    engine, which in float32 is equal to the bit."""
    if dtype == "float32" and same:
        assert_same_logits(np.asarray(got), np.asarray(want), dtype, what)
    else:
        rows_agree(got, want, dtype, what)


def setup(folders, name, dtype, max_tokens=1024):
    folder = folders(name, dtype)
    config, tensors = plain.read_model_folder(folder)
    engine = sakv.Engine(folder, dtype=dtype, max_tokens=max_tokens, poison_freed=True)
    return engine.load_weights(), config, tensors


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_and_every_layer(name, dtype, folders):
    engine, config, tensors = setup(folders, name, dtype)
    for p in prompts_of(name, (1, 2, 63, 201)):
        layers = []
        want = plain.forward(config, tensors, p, layers)
        got, states = engine.forward(p, capture_hidden_states=True)
        compare(got, want, dtype, f"{name}: a prompt of {len(p)}")
        assert states.shape[0] == len(config["layers"]) + 1
        rows_agree(states[0], plain.embed(tensors, p, config["embedding"]), dtype, "embedded")
        for i, s in enumerate(layers[:-1]):      # the stream after each layer but the last
            rows_agree(states[i + 1], s, dtype, f"{name}: after layer {i}")
    assert engine.graph_failure is None


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_pieces_of_a_prompt_and_tokens_one_by_one(name, dtype, folders):
    engine, config, tensors = setup(folders, name, dtype)
    (p,) = prompts_of(name, (230,), seed=1)
    whole = engine.forward(p)
    compare(whole, plain.forward(config, tensors, p), dtype, name)
    for pieces in ([2, 3, 59, 1, 64, 65, 7, 29], [128, 2, 100], [1] * 3 + [190] + [1] * 37):
        (slot,) = engine.open(1)
        rows, at = [], 0
        for n in pieces:
            rows.append(engine.step([slot], [p[at:at + n]], [list(range(n))]).cpu().numpy())
            at += n
        engine.close([slot])
        assert at == len(p)
        compare(np.concatenate(rows), whole, dtype, f"{name}: pieces {pieces[:4]}...", same=True)
    engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_a_long_prompt_whole_in_halves_and_beside_a_short_one(name, dtype, folders):
    engine, config, tensors = setup(folders, name, dtype, max_tokens=2048)
    p, short = prompts_of(name, (610, 30), seed=8)
    want = plain.forward(config, tensors, p)
    whole = engine.forward(p)
    compare(whole, want, dtype, f"{name}: 610 tokens")
    slots = engine.open(2)
    first = engine.step(slots, [p[:321], short], [list(range(321)), list(range(30))]).cpu().numpy()
    rest = engine.step(slots[:1], [p[321:]], [list(range(289))]).cpu().numpy()
    engine.close(slots)
    compare(np.concatenate([first[:321], rest]), whole, dtype, f"{name}: in two steps", same=True)
    compare(first[321:], plain.forward(config, tensors, short), dtype, f"{name}: the short one")
    engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_unequal_batches_with_slots_blocks_and_states_used_again(name, dtype, folders):
    """The cache holds exactly one batch, so every batch gets blocks and slots that the batch
    before gave back (blocks filled with NaN when they were freed, states left as they were:
    a slot's state must be zeroed when the slot is taken)."""
    lengths = (150, 9, 77, 1)
    engine, config, tensors = setup(folders, name, dtype, max_tokens=7 * 64)
    prompts = prompts_of(name, lengths, seed=2)
    alone = [engine.forward(p) for p in prompts]
    for g, w in zip(alone, prompts):
        compare(g, plain.forward(config, tensors, w), dtype, name)
    tails = (6, 3, 9, 0)
    for turn in range(3):
        order = [(i + turn) % 4 for i in range(4)]
        if turn == 1:
            spare, *slots = engine.open(5)
            engine.close([spare])
        else:
            slots = engine.open(4)
        heads = [lengths[i] - tails[i] for i in order]
        out = engine.step(slots, [prompts[i][:h] for i, h in zip(order, heads)],
                          [list(range(h)) for h in heads]).cpu().numpy()
        rows = {i: [out[sum(heads[:k]):sum(heads[:k + 1])]] for k, i in enumerate(order)}
        fed = dict(zip(order, heads))
        live = [(i, s) for i, s in zip(order, slots)]
        while True:
            done = [(i, s) for i, s in live if fed[i] == lengths[i]]
            if done:
                engine.close([s for _, s in done])
            live = [(i, s) for i, s in live if fed[i] < lengths[i]]
            if not live:
                break
            out = engine.step([s for _, s in live], [prompts[i][fed[i]:fed[i] + 1] for i, _ in live])
            for k, (i, _) in enumerate(live):
                rows[i].append(out[k:k + 1].cpu().numpy())
                fed[i] += 1
        for i in range(4):
            compare(np.concatenate(rows[i]), alone[i], dtype, f"{name}: turn {turn}, request {i}",
                    same=True)
        engine.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_mixed_step_starts_goes_on_and_decodes_at_once(dtype, folders):
    """One step in which a sequence starts, one goes on by several tokens and one by one."""
    engine, config, tensors = setup(folders, "mixed", dtype)
    a, b, c = prompts_of("mixed", (70, 101, 40), seed=9)
    want = [plain.forward(config, tensors, p) for p in (a, b, c)]
    sa, sb = engine.open(2)
    first = engine.step([sa, sb], [a[:69], b[:64]], [list(range(69)), list(range(64))]).cpu().numpy()
    (sc,) = engine.open(1)
    second = engine.step([sb, sc, sa], [b[64:], c, a[69:]],
                         [list(range(37)), list(range(40)), [0]]).cpu().numpy()
    engine.close([sa, sb, sc])
    compare(np.concatenate([first[:69], second[77:]]), want[0], dtype, "went on by one")
    compare(np.concatenate([first[69:], second[:37]]), want[1], dtype, "went on by several")
    compare(second[37:77], want[2], dtype, "started")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_long_decoding_past_block_borders_and_temperature_steps(name, dtype, folders):
    engine, config, tensors = setup(folders, name, dtype, max_tokens=512)
    (p,) = prompts_of(name, (300,), seed=3)
    want = plain.forward(config, tensors, p)
    (slot,) = engine.open(1)
    rows = [engine.step([slot], [p[:5]], [list(range(5))]).cpu().numpy()]
    for t in range(5, len(p)):
        rows.append(engine.step([slot], [p[t:t + 1]]).cpu().numpy())
    engine.close([slot])
    compare(np.concatenate(rows), want, dtype, f"{name}: 295 tokens one by one")
    assert engine.graph_failure is None


def far_folder(folder, dtype):
    """A model of two attention layers, the second reading the first one's cache, in which one token
    (number 1) has a key and a value that stand out and another (number 2) asks for that key, in
    both layers and in the head with the flattest slope."""
    import torch
    from semantic_aware_adaptive_kv_cache_precision_b200.weights.safetensors_io import write_safetensors
    from gozolix_configs import attention, dense
    config = {"architecture": "Gozolix", "vocab": 150, "width": 64, "norm": {"eps": 1e-5},
              "embedding": {"scale": 1.0}, "initializer_range": 0.1,
              "layers": [attention(2, 1, 32, 24, 0.5, 30.0, (0.3, 50), dense(40)),
                         attention(2, 1, 32, 24, 0.5, 20.0, None, None, 0)]}
    folder = sakv.write_random_model(folder, config, 77, dtype=dtype)
    _, t = plain.read_model_folder(folder)
    t = {k: np.array(v) for k, v in t.items()}
    rng = np.random.default_rng(0)
    r0, r1 = np.linalg.qr(rng.standard_normal((64, 2)))[0].T
    way, = np.linalg.qr(rng.standard_normal((32, 1)))[0].T
    e = t["embed"]                                # only the two tokens hold r0 and r1
    t["embed"] = e - np.outer(e @ r0, r0) - np.outer(e @ r1, r1)
    t["embed"][1], t["embed"][2] = 3.0 * r0, 3.0 * r1
    t["l0.mix.k"] = t["l0.mix.k"] + 1.5 * np.outer(way, r0)
    v = t["l0.mix.v"]
    t["l0.mix.v"] = v + 0.3 * np.outer(rng.standard_normal(24), r0)
    for i in (0, 1):
        t[f"l{i}.mix.q"][32:] += (1.5, 8.0)[i] * np.outer(way, r1)   # the flat head's queries
    t["l0.mix.o"], t["l1.mix.o"] = 0.5 * t["l0.mix.o"], 2.0 * t["l1.mix.o"]
    stored = torch.float32 if dtype == "float32" else torch.bfloat16
    write_safetensors(folder / "model.safetensors",
                      {k: torch.as_tensor(np.ascontiguousarray(v)).to(stored) for k, v in t.items()})
    return folder, *plain.read_model_folder(folder)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_far_token_shows_in_the_logits(dtype, tmp_path, monkeypatch):
    """The last row depends on the token 419 positions back, in a prompt and decoded, through the
    first layer's cache and through the layer that reads it."""
    n = 420
    folder, cfg, tensors = far_folder(tmp_path / "m", dtype)
    engine = sakv.Engine(folder, dtype=dtype, max_tokens=1024, poison_freed=True).load_weights()
    p = np.random.default_rng(10).integers(3, 150, n).astype(np.int64)
    p[0], p[-1] = 1, 2
    want = plain.forward(cfg, tensors, p)
    soft, calls = plain.causal_softmax, []

    def hidden(which):
        def without(scores):                       # what the model would say without the far key
            calls.append(0)
            scores = scores.copy()
            if (len(calls) - 1) // 2 in which:
                scores[n - 1, 0] = -np.inf
            return soft(scores)
        return without

    for which in ((0, 1), (1,)):                    # in both layers; in the reading layer alone
        calls.clear()
        monkeypatch.setattr(plain, "causal_softmax", hidden(which))
        without = plain.forward(cfg, tensors, p)
        apart = np.sqrt(((want - without) ** 2).mean(-1)) / want.std(-1)
        assert apart[-1] > 0.3, (which, apart[-1])
    monkeypatch.setattr(plain, "causal_softmax", soft)
    (slot,) = engine.open(1)
    head = engine.step([slot], [p[:-3]], [list(range(400, 417))]).cpu().numpy()
    tail = [engine.step([slot], [p[t:t + 1]]).cpu().numpy() for t in range(417, n)]
    engine.close([slot])
    compare(np.concatenate([head] + tail), want[400:], dtype, "before and after a far token")
    compare(tail[-1], want[-1:], dtype, "the far token, decoded")
    compare(engine.forward(p)[-1:], want[-1:], dtype, "the far token, in a prompt")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_token_before_is_part_of_a_sequence_s_state(dtype, folders):
    """Two sequences whose last prompt tokens differ go on with the same token, on slots that other
    sequences left: what their rows add is that of their own pairs."""
    engine, config, tensors = setup(folders, "mixed", dtype)
    slots = engine.open(3)
    engine.step(slots, [[9, 8], [7], [6, 5, 4]], [[], [], []])
    engine.close(slots)
    a, b = engine.open(2)
    engine.step([a, b], [[3, 17], [3, 18]], [[], []])
    got = engine.step([a, b], [[50], [50]]).cpu().numpy()
    want = np.stack([plain.forward(config, tensors, p)[-1] for p in ([3, 17, 50], [3, 18, 50])])
    compare(got, want, dtype, "the same token after different ones")
    assert np.abs(want[0] - want[1]).max() > 0.3 * want.std()


@pytest.mark.parametrize("name", list(CONFIGS))
def test_greedy_generation_through_the_engine(name, folders):
    engine, config, tensors = setup(folders, name, "float32")
    prompts = [p.tolist() for p in prompts_of(name, (7, 40, 1), seed=4)]
    got = engine.generate(prompts, 12, stop_at_eos=False)
    for p, g in zip(prompts, got):
        assert g.tolist() == plain.generate(config, tensors, p, 12)
    assert all(e.state == sakv.COMPLETE for e in engine.endings)
    engine.cache.check()
    assert engine.cache.slots.held == 0


def test_generation_in_bfloat16_follows_the_plain_model(folders):
    engine, config, tensors = setup(folders, "mixed", "bfloat16")
    prompts = [p.tolist() for p in prompts_of("mixed", (33, 5), seed=5)]
    got = engine.generate(prompts, 10, stop_at_eos=False)
    for p, g in zip(prompts, got):         # each token is the plain model's choice or a near tie
        ref = plain.forward(config, tensors, p + g.tolist()[:-1])[len(p) - 1:]
        for k, token in enumerate(g.tolist()):
            assert ref[k].max() - ref[k, token] <= 0.2 * ref[k].std()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_replay_program_runs_a_gozolix_folder(dtype, folders, tmp_path):
    from test_trace_run_gpu import Trace, entry
    folder = folders("mixed", dtype)
    config, tensors = plain.read_model_folder(folder)
    a, b, c = prompts_of("mixed", (90, 41, 3), seed=6)
    want = {k: plain.forward(config, tensors, p) for k, p in (("a", a), ("b", b), ("c", c))}

    def check(got, request, rows, what):
        compare(got, want[request][np.asarray(rows)], dtype, what)

    trace = Trace(folder, dtype, tmp_path / "out", 512)
    got = trace.send([entry("a", a[:80], range(80)), entry("b", b[:40], [0, 39]),
                      entry("c", c, [2])], end=["c"])
    check(got[:80], "a", range(80), "a's prompt")
    check(got[80:82], "b", [0, 39], "b's prompt")
    check(got[82:], "c", [2], "c")
    got = trace.send([entry("a", a[80:81], [0]), entry("b", b[40:], [0])], end=["b"])
    check(got[:1], "a", [80], "a, one token")
    check(got[1:], "b", [40], "b, one token")
    for t in range(81, 90):
        got = trace.send([entry("a", a[t:t + 1], [0])], end=["a"] if t == 89 else [])
        check(got, "a", [t], f"a alone at {t}")
    trace.finish()


def test_the_command_line_writes_and_runs_a_gozolix_folder(tmp_path):
    """`random-model` from a config.json, then `generate` and `throughput` on the folder."""
    import json
    from test_cli import run
    config = tmp_path / "config.json"
    config.write_text(json.dumps(CONFIGS["odd"][0]))
    run("random-model", "--config", str(config), "--seed", "3", "--out", str(tmp_path / "m"),
        "--stored-dtype", "float32")
    cfg, tensors = plain.read_model_folder(tmp_path / "m")
    assert cfg["architecture"] == "Gozolix" and tensors["bigram"].shape == (8, 100)
    assert "l5.mix.k" not in tensors and tensors["l0.mlp.router"].shape == (9, 100)
    (p,) = prompts_of("odd", (11,), seed=7)
    records, _ = run("generate", "--model", str(tmp_path / "m"), "--dtype", "float32",
                     "--ignore-eos", "--prompt-ids", ",".join(map(str, p)), "--new-tokens", "6")
    assert records[0]["tokens"] == plain.generate(cfg, tensors, p.tolist(), 6)
    records, _ = run("throughput", "--model", str(tmp_path / "m"), "--lengths", "70",
                     "--repeat", "1", "--warmup", "1", "--batch", "2")
    assert records[0]["decode_tokens_per_second"] > 0
