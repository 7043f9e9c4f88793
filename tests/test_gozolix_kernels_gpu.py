"""The kernels of the Gozolix mechanisms, each alone against the plain functions, on inputs made so
that a fault shows: pairs of tokens across the pieces of a prompt, a state that still holds a token
hundreds of positions back, tokens whose keys nearly coincide inside a group of four, betas and
decays from 0 to 1, states carried over pieces of every size on slots left dirty, keys far back and
at block borders that stand out among hundreds (in prompts and decoded) in spite of the distance
penalty, scores far beyond the cap, routers whose groups' second best experts decide."""

import numpy as np
import pytest
import torch

import plain_gozolix as plain
from semantic_aware_adaptive_kv_cache_precision_b200 import ops
from semantic_aware_adaptive_kv_cache_precision_b200.ops import mixture
from test_venanex_kernels_gpu import DEV, TYPES, Cache, close, dev, i32, rounded, step_for
from test_zodirax_kernels_gpu import scan_step

pytestmark = pytest.mark.gpu


# -- the table of pairs -----------------------------------------------------------------------

def pairs_step(counts, starts, slots, ids):
    step = scan_step(counts, slots)
    step.token_ids = i32(np.concatenate(ids))
    step.positions = i32(np.concatenate([np.arange(s, s + n) for s, n in zip(starts, counts)]))
    step.token_seq = i32(np.repeat(np.arange(len(counts)), counts))
    return step


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,buckets,mul_prev,mul_cur", [
    (96, 101, 13, 5), (1, 7, 3, 2), (100, 1, 1, 1), (1030, 60000, 2000003, 1999993)])
def test_pairs_of_tokens_over_pieces(dtype, width, buckets, mul_prev, mul_cur):
    """Three sequences in pieces on slots whose last user left another token behind."""
    T = TYPES[dtype]
    rng = np.random.default_rng(width)
    lengths, slots = (40, 1, 17), (4, 0, 2)
    table = rounded(rng.standard_normal((400, width)), T)
    pairs = rounded(rng.standard_normal((buckets + 1, width)), T)
    seqs = [rng.integers(0, 400, n) for n in lengths]
    b = {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}
    want = [plain.embed({"embed": table, "bigram": pairs}, s, {"scale": 3.0, "bigram": b}) for s in seqs]
    for cuts in ((40, 1, 17), (1, 1, 1), (2, 1, 3), (39, 1, 16)):
        last = torch.full((5, 1), 77, dtype=torch.int32, device=DEV)
        at, rows = [0] * 3, [[] for _ in seqs]
        while any(u < n for u, n in zip(at, lengths)):
            live = [i for i in range(3) if at[i] < lengths[i]]
            take = [min(cuts[i], lengths[i] - at[i]) for i in live]
            step = pairs_step(take, [at[i] for i in live], [slots[i] for i in live],
                              [seqs[i][at[i]:at[i] + t] for i, t in zip(live, take)])
            out = ops.embed_pairs(step, dev(table, T), dev(pairs, T), mul_prev, mul_cur, last, scale=3.0)
            for i, t, lo in zip(live, take, np.cumsum([0] + take)):
                rows[i].append(out[lo:lo + t].cpu().numpy())
                at[i] += t
        for i in range(3):
            got = np.concatenate(rows[i])
            assert np.abs(got - want[i]).max() <= 1e-6 * np.abs(want[i]).max(), (cuts, i)
            assert int(last[slots[i], 0]) == seqs[i][-1]
        assert int(last[1, 0]) == int(last[3, 0]) == 77


# -- the square of relu ----------------------------------------------------------------------

@pytest.mark.parametrize("tokens,width,ff", [(1, 96, 128), (8, 256, 520), (40, 128, 384), (64, 200, 30),
                                             (100, 96, 80), (300, 128, 264), (70, 100, 31), (5, 96, 7)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_square_of_relu_in_every_form(dtype, tokens, width, ff):
    T = TYPES[dtype]
    rng = np.random.default_rng(tokens + ff)
    x, w = rounded(rng.standard_normal((tokens, width)), T), rounded(rng.standard_normal((ff, width)), T)
    want = np.maximum(x @ w.T, 0.0) ** 2
    close(ops.dense_up(dev(x, T), dev(w, T)), want, T)
    z = rounded(rng.standard_normal((tokens, ff)), T)
    close(ops.relu_squared(dev(z, T)), np.maximum(z, 0) ** 2, T)


# -- the gated delta rule ---------------------------------------------------------------------

def delta_case(rng, n, heads, kv_heads, dim, vdim):
    """Pre-activations [n, columns] as the device holds them, and where the parts begin."""
    channels = 2 * kv_heads * dim + heads * vdim
    proj = rng.standard_normal((n, channels + 3 + 2 * heads))
    a_off, b_off = channels + 3, channels + 3 + heads
    proj[:, a_off:] *= 3.0
    if n > 100:                   # token 2 writes far more than anything after it, into head 0 above all
        proj[3:, b_off] = -4.0
        proj[2, 2 * kv_heads * dim:channels] = 60.0
        proj[2, b_off:] = 20.0
    return dev(proj).cpu().numpy().astype(np.float64), channels, a_off, b_off


def delta_plain(proj, conv, a, bias, heads, kv_heads, dim, vdim, a_off, b_off):
    n, qk = proj.shape[0], kv_heads * dim
    x = plain.causal_conv(proj[:, :2 * qk + heads * vdim], conv)
    q = plain.unit(x[:, :qk].reshape(n, kv_heads, dim)) * dim ** -0.5
    k = plain.unit(x[:, qk:2 * qk].reshape(n, kv_heads, dim))
    g = np.exp(a * plain.softplus(proj[:, a_off:a_off + heads] + bias))
    beta = plain.sigmoid(proj[:, b_off:b_off + heads])
    o, S = plain.delta_scan(q, k, x[:, 2 * qk:].reshape(n, heads, vdim), g, beta)
    return o.reshape(n, -1), S


@pytest.mark.parametrize("wdtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [
    (4, 2, 24, 16, 4), (3, 3, 7, 10, 6), (5, 1, 20, 12, 1), (1, 1, 4, 50, 2), (4, 2, 128, 128, 4),
    (2, 1, 256, 64, 5), (8, 4, 64, 48, 3), (2, 2, 300, 9, 4), (40, 1, 32, 8, 4), (2, 2, 512, 20, 9),
    (6, 3, 33, 70, 4)])
def test_the_delta_rule_over_pieces_with_a_token_far_back(wdtype, heads, kv_heads, dim, vdim, taps):
    """Head 0 hardly fades, and a token near the start writes far more than those after it; other
    heads fade within a token or two. Pieces down to one token give the same, by groups of four and
    one by one, on slots left dirty by others."""
    rng = np.random.default_rng(dim + vdim + taps)
    lengths, slots = (230, 5, 64), (3, 0, 4)
    a_log = rng.uniform(-2.0, 2.0, heads)
    a_log[0] = -9.0
    a = dev(-np.exp(a_log)).cpu().numpy().astype(np.float64)
    bias = dev(rng.uniform(-4.0, 0.0, heads)).cpu().numpy().astype(np.float64)
    channels = 2 * kv_heads * dim + heads * vdim
    conv = rounded(rng.uniform(-1, 1, (channels, taps)), TYPES[wdtype])
    seqs = []
    for n in lengths:
        proj, channels, a_off, b_off = delta_case(rng, n, heads, kv_heads, dim, vdim)
        seqs.append((proj,) + delta_plain(proj, conv, a, bias, heads, kv_heads, dim, vdim, a_off, b_off))
    bare = seqs[0][0].copy()              # without token 2's values the last token reads otherwise
    bare[2, 2 * kv_heads * dim:channels] = 0.0
    other, _ = delta_plain(bare, conv, a, bias, heads, kv_heads, dim, vdim, a_off, b_off)
    o = seqs[0][1]
    assert np.abs(o[-1, :vdim] - other[-1, :vdim]).max() > 0.05 * np.abs(o[-1, :vdim]).max()
    st = torch.zeros((5, heads, vdim, dim), device=DEV)
    cs = torch.zeros((5, taps - 1, channels), device=DEV)
    exact = None
    for cuts, groups in (((230, 5, 64), False), ((230, 5, 64), True), ((1, 1, 1), False), ((2, 2, 2), True),
                         ((3, 4, 33), True), ((63, 4, 33), False), ((229, 1, 63), True), ((6, 5, 7), True)):
        st.fill_(3.0)
        cs.fill_(3.0)
        st[list(slots)], cs[list(slots)] = 0.0, 0.0
        at, rows = [0] * 3, [[] for _ in lengths]
        while any(u < n for u, n in zip(at, lengths)):
            live = [i for i in range(3) if at[i] < lengths[i]]
            take = [min(cuts[i], lengths[i] - at[i]) for i in live]
            step = scan_step(take, [slots[i] for i in live])
            cat = np.concatenate([seqs[i][0][at[i]:at[i] + t] for i, t in zip(live, take)])
            out = ops.gated_delta(dev(cat), a_off, b_off, dev(conv, TYPES[wdtype]), dev(a), dev(bias), cs, st,
                                  step, heads, kv_heads, dim, vdim, dim ** -0.5, plain.UNIT_EPS,
                                  by_groups=groups)
            for i, t, lo in zip(live, take, np.cumsum([0] + take)):
                rows[i].append(out[lo:lo + t])
                at[i] += t
        for i in range(3):
            close(torch.cat(rows[i]), seqs[i][1], torch.float32, f"cuts {cuts}, groups {groups}, {i}")
            close(st[slots[i]].transpose(1, 2), seqs[i][2], torch.float32, f"state {i}, {cuts}")
        assert (st[1] == 3.0).all() and (cs[2] == 3.0).all()
        if not groups:                    # one by one: the same bits however the tokens come
            now = [torch.cat(r) for r in rows]
            exact = exact or now
            assert all(torch.equal(x, y) for x, y in zip(exact, now)), cuts
    before = st.clone(), cs.clone()       # steps that must leave the state as it was
    for n, groups in ((5, True), (5, False), (1, False)):
        ops.gated_delta(dev(seqs[1][0][:n]), a_off, b_off, dev(conv, TYPES[wdtype]), dev(a), dev(bias), cs, st,
                        scan_step([n], [0]), heads, kv_heads, dim, vdim, dim ** -0.5, plain.UNIT_EPS,
                        keep_state=False, by_groups=groups)
    assert torch.equal(st, before[0]) and torch.equal(cs, before[1])


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 64, 32), (2, 1, 128, 40), (3, 3, 16, 8)])
def test_groups_whose_keys_nearly_coincide_and_betas_at_their_ends(heads, kv_heads, dim, vdim):
    """Inside every group of four the keys are nearly one (the correction between its tokens is as
    large as it gets), betas are nearly 0 or 1, decays nearly 0 or 1."""
    rng = np.random.default_rng(dim)
    n, qk = 50, kv_heads * dim
    proj, channels, a_off, b_off = delta_case(rng, n, heads, kv_heads, dim, vdim)
    base = 2.0 * rng.standard_normal((13, qk))
    proj[:, qk:2 * qk] = np.repeat(base, 4, 0)[:n] + 0.02 * rng.standard_normal((n, qk))
    proj[:, :qk] = proj[:, qk:2 * qk] + 0.1 * rng.standard_normal((n, qk))
    proj[:, b_off:] = rng.choice([-12.0, 12.0, 3.0], (n, heads))
    proj[:, a_off:b_off] = np.where(rng.random((n, heads + b_off - a_off - heads)) < 0.2, 30.0, -12.0)
    proj = dev(proj).cpu().numpy().astype(np.float64)
    conv = np.ones((channels, 1))
    a, bias = -np.ones(heads), np.zeros(heads)
    want, S = delta_plain(proj, conv, a, bias, heads, kv_heads, dim, vdim, a_off, b_off)
    for groups in (False, True):
        st = torch.zeros((1, heads, vdim, dim), device=DEV)
        cs = torch.zeros((1, 0, channels), device=DEV)
        out = ops.gated_delta(dev(proj), a_off, b_off, dev(conv), dev(a), dev(bias), cs, st,
                              scan_step([n], [0]), heads, kv_heads, dim, vdim, dim ** -0.5, plain.UNIT_EPS,
                              by_groups=groups)
        close(out, want, torch.float32, f"groups {groups}")
        close(st[0].transpose(1, 2), S, torch.float32, f"state, groups {groups}")


@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(6, 3, 40, 24), (4, 4, 128, 70), (8, 8, 24, 33),
                                                     (2, 1, 256, 40), (2, 2, 300, 36)])
def test_ninety_sequences_at_once_and_one_alone(heads, kv_heads, dim, vdim):
    """Ninety sequences fill the GPU (by groups a thread then has two columns), one does not. One
    by one every output and state is the same to the bit."""
    g = torch.Generator(device=DEV).manual_seed(heads)
    lengths = [2 + 7 * i % 40 for i in range(90)]
    channels = 2 * kv_heads * dim + heads * vdim
    proj = torch.randn((sum(lengths), channels + 2 * heads), generator=g, device=DEV)
    conv = torch.randn((channels, 4), generator=g, device=DEV)
    a, bias = -torch.rand(heads, generator=g, device=DEV), torch.zeros(heads, device=DEV)

    def run(rows, lengths, slots, groups):
        cs = torch.zeros((len(lengths), 3, channels), device=DEV)
        st = torch.zeros((len(lengths), heads, vdim, dim), device=DEV)
        return ops.gated_delta(rows, channels, channels + heads, conv, a, bias, cs, st,
                               scan_step(lengths, slots), heads, kv_heads, dim, vdim, dim ** -0.5,
                               plain.UNIT_EPS, by_groups=groups), st, cs

    for groups in (False, True):
        out, st, cs = run(proj, lengths, list(range(90)), groups)
        for i in range(0, 90, 9):
            lo = sum(lengths[:i])
            o1, s1, c1 = run(proj[lo:lo + lengths[i]], [lengths[i]], [0], groups)
            assert torch.equal(c1[0], cs[i])
            if groups:
                wide = out[lo:lo + lengths[i]].double().cpu().numpy()
                close(o1, wide, torch.float32, f"sequence {i}")
                close(s1[0], st[i].double().cpu().numpy(), torch.float32, f"state {i}")
            else:
                assert torch.equal(o1, out[lo:lo + lengths[i]]) and torch.equal(s1[0], st[i])


# -- attention with a cap, a linear distance penalty, and another layer's cache -----------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,cap", [
    (4, 2, 32, 24, 9.0), (2, 2, 16, 40, None), (6, 2, 20, 12, 12.0), (5, 1, 12, 36, 20.0),
    (8, 1, 128, 128, 15.0), (1, 1, 64, 320, 1000.0)])
def test_capped_scores_and_a_linear_penalty_with_keys_far_back_and_at_block_borders(
        dtype, heads, kv_heads, dim, vdim, cap):
    """Keys at positions 0, 1, 63, 64, 255 and 256 stand out, each along a direction of its own;
    askers at block borders and behind point at one of them each. The slopes differ by a factor of
    thousands from head to head: in the flat ones a key 600 places back still decides, in the steep
    one only the neighbours count. Scores reach far beyond the cap."""
    T = TYPES[dtype]
    rng = np.random.default_rng(dim + vdim)
    n, scale, group = 700, 0.7, heads // kv_heads
    k = 0.3 * rng.standard_normal((n, kv_heads, dim))
    v = rng.standard_normal((n, kv_heads, vdim))
    q = 0.3 * rng.standard_normal((n, heads, dim))
    special = [0, 1, 63, 64, 255, 256]
    rays = np.linalg.qr(rng.standard_normal((dim, dim)))[0][:len(special)]
    for p, ray in zip(special, rays):
        k[p] = 6.0 * ray
    askers = {63: 0, 64: 1, 65: 2, 256: 4, 257: 5, 320: 3, 511: 2, 640: 5, 698: 0, 699: 1}
    for i, which in askers.items():
        q[i] = 9.0 * rays[which]
    k, v, q = rounded(k, T), rounded(v, T), rounded(q, T)
    slopes = plain.head_slopes(heads) if heads > 1 else np.array([2.0 ** -8])
    slopes = dev(slopes).cpu().numpy().astype(np.float64)
    distance = np.arange(n)[:, None] - np.arange(n)[None, :]
    want, uncapped, flat = (np.empty((n, heads, vdim)) for _ in range(3))
    for h in range(heads):
        s = q[:, h] @ k[:, h // group].T * scale
        want[:, h] = plain.causal_softmax(plain.soft_cap(s, cap) - slopes[h] * distance) @ v[:, h // group]
        uncapped[:, h] = plain.causal_softmax(s - slopes[h] * distance) @ v[:, h // group]
        flat[:, h] = plain.causal_softmax(plain.soft_cap(s, cap)) @ v[:, h // group]
    rows = sorted(askers)
    assert cap is None or cap > 100 or np.abs(want - flat)[rows].max() > 0.05
    assert cap is None or cap > 100 or np.abs(want - uncapped)[rows].max() > 0.05
    want = want.reshape(n, -1)
    cache = Cache(kv_heads, dim, vdim, T, seed=1)
    cache.put(0, k, v)
    table = cache.table([0], n)
    step = step_for([0] * n, np.arange(n))
    more = dict(softcap=cap, linear_slopes=dev(slopes))
    whole = ops.cached_attention(dev(q, T), cache.keys, cache.values, step.positions,
                                 step.token_seq, table, heads, dim, vdim, scale, **more)
    close(whole, want, T, "a prompt")
    some = dev(q[rows], T)
    for first, across in ((False, 1), (True, 1), (True, 3), (True, 16)):
        step = step_for([0] * len(rows), rows)
        got = ops.cached_attention(some, cache.keys, cache.values, step.positions, step.token_seq,
                                   table, heads, dim, vdim, scale, heads_first=first,
                                   key_splits=across, **more)
        close(got, want[rows], T, f"decoded, {across} blocks a token")
    if dtype == "float32":          # a piece of the prompt: the same bits
        step = step_for([0] * 100, np.arange(413, 513))
        part = ops.cached_attention(dev(q[413:513], T), cache.keys, cache.values, step.positions,
                                    step.token_seq, table, heads, dim, vdim, scale, **more)
        assert torch.equal(part, whole[413:513])


def test_a_layer_that_reads_another_s_cache_leaves_it_as_it_is():
    """`qk_prepare` without a cache write makes the queries alone, from a projection that holds
    nothing else."""
    rng = np.random.default_rng(2)
    heads, kv_heads, dim, vdim, n = 4, 2, 20, 12, 70
    proj = dev(rng.standard_normal((n, heads * dim)))
    cache = Cache(kv_heads, dim, vdim, torch.float32, seed=1)
    table = cache.table([0], n)
    cache.keys.normal_()
    cache.values.normal_()
    before = cache.keys.clone(), cache.values.clone()
    step = step_for([0] * n, np.arange(n))
    f = plain.query_temperature(n, {"coef": 0.5, "every": 7})
    got = ops.qk_prepare(proj, 0, 0, 0, heads, kv_heads, dim, vdim, None, None, 0.0, None, None,
                         step.positions, step.token_seq, table, cache.keys, cache.values,
                         torch.float32, write_cache=False, norm=None, temperature=dev(f))
    close(got, proj.cpu().numpy().astype(np.float64) * f[:, None], torch.float32)
    assert torch.equal(cache.keys, before[0]) and torch.equal(cache.values, before[1])


# -- a router over groups scored by their two best experts ----------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,width,experts,top,ff,groups,shared,scale", [
    (77, 96, 8, 3, 48, (4, 2), 40, 2.5), (1, 64, 10, 4, 40, (5, 3), None, 1.0),
    (200, 64, 36, 6, 24, (6, 3), 24, 0.5), (33, 100, 9, 1, 22, (9, 2), 30, 1.0),
    (300, 128, 128, 8, 16, (32, 5), None, 16.0), (90, 64, 5, 2, 130, None, 64, 3.0),
    (70, 48, 4, 4, 32, (2, 2), None, 1.5), (150, 64, 80, 3, 16, (2, 1), 16, 2.0)])
def test_a_router_whose_groups_are_scored_by_their_two_best(dtype, n, width, experts, top, ff, groups,
                                                            shared, scale):
    T = TYPES[dtype]
    rng = np.random.default_rng(n + experts)
    h = rounded(rng.standard_normal((n, width)), T)
    t = {"router": rounded(rng.standard_normal((experts, width)) * 0.2, torch.float32)}
    for e, f in [(f"e{i}", ff) for i in range(experts)] + ([("shared", shared)] if shared else []):
        t[e + ".gate"] = rounded(rng.standard_normal((f, width)) * 0.2, T)
        t[e + ".up"] = rounded(rng.standard_normal((f, width)) * 0.2, T)
        t[e + ".down"] = rounded(rng.standard_normal((width, f)) * 0.2, T)
    router = {"experts": experts, "top": top, "scale": scale}
    count, keep = groups or (1, 1)
    if groups:
        router["groups"] = {"count": count, "keep": keep}
    chosen, weights = plain.route(h, t, "", router)
    logits = mixture.router_logits(dev(h, T), dev(t["router"]))
    how = dict(groups=count, keep_groups=keep, renormalize=True, group_top=2, scale=scale)
    routing = mixture.route(logits, experts, top, **how)
    got = routing.chosen.cpu().numpy()
    same = (got == chosen).all(-1)
    assert same.mean() > 0.97                   # (a close call may fall either way in 32 bits)
    gw = routing.weights.cpu().numpy()
    assert np.allclose(gw[same], weights[same], rtol=3e-5, atol=1e-7)
    assert np.allclose(gw.sum(-1), scale, rtol=1e-5)
    if groups and experts // count > 1 and keep < count and n > 30:    # the second best decides
        best = mixture.route(logits, experts, top, **dict(how, group_top=1))
        assert (np.sort(best.chosen.cpu().numpy(), -1) != np.sort(got, -1)).any()
    if n > mixture.ROUTE_IN_ONE_BLOCK:          # the one-block form and the two-launch form
        part = mixture.route(logits[:50].contiguous(), experts, top, **how)
        assert torch.equal(part.chosen, routing.chosen[:50])
        assert torch.equal(part.weights, routing.weights[:50])
    rows = mixture.gather_rows(dev(h, T), routing, False)
    stack = lambda name: dev(np.stack([t[f"e{e}.{name}"] for e in range(experts)]), T)
    act = mixture.grouped_product(rows, routing, stack("gate"), stack("up"), float("inf"), 1.0, 0.0)
    products = mixture.grouped_product(act, routing, stack("down"), None)
    side = None
    if shared:
        both = ops.linear(dev(h, T), dev(np.concatenate([t["shared.gate"], t["shared.up"]]), T))
        side = ops.linear(mixture.clamped_act(both, float("inf"), 1.0, 0.0), dev(t["shared.down"], T),
                          out_dtype=torch.float32)
    out = mixture.combine(products, routing, True, side)
    want = plain.experts(h, t, "", {"router": router, "shared": shared and {"ff": shared}})
    close(out.cpu()[torch.from_numpy(same)], want[same], T, "the experts")


def test_groups_scored_by_two_with_a_correction_for_the_choice():
    """With a correction a group's score is the sum of its two best corrected scores; the weights
    are not corrected."""
    rng = np.random.default_rng(3)
    z, bias = dev(rng.standard_normal((120, 12))), dev(0.3 * rng.standard_normal(12))
    r = mixture.route(z, 12, 3, bias=bias, groups=3, keep_groups=2, renormalize=True, group_top=2)
    s = plain.sigmoid(z.cpu().numpy().astype(np.float64))
    choice = s + bias.cpu().numpy()
    best = np.sort(choice.reshape(-1, 3, 4), -1)[:, :, -2:].sum(-1)
    kept = np.argsort(-best, -1, kind="stable")[:, :2]
    mask = np.zeros((120, 3), dtype=bool)
    np.put_along_axis(mask, kept, True, -1)
    want = np.argsort(-np.where(np.repeat(mask, 4, -1), choice, -np.inf), -1, kind="stable")[:, :3]
    got = r.chosen.cpu().numpy()
    assert (got == want).all(-1).mean() > 0.97
    w = np.take_along_axis(s, got, -1)
    assert np.allclose(r.weights.cpu().numpy(), w / w.sum(-1, keepdims=True), rtol=3e-5)
