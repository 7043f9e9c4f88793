"""The kernels of the Felovik mechanisms, each alone against the plain functions, on inputs made
so that a fault shows: heads of very different sizes before a norm a head, queries on both
sides of a temperature's step, keys far back and at block borders that stand out among
hundreds (in prompts and decoded), a state that still holds a token hundreds of positions
back, step sizes from tiny to large, states carried over pieces of every size on slots left
dirty, branches of very different sizes before their norms, routers whose groups change the
choice, limits that bind."""

import numpy as np
import pytest
import torch

import plain_felovik as plain
from semantic_aware_adaptive_kv_cache_precision_b200 import ops
from semantic_aware_adaptive_kv_cache_precision_b200.ops import mixture
from test_venanex_kernels_gpu import DEV, TYPES, Cache, close, dev, i32, rounded, step_for
from test_zodirax_kernels_gpu import scan_step

pytestmark = pytest.mark.gpu


# -- learned positions ----------------------------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width", [1, 96, 100, 1000])
def test_embedding_with_a_scale_and_learned_positions(dtype, width):
    T = TYPES[dtype]
    rng = np.random.default_rng(width)
    table, pos = (rounded(rng.standard_normal((r, width)), T) for r in (50, 90))
    ids, positions = rng.integers(0, 50, 70), rng.permutation(90)[:70]
    got = ops.embed(i32(ids), dev(table, T), scale=3.0, positions=i32(positions),
                    position_table=dev(pos, T))
    want = table[ids] * 3.0 + pos[positions]
    assert got.dtype == torch.float32
    assert np.abs(got.cpu().numpy() - want).max() <= 1e-6 * np.abs(want).max()
    # an id or a position outside its table adds nothing
    got = ops.embed(i32([-1, 50, 3]), dev(table, T), scale=2.0, positions=i32([5, 6, 90]),
                    position_table=dev(pos, T)).cpu().numpy()
    assert np.array_equal(got, np.stack([pos[5], pos[6], 2.0 * table[3]]).astype(np.float32))
    plain_rows = ops.embed(i32(ids), dev(table, T))
    assert np.array_equal(plain_rows.cpu().numpy(), table[ids].astype(np.float32))


# -- the norm after the residual sum ----------------------------------------------------------

@pytest.mark.parametrize("width", [1, 7, 96, 100, 256, 1000, 1024, 2050, 4096, 8192, 9000])
@pytest.mark.parametrize("wdtype", [torch.float32, torch.bfloat16])
def test_the_norm_after_the_sum_with_one_output_and_with_two_normed_ones(width, wdtype):
    rng = np.random.default_rng(width)
    n, eps, alpha = 6, 1e-5, 2.7
    x, ya, yb = (dev(s * rng.standard_normal((n, width))) for s in (2.0, 40.0, 0.01))
    yb[3] *= 1e-2                                  # (so small that eps shows)
    w, wa, wb = (rounded(1 + 0.2 * rng.standard_normal(width), wdtype) for _ in range(3))
    x64, a64, b64 = (t.cpu().numpy().astype(np.float64) for t in (x, ya, yb))
    for two in (False, True):
        v = alpha * x64
        if two:
            v = v + 0.5 * (plain.rms_norm(a64, wa, 3e-5) + plain.rms_norm(b64, wb, 3e-5))
        else:
            v = v + a64
        want = plain.rms_norm(v, w, eps)
        more = dict(scale=0.5, branch_weight=dev(wa, wdtype), other=yb, other_weight=dev(wb, wdtype),
                    branch_eps=3e-5) if two else {}
        stream = x.clone()
        low = ops.rms_join(stream, ya, dev(w, wdtype), eps, alpha=alpha, out_dtype=torch.bfloat16,
                           **more)
        assert np.abs(stream.cpu().numpy() - want).max() <= 3e-6 * np.abs(want).max()
        assert torch.equal(low, stream.to(torch.bfloat16))
        alone = x.clone()
        assert ops.rms_join(alone, ya, dev(w, wdtype), eps, alpha=alpha, **more) is None
        assert torch.equal(alone, stream)
        # a row does not depend on what else is in the step
        row = x[2:3].clone()
        if two:
            more["other"] = yb[2:3].contiguous()
        ops.rms_join(row, ya[2:3].contiguous(), dev(w, wdtype), eps, alpha=alpha, **more)
        assert torch.equal(row[0], stream[2])
    both = x.clone()                               # two outputs as they are
    ops.rms_join(both, ya, dev(w, wdtype), eps, other=yb)
    want = plain.rms_norm(x64 + a64 + b64, w, eps)
    assert np.abs(both.cpu().numpy() - want).max() <= 3e-6 * np.abs(want).max()


# -- a norm a head, the temperature, the cache write --------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,temp", [
    (4, 2, 32, 24, {"coef": 0.4, "every": 37}), (6, 2, 20, 12, {"coef": 0.5, "every": 3}),
    (1, 1, 64, 320, None), (5, 1, 7, 36, {"coef": 1.5, "every": 64}), (12, 12, 128, 128, None)])
def test_a_norm_a_head_the_temperature_and_the_cache_write(dtype, heads, kv_heads, dim, vdim, temp):
    """Heads differ in size by a factor of a thousand: a norm over the whole projection, or one
    that mixes heads, would leave the small ones small. One head is so small that eps shows."""
    T = TYPES[dtype]
    rng = np.random.default_rng(dim)
    n, eps = 150, 1e-5
    qc, kc, vc = heads * dim, kv_heads * dim, kv_heads * vdim
    sizes = 10.0 ** rng.uniform(-1.5, 1.5, heads + kv_heads)
    sizes[0] = 3e-3
    per = np.repeat(sizes, dim)
    proj = dev(np.concatenate([rng.standard_normal((n, 5)), rng.standard_normal((n, qc + kc)) * per,
                               rng.standard_normal((n, vc))], 1))
    p64 = proj.cpu().numpy().astype(np.float64)
    q = plain.rms_norm(p64[:, 5:5 + qc].reshape(n, heads, dim), None, eps)
    k = plain.rms_norm(p64[:, 5 + qc:5 + qc + kc].reshape(n, kv_heads, dim), None, eps)
    factor = plain.query_temperature(n, temp)
    q = q * factor[:, None, None]
    cache = Cache(kv_heads, dim, vdim, T, seed=3)
    table = cache.table([0], n)
    step = step_for([0] * n, np.arange(n))
    got = ops.qk_prepare(proj, 5, 5 + qc, 5 + qc + kc, heads, kv_heads, dim, vdim, None, None, eps,
                         None, None, step.positions, step.token_seq, table, cache.keys,
                         cache.values, T, norm="head",
                         temperature=None if temp is None else dev(factor))
    for h in range(heads):                          # (each head against its own size)
        close(got[:, h * dim:(h + 1) * dim], q[:, h], T, f"queries of head {h}")
    rows = table[0].tolist()
    keys = torch.stack([cache.keys[rows[p // 64], :, p % 64] for p in range(n)])
    values = torch.stack([cache.values[rows[p // 64], :, p % 64] for p in range(n)])
    for g in range(kv_heads):
        close(keys[:, g], k[:, g], T, f"keys of head {g}")
    close(values, p64[:, 5 + qc + kc:].reshape(n, kv_heads, vdim), T, "values in the cache")
    # a weight a head's number, the same for all heads, and a rotation after the norm
    from semantic_aware_adaptive_kv_cache_precision_b200.config import RotarySpec
    from semantic_aware_adaptive_kv_cache_precision_b200.parts import RotaryHalf
    if dim % 2 == 0:
        import plain_zodirax
        wq, wk = (rounded(1 + 0.3 * rng.standard_normal(dim), T) for _ in range(2))
        turn = {"base": 500.0, "dims": dim // 2 - dim // 2 % 2 or 2}
        part = RotaryHalf(RotarySpec(dim, turn["dims"], turn["base"], 256), "", dtype)
        part.prepare(DEV, 256)
        got = ops.qk_prepare(proj, 5, 5 + qc, 5 + qc + kc, heads, kv_heads, dim, vdim, dev(wq, T),
                             dev(wk, T), eps, part.cos, part.sin, step.positions, step.token_seq,
                             table, cache.keys, cache.values, T, norm="head",
                             temperature=None if temp is None else dev(factor))
        close(got, plain_zodirax.rotate_front(q * wq, np.arange(n), turn).reshape(n, qc), T,
              "turned queries")


# -- causal attention with an element-wise gate ---------------------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [
    (4, 2, 32, 24), (2, 2, 16, 40), (6, 2, 20, 12), (5, 1, 12, 36), (4, 1, 128, 128), (1, 1, 64, 320)])
def test_keys_far_back_and_at_block_borders_with_an_elementwise_gate(dtype, heads, kv_heads, dim,
                                                                    vdim):
    """Keys at positions 0, 1, 63, 64, 255 and 256 stand out, each along a direction of its own;
    askers at block borders and far behind point at one of them each. The gates' rows are
    strided and differ from number to number."""
    T = TYPES[dtype]
    rng = np.random.default_rng(dim + vdim)
    n, scale, group = 700, 0.4, heads // kv_heads
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
    gates = dev(2.0 * rng.standard_normal((n, heads * vdim + 11)))[:, 5:5 + heads * vdim]
    g64 = gates.cpu().numpy().astype(np.float64)
    want = np.empty((n, heads, vdim))
    for h in range(heads):
        w = plain.causal_softmax(q[:, h] @ k[:, h // group].T * scale)
        for i, which in askers.items():
            assert special[which] <= i and w[i, special[which]] > 0.5
        want[:, h] = w @ v[:, h // group]
    want = want.reshape(n, -1) * plain.sigmoid(g64)
    cache = Cache(kv_heads, dim, vdim, T, seed=1)
    cache.put(0, k, v)
    table = cache.table([0], n)
    step = step_for([0] * n, np.arange(n))
    whole = ops.cached_attention(dev(q, T), cache.keys, cache.values, step.positions,
                                 step.token_seq, table, heads, dim, vdim, scale, elem_gate=gates)
    close(whole, want, T, "a prompt")
    rows = sorted(askers)
    some = dev(q[rows], T)
    for first, across in ((False, 1), (True, 1), (True, 3), (True, 16)):
        step = step_for([0] * len(rows), rows)
        got = ops.cached_attention(some, cache.keys, cache.values, step.positions, step.token_seq,
                                   table, heads, dim, vdim, scale, elem_gate=gates[rows].contiguous(),
                                   heads_first=first, key_splits=across)
        close(got, want[rows], T, f"decoded, {across} blocks a token")
    bare = ops.cached_attention(some, cache.keys, cache.values, step.positions, step.token_seq,
                                table, heads, dim, vdim, scale)
    close(bare, want[rows] / plain.sigmoid(g64[rows]), T, "no gate")


# -- the convolution inside a wider projection, the scan, the gate before the norm -----------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("heads,vdim,state,groups", [
    (4, 16, 24, 2), (3, 24, 16, 1), (5, 12, 7, 5), (3, 10, 1, 1), (6, 8, 40, 3), (2, 64, 160, 2),
    (4, 64, 128, 1), (1, 36, 36, 1), (2, 3, 200, 1), (8, 10, 24, 2), (7, 70, 64, 1)])
def test_dual_scan_over_pieces_with_a_token_far_back(dtype, heads, vdim, state, groups):
    """Head 0 hardly fades and is fed once, at token 2, far more than anything after it; the last
    token's C reads exactly that. Other heads fade within a token or two. Pieces down to one
    token give the same."""
    T = TYPES[dtype]
    rng = np.random.default_rng(vdim + state)
    lengths = (400, 5, 64)
    a_log = rng.uniform(-2.0, 2.5, heads)
    a_log[0] = -9.0
    bias = rng.uniform(-4.0, -1.0, heads)
    d_skip = 1 + 0.3 * rng.standard_normal(heads)
    bias, d_skip = (dev(t).cpu().numpy().astype(np.float64) for t in (bias, d_skip))
    a = dev(-np.exp(a_log)).cpu().numpy().astype(np.float64)
    inner, gn = heads * vdim, groups * state
    seqs = []
    for n in lengths:
        xbc = rng.standard_normal((n, 3 + inner + 2 * gn))               # columns before
        dt = 2.0 * rng.standard_normal((n, heads))
        if n > 100:
            xbc[2, 3:3 + vdim] = 80.0
            dt[2, 0] = 5.0
            xbc[-1, 3 + inner + gn:] = 3.0 * xbc[2, 3 + inner:3 + inner + gn]
        xbc, dt = rounded(xbc, T), dev(dt).cpu().numpy().astype(np.float64)
        x = xbc[:, 3:3 + inner].reshape(n, heads, vdim)
        B, C = (xbc[:, lo:lo + gn].reshape(n, groups, state) for lo in (3 + inner, 3 + inner + gn))
        steps = plain.softplus(dt + bias)
        y, last = plain.dual_scan(x, B, C, steps, np.log(-a), d_skip)
        if n > 100:                                 # the far token is felt at the last one
            bare = x.copy()
            bare[2, 0] = 0.0
            other, _ = plain.dual_scan(bare, B, C, steps, np.log(-a), d_skip)
            assert np.abs(y[-1, 0] - other[-1, 0]).max() > 0.3 * np.abs(y[-1, 0]).max()
        seqs.append((xbc, dt, y.reshape(n, inner), last))
    st = torch.full((5, heads, vdim, state), 3.0, device=DEV)
    # (the second number: tokens a run when a step's part of a sequence is walked in runs)
    for cuts, run in (((400, 5, 64), 0), ((1, 1, 1), 0), ((2, 2, 2), 0), ((63, 4, 33), 0),
                      ((399, 1, 64), 0), ((400, 5, 64), 64), ((400, 5, 64), 16), ((130, 5, 33), 32),
                      ((399, 1, 64), 7)):
        slots = [3, 0, 4]
        st[slots] = 0.0
        at = [0] * 3
        rows = [[] for _ in lengths]
        while any(u < n for u, n in zip(at, lengths)):
            live = [i for i in range(3) if at[i] < lengths[i]]
            take = [min(cuts[i], lengths[i] - at[i]) for i in live]
            step = scan_step(take, [slots[i] for i in live])
            cat = lambda j: np.concatenate([seqs[i][j][at[i]:at[i] + t] for i, t in zip(live, take)])
            wide = dev(np.concatenate([np.ones((sum(take), 2)), cat(1)], 1))        # strided rows
            out = ops.dual_scan(dev(cat(0), T), 3, 3 + inner, 3 + inner + gn, wide[:, 2:],
                                dev(bias), dev(a), dev(d_skip), heads, groups, state, vdim, st,
                                step, run=run)
            assert out.dtype == torch.float32
            for i, t, lo in zip(live, take, np.cumsum([0] + take)):
                rows[i].append(out[lo:lo + t])
                at[i] += t
        for i in range(3):                          # (fp32 sums of exact products in both types)
            close(torch.cat(rows[i]), seqs[i][2], torch.float32, f"cuts {cuts}, runs of {run}, {i}")
            close(st[slots[i]].transpose(1, 2), seqs[i][3], torch.float32, f"state {i}, {cuts}")
    before = st.clone()                             # a step that must leave the state as it was
    ops.dual_scan(dev(seqs[1][0], T), 3, 3 + inner, 3 + inner + gn, dev(seqs[1][1]), dev(bias),
                  dev(a), dev(d_skip), heads, groups, state, vdim, st, scan_step([5], [0]),
                  keep_state=False, run=2)
    assert torch.equal(st, before)


@pytest.mark.parametrize("heads,vdim,state,groups", [(6, 24, 40, 2), (4, 70, 128, 1), (8, 9, 16, 8)])
def test_a_full_step_and_single_sequences_give_the_same_bits(heads, vdim, state, groups):
    """Ninety sequences fill the GPU (several columns a thread), one does not (one column a
    thread): every output and state is the same to the bit."""
    g = torch.Generator(device=DEV).manual_seed(heads)
    lengths = [1 + 7 * i % 40 for i in range(90)]
    n, inner, gn = sum(lengths), heads * vdim, groups * state
    rand = lambda *shape: torch.randn(shape, generator=g, device=DEV)
    xbc, dt = rand(n, inner + 2 * gn), rand(n, heads)
    bias, a, skip = rand(heads) - 2.0, -torch.exp(rand(heads)), rand(heads)

    def run(x, d, lengths, slots, state_t):
        return ops.dual_scan(x, 0, inner, inner + gn, d, bias, a, skip, heads, groups, state, vdim,
                             state_t, scan_step(lengths, slots))

    together = torch.zeros((90, heads, vdim, state), device=DEV)
    out = run(xbc, dt, lengths, list(range(90)), together)
    at = 0
    for i, m in enumerate(lengths):
        if i % 9 == 0:
            alone = torch.zeros((1, heads, vdim, state), device=DEV)
            got = run(xbc[at:at + m], dt[at:at + m], [m], [0], alone)
            assert torch.equal(got, out[at:at + m]) and torch.equal(alone[0], together[i])
        at += m


def test_the_convolution_reads_columns_inside_a_wider_projection():
    rng = np.random.default_rng(5)
    n, channels = 90, 52
    wide = dev(rng.standard_normal((n, 20 + channels + 7)))
    w, b = dev(rng.standard_normal((channels, 4))), dev(rng.standard_normal(channels))
    x = wide.cpu().numpy().astype(np.float64)[:, 20:20 + channels]
    want = plain.causal_conv(x, w.cpu().numpy().astype(np.float64), b.cpu().numpy().astype(np.float64))
    state = torch.zeros((2, 3, channels), device=DEV)
    rows = []
    for lo, hi in ((0, 50), (50, 51), (51, 53), (53, 90)):
        rows.append(ops.causal_conv(wide[lo:hi, 20:20 + channels], channels, w, b, state,
                                    scan_step([hi - lo], [1]), torch.float32))
    close(torch.cat(rows), want, torch.float32)
    assert not state[0].any()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("width,parts", [(64, 2), (60, 5), (30, 10), (256, 1), (2048, 2), (96, 32),
                                         (3000, 1), (4096, 8), (4096, 16)])
def test_the_gate_comes_before_a_norm_in_parts(dtype, width, parts):
    T = TYPES[dtype]
    rng = np.random.default_rng(width + parts)
    n, eps = 7, 1e-5
    y = dev(rng.standard_normal((n, width)) * np.repeat(10.0 ** rng.uniform(-2, 2, parts), width // parts))
    z = dev(2.0 * rng.standard_normal((n, width + 3)))[:, 1:1 + width]
    w = rounded(1 + 0.2 * rng.standard_normal(width), T)
    y64, z64 = (t.cpu().numpy().astype(np.float64) for t in (y, z))
    got = ops.norm_gate(y, dev(w, T), z, eps, 1.0, T, group=width // parts, gate_silu=True,
                        gate_first=True)
    close(got, plain.gate_then_norm(y64, z64, w, parts, eps), T)
    after = ops.norm_gate(y, dev(w, T), z, eps, 1.0, T, group=width // parts, gate_silu=True)
    want = plain.rms_norm(y64.reshape(n, parts, -1), None, eps).reshape(n, width) * w * plain.silu(z64)
    close(after, want, T, "the gate after the norm")
    assert not torch.equal(after, got)


# -- the router over groups of experts, plain gated experts -----------------------------------------

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("n,width,experts,top,ff,groups", [
    (77, 96, 8, 3, 48, (4, 2)), (1, 64, 10, 4, 40, (5, 3)), (200, 64, 36, 6, 24, (6, 3)),
    (33, 100, 9, 1, 22, (9, 2)), (5, 72, 6, 4, 50, (3, 2)), (300, 128, 128, 8, 16, (64, 5)),
    (90, 64, 5, 2, 130, None), (70, 48, 4, 4, 32, (2, 2)), (150, 64, 80, 3, 16, (2, 1)),
    (64, 64, 80, 5, 16, (40, 7))])
def test_a_router_over_groups_with_weights_over_their_sum(dtype, n, width, experts, top, ff, groups):
    T = TYPES[dtype]
    rng = np.random.default_rng(n + experts)
    h = rounded(rng.standard_normal((n, width)), T)
    t = {"router": rounded(rng.standard_normal((experts, width)) * 0.3, torch.float32)}
    for e in range(experts):
        t[f"e{e}.gate"] = rounded(rng.standard_normal((ff, width)) * 0.2, T)
        t[f"e{e}.up"] = rounded(rng.standard_normal((ff, width)) * 0.2, T)
        t[f"e{e}.down"] = rounded(rng.standard_normal((width, ff)) * 0.2, T)
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    chosen, weights = plain.route(h, t, "", router)
    free, _ = plain.route(h, t, "", {"experts": experts, "top": top})
    if groups and n > 30 and groups[1] < min(groups[0], top):
        assert (np.sort(chosen, -1) != np.sort(free, -1)).any()        # the groups matter
    logits = mixture.router_logits(dev(h, T), dev(t["router"]))
    count, keep = groups or (1, 1)
    routing = mixture.route(logits, experts, top, softmax=True, groups=count, keep_groups=keep,
                            renormalize=True)
    got = routing.chosen.cpu().numpy()
    same = (got == chosen).all(-1)
    assert same.mean() > 0.97                   # (a close call may fall either way in 32 bits)
    gw = routing.weights.cpu().numpy()
    assert np.allclose(gw[same], weights[same], rtol=3e-5, atol=1e-7)
    assert np.allclose(gw.sum(-1), 1.0, atol=1e-5)
    assert all(len(set(row)) == top for row in got.tolist())
    if groups:
        size = experts // count
        assert all(len(set(e // size for e in row)) <= keep for row in got.tolist())
    # the one-block form and the two-launch form choose alike
    if n > mixture.ROUTE_IN_ONE_BLOCK:
        part = mixture.route(logits[:50].contiguous(), experts, top, softmax=True, groups=count,
                             keep_groups=keep, renormalize=True)
        assert torch.equal(part.chosen, routing.chosen[:50])
        assert torch.equal(part.weights, routing.weights[:50])
    rows = mixture.gather_rows(dev(h, T), routing, False)
    stack = lambda name: dev(np.stack([t[f"e{e}.{name}"] for e in range(experts)]), T)
    act = mixture.grouped_product(rows, routing, stack("gate"), stack("up"), float("inf"), 1.0, 0.0)
    products = mixture.grouped_product(act, routing, stack("down"), None)
    out = mixture.combine(products, routing, True)
    want = plain.experts(h, t, "", {"router": router})
    close(out.cpu()[torch.from_numpy(same)], want[same], T, "the routed experts")


def test_groups_and_a_correction_for_the_choice_together():
    """With a correction a group's score is its largest corrected score; the weights are not
    corrected."""
    rng = np.random.default_rng(3)
    z, bias = dev(rng.standard_normal((120, 12))), dev(0.3 * rng.standard_normal(12))
    r = mixture.route(z, 12, 3, softmax=True, bias=bias, groups=4, keep_groups=2, renormalize=True)
    z64 = z.cpu().numpy().astype(np.float64)
    s = np.exp(z64) / np.exp(z64).sum(-1, keepdims=True)
    choice = s + bias.cpu().numpy()
    best = choice.reshape(-1, 4, 3).max(-1)
    kept = np.argsort(-best, -1, kind="stable")[:, :2]
    mask = np.zeros((120, 4), dtype=bool)
    np.put_along_axis(mask, kept, True, -1)
    want = np.argsort(-np.where(np.repeat(mask, 3, -1), choice, -np.inf), -1, kind="stable")[:, :3]
    got = r.chosen.cpu().numpy()
    assert (got == want).all(-1).mean() > 0.97
    w = np.take_along_axis(s, got, -1)
    assert np.allclose(r.weights.cpu().numpy(), w / w.sum(-1, keepdims=True), rtol=3e-5)


# -- the clamped dense feed-forward --------------------------------------------------------------

@pytest.mark.parametrize("tokens,width,ff", [(1, 96, 128), (8, 256, 512), (40, 128, 384), (64, 200, 128),
                                             (100, 96, 80), (256, 256, 512), (300, 128, 264),
                                             (200, 512, 1024), (70, 100, 30), (5, 96, 80)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_clamped_product_in_every_form(dtype, tokens, width, ff):
    """Gates and ups reach far beyond the limit on both sides: the gate is bounded above only."""
    T = TYPES[dtype]
    rng = np.random.default_rng(tokens + ff)
    limit, alpha, plus = 1.5, 1.702, 1.0
    x = rounded(rng.standard_normal((tokens, width)), T)
    gate, up = (rounded(rng.standard_normal((ff, width)) * 3.0 / width ** 0.5, T) for _ in range(2))
    g, u = x @ gate.T, x @ up.T
    assert (g > limit).any() and (g < -limit).any() and (np.abs(u) > limit).any()
    gc = np.minimum(g, limit)
    want = gc * plain.sigmoid(alpha * gc) * (np.clip(u, -limit, limit) + plus)
    w = dev(np.concatenate([gate, up]), T)
    close(ops.gated_up(dev(x, T), w, (limit, alpha, plus)), want, T, "clamped")
    # an infinite limit, 1 and 0: the gated silu
    silu = ops.gated_up(dev(x, T), w, (float("inf"), 1.0, 0.0))
    close(silu, plain.silu(g) * u, T, "as the gated silu")
    close(ops.gated_up(dev(x, T), w), plain.silu(g) * u, T, "the gated silu")


# -- two branches with norms, as any block asks for them -------------------------------------------

def test_the_mixer_sums_its_branches_norms_for_a_block_that_does_not_join():
    """`produce` (the sum of the normed branches times the scale) is what `produce_branches` and
    the norms give, through a cache of its own."""
    from semantic_aware_adaptive_kv_cache_precision_b200 import Engine
    from felovik_configs import MIXED
    engine = Engine(config=dict(MIXED), dtype="float32", random_seed=3, max_tokens=256).load_weights()
    mixer = engine.model.blocks[0].mixer
    cache = engine._need_cache()
    h = torch.randn((9, 96), device=DEV)
    out = []
    for ask in (mixer.produce, mixer.produce_branches):
        (slot,) = engine.open(1)
        cache.reserve([slot], [9])
        ctx = engine._stager.build([slot], [list(range(9))], [0], [], cache.tables_for([slot]))
        out.append(ask(h, ctx, cache.entry_view(0, ctx.tables)))
        engine.close([slot])
    ya, yb = (y.cpu().numpy().astype(np.float64) for y in out[1])
    wa, wb = (n.weight.float().cpu().numpy().astype(np.float64) for n in mixer.norms)
    want = 0.5 * (plain.rms_norm(ya, wa, 1e-5) + plain.rms_norm(yb, wb, 1e-5))
    close(out[0], want, torch.float32)
