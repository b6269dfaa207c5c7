"""The mechanisms of the Sosepel design one by one, each built from its own parameters with weights of its own, against the
plain functions: differential attention (sizes, portions, far keys, block borders, cap, temperature), the pair embedding and
its state, sigmoid routing in groups with shares, the gated shared expert, and the kernel that joins a block's branches."""
import numpy as np
import pytest
import torch

import helpers
from plain import sosepel_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def _name(dtype):
    return "float32" if dtype == torch.float32 else "bfloat16"


def _context(cache, slot_tokens, dtype, vocab=10):
    from hymt2sharp_b200.engine.engine import StepEntry, make_context
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    entries = [StepEntry(s, t if isinstance(t, list) else [0] * t, []) for s, t in slot_tokens]
    ctx, _, _, plan = make_context(cache, entries, vocab, dtype, DEV, status)
    return ctx, plan


def _cache(mixer, dtype, tokens=4096, slots=4, state_bytes=0):
    from hymt2sharp_b200.cache import GroupSpec, PagedCache
    from hymt2sharp_b200.parts import MixerSlot
    n = mixer.cache_need()
    cache = PagedCache([GroupSpec(n.kind, n.kv_heads, n.head_dim, 1, n.window, n.streams, n.value_dim)], dtype, DEV, tokens, max_slots=slots,
                       state_bytes=state_bytes)
    slot = MixerSlot()
    slot.group, slot.plane = 0, 0
    return cache, slot


def _attention(hidden, m, eps=1e-5):
    from hymt2sharp_b200.parts import PartSpec, build_part
    temp = m.get("q_temp") or dict(coef=0.0, every=1)
    return build_part("mixer", PartSpec("diff_attention", dict(
        hidden=hidden, heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], vdim=m["vdim"], scale=m["scale"], eps=eps, diff=m["diff"],
        softcap=m.get("softcap"), temp_coef=temp["coef"], temp_every=temp["every"], q_proj="q", k_proj="k", v_proj="v", o_proj="o",
        lambdas=["lq1", "lk1", "lq2", "lk2"])))


def _weights(part, scale=0.1):
    return {n: (torch.randn(s.shape) * (scale if len(s.shape) == 2 else 0.4 / s.shape[0] ** 0.5)).to(torch.bfloat16) for n, s in part.tensors().items()}


def _run(part, cache, mslot, schedule, xs, dtype):
    """schedule: [[(sequence index, tokens), ...], ...]; xs[i] [T_i, hidden]; returns per sequence what the mixer wrote."""
    slots, at, outs = {}, {i: 0 for i in range(len(xs))}, {i: [] for i in range(len(xs))}
    for step in schedule:
        for i, _ in step:
            if i not in slots:
                slots[i] = cache.alloc_slots(1)[0]
        ctx, plan = _context(cache, [(slots[i], n) for i, n in step], dtype)
        x = torch.cat([xs[i][at[i]:at[i] + n] for i, n in step]).to(DEV).to(dtype)
        res = torch.full((x.shape[0], xs[0].shape[1]), float("nan"), dtype=torch.float32, device=DEV)
        part.forward(x, res, ctx, mslot, store=True)
        cache.end_step(plan)
        assert int(ctx.status[0]) == 0
        from hymt2sharp_b200.kernels import ops
        assert int(ops.device_status(torch.device(DEV))[0]) == 0
        o = 0
        for i, n in step:
            outs[i].append(res[o:o + n].cpu()); o += n; at[i] += n
    cache.free_slots(list(slots.values()))
    return [torch.cat(outs[i]) for i in range(len(xs))]


MIXERS = {
    "odd": (44, dict(heads=3, kv_heads=1, dim=5, vdim=6, scale=3.0, diff=0.2, softcap=4.0, q_temp=dict(coef=0.7, every=3))),
    "wide": (64, dict(heads=2, kv_heads=2, dim=136, vdim=264, scale=0.3, diff=0.5, softcap=3.0, q_temp=dict(coef=-0.1, every=10))),
    "tc 64/128": (128, dict(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.6, diff=0.3, softcap=9.0, q_temp=dict(coef=0.3, every=64))),
    "tc 64/128, 8 heads on one": (96, dict(heads=8, kv_heads=1, dim=64, vdim=128, scale=0.6, diff=0.4, softcap=30.0, q_temp=dict(coef=0.2, every=50))),
    "tc 64/128, 3 heads on each": (128, dict(heads=6, kv_heads=2, dim=64, vdim=128, scale=0.5, diff=0.35, softcap=15.0, q_temp=dict(coef=0.1, every=7))),
    "tc 64/128, no cap": (128, dict(heads=2, kv_heads=1, dim=64, vdim=128, scale=0.3, diff=0.3)),
    "tc 64/128, a cap too wide for a fixed offset": (128, dict(heads=2, kv_heads=1, dim=64, vdim=128, scale=0.6, diff=0.3, softcap=90.0, q_temp=dict(coef=0.2, every=20))),
    "tc 32/64": (96, dict(heads=6, kv_heads=2, dim=32, vdim=64, scale=0.9, diff=0.25, softcap=6.0, q_temp=dict(coef=0.3, every=40))),
    "tc 32/128": (64, dict(heads=2, kv_heads=1, dim=32, vdim=128, scale=0.9, diff=0.7, softcap=20.0)),
    "tc 128/64": (128, dict(heads=2, kv_heads=1, dim=128, vdim=64, scale=0.4, diff=0.3, softcap=7.0, q_temp=dict(coef=0.5, every=100))),
    "tc 128/128": (128, dict(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.4, diff=0.3, softcap=25.0)),
}

SCHEDULES = {
    "whole": lambda n, m: [[(0, n), (1, m)]],
    "portions down to two tokens": lambda n, m: [[(0, 2), (1, 3)], [(0, 67), (1, 2)], [(0, n - 69), (1, m - 5)]],
    "a prompt and single tokens": lambda n, m: [[(0, n - 40), (1, m - 10)]] + [[(0, 1), (1, 1)]] * 10 + [[(0, 1)]] * 30,
}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_differential_attention_in_every_schedule(name, dtype):
    """Two unequal sequences, in a cache that was poisoned and whose slots and blocks another, longer pair held before."""
    hidden, m = MIXERS[name]
    torch.manual_seed(len(name))
    part = _attention(hidden, m)
    w = _weights(part)
    part.load(w, DEV, dtype)
    cache, slot = _cache(part, dtype)
    for s in cache.storage:
        s.fill_(float("nan"))
    xs = [torch.randn(n, hidden).to(torch.bfloat16).float() for n in (333, 29)]
    w64 = {k: v.to(F64) for k, v in w.items()}
    refs = [plain.attention(x.to(F64), w64, "", m, 1e-5) for x in xs]
    _run(part, cache, slot, [[(0, 400), (1, 190)]], [torch.randn(400, hidden), torch.randn(190, hidden)], dtype)
    for what, cuts in SCHEDULES.items():
        for x, got, ref in zip(xs, _run(part, cache, slot, cuts(333, 29), xs, dtype), refs):
            helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} {what} ({len(x)})", factor=2.0)
    cache.book.audit()


def _standing_out(m, hidden, T, query, key):
    """Inputs and weights in which `query`'s scores for `key` stand out in map 1 and nothing else does: channel 0 is on at the
    query alone, channel 1 at the key alone; map 1's first entries read them."""
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    x = torch.randn(T, hidden).to(torch.bfloat16).float() * 0.5
    x[:, :2] = 0.0
    x[query, 0], x[key, 1] = 1.0, 1.0
    part = _attention(hidden, m)
    w = {k: v.float() for k, v in _weights(part, scale=0.05).items()}
    for h in range(H):
        w["q"][h * 2 * d, :] = 0.0
        w["q"][h * 2 * d, 0] = 12.0
    for g in range(G):
        w["k"][g * 2 * d, :] = 0.0
        w["k"][g * 2 * d, 1] = 12.0
    return part, {k: v.to(torch.bfloat16) for k, v in w.items()}, x


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["odd", "tc 64/128", "tc 32/64"])
@pytest.mark.parametrize("query, key", [(299, 0), (299, 1), (299, 63), (299, 64), (300, 127), (300, 128), (319, 255), (319, 256), (319, 319), (320, 319),
                                        (256, 255), (128, 0), (127, 64)])
def test_far_keys_and_block_borders(name, dtype, query, key):
    """One key whose score stands out, at the edges of blocks, tiles and splits and at the sequence's beginning, for a query that
    is the last of a prompt and for one that is decoded; the tokens in front of the query are there to hide it."""
    hidden, m = MIXERS[name]
    m = dict(m, scale=0.06)
    torch.manual_seed(query + key)
    part, w, x = _standing_out(m, hidden, query + 1, query, key)
    part.load(w, DEV, dtype)
    cache, slot = _cache(part, dtype)
    w64 = {k: v.to(F64) for k, v in w.items()}
    ref = plain.attention(x.to(F64), w64, "", m, 1e-5)[query]
    blind = plain.attention(torch.cat([x[:key], x[key:] * torch.tensor([1.0, 0.0] + [1.0] * (hidden - 2))]).to(F64), w64, "", m, 1e-5)[query]
    assert float((ref - blind).norm() / ref.norm()) > 0.2          # leaving the key out would show
    for what, cuts in (("prompt", [[(0, query + 1)]]), ("decoded", [[(0, query)], [(0, 1)]] if query else [[(0, 1)]]),
                       ("portion of two", [[(0, query - 1)], [(0, 2)]])):
        got = _run(part, cache, slot, cuts, [x], dtype)[0][query]
        helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} {what}: query {query}, key {key}", factor=2.0)


@pytest.mark.parametrize("name", ["odd", "tc 64/128"])
def test_a_score_far_beyond_the_cap(name):
    """Scores of several hundred, capped; without the cap, or with the cap in front of the scale, the result is another."""
    hidden, m = MIXERS[name]
    torch.manual_seed(5)
    m = dict(m, scale=3.0)
    part, w, x = _standing_out(m, hidden, 200, 199, 17)
    w64 = {k: v.to(F64) for k, v in w.items()}
    ref = plain.attention(x.to(F64), w64, "", m, 1e-5)
    for dtype in (torch.float32, torch.bfloat16):
        part.load(w, DEV, dtype)
        cache, slot = _cache(part, dtype)
        for cuts in ([[(0, 200)]], [[(0, 150)]] + [[(0, 1)]] * 50):
            got = _run(part, cache, slot, cuts, [x], dtype)[0]
            helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} beyond the cap", factor=2.0)


@pytest.mark.parametrize("name", ["odd", "tc 64/128"])
def test_many_sequences_decode_together_and_alone(name):
    """Decode steps of more sequences than one, with lengths from 1 to several splits, against each of them alone (bfloat16:
    which other rows are in the batch does not show beyond rounding)."""
    hidden, m = MIXERS[name]
    torch.manual_seed(9)
    part = _attention(hidden, m)
    w = _weights(part)
    lens = [1, 2, 63, 64, 65, 127, 128, 129, 300, 517, 40, 7]
    xs = [torch.randn(n + 3, hidden).to(torch.bfloat16).float() for n in lens]
    for dtype in (torch.float32, torch.bfloat16):
        part.load(w, DEV, dtype)
        cache, slot = _cache(part, dtype, tokens=8192, slots=16)
        together = _run(part, cache, slot, [[(i, n) for i, n in enumerate(lens)]] + [[(i, 1) for i in range(len(lens))]] * 3, xs, dtype)
        for i, n in enumerate(lens):
            alone = _run(part, cache, slot, [[(0, n)]] + [[(0, 1)]] * 3, [xs[i]], dtype)[0]
            helpers.assert_close(together[i].numpy(), alone.numpy(), _name(dtype), f"{name} sequence of {n}", factor=1.0)


def test_temperature_changes_where_it_should():
    """With keys and values of which the maps find only the size, the temperature shows in the scores alone: the same sequence with
    a temperature that changes every 1, 4 or 1000 positions, against the plain function at every position."""
    for every in (1, 4, 1000):
        hidden, m = MIXERS["odd"]
        m = dict(m, q_temp=dict(coef=1.5, every=every))
        torch.manual_seed(every)
        part = _attention(hidden, m)
        w = _weights(part, scale=0.2)
        part.load(w, DEV, torch.float32)
        cache, slot = _cache(part, torch.float32)
        x = torch.randn(70, hidden)
        ref = plain.attention(x.to(F64), {k: v.to(F64) for k, v in w.items()}, "", m, 1e-5)
        got = _run(part, cache, slot, [[(0, 50)]] + [[(0, 1)]] * 20, [x], torch.float32)[0]
        helpers.assert_close(got.numpy(), ref.numpy(), "float32", f"every {every}", factor=2.0)


# -- the pair embedding ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_pair_embedding_over_steps_batches_and_reused_slots(dtype):
    """Portions of every size down to one token, sequences that begin and go on side by side, state rows that were poisoned."""
    from hymt2sharp_b200.kernels import ops
    from hymt2sharp_b200.cache import GroupSpec, PagedCache
    V, W, buckets, mp, mc, scale = 53, 37, 19, 1234567, 891, 2.5
    torch.manual_seed(1)
    w = dict(embed=torch.randn(V, W).to(torch.bfloat16), bigram=torch.randn(buckets + 1, W).to(torch.bfloat16))
    cfg = dict(embedding=dict(scale=scale, bigram=dict(buckets=buckets, mul_prev=mp, mul_cur=mc)))
    w64 = {k: v.to(F64) for k, v in w.items()}
    table, pairs = (w[k].to(DEV).to(dtype) for k in ("embed", "bigram"))
    cache = PagedCache([GroupSpec("full", 1, 8, 1)], dtype, DEV, 1024, max_slots=4, state_bytes=20)
    seqs = [helpers.random_tokens(V, n, n) for n in (40, 9, 1)]
    refs = [plain.embed(s, w64, cfg) for s in seqs]
    for cuts in ([[40, 9, 1]], [[1, 1, 1], [1, 2, 0], [2, 6, 0], [36, 0, 0]], [[7, 0, 0], [3, 4, 0], [30, 5, 1]]):
        slots = cache.alloc_slots(3)
        cache.state.fill_(170)
        at, rows = [0, 0, 0], [[], [], []]
        for step in cuts:
            live = [(i, n) for i, n in enumerate(step) if n]
            ctx, plan = _context(cache, [(slots[i], seqs[i][at[i]:at[i] + n]) for i, n in live], dtype, V)
            out = torch.empty(ctx.num_tokens, W, device=DEV)
            ops.embed_pairs(out, table, pairs, ctx.tokens, ctx.token_seq, ctx.token_pos, ctx.cu_seqlens, ctx.slot_ids, cache.state, 16, scale, mp, mc, ctx.status)
            cache.end_step(plan)
            assert int(ctx.status[0]) == 0
            o = 0
            for i, n in live:
                rows[i].append(out[o:o + n].cpu()); o += n; at[i] += n
        cache.free_slots(slots)
        for r, ref in zip(rows, refs):
            helpers.assert_close(torch.cat(r).numpy(), ref.numpy(), "float32", f"pair embedding {cuts}", factor=0.1)


# -- routing and the mixture -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E, top, groups", [(6, 2, (3, 2)), (10, 4, (5, 3)), (5, 1, (5, 3)), (7, 7, None), (64, 6, (8, 3)), (130, 5, (65, 4)), (12, 3, (2, 1))])
@pytest.mark.parametrize("T", [1, 5, 300])
def test_sigmoid_routing_in_groups(T, E, top, groups):
    from hymt2sharp_b200.kernels import ops
    torch.manual_seed(T + E)
    logits = torch.randn(T, E + 3) * 2                       # columns behind the router's are another product's
    rule = ops.RouteRule("sigmoid", True, 1e-20, *(groups or (1, 1)))
    chosen = torch.empty(T, top, dtype=torch.int32, device=DEV)
    weight = torch.empty(T, top, dtype=torch.float32, device=DEV)
    dev = logits.to(DEV)
    ops.moe_route(chosen, weight, dev, None, rule=rule, outputs=E)
    small = None
    if T * top <= ops.MOE_SMALL_PAIRS:
        tile, tiles = 8, ops.moe_tiles(T, top, E, 8)
        small = (torch.empty_like(chosen), torch.empty_like(weight))
        ints = [torch.empty(n, dtype=torch.int32, device=DEV) for n in (tiles * tile, tiles + 1)]
        ops.moe_route_place(*small, torch.empty_like(chosen), *ints, dev, None, E, tile, rule=rule, outputs=E)
    g = dict(count=groups[0], keep=groups[1]) if groups else None
    for t in range(T):
        s = torch.sigmoid(logits[t, :E].to(F64))
        want = plain.choose(s.tolist(), top, g)
        picked = s[want] / (s[want].sum() + 1e-20)
        for c, v in ((chosen, weight),) + ((small,) if small else ()):
            assert c[t].tolist() == want
            assert np.allclose(v[t].cpu().numpy(), picked.numpy(), rtol=2e-6, atol=1e-9)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, W, E, top, groups, ff, shared", [(3, 44, 6, 2, (3, 2), 9, 7), (200, 64, 10, 4, (5, 3), 24, 40), (9, 128, 12, 3, (4, 2), 48, 48),
                                                              (260, 128, 8, 4, None, 64, 96), (5, 64, 4, 2, None, 24, None)])
def test_mixture_with_a_gated_shared_expert(dtype, T, W, E, top, groups, ff, shared):
    """Stored and added; every expert has its own size of weights, so that a wrong one shows."""
    from hymt2sharp_b200.parts import PartSpec, build_part
    from types import SimpleNamespace
    torch.manual_seed(T + E)
    params = dict(hidden=W, experts=E, identity=0, top=top, intermediate=ff, activation="silu", router="router", scores="sigmoid", weights="chosen_share",
                  share_eps=1e-20, gate_proj="e{}.gate", up_proj="e{}.up", down_proj="e{}.down")
    if groups:
        params.update(groups=groups[0], keep=groups[1])
    if shared:
        params.update(shared=PartSpec("swiglu", dict(hidden=W, intermediate=shared, activation="silu", gate_proj="shared.gate", up_proj="shared.up",
                                                     down_proj="shared.down")), shared_gate="shared.sg")
    part = build_part("feed_forward", PartSpec("routed_experts", params))
    w = {n: torch.randn(s.shape) * 0.2 for n, s in part.tensors().items()}
    for e in range(E):
        w[f"e{e}.down"] *= 1.0 + e
    w["router"] *= 3.0
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    part.load(w, DEV, dtype)
    x = torch.randn(T, W).to(torch.bfloat16).float()
    mlp = dict(router=dict(top=top, groups=dict(count=groups[0], keep=groups[1]) if groups else None), shared=dict(ff=shared) if shared else None)
    ref = plain.mixture(x.to(F64), {k: v.to(F64) for k, v in w.items()}, "", mlp)
    ctx = SimpleNamespace(prenormed=None, norm_ahead=None)
    out = torch.full((T, W), float("nan"), device=DEV)
    part.forward(x.to(DEV).to(dtype), out, ctx, store=True)
    helpers.assert_close(out.cpu().numpy(), ref.numpy(), _name(dtype), "stored", factor=1.5)
    base = torch.randn(T, W)
    out = base.to(DEV).clone()
    part.forward(x.to(DEV).to(dtype), out, ctx)
    helpers.assert_close(out.cpu().numpy(), (base.to(F64) + ref).numpy(), _name(dtype), "added", factor=1.5)


# -- the sum at a block's end ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, W", [(3, 44), (70, 128), (2, 1030), (5, 2048), (2, 3000), (3, 6144)])
@pytest.mark.parametrize("form", ["two branches", "one branch", "a mixture", "a mixture and a shared expert", "a mixture and a gated shared expert"])
def test_branches_join_the_residual_and_the_next_norm_reads_it(dtype, T, W, form):
    from hymt2sharp_b200.kernels import ops
    torch.manual_seed(W + T)
    x, y0, y1 = (torch.randn(T, W) for _ in range(3))
    g0, g1, gn = (0.5 + torch.rand(W) for _ in range(3))
    top, rows = 3, 11
    routed, pair_row, weight = torch.randn(rows, W), torch.randint(0, rows, (T, top), dtype=torch.int32), torch.rand(T, top)
    shared, z = torch.randn(T, W), torch.randn(T, 4)
    ref = x.to(F64) + g0.to(F64) * y0.to(F64)
    branches, mixture = [(y0.to(DEV), g0.to(DEV))], None
    if form == "two branches":
        branches.append((y1.to(DEV), g1.to(DEV)))
        ref = ref + g1.to(F64) * y1.to(F64)
    elif form != "one branch":
        mix = (weight.to(F64)[:, :, None] * routed.to(F64)[pair_row.long()]).sum(1)
        zd = None
        if "shared" in form:
            zd = z.to(DEV)[:, 2:3] if "gated" in form else None
            mix = mix + (torch.sigmoid(z[:, 2:3].to(F64)) if zd is not None else 1.0) * shared.to(F64)
        mixture = (routed.to(DEV), pair_row.to(DEV), weight.to(DEV), g1.to(DEV), shared.to(DEV) if "shared" in form else None, zd)
        ref = ref + g1.to(F64) * mix
    plain_x = x.to(DEV).clone()
    assert ops.join_branches(plain_x, branches, mixture) is None
    helpers.assert_close(plain_x.cpu().numpy(), ref.numpy(), "float32", form, factor=0.2)
    normed_x, out = x.to(DEV).clone(), torch.empty(T, W, dtype=dtype, device=DEV)
    h = ops.join_branches(normed_x, branches, mixture, (gn.to(DEV).to(dtype), 1e-5, out))
    assert torch.equal(normed_x, plain_x)
    gain = gn.to(dtype).to(F64)
    helpers.assert_close(h.float().cpu().numpy(), plain.norm(ref, gain, 1e-5).numpy(), _name(dtype), f"{form}, normed", factor=0.5)


def test_rows_are_placed_beside_others():
    from hymt2sharp_b200.kernels import ops
    for W, dtype in ((44, torch.float32), (46, torch.bfloat16), (64, torch.bfloat16)):
        both = torch.zeros(5, 2 * W, dtype=dtype, device=DEV)
        x = torch.randn(5, W, device=DEV)
        ops.place_rows(both[:, W:], x)
        assert torch.equal(both[:, W:], x.to(dtype)) and not both[:, :W].any()
        ops.place_rows(both[:, :W], 2 * x)
        assert torch.equal(both[:, W:], x.to(dtype)) and torch.equal(both[:, :W], (2 * x).to(dtype))
