"""The mechanisms of the Gomerax design one by one, each built from its own parameters with weights of its own, against the
plain functions: latent attention with a latent vector of the queries, a window and a sink a head (sizes, portions, far keys,
block borders, window edges, the share of the sink), the table of positions, routing by a group's best choice score, clamped
experts, gated products with rules and biases in their epilogue, the sum at a block's end, and runs that add the embedding's
output."""
import numpy as np
import pytest
import torch

import helpers
from plain import gomerax_plain as plain

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


def _name(dtype):
    return "float32" if dtype == torch.float32 else "bfloat16"


def _w64(w):
    return {k: v.to(F64) for k, v in w.items()}


def _context(cache, slot_tokens, dtype, vocab=10):
    from hymt2sharp_b200.engine.engine import StepEntry, make_context
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    entries = [StepEntry(s, t if isinstance(t, list) else [0] * t, []) for s, t in slot_tokens]
    ctx, _, _, plan = make_context(cache, entries, vocab, dtype, DEV, status)
    return ctx, plan


def _cache(mixer, dtype, tokens=4096, slots=4):
    from hymt2sharp_b200.cache import GroupSpec, PagedCache
    from hymt2sharp_b200.parts import MixerSlot
    n = mixer.cache_need()
    cache = PagedCache([GroupSpec(n.kind, n.kv_heads, n.head_dim, 1, n.window, n.streams, n.value_dim)], dtype, DEV, tokens, max_slots=slots)
    return cache, MixerSlot(group=0, plane=0)


def _attention(hidden, m, eps=1e-5, sink="sink"):
    from hymt2sharp_b200.parts import PartSpec, build_part
    position = PartSpec("yarn_interleaved", dict(dims=m["rot"]["dims"], base=m["rot"]["base"]))
    return build_part("mixer", PartSpec("latent_attention", dict(
        hidden=hidden, heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], kv_rank=m["kv_rank"], scale=m["scale"], eps=eps,
        position=position, gate=None, window=(m.get("mask") or {}).get("size"), q_rank=m["q_rank"], dq_proj="dq", dq_norm="dq.norm", q_proj="uq",
        dkv_proj="dkv", dkv_norm="dkv.norm", uk_proj="uk", uv_proj="uv", o_proj="o", sink=sink)))


def _weights(part, scale=0.15):
    w = {}
    for n, s in part.tensors().items():
        x = torch.randn(s.shape)
        w[n] = (1.0 + 0.3 * x if n.endswith("norm") else x if n == "sink" else x * scale).to(torch.bfloat16)
    return w


def _run(part, cache, mslot, schedule, xs, dtype):
    """schedule: [[(sequence index, tokens), ...], ...]; xs[i] [T_i, hidden]; returns per sequence what the mixer wrote."""
    from hymt2sharp_b200.kernels import ops
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
        assert int(ctx.status[0]) == 0 and int(ops.device_status(torch.device(DEV))[0]) == 0
        o = 0
        for i, n in step:
            outs[i].append(res[o:o + n].cpu()); o += n; at[i] += n
    cache.free_slots(list(slots.values()))
    return [torch.cat(outs[i]) for i in range(len(xs))]


def _m(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window=None, base=1000.0):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=dict(dims=rot_dim, base=base))
    if window:
        m["mask"] = dict(size=window)
    return m


MIXERS = {
    "odd": (44, _m(3, 5, 6, 7, 11, 9, 1.5, 70)),
    "odd, one head, no window": (50, _m(1, 3, 2, 5, 6, 7, 2.0)),
    "wide": (64, _m(2, 200, 40, 264, 72, 320, 0.2, 150)),
    "pieces of 16": (96, _m(6, 16, 16, 16, 48, 32, 0.9, 65)),
    "pieces of 16, 20 heads": (96, _m(20, 48, 16, 48, 32, 80, 0.4)),
    "64 + 64": (128, _m(4, 64, 64, 64, 96, 64, 0.3, 64)),
    "64 + 32, values of 128": (96, _m(5, 64, 32, 128, 48, 96, 0.3, 100)),
    "40 + 24, values of 64": (64, _m(3, 40, 24, 64, 40, 48, 0.4)),
    "128 + 64": (128, _m(2, 128, 64, 128, 64, 256, 0.2, 190)),
    "80 + 48, values of 112": (80, _m(3, 80, 48, 112, 40, 64, 0.3, 130, 50.0)),
    "32 + 32, no window": (64, _m(8, 32, 32, 32, 24, 48, 0.6)),
}

SCHEDULES = {
    "whole": lambda n, m: [[(0, n), (1, m)]],
    "portions down to two tokens": lambda n, m: [[(0, 2), (1, 3)], [(0, 67), (1, 2)], [(0, n - 69), (1, m - 5)]],
    "a prompt and single tokens": lambda n, m: [[(0, n - 40), (1, m - 10)]] + [[(0, 1), (1, 1)]] * 10 + [[(0, 1)]] * 30,
}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", sorted(MIXERS))
def test_latent_attention_in_every_schedule(name, dtype):
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
    refs = [plain.attention(x.to(F64), _w64(w), "", m, 1e-5) for x in xs]
    _run(part, cache, slot, [[(0, 400), (1, 190)]], [torch.randn(400, hidden), torch.randn(190, hidden)], dtype)
    for what, cuts in SCHEDULES.items():
        for x, got, ref in zip(xs, _run(part, cache, slot, cuts(333, 29), xs, dtype), refs):
            helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} {what} ({len(x)})", factor=2.0)
    cache.book.audit()


def _standing_out(m, hidden, T, query, key, score=9.0):
    """Inputs and weights in which `query`'s scores for `key` stand out (about `score`) and nothing else does: channel 0 is on at the
    query alone, channel 1 at the key alone; the first latent entries read them."""
    H, d, rot = m["heads"], m["dim"], m["rot_dim"]
    x = torch.randn(T, hidden).to(torch.bfloat16).float() * 0.5
    x[:, :2] = 0.0
    x[query, 0], x[key, 1] = 30.0, 30.0
    part = _attention(hidden, m)
    w = {k: v.float() for k, v in _weights(part, scale=0.05).items()}
    w["dq.norm"][0] = w["dkv.norm"][0] = 1.0
    w["sink"][:] = 0.5
    for name, channel in (("dq", 0), ("dkv", 1)):
        w[name][:, :2] = 0.0
        w[name][0, :] = 0.0
        w[name][0, channel] = 1.0
    # a normed latent vector whose first entry alone is large holds about sqrt(rank) there
    at = torch.arange(H) * (d + rot)
    w["uq"][at, :] = 0.0
    w["uq"][at, 0] = score / (m["scale"] * (m["q_rank"] * m["kv_rank"]) ** 0.5)
    w["uk"][torch.arange(H) * d, :] = 0.0
    w["uk"][torch.arange(H) * d, 0] = 1.0
    return part, {k: v.to(torch.bfloat16) for k, v in w.items()}, x


def _without(x, key):
    y = x.clone()
    y[key, 1] = 0.0
    return y


CUTS = (("prompt", lambda q: [[(0, q + 1)]]), ("decoded", lambda q: [[(0, q)], [(0, 1)]]), ("portion of two", lambda q: [[(0, q - 1)], [(0, 2)]]))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["odd", "pieces of 16", "64 + 64", "128 + 64", "40 + 24, values of 64"])
@pytest.mark.parametrize("query, key", [(299, 0), (299, 1), (299, 63), (299, 64), (300, 127), (300, 128), (319, 255), (319, 256), (319, 319), (320, 319),
                                        (256, 255), (128, 0), (127, 64)])
def test_far_keys_and_block_borders(name, dtype, query, key):
    """One key whose score stands out, at the edges of blocks, tiles and splits and at the sequence's beginning, for a query that
    is the last of a prompt and for one that is decoded; the tokens in front of the query are there to hide it."""
    hidden, m = MIXERS[name]
    m = {k: v for k, v in m.items() if k != "mask"}
    torch.manual_seed(query + key)
    part, w, x = _standing_out(m, hidden, query + 1, query, key)
    part.load(w, DEV, dtype)
    cache, slot = _cache(part, dtype)
    ref = plain.attention(x.to(F64), _w64(w), "", m, 1e-5, [query])[query]
    blind = plain.attention(_without(x, key).to(F64), _w64(w), "", m, 1e-5, [query])[query]
    assert float((ref - blind).norm() / ref.norm()) > 0.2          # leaving the key out would show
    for what, cuts in CUTS:
        got = _run(part, cache, slot, cuts(query), [x], dtype)[0][query]
        helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} {what}: query {query}, key {key}", factor=2.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["odd", "pieces of 16", "64 + 32, values of 128"])
@pytest.mark.parametrize("window", [2, 63, 64, 65, 128, 129, 200])
def test_window_edges(name, dtype, window):
    """The key `window` - 1 places back is seen, the one `window` back is not, wherever the edge falls."""
    hidden, m = MIXERS[name]
    m = dict(m, mask=dict(size=window))
    wider = dict(m, mask=dict(size=window + 1))
    for query in (260, 320):
        for back in (window - 1, window):
            torch.manual_seed(query + back)
            part, w, x = _standing_out(m, hidden, query + 1, query, query - back)
            part.load(w, DEV, dtype)
            cache, slot = _cache(part, dtype)
            ref = plain.attention(x.to(F64), _w64(w), "", m, 1e-5, [query])[query]
            other = plain.attention((x if back == window else _without(x, query - back)).to(F64), _w64(w), "", wider, 1e-5, [query])[query]
            assert float((ref - other).norm() / ref.norm()) > 0.2  # an edge one off would show
            for what, cuts in CUTS:
                got = _run(part, cache, slot, cuts(query), [x], dtype)[0][query]
                helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} {what}: window {window}, {back} back", factor=2.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["odd", "pieces of 16, 20 heads", "128 + 64", "64 + 64", "40 + 24, values of 64", "32 + 32, no window"])
def test_sinks_of_every_size(name, dtype):
    """Sinks far above, among and far below the scores, another one a head; whole prompts, whose first rows have few keys beside
    the sink, and decode steps with and without splits.  Without a sink the result is another."""
    hidden, m = MIXERS[name]
    m = {k: v for k, v in m.items() if k != "mask"}
    torch.manual_seed(3)
    part = _attention(hidden, m)
    w = _weights(part)
    w["sink"] = (torch.linspace(-20.0, 12.0, m["heads"]) if m["heads"] > 2 else torch.linspace(5.0, 8.0, m["heads"])).to(torch.bfloat16)
    part.load(w, DEV, dtype)
    cache, slot = _cache(part, dtype)
    x = torch.randn(310, hidden).to(torch.bfloat16).float()
    ref = plain.attention(x.to(F64), _w64(w), "", m, 1e-5)
    none = plain.attention(x.to(F64), {k: v for k, v in _w64(w).items() if k != "sink"}, "", m, 1e-5)
    assert float((ref - none).norm() / none.norm()) > 0.1           # leaving the sinks out would show
    for cuts in ([[(0, 310)]], [[(0, 1)]] + [[(0, 1)]] * 309, [[(0, 200)], [(0, 70)], [(0, 40)]]):
        got = _run(part, cache, slot, cuts, [x], dtype)[0]
        helpers.assert_close(got.numpy(), ref.numpy(), _name(dtype), f"{name} {len(cuts)} steps", factor=2.0)
    # no stored sink: the same part without the term
    part = _attention(hidden, m, sink=None)
    part.load(w, DEV, dtype)
    for cuts in ([[(0, 310)]], [[(0, 290)]] + [[(0, 1)]] * 20):
        got = _run(part, cache, slot, cuts, [x], dtype)[0]
        helpers.assert_close(got.numpy(), none.numpy(), _name(dtype), f"{name} without a sink", factor=2.0)


@pytest.mark.parametrize("name", ["odd", "pieces of 16", "64 + 64", "128 + 64"])
def test_many_sequences_decode_together_and_alone(name):
    """Decode steps of more sequences than one, with lengths from 1 to several splits, against each of them alone: which other
    rows are in the batch does not show beyond rounding.  Prompts likewise."""
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


# -- the table of positions --------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("W", [37, 64])
def test_embedding_with_a_table_of_positions(dtype, W):
    """Portions of sequences side by side; the second copy; a position outside the table is flagged and nothing else is."""
    from hymt2sharp_b200.kernels import ops
    V, P, scale = 53, 45, 2.5
    torch.manual_seed(1)
    w = dict(embed=torch.randn(V, W).to(torch.bfloat16), pos=torch.randn(P, W).to(torch.bfloat16))
    table, positions = (w[k].to(DEV).to(dtype) for k in ("embed", "pos"))
    seqs = [helpers.random_tokens(V, n, n) for n in (45, 9, 1)]
    refs = [plain.embed(s, _w64(w), dict(embedding=dict(scale=scale))) for s in seqs]
    status = torch.zeros(4, dtype=torch.int32, device=DEV)
    for pieces in ([(0, 0, 45), (1, 0, 9), (2, 0, 1)], [(1, 3, 4), (0, 40, 45)], [(0, 44, 45)]):
        ids = torch.tensor([t for i, a, b in pieces for t in seqs[i][a:b]], dtype=torch.int32, device=DEV)
        pos = torch.tensor([p for i, a, b in pieces for p in range(a, b)], dtype=torch.int32, device=DEV)
        out, copy = torch.empty(len(ids), W, device=DEV), torch.full((len(ids), W), float("nan"), device=DEV)
        ops.embed_positions(out, table, positions, ids, pos, status, scale, copy)
        ref = torch.cat([refs[i][a:b] for i, a, b in pieces])
        helpers.assert_close(out.cpu().numpy(), ref.numpy(), "float32", "embedding", factor=0.1)
        assert torch.equal(out, copy) and int(status[0]) == 0
    pos = torch.tensor([P], dtype=torch.int32, device=DEV)
    ops.embed_positions(out[:1], table, positions, ids[:1], pos, status, scale)
    assert int(status[0]) == 3 and not out[0].any()


# -- gated products ----------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, W, F", [(1, 44, 21), (9, 46, 33), (1, 128, 96), (8, 256, 200), (40, 512, 264), (100, 2048, 136), (130, 128, 320), (300, 256, 72)])
@pytest.mark.parametrize("kind", ["biased", "clamped", "clamped and biased"])
def test_gated_feed_forward_with_a_rule_and_biases_in_its_epilogue(dtype, T, W, F, kind):
    """Stored, added, and with the output's bias left to the block; clamps that bite, biases as large as the sums."""
    from types import SimpleNamespace
    from hymt2sharp_b200.parts import PartSpec, build_part
    torch.manual_seed(T + W)
    names = dict(hidden=W, intermediate=F, gate_proj="gate", up_proj="up", down_proj="down")
    if "biased" in kind:
        names.update(gate_bias="gate.b", up_bias="up.b", down_bias="down.b")
    part = build_part("feed_forward", PartSpec("clamped_glu", dict(names, limit=0.9, alpha=1.702)) if "clamped" in kind else PartSpec("swiglu", names))
    w = {n: (torch.randn(s.shape) * (1.5 / s.shape[1] ** 0.5 if len(s.shape) == 2 else 0.7)).to(torch.bfloat16) for n, s in part.tensors().items()}
    assert ("up.b" in w) == ("biased" in kind)
    part.load(w, DEV, dtype)
    x = torch.randn(T, W).to(torch.bfloat16).float()
    full = _w64(w)
    if kind == "clamped":
        ref = plain.clamped(x.to(F64), full, "", 0.9)
    elif kind == "biased":
        ref = plain.dense(x.to(F64), full, "")
    else:    # the plain clamped expert on an input with one more entry, whose column is the bias
        x1 = torch.cat([x.to(F64), torch.ones(T, 1, dtype=F64)], 1)
        ext = {k: torch.cat([full[k], full[k + ".b"][:, None]], 1) for k in ("gate", "up")}
        ref = plain.clamped(x1, dict(ext, down=full["down"]), "", 0.9) + full["down.b"]
    ctx = SimpleNamespace(prenormed=None, norm_ahead=None)
    xd = x.to(DEV).to(dtype)
    out = torch.full((T, W), float("nan"), device=DEV)
    part.forward(xd, out, ctx, store=True)
    helpers.assert_close(out.cpu().numpy(), ref.numpy(), _name(dtype), "stored")
    base = torch.randn(T, W)
    out = base.to(DEV).clone()
    part.forward(xd, out, ctx)
    helpers.assert_close(out.cpu().numpy(), (base.to(F64) + ref).numpy(), _name(dtype), "added")
    if "biased" in kind:
        part.forward(xd, out, ctx, store=True, bias_later=True)
        helpers.assert_close((out + part.output_bias).cpu().numpy(), ref.numpy(), _name(dtype), "bias left out")


# -- routing and the mixture -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("E, top, groups", [(6, 2, (3, 2)), (10, 4, (5, 3)), (5, 1, (5, 3)), (7, 7, None), (64, 6, (8, 3)), (130, 5, (65, 4)), (12, 3, (2, 1))])
@pytest.mark.parametrize("T", [1, 5, 300])
def test_softmax_routing_by_a_groups_best_choice_score(T, E, top, groups):
    """Corrections that decide, choice scores of both signs (an excluded expert's is below every one of them), a factor of the
    weights; both routing kernels."""
    from hymt2sharp_b200.kernels import ops
    torch.manual_seed(T + E)
    logits, correction = torch.randn(T, E) * 2, torch.randn(E) * 0.4 - 0.3
    rule = ops.RouteRule("softmax", True, 1e-20, *(groups or (1, 1)), group_best=1, weight_scale=2.5)
    chosen = torch.empty(T, top, dtype=torch.int32, device=DEV)
    weight = torch.empty(T, top, dtype=torch.float32, device=DEV)
    dev, corr = logits.to(DEV), correction.to(DEV)
    ops.moe_route(chosen, weight, dev, corr, rule=rule)
    small = None
    if T * top <= ops.MOE_SMALL_PAIRS:
        tile, tiles = 8, ops.moe_tiles(T, top, E, 8)
        small = (torch.empty_like(chosen), torch.empty_like(weight))
        ints = [torch.empty(n, dtype=torch.int32, device=DEV) for n in (tiles * tile, tiles + 1)]
        ops.moe_route_place(*small, torch.empty_like(chosen), *ints, dev, corr, E, tile, rule=rule)
    g = dict(count=groups[0], keep=groups[1]) if groups else None
    other = 0
    for t in range(T):
        s = torch.softmax(logits[t].to(F64), 0)
        choice = (s + correction.to(F64)).tolist()
        want = plain.choose(choice, top, g)
        if g:    # (ranked by the two best together other groups would be kept, now and then)
            per = E // g["count"]
            worth = [sum(sorted(choice[i * per:(i + 1) * per])[-2:]) for i in range(g["count"])]
            kept = sorted(range(g["count"]), key=lambda i: -worth[i])[:g["keep"]]
            other += any(e // per not in kept for e in want)
        picked = s[want] / (s[want].sum() + 1e-20) * 2.5
        for c, v in ((chosen, weight),) + ((small,) if small else ()):
            assert c[t].tolist() == want
            assert np.allclose(v[t].cpu().numpy(), picked.numpy(), rtol=4e-6, atol=1e-9)
    assert not (g and T == 300 and E // g["count"] > 1) or other > 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, W, E, top, groups, ff, shared", [(3, 44, 6, 2, (3, 2), 9, 7), (200, 64, 10, 4, (5, 3), 24, 40), (9, 128, 12, 3, (4, 2), 48, 48),
                                                              (260, 128, 8, 4, (2, 2), 64, 96), (5, 64, 4, 2, None, 24, None), (150, 46, 6, 1, None, 10, 12)])
def test_mixture_of_clamped_experts(dtype, T, W, E, top, groups, ff, shared):
    """Stored and added, on every grouped kernel; every expert has its own size of weights, so that a wrong one shows, and the
    shared expert a limit of its own."""
    from types import SimpleNamespace
    from hymt2sharp_b200.parts import PartSpec, build_part
    torch.manual_seed(T + E)
    params = dict(hidden=W, experts=E, identity=0, top=top, intermediate=ff, activation="clamped", limit=0.6, alpha=1.702, router="router",
                  correction="correction", scores="softmax", weights="chosen_share", share_eps=1e-20, weight_scale=1.4, group_best=1,
                  gate_proj="e{}.gate", up_proj="e{}.up", down_proj="e{}.down")
    if groups:
        params.update(groups=groups[0], keep=groups[1])
    if shared:
        params.update(shared=PartSpec("clamped_glu", dict(hidden=W, intermediate=shared, limit=1.1, alpha=1.702, gate_proj="shared.gate",
                                                          up_proj="shared.up", down_proj="shared.down")))
    part = build_part("feed_forward", PartSpec("routed_experts", params))
    w = {n: torch.randn(s.shape) * 0.2 for n, s in part.tensors().items()}
    for e in range(E):
        w[f"e{e}.down"] *= 1.0 + e
    w["router"] *= 3.0
    w = {k: v.to(torch.bfloat16) for k, v in w.items()}
    part.load(w, DEV, dtype)
    x = torch.randn(T, W).to(torch.bfloat16).float()
    mlp = dict(router=dict(top=top, scale=1.4, groups=dict(count=groups[0], keep=groups[1]) if groups else None), expert=dict(limit=0.6),
               shared=dict(limit=1.1) if shared else None)
    ref = plain.mixture(x.to(F64), _w64(w), "", mlp)
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
@pytest.mark.parametrize("T, W", [(3, 44), (70, 128), (2, 1030), (5, 2048), (3, 6144)])
@pytest.mark.parametrize("form", ["three branches, one biased", "a biased branch with a gain", "a mixture, a shared expert and rows to add", "rows alone"])
def test_branches_without_gains_join_the_residual(dtype, T, W, form):
    from hymt2sharp_b200.kernels import ops
    torch.manual_seed(W + T)
    x, y0, y1, y2 = (torch.randn(T, W) for _ in range(4))
    g, b, gn = 0.5 + torch.rand(W), torch.randn(W), torch.randn(W) * 0.3
    top, rows = 3, 11
    routed, pair_row, weight = torch.randn(rows, W), torch.randint(0, rows, (T, top), dtype=torch.int32), torch.rand(T, top)
    d = lambda t: t.to(DEV)
    ref, mixture = x.to(F64) + y0.to(F64), None
    branches = [(d(y0), None)]
    if form.startswith("three"):
        branches += [(d(y1), None, d(b)), (d(y2), None)]
        ref = ref + y1.to(F64) + b.to(F64) + y2.to(F64)
    elif form.startswith("a biased"):
        branches += [(d(y1), d(g), d(b))]
        ref = ref + g.to(F64) * (y1.to(F64) + b.to(F64))
    elif form.startswith("a mixture"):
        branches += [(d(y2), None)]
        mixture = (d(routed), d(pair_row), d(weight), None, d(y1), None)
        ref = ref + y2.to(F64) + (weight.to(F64)[:, :, None] * routed.to(F64)[pair_row.long()]).sum(1) + y1.to(F64)
    plain_x = d(x).clone()
    assert ops.join_branches(plain_x, branches, mixture) is None
    helpers.assert_close(plain_x.cpu().numpy(), ref.numpy(), "float32", form, factor=0.2)
    normed_x, out = d(x).clone(), torch.empty(T, W, dtype=dtype, device=DEV)
    h = ops.join_branches(normed_x, branches, mixture, (d(1.0 + gn), 1e-5, out))     # (a gain in float32 beside rows of either type)
    assert torch.equal(normed_x, plain_x)
    helpers.assert_close(h.float().cpu().numpy(), plain.norm_around_zero(ref, gn.to(F64), 1e-5).numpy(), _name(dtype), f"{form}, normed", factor=0.5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_runs_that_add_the_embedding_work_with_other_blocks(dtype, tmp_path):
    """The same layers as pre-norm blocks, which know nothing of rows to add: the model adds them itself."""
    import gomerax_models
    from hymt2sharp_b200.config import GomeraxConfig
    from hymt2sharp_b200.engine.engine import Engine, StepEntry
    from hymt2sharp_b200.engine.gomerax import build_spec
    from hymt2sharp_b200.engine.spec import Run
    from hymt2sharp_b200.parts import PartSpec

    def other_blocks(cfg: GomeraxConfig):
        spec = build_spec(cfg)
        spec.layers = [PartSpec("pre_norm", dict(norm1=b.params["norm"], mixer=b.params["mixer"], norm2=b.params["norm"],
                                                 feed_forward=b.params["feed_forward"])) for b in spec.layers]
        spec.order = [Run(0), Run(1), Run(0, adds=True), Run(1), Run(1, adds=True)]
        return spec
    folder = gomerax_models.make_model_dir(str(tmp_path), "bare")
    cfg, w = plain.read_model(folder)
    tokens = helpers.random_tokens(cfg["vocab"], 90, 2)
    eps = cfg["norm"]["eps"]
    x = x0 = plain.embed(tokens, w, cfg)
    for i, again in ((0, 0), (1, 0), (0, 1), (1, 0), (1, 1)):
        x, p, spec = x + again * x0, f"l{i}.", cfg["layers"][i]
        x = x + plain.attention(plain.norm_around_zero(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps)
        x = x + plain.feed_forward(plain.norm_around_zero(x, w[p + "norm1"], eps), w, p + "mlp.", spec["mlp"])
    ref = (plain.norm_around_zero(x, w["final.norm"], eps) @ w["embed"].T).numpy()
    engine = Engine(folder, dtype=dtype, max_tokens=512, spec_override=other_blocks)
    for cuts in ([90], [60] + [1] * 30):
        slot, rows, at = engine.alloc_slots(1)[0], [], 0
        for n in cuts:
            rows.append(engine.step([StepEntry(slot, tokens[at:at + n], list(range(n)))]).cpu().numpy()); at += n
        engine.check()
        engine.free_slots([slot])
        got = np.concatenate(rows)
        if dtype == "float32":
            helpers.assert_close(got, ref, dtype, f"{len(cuts)} steps", factor=4.0)
        else:
            e = np.sqrt(((got - ref) ** 2).mean(1)) / ref.std()
            assert np.median(e) < 0.08 and (e > 0.35).mean() <= 0.1
