"""The Gomerax design without a GPU: its configuration (every size read, errors that name their key), the registry, the tensor
list, the memory plan of a looped order, and the plain implementation's mechanisms against values worked out by hand."""
import copy
import math

import pytest
import torch

import gomerax_models
from plain import gomerax_plain as plain

F64 = torch.float64


def _cfg(name="odd"):
    return copy.deepcopy(gomerax_models.CONFIGS[name]["config"])


def test_every_size_is_read_and_written_back():
    from hymt2sharp_b200.config import GomeraxConfig
    for name in gomerax_models.CONFIGS:
        raw = _cfg(name)
        cfg = GomeraxConfig.from_dict(raw)
        assert cfg.to_dict() == raw
        assert GomeraxConfig.from_dict(cfg.to_dict()) == cfg
    cfg = GomeraxConfig.from_dict(_cfg("odd"))
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.max_positions, cfg.embedding_scale) == (103, 44, 1e-5, 400, 3.5)
    m = cfg.layers[0].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.window, m.rot_dims, m.rot_base) == (3, 5, 6, 7, 11, 9, 0.9, 5, 6, 300.0)
    f = cfg.layers[0].mlp
    assert (f.kind, f.experts, f.top, f.ff, f.limit, f.scale, f.groups, f.keep, f.shared_ff, f.shared_limit) == ("moe", 6, 2, 9, 0.8, 1.7, 3, 2, 7, 0.4)
    assert cfg.layers[1].mlp is None and cfg.layers[2].mlp.ff == 13
    want = [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert cfg.runs() == want == plain.layer_runs(_cfg("odd"))
    bare = GomeraxConfig.from_dict(_cfg("bare"))
    assert bare.loop is None and bare.runs() == [(0, False), (1, False)] and bare.layers[0].mixer.window is None
    assert (bare.layers[1].mlp.groups, bare.layers[1].mlp.shared_ff) == (1, None)


@pytest.mark.parametrize("change, key", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["layers"][0].update(type="attention"), "type 'attention'"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "mixer.q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "mixer.scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "mixer.rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mixer.mask.size"),
    (lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"), "mlp.expert.limit"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("limit"), "mlp.shared.limit"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "mlp.router.top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "mlp.router.groups.count"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "mlp.router.groups.keep"),
    (lambda c: c["layers"][2]["mlp"].update(kind="glu"), "mlp.kind 'glu'"),
    (lambda c: c["loop"].update(stop=9), "loop.stop"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
])
def test_errors_name_their_key(change, key):
    from hymt2sharp_b200.config import ConfigError, GomeraxConfig
    raw = _cfg("odd")
    change(raw)
    with pytest.raises(ConfigError, match=key.replace(".", r"\.")):
        GomeraxConfig.from_dict(raw)


def test_registry_tensor_list_and_memory_plan():
    from hymt2sharp_b200.config import GomeraxConfig, get_architecture
    from hymt2sharp_b200.engine.model import DecoderModel
    arch = get_architecture("Gomerax")
    cfg = GomeraxConfig.from_dict(_cfg("odd"))
    shapes = {n: s.shape for n, s in arch.tensor_shapes(cfg).items()}
    assert shapes["embed"] == (103, 44) and shapes["pos"] == (400, 44) and "head" not in shapes and shapes["final.norm"] == (44,)
    assert {n[len("l0.mix."):]: s for n, s in shapes.items() if n.startswith("l0.mix.")} == {
        "dq": (11, 44), "dq.norm": (11,), "uq": (33, 11), "dkv": (15, 44), "dkv.norm": (9,), "uk": (15, 9), "uv": (21, 9), "sink": (3,), "o": (44, 21)}
    assert shapes["l0.mlp.router"] == (6, 44) and shapes["l0.mlp.correction"] == (6,) and shapes["l0.mlp.e5.down"] == (44, 9)
    assert shapes["l0.mlp.shared.gate"] == (7, 44) and not [n for n in shapes if n.startswith("l1.mlp")]
    assert {n[len("l2.mlp."):]: s for n, s in shapes.items() if n.startswith("l2.mlp.")} == {
        "gate": (13, 44), "gate.b": (13,), "up": (13, 44), "up.b": (13,), "down": (44, 13), "down.b": (44,)}
    assert not [n for n in shapes if n.endswith("norm2")]
    bare = arch.tensor_shapes(GomeraxConfig.from_dict(_cfg("bare")))
    assert not [n for n in bare if "shared" in n] and "l1.mlp.correction" in bare
    # three passes over layers 1 and 2: three cache planes of each; one row a token for all heads; no state
    model = DecoderModel(arch.build_spec(cfg))
    assert [(g.kind, g.window, g.planes, g.kv_heads, g.head_dim, g.streams) for g in model.groups] == \
        [("window", 5, 1, 1, 15, 1), ("window", 150, 3, 1, 15, 1), ("window", 33, 3, 1, 7, 1), ("window", 64, 1, 1, 27, 1)]
    assert [(r.layer, r.adds) for r in model.spec.order] == cfg.runs() and model.state_bytes == 0 and model.spec.max_positions == 400
    assert [row[0].plane for row in model.slots] == [0, 0, 0, 1, 1, 2, 2, 0]
    assert [g.kind for g in DecoderModel(arch.build_spec(GomeraxConfig.from_dict(_cfg("bare")))).groups] == ["full", "full"]


def test_parts_refuse_what_they_cannot_do():
    from hymt2sharp_b200.engine.spec import ModelSpec, Run
    from hymt2sharp_b200.parts import PartSpec, build_part
    latent = dict(hidden=8, heads=2, dim=4, rot_dim=2, vdim=4, kv_rank=4, scale=1.0, eps=1e-5, position=None, gate=None, q_proj="q", dkv_proj="d",
                  dkv_norm="n", uk_proj="k", uv_proj="v", o_proj="o")
    with pytest.raises(ValueError, match="latent vector of the queries"):
        build_part("mixer", PartSpec("latent_attention", dict(latent, q_rank=4)))
    moe = dict(hidden=8, experts=6, identity=0, top=2, intermediate=4, activation="clamped", limit=1.0, alpha=1.7, router="r", gate_proj="g{}", up_proj="u{}",
               down_proj="d{}")
    build_part("feed_forward", PartSpec("routed_experts", moe))
    for bad, match in ((dict(limit=0.0), "positive"), (dict(group_best=3), "best score")):
        with pytest.raises(ValueError, match=match):
            build_part("feed_forward", PartSpec("routed_experts", dict(moe, **bad)))
    glu = dict(hidden=8, intermediate=4, gate_proj="g", up_proj="u", down_proj="d")
    for bad in (dict(gate_bias="gb"), dict(gate_bias="gb", up_bias="ub", activation="gelu_tanh")):
        with pytest.raises(ValueError, match="bias"):
            build_part("feed_forward", PartSpec("swiglu", dict(glu, **bad)))
    base = dict(vocab=4, hidden=8, embedding="e", layers=[PartSpec("parallel")], final_norm=PartSpec("rmsnorm"), head=None)
    for bad, match in ((dict(order=[Run(0, adds=True)]), "first run"), (dict(positions="p"), "length"),
                       (dict(order=[Run(0), Run(0, adds=True, joins=True)], join="j"), "either")):
        with pytest.raises(ValueError, match=match):
            ModelSpec(**base, **bad)


# -- the plain implementation against values worked out by hand ------------------------------------------------------------
def test_plain_embedding_and_norms():
    w = dict(embed=torch.tensor([[1.0], [2.0]], dtype=F64), pos=torch.tensor([[10.0], [20.0], [30.0]], dtype=F64))
    assert plain.embed([1, 0, 1], w, dict(embedding=dict(scale=3.0))).flatten().tolist() == [16.0, 23.0, 36.0]    # the position is not scaled
    x = torch.tensor([[3.0, 4.0]], dtype=F64)
    r = math.sqrt(12.5 + 0.5)
    assert plain.norm_around_zero(x, torch.tensor([0.5, -1.0], dtype=F64), 0.5).tolist()[0] == pytest.approx([4.5 / r, 0.0])
    assert plain.norm_plain(x, torch.tensor([0.5, -1.0], dtype=F64), 0.5).tolist()[0] == pytest.approx([1.5 / r, -4.0 / r])


def test_plain_rotation_window_and_sink():
    v = torch.tensor([1.0, 0.0, 0.0, 2.0, 7.0], dtype=F64)
    a, b = 3.0, 3.0 * 100.0 ** -0.5                                  # position 3, frequencies 1 and 1/10; the fifth entry stays
    assert plain.turn(v, 3, 4, 100.0).tolist() == pytest.approx([math.cos(a), math.sin(a), -2 * math.sin(b), 2 * math.cos(b), 7.0])
    assert [j for j in range(12) if plain.sees(8, j, 3)] == [6, 7, 8] and [j for j in range(12) if plain.sees(2, j, None)] == [0, 1, 2]
    p = plain.weights_with_sink(torch.tensor([0.0, math.log(2.0)], dtype=F64), torch.tensor(math.log(5.0), dtype=F64))
    assert p.tolist() == pytest.approx([1 / 8, 2 / 8])
    # the sink's score is not scaled: two keys of score ln 4 / 2 after the scale
    one = torch.ones(2, 1, dtype=F64)
    out = plain.attend(one * math.log(4.0), one, one, 0.5, 2, torch.tensor(math.log(3.0), dtype=F64))
    assert out.flatten().tolist() == pytest.approx([2 / 5, 4 / 7])


def test_plain_clamped_expert_and_biased_dense():
    eye = torch.eye(2, dtype=F64)
    w = {"gate": eye, "up": -eye, "down": eye}
    y = plain.clamped(torch.tensor([[5.0, -5.0]], dtype=F64), w, "", 2.0)
    g = [2.0, -5.0]                                                # the gate is cut from above only, the up entry from both sides
    want = [g[0] / (1 + math.exp(-1.702 * g[0])) * (-2.0 + 1), g[1] / (1 + math.exp(-1.702 * g[1])) * (2.0 + 1)]
    assert y.tolist()[0] == pytest.approx(want)
    b = {k + ".b": torch.tensor(v, dtype=F64) for k, v in (("gate", [1.0, 0.0]), ("up", [0.0, 3.0]), ("down", [-1.0, 0.5]))}
    y = plain.dense(torch.tensor([[1.0, 2.0]], dtype=F64), dict(w, **b), "")
    sig = lambda z: 1 / (1 + math.exp(-z))
    assert y.tolist()[0] == pytest.approx([2 * sig(2) * -1.0 - 1.0, 2 * sig(2) * 1.0 + 0.5])


def test_plain_choice_in_groups_and_weights():
    c = [0.3, 0.3, 0.4, -0.9, -0.1, -0.2]
    assert plain.choose(c, 2) == [2, 0]
    # groups (0, 1), (2, 3), (4, 5): worth 0.3, 0.4, -0.1 (not what their two best add up to)
    assert plain.choose(c, 2, dict(count=3, keep=1)) == [2, 3]
    assert plain.choose(c, 2, dict(count=3, keep=2)) == [2, 0]
    assert plain.choose([-5.0, -4.0, -1.0, -2.0], 2, dict(count=2, keep=1)) == [2, 3]      # negative scores of a kept group stay choosable
    router = torch.tensor([[1.0], [0.0], [2.0]], dtype=F64)
    chosen, weight = plain.route(torch.tensor([1.0], dtype=F64), router, torch.tensor([0.0, 2.0, 0.0], dtype=F64), 2, 3.0)
    e = [math.exp(1), 1.0, math.exp(2)]
    assert chosen == [1, 2] and weight.tolist() == pytest.approx([3 * e[1] / (e[1] + e[2]), 3 * e[2] / (e[1] + e[2])])   # weights without the correction


def test_plain_layer_and_loop():
    torch.manual_seed(0)
    shapes = {"l0.norm1": (4,), "l0.mix.dq": (3, 4), "l0.mix.dq.norm": (3,), "l0.mix.uq": (8, 3), "l0.mix.dkv": (5, 4), "l0.mix.dkv.norm": (3,),
              "l0.mix.uk": (4, 3), "l0.mix.uv": (6, 3), "l0.mix.sink": (2,), "l0.mix.o": (4, 6), "l0.mlp.gate": (5, 4), "l0.mlp.gate.b": (5,),
              "l0.mlp.up": (5, 4), "l0.mlp.up.b": (5,), "l0.mlp.down": (4, 5), "l0.mlp.down.b": (4,), "embed": (6, 4), "pos": (9, 4), "final.norm": (4,)}
    w = {n: torch.randn(s, dtype=F64) for n, s in shapes.items()}
    mixer = dict(heads=2, dim=2, rot_dim=2, vdim=3, q_rank=3, kv_rank=3, scale=0.7, rot=dict(dims=2, base=10.0), mask=dict(size=2))
    cfg = dict(norm=dict(eps=1e-5), embedding=dict(scale=2.0), layers=[dict(mixer=mixer, mlp=dict(kind="dense", ff=5))], loop=dict(start=0, stop=1, times=2))
    x = torch.randn(3, 4, dtype=F64)
    h = x / torch.sqrt((x * x).mean(1, keepdim=True) + 1e-5) * (1 + w["l0.norm1"])
    step = lambda x, h: x + plain.attention(h, w, "l0.mix.", mixer, 1e-5) + plain.dense(h, w, "l0.mlp.")
    assert torch.allclose(plain.layer(x, w, 0, cfg["layers"][0], 1e-5), step(x, h))
    tokens = [5, 0, 3]
    x0 = torch.stack([w["embed"][t] * 2 + w["pos"][i] for i, t in enumerate(tokens)])
    x1 = plain.layer(x0, w, 0, cfg["layers"][0], 1e-5)
    x2 = plain.layer(x1 + x0, w, 0, cfg["layers"][0], 1e-5)
    logits, seen = plain.forward(cfg, w, tokens, True)
    assert torch.allclose(seen[0], x1) and torch.allclose(seen[1], x2)
    assert torch.allclose(logits, plain.norm_around_zero(x2, w["final.norm"], 1e-5) @ w["embed"].T)
