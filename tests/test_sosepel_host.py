"""The Sosepel design without a GPU: its configuration (every size read, errors that name their key), the registry, the tensor
list, the memory plan of a looped order, and the plain implementation's mechanisms against values worked out by hand."""
import copy
import math

import pytest
import torch

import sosepel_models
from plain import sosepel_plain as plain

F64 = torch.float64


def _cfg(name="odd"):
    return copy.deepcopy(sosepel_models.CONFIGS[name]["config"])


def test_every_size_is_read_and_written_back():
    from hymt2sharp_b200.config import SosepelConfig
    for name in sosepel_models.CONFIGS:
        raw = _cfg(name)
        cfg = SosepelConfig.from_dict(raw)
        assert cfg.to_dict() == raw
        assert SosepelConfig.from_dict(cfg.to_dict()) == cfg
    cfg = SosepelConfig.from_dict(_cfg("odd"))
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.logit_softcap, cfg.embedding_scale) == (101, 44, 1e-5, 7.0, 3.5)
    assert (cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur) == (37, 131, 29)
    m = cfg.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.diff, m.softcap, m.q_temp.coef, m.q_temp.every) == (3, 1, 5, 6, 2.5, 0.2, 4.0, 0.7, 3)
    f = cfg.layers[0].mlp
    assert (f.kind, f.experts, f.top, f.ff, f.groups, f.keep, f.shared_ff) == ("moe", 6, 2, 9, 3, 2, 7)
    assert cfg.layers[1].mlp is None and cfg.layers[2].mlp.ff == 13
    assert cfg.runs() == [(0, False), (1, True), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)] == plain.layer_runs(_cfg("odd"))
    bare = SosepelConfig.from_dict(_cfg("bare"))
    assert bare.loop is None and bare.bigram is None and bare.logit_softcap is None and bare.runs() == [(0, False), (1, False)]
    assert bare.layers[0].mixer.softcap is None and bare.layers[0].mixer.q_temp is None
    assert (bare.layers[1].mlp.groups, bare.layers[1].mlp.shared_ff) == (1, None)


@pytest.mark.parametrize("change, key", [
    (lambda c: c.pop("width"), "width"),
    (lambda c: c["layers"][0].update(type="conv"), "type 'conv'"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=2), "mixer.kv_heads"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "mixer.scale"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "mixer.diff"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].pop("every"), "mixer.q_temp.every"),
    (lambda c: c["layers"][0]["mixer"].update(softcap=0), "mixer.softcap"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=5), "mlp.router.top"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=4), "mlp.router.groups.count"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=4), "mlp.router.groups.keep"),
    (lambda c: c["layers"][2]["mlp"].update(kind="glu"), "mlp.kind 'glu'"),
    (lambda c: c["loop"].update(stop=9), "loop.stop"),
    (lambda c: c["embedding"]["bigram"].pop("mul_prev"), "embedding.bigram.mul_prev"),
    (lambda c: c["norm"].pop("eps"), "norm.eps"),
])
def test_errors_name_their_key(change, key):
    from hymt2sharp_b200.config import ConfigError, SosepelConfig
    raw = _cfg("odd")
    change(raw)
    with pytest.raises(ConfigError, match=key.replace(".", r"\.")):
        SosepelConfig.from_dict(raw)


def test_registry_tensor_list_and_memory_plan():
    from hymt2sharp_b200.config import SosepelConfig, get_architecture
    from hymt2sharp_b200.engine.model import DecoderModel
    arch = get_architecture("Sosepel")
    cfg = SosepelConfig.from_dict(_cfg("odd"))
    shapes = arch.tensor_shapes(cfg)
    assert shapes["embed"].shape == (101, 44) and shapes["bigram"].shape == (38, 44) and shapes["loop.in"].shape == (44, 88) and "head" not in shapes
    assert shapes["l0.mix.q"].shape == (30, 44) and shapes["l0.mix.k"].shape == (10, 44) and shapes["l0.mix.v"].shape == (6, 44)
    assert shapes["l0.mix.o"].shape == (44, 18) and shapes["l1.mix.lk2"].shape == (7,)
    assert shapes["l0.mlp.router"].shape == (6, 44) and shapes["l0.mlp.e5.down"].shape == (44, 9) and shapes["l0.mlp.shared.sg"].shape == (1, 44)
    assert shapes["l2.mlp.up"].shape == (13, 44) and "l2.mlp.gate" not in shapes and shapes["l2.ls2"].shape == (44,)
    assert "l1.ls2" not in shapes and shapes["l1.ls1"].shape == (44,) and not [n for n in shapes if n.startswith("l1.mlp")]
    assert not [n for n in shapes if n.endswith("norm2")]
    bare = arch.tensor_shapes(SosepelConfig.from_dict(_cfg("bare")))
    assert "bigram" not in bare and "loop.in" not in bare and not [n for n in bare if "shared" in n]
    # three passes over layers 1 and 2: three cache planes of each; two keys of a head are one row; the token in front is state
    model = DecoderModel(arch.build_spec(cfg))
    assert [(g.kind, g.planes, g.kv_heads, g.head_dim, g.value_width) for g in model.groups] == \
        [("full", 1, 1, 10, 6), ("full", 3, 2, 14, 10), ("full", 3, 2, 12, 12), ("full", 1, 3, 6, 5)]
    assert [(r.layer, r.joins) for r in model.spec.order] == cfg.runs()
    assert model.state_bytes == 4 and DecoderModel(arch.build_spec(SosepelConfig.from_dict(_cfg("bare")))).state_bytes == 0
    assert [row[0].plane for row in model.slots] == [0, 0, 0, 1, 1, 2, 2, 0]


def test_parts_refuse_what_they_cannot_do():
    from hymt2sharp_b200.engine.spec import ModelSpec, Run
    from hymt2sharp_b200.parts import PartSpec, build_part
    names = dict(q_proj="q", k_proj="k", v_proj="v", o_proj="o")
    with pytest.raises(ValueError, match="kv heads"):
        build_part("mixer", PartSpec("diff_attention", dict(hidden=8, heads=3, kv_heads=2, dim=4, vdim=4, scale=1.0, eps=1e-5, diff=0.1, lambdas=list("abcd"), **names)))
    moe = dict(hidden=8, experts=6, identity=0, top=2, intermediate=4, activation="silu", router="r", gate_proj="g{}", up_proj="u{}", down_proj="d{}")
    for bad, match in ((dict(groups=4), "groups"), (dict(groups=3, keep=4), "groups"), (dict(groups=6, keep=1), "choices"),
                       (dict(scores="sigmoid", weights="chosen_softmax"), "softmax"), (dict(shared_gate="s"), "shared expert")):
        with pytest.raises(ValueError, match=match):
            build_part("feed_forward", PartSpec("routed_experts", dict(moe, **bad)))
    with pytest.raises(ValueError, match="gain"):
        build_part("block", PartSpec("parallel", dict(norm=PartSpec("rmsnorm", dict(dim=8, eps=1e-5, weight="n")), mixer=PartSpec(
            "diff_attention", dict(hidden=8, heads=2, kv_heads=2, dim=4, vdim=4, scale=1.0, eps=1e-5, diff=0.1, lambdas=list("abcd"), **names)), mixer_gain="m",
            ff_gain="f")))
    with pytest.raises(ValueError, match="matrix"):
        ModelSpec(vocab=4, hidden=8, embedding="e", layers=[PartSpec("parallel")], final_norm=PartSpec("rmsnorm"), head=None, order=[Run(0, joins=True)])


# -- the plain implementation against values worked out by hand ------------------------------------------------------------
def test_plain_pair_rows_and_embedding():
    assert plain.bigram_row(None, 5, 7, 3, 2) == 7                       # the first token: the last row
    assert plain.bigram_row(4, 5, 7, 3, 2) == (12 + 10) % 7 == 1
    w = dict(embed=torch.tensor([[1.0], [2.0]], dtype=F64), bigram=torch.tensor([[10.0], [20.0], [30.0], [40.0]], dtype=F64))
    cfg = dict(embedding=dict(scale=2.0, bigram=dict(buckets=3, mul_prev=2, mul_cur=1)))
    # tokens 1, 0, 1: rows 3 (first), (2 + 0) mod 3 = 2, (0 + 1) mod 3 = 1; the pair's row is not scaled
    assert plain.embed([1, 0, 1], w, cfg).flatten().tolist() == [4.0 + 40.0, 2.0 + 30.0, 4.0 + 20.0]


def test_plain_temperature_cap_and_lambda():
    # floor((p + 1) / 3): 0, 0, 1, 1, 1, 2 at positions 0 .. 5
    want = [1 + 0.5 * math.log(n + 1) for n in (0, 0, 1, 1, 1, 2)]
    assert [plain.query_temperature(p, 3, 0.5) for p in range(6)] == pytest.approx(want)
    z = torch.tensor([-100.0, 0.0, 1.0], dtype=F64)
    assert plain.soft_cap(z, 2.0).tolist() == pytest.approx([-2.0, 0.0, 2 * math.tanh(0.5)]) and plain.soft_cap(z, None) is z
    a, b = torch.tensor([1.0, 2.0]), torch.tensor([0.5, 0.25])
    assert plain.lambda_of(a, b, b, b, 0.3) == pytest.approx(math.exp(1.0) - math.exp(0.3125) + 0.3)


def test_plain_two_maps_of_one_head():
    # one key that map 1 finds and map 2 does not; values that name their position
    k = torch.tensor([[20.0], [0.0], [0.0]], dtype=F64)
    v = torch.tensor([[1.0, 0.0], [0.0, 3.0], [0.0, 3.0]], dtype=F64)
    a1 = plain.one_map(torch.ones(3, 1, dtype=F64), k, v, 1.0, None)
    a2 = plain.one_map(torch.zeros(3, 1, dtype=F64), k, v, 1.0, None)
    assert torch.allclose(a1[2], torch.tensor([1.0, 0.0], dtype=F64), atol=1e-6)
    assert torch.allclose(a2[2], torch.tensor([1.0 / 3.0, 2.0], dtype=F64))
    o = plain.differential(a1[2], a2[2], 0.5, 0.2, 0.0)
    d = torch.tensor([1.0 - 1.0 / 6.0, -1.0], dtype=F64)
    assert torch.allclose(o, 0.8 * d / torch.sqrt((d * d).mean()), atol=1e-5)


def test_plain_choice_in_groups_and_weights():
    s = [0.9, 0.1, 0.6, 0.55, 0.2, 0.8]
    assert plain.choose(s, 2) == [0, 5]
    # groups (0, 1), (2, 3), (4, 5): worth 1.0, 1.15, 1.0; of the equals the first stays
    assert plain.choose(s, 2, dict(count=3, keep=1)) == [2, 3]
    assert plain.choose(s, 2, dict(count=3, keep=2)) == [0, 2]
    assert plain.choose(s, 3, dict(count=6, keep=3)) == [0, 5, 2]           # groups of one: their own score
    router = torch.tensor([[1.0], [-1.0], [0.5]], dtype=F64)
    chosen, weight = plain.route(torch.tensor([2.0], dtype=F64), router, 2)
    sig = lambda z: 1 / (1 + math.exp(-z))
    assert chosen == [0, 2] and weight.tolist() == pytest.approx([sig(2) / (sig(2) + sig(1)), sig(1) / (sig(2) + sig(1))])


def test_plain_layer_sums_both_sublayers_of_one_norm():
    torch.manual_seed(0)
    w = {n: torch.randn(s, dtype=F64) for n, s in {"l0.norm1": (4,), "l0.ls1": (4,), "l0.ls2": (4,), "l0.mix.q": (4, 4), "l0.mix.k": (4, 4), "l0.mix.v": (3, 4),
         "l0.mix.o": (4, 3), "l0.mix.lq1": (2,), "l0.mix.lk1": (2,), "l0.mix.lq2": (2,), "l0.mix.lk2": (2,), "l0.mlp.up": (5, 4), "l0.mlp.down": (4, 5)}.items()}
    spec = dict(mixer=dict(heads=1, kv_heads=1, dim=2, vdim=3, scale=0.7, diff=0.3), mlp=dict(kind="dense", ff=5))
    x = torch.randn(3, 4, dtype=F64)
    h = x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-5) * w["l0.norm1"]
    ff = torch.clamp(h @ w["l0.mlp.up"].T, min=0) ** 2 @ w["l0.mlp.down"].T
    want = x + plain.attention(h, w, "l0.mix.", spec["mixer"], 1e-5) * w["l0.ls1"] + ff * w["l0.ls2"]
    assert torch.allclose(plain.layer(x, w, 0, spec, 1e-5), want)
    j = plain.join_input(x, 2 * x, torch.cat([torch.eye(4, dtype=F64), 10 * torch.eye(4, dtype=F64)], dim=1))
    assert torch.allclose(j, 21 * x)
