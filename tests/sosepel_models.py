"""Tiny Sosepel configurations for the tests, and their model folders with random weights."""
from __future__ import annotations

ARCH = "Sosepel"


def _layer(heads, kv_heads, dim, vdim, scale, diff, softcap=None, temp=None, mlp=None):
    mixer = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff)
    if softcap is not None:
        mixer["softcap"] = softcap
    if temp is not None:
        mixer["q_temp"] = dict(coef=temp[0], every=temp[1])
    return dict(type="attention", mixer=mixer, mlp=mlp)


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(experts, top, ff, groups=None, shared=None):
    router = dict(experts=experts, top=top)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    mlp = dict(kind="moe", expert=dict(ff=ff), router=router)
    if shared is not None:
        mlp["shared"] = dict(ff=shared)
    return mlp


CONFIGS = {
    # odd sizes all round, nothing a multiple of 8: a loop over the two middle layers, three times; one kv head, and as many kv
    # heads as heads; a cap that bites and a temperature that changes every three positions; groups of two and of one expert;
    # one chosen expert; a layer without feed-forward; a pair table smaller than the multipliers
    "odd": dict(config=dict(architecture=ARCH, vocab=101, width=44, norm=dict(eps=1e-5), logit_softcap=7.0,
                            embedding=dict(scale=3.5, bigram=dict(buckets=37, mul_prev=131, mul_cur=29)), loop=dict(start=1, stop=3, times=3), layers=[
        _layer(3, 1, 5, 6, 2.5, 0.2, 4.0, (0.7, 3), mlp=_moe(6, 2, 9, groups=(3, 2), shared=7)),
        _layer(2, 2, 7, 10, 1.5, 0.4, 3.0, (0.2, 50)),
        _layer(4, 2, 6, 12, 2.0, -0.1, 9.0, (-0.1, 7), mlp=_dense(13)),
        _layer(3, 3, 3, 5, 4.0, 0.8, 6.0, (0.05, 1), mlp=_moe(5, 1, 5, groups=(5, 3), shared=11)),
    ]), seed=41, sigma=0.12),
    # sizes in multiples of 16, among them those that the bfloat16 engine's tensor-core attention takes; the loop begins with
    # the first layer; 12 experts in four groups of which two are kept; a shared expert as wide as the others, and one wider
    "even": dict(config=dict(architecture=ARCH, vocab=512, width=128, norm=dict(eps=1e-6), logit_softcap=20.0,
                             embedding=dict(scale=8.0, bigram=dict(buckets=255, mul_prev=1009, mul_cur=31)), loop=dict(start=0, stop=2, times=2), layers=[
        _layer(4, 2, 64, 128, 0.5, 0.3, 12.0, (0.3, 64), mlp=_moe(12, 3, 48, groups=(4, 2), shared=48)),
        _layer(4, 1, 32, 64, 0.6, 0.5, 25.0, (0.1, 100), mlp=_dense(320)),
        _layer(2, 2, 128, 64, 0.3, 0.2, 5.0, (0.2, 33), mlp=_moe(8, 4, 64, groups=(2, 1), shared=96)),
        _layer(8, 2, 16, 32, 0.9, 0.6, 8.0, (0.2, 128), mlp=_dense(192)),
    ]), seed=42, sigma=0.09),
    # the keys that may be absent are absent: no loop, no pair table, no caps, no temperature, no groups, no shared expert
    "bare": dict(config=dict(architecture=ARCH, vocab=200, width=64, norm=dict(eps=1e-5), embedding=dict(scale=1.0), layers=[
        _layer(2, 1, 64, 128, 0.4, 0.3, mlp=_dense(96)),
        _layer(2, 2, 16, 24, 0.8, 0.1, mlp=_moe(4, 2, 24)),
    ]), seed=43, sigma=0.12),
}

ROUTER_SPREAD = 2.5    # a choice between two experts that rests on the last bits would compare two different sums
LAMBDA_SPREAD = 4.0    # so that exp(lq1 . lk1) and exp(lq2 . lk2) are not both nearly 1


def make_model_dir(folder: str, name: str) -> str:
    import os
    import torch
    from safetensors.torch import load_file, save_file
    from hymt2sharp_b200.config import SosepelConfig
    from hymt2sharp_b200.weights import write_random_model
    spec = CONFIGS[name]
    write_random_model(folder, SosepelConfig.from_dict(spec["config"]), spec["seed"], spec["sigma"])
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    gen = torch.Generator().manual_seed(spec["seed"])
    for k in sorted(tensors):
        t, leaf = tensors[k], k.rsplit(".", 1)[-1]
        if leaf == "router":
            tensors[k] = (t.float() * ROUTER_SPREAD).to(t.dtype)
        elif leaf in ("lq1", "lk1", "lq2", "lk2"):
            tensors[k] = (torch.randn(t.shape, generator=gen) * LAMBDA_SPREAD / t.numel() ** 0.5 * 0.2).to(t.dtype)
        elif leaf in ("ls1", "ls2"):
            tensors[k] = (0.2 + torch.rand(t.shape, generator=gen)).to(t.dtype)      # gains far from 1 and from each other
        elif k == "loop.in":
            W = t.shape[0]                                                           # [x; x0]: both halves matter, neither explodes
            tensors[k] = (t.float() + 0.8 * torch.eye(W, 2 * W)).to(t.dtype)
    save_file(tensors, path)
    return folder
