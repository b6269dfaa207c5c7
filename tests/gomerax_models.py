"""Tiny Gomerax configurations for the tests, and their model folders with random weights."""
from __future__ import annotations

ARCH = "Gomerax"


def _layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, window=None, base=10000.0, mlp=None):
    mixer = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, scale=scale, rot=dict(dims=rot_dim, base=base))
    if window is not None:
        mixer["mask"] = dict(size=window)
    return dict(type="latent_attention", mixer=mixer, mlp=mlp)


def _dense(ff):
    return dict(kind="dense", ff=ff)


def _moe(experts, top, ff, limit, scale, groups=None, shared=None):
    router = dict(experts=experts, top=top, scale=scale)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    mlp = dict(kind="moe", expert=dict(ff=ff, limit=limit), router=router)
    if shared is not None:
        mlp["shared"] = dict(ff=shared[0], limit=shared[1])
    return mlp


CONFIGS = {
    # odd sizes all round, nothing a multiple of 8: a loop of three passes over two middle layers, windows of 5 to 150, one head,
    # more latent than head entries and fewer, groups of two and of one expert, one chosen expert, a layer without feed-forward
    "odd": dict(config=dict(architecture=ARCH, vocab=103, width=44, max_positions=400, norm=dict(eps=1e-5), embedding=dict(scale=3.5),
                            loop=dict(start=1, stop=3, times=3), layers=[
        _layer(3, 5, 6, 7, 11, 9, 0.9, 5, 300.0, mlp=_moe(6, 2, 9, 0.8, 1.7, groups=(3, 2), shared=(7, 0.4))),
        _layer(1, 7, 2, 4, 5, 13, 1.4, 150, 20000.0),
        _layer(4, 6, 4, 12, 21, 3, 1.1, 33, 1000.0, mlp=_dense(13)),
        _layer(2, 3, 10, 5, 9, 17, 0.7, 64, 50.0, mlp=_moe(5, 1, 5, 1.3, 0.6, groups=(5, 3), shared=(11, 2.0))),
    ]), seed=51, sigma=0.15),
    # sizes in multiples of 16, on which the bfloat16 engine runs its tensor-core kernels: the per-head prompt kernel's shapes with
    # one and two boxes of unrotated entries, values narrower and wider than a box; the loop begins with the first layer and
    # there are no layers behind it but one; all groups kept; windows at and beside the cache block's 64
    "even": dict(config=dict(architecture=ARCH, vocab=512, width=128, max_positions=1000, norm=dict(eps=1e-6), embedding=dict(scale=8.0),
                             loop=dict(start=0, stop=3, times=2), layers=[
        _layer(5, 64, 32, 64, 80, 96, 0.08, 64, 10000.0, mlp=_moe(12, 3, 48, 1.0, 2.0, groups=(4, 2), shared=(48, 0.7))),
        _layer(4, 128, 64, 128, 64, 192, 0.05, 129, 5000.0, mlp=_dense(320)),
        _layer(16, 16, 16, 32, 48, 64, 0.15, 63, 700.0, mlp=_moe(8, 4, 64, 3.0, 0.5, groups=(2, 2), shared=(96, 1.5))),
        _layer(2, 80, 48, 112, 136, 128, 0.07, 300, 100000.0, mlp=_dense(192)),
    ]), seed=52, sigma=0.09),
    # the keys that may be absent are absent: no loop, no groups, no shared expert, no window
    "bare": dict(config=dict(architecture=ARCH, vocab=200, width=64, max_positions=512, norm=dict(eps=1e-5), embedding=dict(scale=1.0), layers=[
        _layer(2, 32, 16, 24, 24, 40, 0.4, mlp=_dense(96)),
        _layer(3, 24, 8, 16, 40, 32, 0.5, mlp=_moe(4, 2, 24, 1.0, 1.0)),
    ]), seed=53, sigma=0.15),
}

ROUTER_SPREAD = 4.0       # a choice between two experts that rests on the last bits would compare two different sums
QUERY_SPREAD = 4.0        # queries long enough for scores that pick among keys


def make_model_dir(folder: str, name: str) -> str:
    import os
    import torch
    from safetensors.torch import load_file, save_file
    from hymt2sharp_b200.config import GomeraxConfig
    from hymt2sharp_b200.weights import write_random_model
    spec = CONFIGS[name]
    write_random_model(folder, GomeraxConfig.from_dict(spec["config"]), spec["seed"], spec["sigma"])
    path = os.path.join(folder, "model.safetensors")
    tensors = load_file(path)
    gen = torch.Generator().manual_seed(spec["seed"])
    draw = lambda t: torch.randn(t.shape, generator=gen)
    for k in sorted(tensors):
        t, leaf = tensors[k], k.rsplit(".", 1)[-1]
        if leaf == "router":
            new = t.float() * ROUTER_SPREAD
        elif leaf == "correction":
            new = draw(t) * 0.25 - 0.3               # choice scores of both signs, and larger than the scores' differences
        elif leaf == "sink":
            new = draw(t) * 1.5 + 1.0                # a sink that takes a good share of a row
        elif leaf == "b":
            new = draw(t) * 0.4
        elif leaf == "norm1" or k == "final.norm":
            new = draw(t) * 0.3                      # around zero
        elif leaf == "uq":
            new = t.float() * QUERY_SPREAD
        elif k == "pos":
            new = draw(t) * 0.7                      # as long as the scaled embedding
        else:
            continue
        tensors[k] = new.to(t.dtype)
    save_file(tensors, path)
    return folder
