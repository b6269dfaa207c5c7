"""Sosepel: from its configuration to a ModelSpec.

Every layer is a parallel block: one norm's output is read by both sublayers, and their outputs join the residual together,
each multiplied entry by entry by a stored vector.  The mixer is differential attention (two softmax maps a head over the
same values, scores capped, queries with a temperature that grows with the position).  The feed-forward is dense with the
square of relu, a mixture of SiLU-gated experts chosen by sigmoid scores within groups beside a shared expert with a gate per
token, or absent.  A stretch of layers runs several times in a row with the same weights, every pass with its own cache
planes, and every pass begins by joining the residual with the embedding's output through a stored matrix.  The embedding is
scaled and adds a row of a table of token pairs; the head is the embedding table; the logits are capped.  Tensor names are
those of the design's checkpoints: 'l<i>.' in front of a layer's, '.mix.' for its mixer, '.mlp.' for its feed-forward.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.sosepel import ARCHITECTURE, SosepelConfig
from ..parts.base import PartSpec
from .spec import Bigram, ModelSpec, Run

DENSE_ACTIVATION = "relu2"     # constants of the design
EXPERT_ACTIVATION = "silu"
ROUTER_EPS = 1e-20             # in the sum that the chosen scores are divided by


def build_spec(cfg: SosepelConfig) -> ModelSpec:
    W = cfg.width

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", dict(dim=W, eps=cfg.norm_eps, weight=name))

    layers, unread = [], []
    for i, layer in enumerate(cfg.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        x, y = p + "mix.", p + "mlp."
        mixer = PartSpec("diff_attention", dict(
            hidden=W, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, eps=cfg.norm_eps, diff=m.diff,
            softcap=m.softcap, temp_coef=m.q_temp.coef if m.q_temp else 0.0, temp_every=m.q_temp.every if m.q_temp else 1,
            q_proj=x + "q", k_proj=x + "k", v_proj=x + "v", o_proj=x + "o", lambdas=[x + n for n in ("lq1", "lk1", "lq2", "lk2")]))
        params = dict(norm=norm(p + "norm1"), mixer=mixer, mixer_gain=p + "ls1")
        if f is None:
            # a layer without a feed-forward reads none of its tensors, should a checkpoint hold them
            unread.append(rf"l{i}\.(ls2|mlp\..*)")
        else:
            params["ff_gain"] = p + "ls2"
            if f.kind == "dense":
                params["feed_forward"] = PartSpec("dense_mlp", dict(hidden=W, intermediate=f.ff, activation=DENSE_ACTIVATION,
                                                                    up_proj=y + "up", down_proj=y + "down"))
            else:
                shared = None
                if f.shared_ff is not None:
                    shared = PartSpec("swiglu", dict(hidden=W, intermediate=f.shared_ff, activation=EXPERT_ACTIVATION,
                                                     gate_proj=y + "shared.gate", up_proj=y + "shared.up", down_proj=y + "shared.down"))
                params["feed_forward"] = PartSpec("routed_experts", dict(
                    hidden=W, experts=f.experts, identity=0, top=f.top, intermediate=f.ff, activation=EXPERT_ACTIVATION,
                    router=y + "router", scores="sigmoid", weights="chosen_share", share_eps=ROUTER_EPS, groups=f.groups, keep=f.keep,
                    gate_proj=y + "e{}.gate", up_proj=y + "e{}.up", down_proj=y + "e{}.down", shared=shared,
                    shared_gate=y + "shared.sg" if shared is not None else None))
        layers.append(PartSpec("parallel", params))
    bigram = None
    if cfg.bigram is not None:
        bigram = Bigram("bigram", cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur)
    return ModelSpec(vocab=cfg.vocab, hidden=W, embedding="embed", layers=layers, order=[Run(i, joins=begins) for i, begins in cfg.runs()],
                     final_norm=norm("final.norm"), head=None, embed_scale=cfg.embedding_scale, bigram=bigram,
                     join="loop.in" if cfg.loop is not None else None, logit_softcap=cfg.logit_softcap, ignorable_tensors=unread)


def tensor_shapes(cfg: SosepelConfig):
    from .model import DecoderModel
    return DecoderModel(build_spec(cfg)).tensors()


register_architecture(ARCHITECTURE, SosepelConfig, build_spec, tensor_shapes)
