"""Gomerax: from its configuration to a ModelSpec.

Every layer is a parallel block: one norm's output (its weight stored around zero) is read by both sublayers, and their outputs
join the residual together as they are.  The mixer is latent attention whose queries come out of a latent vector of their own,
in a sliding window, with a sink a head.  The feed-forward is dense (SiLU-gated, every projection with a bias), a mixture of
clamped gated experts (softmax scores, choice by score plus correction within the groups of the best single scores, the chosen
scores' shares times a factor) beside a shared expert of the same form, or absent.  A stretch of layers runs several times in
a row with the same weights, every pass with its own cache planes, and every pass but the first begins by adding the
embedding's output to the residual.  The embedding is scaled and adds a stored vector of the position; the head is the
embedding table.  Tensor names are those of the design's checkpoints: 'l<i>.' in front of a layer's, '.mix.' for its mixer,
'.mlp.' for its feed-forward.
"""
from __future__ import annotations

from ..config.gomerax import ARCHITECTURE, GomeraxConfig
from ..config.registry import register_architecture
from ..parts.base import PartSpec
from .spec import ModelSpec, Run

EXPERT_SLOPE = 1.702           # constants of the design: the factor in the experts' sigmoid,
ROUTER_EPS = 1e-20             # and what is added to the sum that the chosen scores are divided by


def build_spec(cfg: GomeraxConfig) -> ModelSpec:
    W = cfg.width

    def norm(name: str) -> PartSpec:
        return PartSpec("rmsnorm", dict(dim=W, eps=cfg.norm_eps, weight=name, offset=1.0))

    layers, unread = [], []
    for i, layer in enumerate(cfg.layers):
        p, m, f = f"l{i}.", layer.mixer, layer.mlp
        x, y = p + "mix.", p + "mlp."
        position = PartSpec("yarn_interleaved", dict(dims=m.rot_dims, base=m.rot_base)) if m.rot_dims else None
        params = dict(norm=norm(p + "norm1"), mixer=PartSpec("latent_attention", dict(
            hidden=W, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale, eps=cfg.norm_eps,
            position=position, gate=None, window=m.window, q_rank=m.q_rank, dq_proj=x + "dq", dq_norm=x + "dq.norm", q_proj=x + "uq",
            dkv_proj=x + "dkv", dkv_norm=x + "dkv.norm", uk_proj=x + "uk", uv_proj=x + "uv", o_proj=x + "o", sink=x + "sink")))
        if f is None:
            unread.append(rf"l{i}\.mlp\..*")    # (a layer without a feed-forward reads none, should a checkpoint hold one)
        elif f.kind == "dense":
            params["feed_forward"] = PartSpec("swiglu", dict(
                hidden=W, intermediate=f.ff, gate_proj=y + "gate", up_proj=y + "up", down_proj=y + "down", gate_bias=y + "gate.b",
                up_bias=y + "up.b", down_bias=y + "down.b"))
        else:
            shared = None
            if f.shared_ff is not None:
                shared = PartSpec("clamped_glu", dict(hidden=W, intermediate=f.shared_ff, limit=f.shared_limit, alpha=EXPERT_SLOPE,
                                                      gate_proj=y + "shared.gate", up_proj=y + "shared.up", down_proj=y + "shared.down"))
            params["feed_forward"] = PartSpec("routed_experts", dict(
                hidden=W, experts=f.experts, identity=0, top=f.top, intermediate=f.ff, activation="clamped", limit=f.limit, alpha=EXPERT_SLOPE,
                router=y + "router", correction=y + "correction", scores="softmax", weights="chosen_share", share_eps=ROUTER_EPS,
                weight_scale=f.scale, groups=f.groups, keep=f.keep, group_best=1, gate_proj=y + "e{}.gate", up_proj=y + "e{}.up",
                down_proj=y + "e{}.down", shared=shared))
        layers.append(PartSpec("parallel", params))
    return ModelSpec(vocab=cfg.vocab, hidden=W, embedding="embed", layers=layers, order=[Run(i, adds=again) for i, again in cfg.runs()],
                     final_norm=norm("final.norm"), head=None, embed_scale=cfg.embedding_scale, positions="pos", max_positions=cfg.max_positions,
                     ignorable_tensors=unread)


def tensor_shapes(cfg: GomeraxConfig):
    from .model import DecoderModel
    return DecoderModel(build_spec(cfg)).tensors()


register_architecture(ARCHITECTURE, GomeraxConfig, build_spec, tensor_shapes)
