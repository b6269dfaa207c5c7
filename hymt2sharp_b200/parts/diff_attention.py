"""Differential attention over the paged cache, as a mixer part: every head has two softmax maps over the same values.

q = W_q x (heads x 2 x dim), k = W_k x (kv_heads x 2 x dim), v = W_v x (kv_heads x vdim), no biases, no rotation; a head's
query and key rows hold map 1's entries, then map 2's.  With the query temperature of a position p,
tau(p) = 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1) (temp_coef 0: tau = 1),

    s_m(i, j) = cap(tau(i) * scale * q_m(i) . k_m(j)),   cap(s) = softcap * tanh(s / softcap)      (no softcap: s itself)
    a_m(i)    = sum_{j <= i} softmax_j(s_m(i, .)) v(j)                                             m = 1, 2
    o         = a_1 - lambda * a_2,   y = o / sqrt(mean(o^2) + eps) * (1 - diff)                   over a head's vdim entries
    lambda    = exp(sum lq1 * lk1) - exp(sum lq2 * lk2) + diff                                     worked out once, at load

and W_o projects the heads side by side.  Head h reads key/value head h // (heads / kv_heads).  Scores, temperature, softmax,
lambda and the combination of the two maps are float32.  The cache keeps a token's two keys of a head as one row of 2 * dim
entries beside its value row.
"""
from __future__ import annotations

import math

import torch

from ..cache.allocator import GroupSpec
from ..kernels import fast, ops
from ..weights.loader import TensorSpec
from .attention import SPLIT_KEYS
from .base import MixerSlot, RotaryEpilogue, register_part
from .linear import Linear, compute_form

MAPS = 2


class DiffAttention:
    graph_safe = True
    can_store = True

    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, diff: float, q_proj: str,
                 k_proj: str, v_proj: str, o_proj: str, lambdas: list, softcap: float | None = None, temp_coef: float = 0.0, temp_every: int = 1):
        """`lambdas`: the names of the stored vectors lq1, lk1, lq2, lk2 [dim]."""
        if heads % kv_heads:
            raise ValueError(f"{heads} heads are not a multiple of {kv_heads} kv heads")
        if len(lambdas) != 4 or temp_every < 1:
            raise ValueError("the weight of the second map comes from four stored vectors, and a temperature changes every 1 position or more")
        self.hidden, self.heads, self.kv_heads, self.dim, self.vdim = int(hidden), int(heads), int(kv_heads), int(dim), int(vdim)
        self.scale, self.eps, self.diff, self.softcap = float(scale), float(eps), float(diff), float(softcap or 0.0)
        self.temp_coef, self.temp_every = float(temp_coef), int(temp_every)
        self.names = dict(q=q_proj, k=k_proj, v=v_proj, o=o_proj)
        self.lambdas = list(lambdas)
        self.qkv = self.out = self.out_store = self.lam = None

    def tensors(self):
        n, h = self.names, self.hidden
        t = {n["q"]: TensorSpec((self.heads * MAPS * self.dim, h)), n["k"]: TensorSpec((self.kv_heads * MAPS * self.dim, h)),
             n["v"]: TensorSpec((self.kv_heads * self.vdim, h)), n["o"]: TensorSpec((h, self.heads * self.vdim))}
        for name in self.lambdas:
            t[name] = TensorSpec((self.dim,))
        return t

    def cache_need(self):
        row = MAPS * self.dim
        return GroupSpec("full", self.kv_heads, row, planes=0, value_dim=0 if self.vdim == row else self.vdim)

    def state_bytes(self) -> int:
        return 0

    def load(self, weights, device, dtype):
        n = self.names
        self.qkv = Linear(compute_form(torch.cat([weights[n["q"]], weights[n["k"]], weights[n["v"]]], dim=0), device, dtype), role="qkv")
        self.out = Linear(compute_form(weights[n["o"]], device, dtype), ops.EPILOGUE_ACCUMULATE, role="o_proj")
        self.out_store = Linear(self.out.weight, ops.EPILOGUE_STORE, role="o_proj")
        q1, k1, q2, k2 = (weights[name].double() for name in self.lambdas)
        self.lam = math.exp(float((q1 * k1).sum())) - math.exp(float((q2 * k2).sum())) + self.diff

    def first_weights(self):
        return self.qkv.weight if self.qkv is not None else None

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, slot: MixerSlot, store: bool = False) -> None:
        T, H, G, d, dv = ctx.num_tokens, self.heads, self.kv_heads, self.dim, self.vdim
        k_plane, v_plane = ctx.cache.plane(slot.group, slot.plane)
        table = ctx.cache.tables[slot.group]
        planes = (k_plane, v_plane) if slot.writes else (None, None)
        q = None
        if MAPS * d == dv:      # projection and cache append as one kernel, where the kernels have one for the shape
            q = fast.try_project_rope_kv(x, self.qkv.weight, RotaryEpilogue.none(), ctx, planes, k_plane.dtype, table, None, None, self.eps, H, G, dv)
        if q is None:
            proj = self.qkv(x, ctx=ctx)
            q = torch.empty((T, H * MAPS * d), dtype=proj.dtype, device=proj.device)
            ops.rope_kv_general(proj, q, *planes, table, ctx.cache.block_tokens, ctx.token_seq, ctx.token_pos, ctx.slot_ids, None, 0, None, None,
                                ops.NORM_NONE, self.eps, H, G, MAPS * d, dv, True)
        out = torch.empty((T, H * dv), dtype=q.dtype, device=q.device)
        self.attend(out, q, k_plane, v_plane, table, ctx)
        if store:
            self.out_store(out, out=residual)
            ctx.prenormed = None
        else:
            self.out.add_then_norm(out, residual, getattr(ctx, "norm_ahead", None), ctx)

    def attend(self, out, q, k_plane, v_plane, table, ctx) -> None:
        T, H, G, d, dv = ctx.num_tokens, self.heads, self.kv_heads, self.dim, self.vdim
        if fast.try_diff_attention(out, q, k_plane, v_plane, table, ctx, H, G, d, dv, self.scale, self.softcap, self.temp_coef, self.temp_every,
                                   self.lam, self.eps, 1.0 - self.diff):
            return
        split, max_splits, acc, ml = 0, 0, None, None
        if ctx.decode and ctx.max_kv_len > SPLIT_KEYS:
            split, max_splits = SPLIT_KEYS, -(-ctx.max_kv_len // SPLIT_KEYS)
            na, nm = ops.attention_simt_scratch(T, H * MAPS, dv, max_splits)
            acc = torch.empty(na, dtype=torch.float32, device=out.device)
            ml = torch.empty(nm, dtype=torch.float32, device=out.device)
        maps = torch.empty((T, H * MAPS * dv), dtype=torch.float32, device=out.device)
        ops.attention_simt_maps(maps, q, k_plane, v_plane, table, ctx.cu_seqlens, ctx.slot_ids, ctx.kv_lens, ctx.num_seqs, ctx.max_new_tokens,
                                H, G, MAPS, d, dv, self.scale, self.softcap, self.temp_coef, self.temp_every, split, max_splits, acc, ml)
        ops.diff_combine(out, maps, H, dv, self.lam, self.eps, 1.0 - self.diff)


register_part("mixer", "diff_attention", DiffAttention)
