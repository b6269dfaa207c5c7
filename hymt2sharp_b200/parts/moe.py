"""A mixture of small feed-forward experts with a router: residual += sum over a token's chosen experts of weight * expert(x).

The router's outputs z = W_router x are float32 (float32 sums of the products in both engines); the scores are their
softmax over ALL outputs.  The first `experts` outputs name experts with tensors, expert(x) = W_down act(W_up x); the last
`identity` outputs name identity experts, whose output is x itself.  The `top` outputs with the largest score + correction
are chosen (`correction`: a stored vector, one entry per output; None: none); a chosen output's weight is its score, without
the correction and not renormalised.  A shared expert (any feed-forward part) runs for every token with weight 1.

Chosen by parameters beyond that: a bias of the router (`router_bias`, a stored vector added to z); weights that are the
softmax over the CHOSEN outputs only (`weights="chosen_softmax"`; the choice by score is then the choice by z); and gated
experts, expert(x) = W_down (act(W_gate x) * (W_up x)) (`gate_proj` given; act "silu", "gelu_tanh", or "clamped": with g = min(W_gate x, limit)
and u = clamp(W_up x, -limit, limit), W_down (g * sigmoid(alpha * g) * (u + 1))): gate and up are one grouped product over the
stacked matrices, whose epilogue applies the activation and multiplies (the general CUDA-core kernel, and "gelu_tanh":
a small kernel behind it).  The scores may be the sigmoid of each output
(`scores="sigmoid"`), the weights the chosen scores' shares of their sum (`weights="chosen_share"`, `share_eps` added to the
sum), and the choice limited to groups: outputs side by side are cut into `groups` runs of equal length, the runs are ranked by
what their two best scores (with the correction) add up to, or by their best one (`group_best=1`), and the choice is among the outputs of
the first `keep` runs.  `weight_scale` multiplies the weights at the end.  The shared expert may have a gate per token
(`shared_gate`, a stored [1, hidden] matrix): its output is multiplied by sigmoid(W x); that product is one more row of the
router's.

How a step runs: router product; `moe_route` (softmax, choice); `moe_place` sorts the (token, choice) pairs by expert, each
expert's rows padded to whole row tiles; one grouped product per projection over the sorted rows (the first gathers its
input rows by token, its epilogue is the activation); `moe_combine` adds a token's rows up in the order they were chosen.
Nothing uses atomics and every sum has a fixed order, so a token's result does not depend on the other tokens of the step.
"""
from __future__ import annotations

import torch

from ..kernels import ops
from ..weights.loader import TensorSpec
from .base import PartSpec, build_part, register_part
from .linear import Linear, compute_form

ACTIVATIONS = {"relu2": ops.EPILOGUE_RELU_SQUARED}      # experts without a gate: an epilogue of the grouped product
GATED_ACTIVATIONS = {"silu": ops.GATED_SILU, "gelu_tanh": ops.GATED_GELU_TANH, "clamped": None}   # (None: a kernel of its own)
WEIGHTS = ("scores", "chosen_softmax", "chosen_share")
SKINNY_MAX_PAIRS = 512        # up to this many (token, choice) pairs in a step the kernel for few rows runs the experts,
SKINNY_PAIRS_BESIDE_TC = 64   # where the tensor cores take the operands only up to this many: beyond, most experts meet several
                              # rows, and a row tile of 128 on the tensor cores, mostly empty, still reads each expert once


class RoutedExperts:
    graph_safe = True  # its forward only launches kernels on the current stream
    can_store = True   # forward(..., store=True) overwrites `residual` with its output instead of adding to it

    def __init__(self, hidden: int, experts: int, identity: int, top: int, intermediate: int, activation: str, router: str,
                 up_proj: str, down_proj: str, correction: str | None = None, shared: PartSpec | None = None,
                 gate_proj: str | None = None, router_bias: str | None = None, weights: str = "scores", scores: str = "softmax",
                 share_eps: float = 0.0, groups: int = 1, keep: int = 1, shared_gate: str | None = None, group_best: int = 2,
                 weight_scale: float = 1.0, limit: float = 0.0, alpha: float = 1.0):
        """`up_proj` / `down_proj` / `gate_proj`: the tensor names of expert e with `{}` in place of e."""
        known = GATED_ACTIVATIONS if gate_proj is not None else ACTIVATIONS
        if activation not in known:
            raise ValueError(f"activation '{activation}' is not known for experts {'with' if gate_proj else 'without'} a gate "
                             f"(known: {', '.join(known)})")
        if weights not in WEIGHTS:
            raise ValueError(f"weights '{weights}' is not known (known: {', '.join(WEIGHTS)})")
        if scores not in ops.SCORES or (weights == "chosen_softmax" and scores != "softmax"):
            raise ValueError(f"scores '{scores}' with weights '{weights}': known scores are {', '.join(ops.SCORES)}, and the softmax over the "
                             f"chosen outputs comes from softmax scores")
        outputs = experts + identity
        if groups < 1 or outputs % groups or not (0 < keep <= groups) or (groups > 1 and top > keep * (outputs // groups)):
            raise ValueError(f"{outputs} outputs in {groups} groups of which {keep} are kept cannot give {top} choices")
        if group_best not in (1, 2):
            raise ValueError(f"groups are ranked by their best score or by the sum of their two best, not of {group_best}")
        if activation == "clamped" and not limit > 0:
            raise ValueError(f"a clamp at {limit}: the limit must be positive")
        if shared_gate is not None and shared is None:
            raise ValueError("a gate of the shared expert needs a shared expert")
        self.gated = gate_proj is not None
        self.rule = ops.RouteRule(scores=scores, renormalise=weights != "scores", share_eps=float(share_eps), groups=int(groups), keep=int(keep),
                                  group_best=int(group_best), weight_scale=float(weight_scale))
        self.glu = ops.GluRule("clamped", float(limit), float(alpha)) if activation == "clamped" else ops.GLU_SILU
        if experts < 0 or identity < 0 or not (0 < top <= experts + identity):
            raise ValueError(f"{top} of {experts} + {identity} experts cannot be chosen")
        self.hidden, self.experts, self.identity, self.top = int(hidden), int(experts), int(identity), int(top)
        self.intermediate, self.activation = int(intermediate), activation
        self.names = dict(r=router, c=correction, u=up_proj, d=down_proj, g=gate_proj, b=router_bias, sg=shared_gate)
        self.bias = None
        self.shared = build_part("feed_forward", shared) if shared is not None else None
        self.router = self.correction = self.up = self.down = None

    @property
    def outputs(self) -> int:
        return self.experts + self.identity

    def tensors(self):
        n = self.names
        t = {n["r"]: TensorSpec((self.outputs, self.hidden))}
        if n["c"] is not None:
            t[n["c"]] = TensorSpec((self.outputs,))
        if n["b"] is not None:
            t[n["b"]] = TensorSpec((self.outputs,))
        for e in range(self.experts):
            if self.gated:
                t[n["g"].format(e)] = TensorSpec((self.intermediate, self.hidden))
            t[n["u"].format(e)] = TensorSpec((self.intermediate, self.hidden))
            t[n["d"].format(e)] = TensorSpec((self.hidden, self.intermediate))
        if self.shared is not None:
            t.update(self.shared.tensors())
        if n["sg"] is not None:
            t[n["sg"]] = TensorSpec((1, self.hidden))
        return t

    def load(self, weights, device, dtype):
        n = self.names
        rows = weights[n["r"]]
        if n["sg"] is not None:    # the shared expert's gate is one more row of the router's product
            rows = torch.cat([rows, weights[n["sg"]].to(rows.dtype)], dim=0)
        self.router = Linear(compute_form(rows, device, dtype), role="router")
        self.correction = weights[n["c"]].to(device).float().contiguous() if n["c"] is not None else None
        self.bias = weights[n["b"]].to(device).float().contiguous() if n["b"] is not None else None
        if self.experts:
            # every expert's matrix of a kind in one tensor [experts, out, in]: a grouped product picks its expert by index
            # (gated experts: an expert's gate rows, then its up rows)
            ups = [torch.cat([weights[n["g"].format(e)], weights[n["u"].format(e)]]) if self.gated else weights[n["u"].format(e)]
                   for e in range(self.experts)]
            self.up = compute_form(torch.stack(ups), device, dtype)
            self.down = compute_form(torch.stack([weights[n["d"].format(e)] for e in range(self.experts)]), device, dtype)
        if self.shared is not None:
            self.shared.load(weights, device, dtype)

    def first_weights(self):
        return self.router.weight if self.router is not None else None

    def _grouped_kernel(self, x: torch.Tensor, tokens: int) -> str:
        """Which grouped product runs the experts: few (token, choice) pairs meet mostly different experts, and the step costs
        what reading those experts' weights costs (the kernel for few rows); many pairs go to the tensor cores where the
        operands are bfloat16 with rows in whole 16-byte pieces; everything else to the general CUDA-core kernel."""
        same = self.up is not None and x.dtype == self.up.dtype
        pairs = tokens * self.top
        tensor_cores = same and x.dtype == torch.bfloat16 and self.hidden % 8 == 0 and self.intermediate % 8 == 0
        if same and pairs <= (SKINNY_PAIRS_BESIDE_TC if tensor_cores else SKINNY_MAX_PAIRS):
            return "skinny"
        return "tc" if tensor_cores else "simt"

    def _experts(self, x: torch.Tensor, ctx):
        """Routing, the sorted rows and the experts' products: (y, pair_row, weight, z), y float32 [sorted rows, hidden], z float32
        [T, 1] the shared expert's gate in front of its sigmoid (None without one)."""
        T, dev = x.shape[0], x.device
        logits = self.router(x, out_dtype=torch.float32, ctx=ctx)
        z = logits[:, self.outputs:] if self.names["sg"] is not None else None
        chosen = torch.empty((T, self.top), dtype=torch.int32, device=dev)
        weight = torch.empty((T, self.top), dtype=torch.float32, device=dev)
        kernel = self._grouped_kernel(x, T)
        tile = ops.gemm_group_tile(kernel)
        tiles = ops.moe_tiles(T, self.top, self.experts, tile)
        ints = torch.empty(T * self.top + tiles * tile + tiles + 1 + max(self.experts, 1), dtype=torch.int32, device=dev)
        pair_row = ints[: T * self.top].view(T, self.top)
        row_token = ints[T * self.top: T * self.top + tiles * tile]
        tile_group = ints[T * self.top + tiles * tile: T * self.top + tiles * tile + tiles + 1]   # and the number of tiles in use
        counts = ints[T * self.top + tiles * tile + tiles + 1:]
        if T * self.top <= ops.MOE_SMALL_PAIRS and self.outputs <= 512:
            ops.moe_route_place(chosen, weight, pair_row, row_token, tile_group, logits, self.correction, self.experts, tile,
                                self.bias, rule=self.rule, outputs=self.outputs)
        else:
            ops.moe_route(chosen, weight, logits, self.correction, self.bias, rule=self.rule, outputs=self.outputs)
            ops.moe_place(pair_row, row_token, tile_group, counts, chosen, self.experts, tile)
        if not self.experts:
            return torch.empty((1, self.hidden), dtype=torch.float32, device=dev), pair_row, weight, z   # y is never read
        rows, gather = x, True
        if kernel == "tc":     # its tiles come by TMA, which reads rows side by side
            rows, gather = torch.empty((tiles * tile, self.hidden), dtype=x.dtype, device=dev), False
            ops.moe_gather(rows, x, row_token)
        ops.tag = "experts_up"
        if self.gated and self.activation in ("silu", "clamped") and kernel != "simt":
            act = torch.empty((tiles * tile, self.intermediate), dtype=x.dtype, device=dev)
            ops.gemm_grouped(kernel, act, rows, self.up, tile_group, row_token, gather, ops.EPILOGUE_SWIGLU, self.glu)
        elif self.gated:
            both = torch.empty((tiles * tile, 2 * self.intermediate), dtype=x.dtype, device=dev)
            ops.gemm_grouped(kernel, both, rows, self.up, tile_group, row_token, gather, ops.EPILOGUE_STORE)
            act = torch.empty((tiles * tile, self.intermediate), dtype=x.dtype, device=dev)
            # (rows of tiles not in use hold whatever was there: nobody reads them)
            if self.activation == "clamped":
                ops.clamped_glu(act, both, None, self.glu.limit, self.glu.alpha)
            else:
                ops.gated_act(act, both, GATED_ACTIVATIONS[self.activation])
        else:
            act = torch.empty((tiles * tile, self.intermediate), dtype=x.dtype, device=dev)
            ops.gemm_grouped(kernel, act, rows, self.up, tile_group, row_token, gather, ACTIVATIONS[self.activation])
        y = torch.empty((tiles * tile, self.hidden), dtype=torch.float32, device=dev)
        ops.tag = "experts_down"
        ops.gemm_grouped(kernel, y, act, self.down, tile_group, row_token, False, ops.EPILOGUE_STORE)
        ops.tag = None
        return y, pair_row, weight, z

    def _shared_rows(self, x: torch.Tensor, ctx):
        """The shared expert's output as float32 rows of its own."""
        rows = torch.empty((x.shape[0], self.hidden), dtype=torch.float32, device=x.device)
        if getattr(self.shared, "can_store", False):
            self.shared.forward(x, rows, ctx, store=True)
        else:
            rows.zero_()
            self.shared.forward(x, rows, ctx)
        return rows

    def pieces(self, x: torch.Tensor, ctx):
        """What is left to add up: (y, pair_row, weight, shared, z) for ops.join_branches, a block's own sum.  None: this mixture has
        outputs that are no rows of y (identity experts), or more choices than that kernel takes."""
        if self.identity or self.top > ops.JOIN_MAX_TOP or not self.experts:
            return None
        y, pair_row, weight, z = self._experts(x, ctx)
        shared = self._shared_rows(x, ctx) if self.shared is not None else None
        ctx.prenormed = None
        return y, pair_row, weight, shared, z

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, store: bool = False) -> None:
        if self.names["sg"] is not None:
            # the gated shared expert's rows are added up with the experts' by the kernel that a block uses for its own sum
            pieces = self.pieces(x, ctx)
            if pieces is None:
                raise ValueError("a gate of the shared expert beside identity experts, or beside this many choices, is not built")
            if store:
                residual.zero_()
            y, pair_row, weight, shared, z = pieces
            ops.join_branches(residual, [], (y, pair_row, weight, None, shared, z))
            return
        y, pair_row, weight, _ = self._experts(x, ctx)
        ops.moe_combine(residual, y, x, pair_row, weight, add=not store)
        if self.shared is not None:
            self.shared.forward(x, residual, ctx)
        ctx.prenormed = None

    def forward_then_norm(self, x: torch.Tensor, residual: torch.Tensor, norm, ctx, rows_dtype=None):
        """residual += norm(mixture(x)) for a block whose norm stands behind the sublayer: the experts' rows are added up,
        normed and added to the residual by one kernel.  Returns the new residual rows rounded to `rows_dtype` (None: not
        wanted), or False when this part cannot do it for this norm (the block then goes the long way)."""
        if getattr(norm, "groups", 1) != 1 or self.hidden > ops.MOE_COMBINE_NORM_MAX_WIDTH or norm.dim != self.hidden:
            return False
        if self.names["sg"] is not None:
            return False
        branch = self._shared_rows(x, ctx) if self.shared is not None else None
        y, pair_row, weight, _ = self._experts(x, ctx)
        rows = torch.empty(residual.shape, dtype=rows_dtype, device=residual.device) if rows_dtype is not None else None
        ops.moe_combine_norm(residual, rows, branch, y, x, pair_row, weight, norm.gain, norm.eps)
        ctx.prenormed = None
        return rows


register_part("feed_forward", "routed_experts", RoutedExperts)
