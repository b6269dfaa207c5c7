"""Plain, slow forward pass of the Gomerax design: whole sequences, no cache, CPU only.

One function per mechanism, written from the design's equations, computing with torch on
the CPU in float64 (or float32).  It shares no code with the product package: it reads
config.json with json and the weights with the `safetensors` library.

Notation: x is the residual [T, width]; h is what both sublayers of a layer read; t is a
token's index in its sequence (its position, from 0); W is a weight stored [out, in] and
applied as W h.
"""
from __future__ import annotations

import json
import math
import os

import torch

EXPERT_SLOPE = 1.702     # in the sigmoid of an expert's activation
SHARE_EPS = 1e-20        # in the sum that the chosen scores are divided by


def read_model(folder: str, dtype=torch.float64):
    from safetensors.torch import load_file
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    weights = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    return config, weights


# -- small pieces ---------------------------------------------------------------------------------
def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """Over the last axis: x / sqrt(mean(x^2) + eps)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_around_zero(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * (1.0 + w)


def norm_plain(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# -- the embedding and the loop ---------------------------------------------------------------------
def embed(tokens: list, w: dict, config: dict) -> torch.Tensor:
    scale = config["embedding"].get("scale", 1.0)
    return torch.stack([w["embed"][t] * scale + w["pos"][p] for p, t in enumerate(tokens)])


def layer_runs(config: dict) -> list:
    """[(layer, the embedding's output is added in front of it), ...] in the order they run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(loop["start"])]
    for k in range(loop["times"]):
        runs += [(i, k > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


# -- latent attention ---------------------------------------------------------------------------------
def turn(v: torch.Tensor, position, dims: int, base: float) -> torch.Tensor:
    """The first `dims` entries of v [.., n] in neighbouring pairs, pair i by position * base^(-2i/dims).  `position`: one number, or
    one for each v[t]."""
    out = v.clone()
    p = torch.as_tensor(position, dtype=v.dtype)
    p = p.reshape(-1, *[1] * (v.dim() - 2)) if p.dim() else p
    for i in range(dims // 2):
        a = p * base ** (-2.0 * i / dims)
        c, s = torch.cos(a), torch.sin(a)
        out[..., 2 * i] = v[..., 2 * i] * c - v[..., 2 * i + 1] * s
        out[..., 2 * i + 1] = v[..., 2 * i + 1] * c + v[..., 2 * i] * s
    return out


def sees(i: int, j: int, window) -> bool:
    return 0 <= i - j and (not window or i - j < window)


def weights_with_sink(s: torch.Tensor, sink) -> torch.Tensor:
    """exp(s_j) / (exp(sink) + sum_j exp(s_j)); sink None: no such term."""
    terms = s if sink is None else torch.cat([s, sink.reshape(1).to(s.dtype)])
    return torch.softmax(terms, dim=0)[:s.shape[0]]


def queries(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    """[T, heads, dim + rot_dim], the last rot_dim of a head turned."""
    T = h.shape[0]
    c = norm_plain(h @ w[p + "dq"].T, w[p + "dq.norm"], eps)
    q = (c @ w[p + "uq"].T).view(T, m["heads"], m["dim"] + m["rot_dim"])
    return torch.cat([q[..., :m["dim"]], turn(q[..., m["dim"]:], list(range(T)), m["rot"]["dims"], m["rot"]["base"])], dim=-1)


def compressed(h: torch.Tensor, w: dict, p: str, m: dict, eps: float):
    """The latent vectors [T, kv_rank] and the shared rotated key parts [T, rot_dim]."""
    z = h @ w[p + "dkv"].T
    k = turn(z[:, m["kv_rank"]:], list(range(h.shape[0])), m["rot"]["dims"], m["rot"]["base"])
    return norm_plain(z[:, :m["kv_rank"]], w[p + "dkv.norm"], eps), k


def attend(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, window, sink, only=None) -> torch.Tensor:
    """One head: q, k [T, d], v [T, dv] -> [T, dv] (`only`: zeros but for these tokens' rows)."""
    out = torch.zeros((q.shape[0], v.shape[1]), dtype=q.dtype)
    for i in range(q.shape[0]) if only is None else only:
        seen = [j for j in range(i + 1) if sees(i, j, window)]
        a, b = seen[0], i + 1
        out[i] = weights_with_sink((k[a:b] @ q[i]) * scale, sink) @ v[a:b]
    return out


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float, only=None) -> torch.Tensor:
    T, H = h.shape[0], m["heads"]
    q = queries(h, w, p, m, eps)
    c, kr = compressed(h, w, p, m, eps)
    k = (c @ w[p + "uk"].T).view(T, H, m["dim"])
    v = (c @ w[p + "uv"].T).view(T, H, m["vdim"])
    window = (m.get("mask") or {}).get("size")
    sink = w.get(p + "sink")
    heads = [attend(q[:, a], torch.cat([k[:, a], kr], dim=1), v[:, a], m["scale"], window, None if sink is None else sink[a], only)
             for a in range(H)]
    return torch.cat(heads, dim=-1) @ w[p + "o"].T


# -- feed-forwards --------------------------------------------------------------------------------
def dense(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    z = silu(h @ w[p + "gate"].T + w[p + "gate.b"]) * (h @ w[p + "up"].T + w[p + "up.b"])
    return z @ w[p + "down"].T + w[p + "down.b"]


def clamped(h: torch.Tensor, w: dict, p: str, limit: float) -> torch.Tensor:
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * torch.sigmoid(EXPERT_SLOPE * g) * (u + 1.0)) @ w[p + "down"].T


def choose(choice: list, top: int, groups=None) -> list:
    """The `top` outputs with the largest choice scores, in falling order (ties: lower index); with groups ({count, keep}: equal
    groups of neighbours) only those of the `keep` groups whose largest choice scores are the largest."""
    allowed = range(len(choice))
    if groups:
        per = len(choice) // groups["count"]
        worth = [max(choice[g * per:(g + 1) * per]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: (-worth[g], g))[:groups["keep"]]
        allowed = [e for e in allowed if e // per in kept]
    return sorted(allowed, key=lambda e: (-choice[e], e))[:top]


def route(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, top: int, scale: float, groups=None):
    """One token: its experts and their weights."""
    s = torch.softmax(router @ h, dim=0)
    chosen = choose([float(v) for v in s + correction], top, groups)
    picked = torch.stack([s[e] for e in chosen])
    return chosen, picked / (picked.sum() + SHARE_EPS) * scale


def mixture(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weight = route(h[t], w[p + "router"], w[p + "correction"], r["top"], r.get("scale", 1.0), r.get("groups"))
        for e, g in zip(chosen, weight):
            out[t] += g * clamped(h[t:t + 1], w, f"{p}e{e}.", mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        out = out + clamped(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


def feed_forward(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


# -- the model ---------------------------------------------------------------------------------
def layer(x: torch.Tensor, w: dict, i: int, spec: dict, eps: float) -> torch.Tensor:
    """Both sublayers read one norm's output and join the residual together."""
    p = f"l{i}."
    h = norm_around_zero(x, w[p + "norm1"], eps)
    y = attention(h, w, p + "mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        y = y + feed_forward(h, w, p + "mlp.", spec["mlp"])
    return x + y


def forward(config: dict, w: dict, tokens: list, layers_out: bool = False):
    """Logits [T, vocab] of one sequence (and, asked for, the residual after every layer run)."""
    eps = config["norm"]["eps"]
    x0 = x = embed(tokens, w, config)
    seen = []
    for i, again in layer_runs(config):
        if again:
            x = x + x0
        x = layer(x, w, i, config["layers"][i], eps)
        seen.append(x)
    logits = norm_around_zero(x, w["final.norm"], eps) @ w["embed"].T
    return (logits, torch.stack(seen)) if layers_out else logits


def greedy(config: dict, weights: dict, prompt, new_tokens: int) -> list:
    tokens, out = list(prompt), []
    for _ in range(new_tokens):
        nxt = int(torch.argmax(forward(config, weights, tokens)[-1]))
        out.append(nxt)
        tokens.append(nxt)
    return out
