"""Plain, slow forward pass of the Sosepel design: whole sequences, no cache, CPU only.

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


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w


def soft_cap(z: torch.Tensor, cap) -> torch.Tensor:
    return z if not cap else cap * torch.tanh(z / cap)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# -- the embedding ----------------------------------------------------------------------------------
def bigram_row(previous, token: int, buckets: int, mul_prev: int, mul_cur: int) -> int:
    """Which row of the bigram table belongs to `token` behind `previous` (None: the token is its sequence's first)."""
    if previous is None:
        return buckets
    return (previous * mul_prev + token * mul_cur) % buckets


def embed(tokens: list, w: dict, config: dict) -> torch.Tensor:
    e = config["embedding"]
    x = torch.stack([w["embed"][t] * e.get("scale", 1.0) for t in tokens])
    b = e.get("bigram")
    if b:
        rows = [bigram_row(tokens[i - 1] if i else None, t, b["buckets"], b["mul_prev"], b["mul_cur"]) for i, t in enumerate(tokens)]
        x = x + torch.stack([w["bigram"][r] for r in rows])
    return x


# -- the loop -----------------------------------------------------------------------------------------
def layer_runs(config: dict) -> list:
    """[(layer, a pass of the loop begins here), ...] in the order they run."""
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return [(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * times + [(i, False) for i in range(b, n)]


def join_input(x: torch.Tensor, x0: torch.Tensor, w_in: torch.Tensor) -> torch.Tensor:
    return torch.cat([x, x0], dim=-1) @ w_in.T


# -- differential attention -------------------------------------------------------------------------
def query_temperature(position: int, every: int, coef: float) -> float:
    return 1.0 + coef * math.log((position + 1) // every + 1)


def lambda_of(lq1, lk1, lq2, lk2, diff: float) -> float:
    return math.exp(float((lq1.double() * lk1.double()).sum())) - math.exp(float((lq2.double() * lk2.double()).sum())) + diff


def one_map(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, cap) -> torch.Tensor:
    """q [T, d] (its temperature already in it), k [T, d], v [T, dv] -> [T, dv]: token t sees the tokens up to itself."""
    out = torch.zeros((q.shape[0], v.shape[-1]), dtype=q.dtype)
    for t in range(q.shape[0]):
        s = soft_cap((k[:t + 1] @ q[t]) * scale, cap)
        out[t] = torch.softmax(s, dim=0) @ v[:t + 1]
    return out


def differential(a1: torch.Tensor, a2: torch.Tensor, lam: float, diff: float, eps: float) -> torch.Tensor:
    """The two maps' outputs [.., dv] of one head."""
    return unit_rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention(h: torch.Tensor, w: dict, p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, 2, d)
    k = (h @ w[p + "k"].T).view(T, G, 2, d)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    if m.get("q_temp"):
        temp = torch.tensor([query_temperature(t, m["q_temp"]["every"], m["q_temp"]["coef"]) for t in range(T)], dtype=h.dtype)
        q = q * temp[:, None, None, None]
    lam = lambda_of(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    heads = []
    for a in range(H):
        g = a // (H // G)
        a1, a2 = (one_map(q[:, a, i], k[:, g, i], v[:, g], m["scale"], m.get("softcap")) for i in (0, 1))
        heads.append(differential(a1, a2, lam, m["diff"], eps))
    return torch.cat(heads, dim=-1) @ w[p + "o"].T


# -- feed-forwards --------------------------------------------------------------------------------
def dense(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return torch.relu(h @ w[p + "up"].T) ** 2 @ w[p + "down"].T


def expert(h: torch.Tensor, w: dict, p: str) -> torch.Tensor:
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def choose(s: list, top: int, groups=None) -> list:
    """The `top` outputs with the largest scores, in falling order (ties: lower index); with groups ({count, keep}: equal
    groups of neighbours) only those of the `keep` groups whose two largest scores have the largest sums."""
    allowed = range(len(s))
    if groups:
        per = len(s) // groups["count"]
        worth = [sum(sorted(s[g * per:(g + 1) * per], reverse=True)[:2]) for g in range(groups["count"])]
        kept = sorted(range(groups["count"]), key=lambda g: (-worth[g], g))[:groups["keep"]]
        allowed = [e for e in allowed if e // per in kept]
    return sorted(allowed, key=lambda e: (-s[e], e))[:top]


def route(h: torch.Tensor, router: torch.Tensor, top: int, groups=None):
    """One token: its experts and their weights."""
    s = torch.sigmoid(router @ h)
    chosen = choose([float(v) for v in s], top, groups)
    picked = torch.stack([s[e] for e in chosen])
    return chosen, picked / (picked.sum() + 1e-20)


def mixture(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    r = mlp["router"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weight = route(h[t], w[p + "router"], r["top"], r.get("groups"))
        for e, g in zip(chosen, weight):
            out[t] += g * expert(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * expert(h, w, p + "shared.")
    return out


def feed_forward(h: torch.Tensor, w: dict, p: str, mlp: dict) -> torch.Tensor:
    return dense(h, w, p) if mlp["kind"] == "dense" else mixture(h, w, p, mlp)


# -- the model ---------------------------------------------------------------------------------
def layer(x: torch.Tensor, w: dict, i: int, spec: dict, eps: float) -> torch.Tensor:
    """Both sublayers read one norm's output; each result is scaled entry by entry before the sum."""
    p = f"l{i}."
    h = norm(x, w[p + "norm1"], eps)
    y = attention(h, w, p + "mix.", spec["mixer"], eps) * w[p + "ls1"]
    if spec.get("mlp") is not None:
        y = y + feed_forward(h, w, p + "mlp.", spec["mlp"]) * w[p + "ls2"]
    return x + y


def forward(config: dict, w: dict, tokens: list, layers_out: bool = False):
    """Logits [T, vocab] of one sequence (and, asked for, the residual after every layer run)."""
    eps = config["norm"]["eps"]
    x0 = x = embed(tokens, w, config)
    seen = []
    for i, begins in layer_runs(config):
        if begins:
            x = join_input(x, x0, w["loop.in"])
        x = layer(x, w, i, config["layers"][i], eps)
        seen.append(x)
    logits = soft_cap(norm(x, w["final.norm"], eps) @ w["embed"].T, config.get("logit_softcap"))
    return (logits, torch.stack(seen)) if layers_out else logits


def greedy(config: dict, weights: dict, prompt, new_tokens: int) -> list:
    tokens, out = list(prompt), []
    for _ in range(new_tokens):
        nxt = int(torch.argmax(forward(config, weights, tokens)[-1]))
        out.append(nxt)
        tokens.append(nxt)
    return out
