"""Plain CPU statement of the Temuvik decoder: one function per mechanism, whole score rows for attention, one token and one
expert at a time for the routed feed-forward.  No caches, no batches, no blocking, no absorbed projections; float64 by
default so that a comparison measures the product's rounding only.  TEST INFRASTRUCTURE ONLY.

Notation: x [T, width] is the residual stream of one sequence, t / i / j are positions from 0.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional

import torch

Weights = Dict[str, torch.Tensor]


# ---- mechanisms ----------------------------------------------------------------------------------------------
def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def turn(u: torch.Tensor, v: torch.Tensor, base: float, dims: int, i: int):
    """Pair i of a head at every position t: turned by t * base^(-2 i / dims).  u, v [T, heads]."""
    a = torch.arange(u.shape[0], dtype=u.dtype)[:, None] * base ** (-2.0 * i / dims)
    return u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)


def rotate_half(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """x [T, heads, D]: channels i and i + dims / 2 are pair i; channels >= dims pass."""
    out = x.clone()
    for i in range(dims // 2):
        out[:, :, i], out[:, :, i + dims // 2] = turn(x[:, :, i], x[:, :, i + dims // 2], base, dims, i)
    return out


def rotate_pairs(x: torch.Tensor, base: float, dims: int) -> torch.Tensor:
    """The same with the neighbours 2 i and 2 i + 1 as pair i."""
    out = x.clone()
    for i in range(dims // 2):
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = turn(x[:, :, 2 * i], x[:, :, 2 * i + 1], base, dims, i)
    return out


def visible(i: int, size: Optional[int], keep: int) -> torch.Tensor:
    """Which of the keys 0 .. i position i sees: the last `size` (itself among them) and the first `keep` of the sequence."""
    j = torch.arange(i + 1)
    if size is None:
        return torch.ones(i + 1, dtype=torch.bool)
    return (i - j < size) | (j < keep)


def sink_softmax(s: torch.Tensor, sink: Optional[torch.Tensor]) -> torch.Tensor:
    """softmax over s with exp(sink) as one more term of the denominator."""
    if sink is None:
        return torch.softmax(s, 0)
    top = torch.maximum(s.max(), sink)
    e = torch.exp(s - top)
    return e / (e.sum() + torch.exp(sink - top))


def attention(q, k, v, *, scale: float, size: Optional[int], keep: int = 0, sink=None) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            see = visible(i, size, keep)
            s = (k[:i + 1, g][see] @ q[i, h]) * scale
            out[i, h] = sink_softmax(s, None if sink is None else sink[h]) @ v[:i + 1, g][see]
    return out


def route(z: torch.Tensor, top: int, groups: int, keep: int):
    """One token's router logits -> (chosen experts, their weights).  Scores softmax(z); only experts of the `keep` groups with
    the largest best score can be chosen; the weights are the scores as they are."""
    s = torch.softmax(z, 0)
    per = s.shape[0] // groups
    best = torch.stack([s[g * per:(g + 1) * per].max() for g in range(groups)])
    open_ = torch.topk(best, keep).indices.tolist()
    allowed = [e for e in range(s.shape[0]) if e // per in open_]
    chosen = sorted(allowed, key=lambda e: (-float(s[e]), e))[:top]
    return chosen, s[chosen]


def expert(h, gate, up, down):
    z = gate @ h
    return down @ (z * torch.sigmoid(z) * (up @ h))


def expert_mlp(h, W, p, mlp):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, w = route(W[p + "router"] @ h[t], r["top"], groups["count"], groups["keep"])
        for e, s in zip(chosen, w):
            out[t] += s * expert(h[t], W[f"{p}e{e}.gate"], W[f"{p}e{e}.up"], W[f"{p}e{e}.down"])
    return out


# ---- layers --------------------------------------------------------------------------------------------------
def attention_mixer(h, W, p, m, eps):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, D)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, D)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, Dv)
    q, k = (rms(rotate_half(x, m["rot"]["base"], m["rot"]["dims"]), eps) for x in (q, k))
    mask = m.get("mask") or {}
    o = attention(q, k, v, scale=m["scale"], size=mask.get("size"), keep=mask.get("keep_first", 0))
    return o.reshape(T, H * Dv) @ W[p + "o"].T


def latent_mixer(h, W, p, m, eps):
    T, H, D, R, Dv, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = ((rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, D + R)
    down = h @ W[p + "dkv"].T
    c = rms(down[:, :L], eps) * W[p + "dkv.norm"]
    kr = rotate_pairs(down[:, None, L:], base, R).expand(T, H, R)
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, D), kr], -1)
    q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], base, R)], -1)
    v = (c @ W[p + "uv"].T).view(T, H, Dv)
    mask = m.get("mask") or {}
    o = attention(q, k, v, scale=m["scale"], size=mask.get("size"), keep=mask.get("keep_first", 0), sink=W[p + "sink"])
    return (o.reshape(T, H * Dv) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


MIXERS: Dict[str, Callable] = {"attention": attention_mixer, "latent_attention": latent_mixer}


def layer_order(config: dict) -> List[int]:
    """Layer of every run: layers start .. stop - 1 run `times` times in a row."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + loop["times"] * list(range(loop["start"], loop["stop"])) + list(range(loop["stop"], n))


@dataclass
class Run:
    logits: torch.Tensor                        # [T, vocab]
    layers: List[torch.Tensor] = field(default_factory=list)   # residual stream after every layer run


def forward(config: dict, weights: Weights, tokens, dtype=torch.float64) -> Run:
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    x = W["embed"][ids] * config["embedding"]["scale"]
    out = []
    for i in layer_order(config):
        layer, p = config["layers"][i], f"l{i}."
        y = MIXERS[layer["type"]](rms(x, eps) * W[p + "norm1"], W, p + "mix.", layer["mixer"], eps)
        x = x + rms(y, eps) * W[p + "norm1b"]
        if layer["mlp"] is not None:
            y = expert_mlp(rms(x, eps) * W[p + "norm2"], W, p + "mlp.", layer["mlp"])
            x = x + rms(y, eps) * W[p + "norm2b"]
        out.append(x)
    return Run((rms(x, eps) * W["final.norm"]) @ W["head"].T, out)
