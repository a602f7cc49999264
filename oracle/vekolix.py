"""Plain CPU statement of the Vekolix decoder: one function per mechanism, whole score rows for attention, one token at a time
for the recurrence and the routed feed-forward.  No caches, no batches, no chunks, no absorbed projections; float64 by default
so that a comparison measures the product's rounding only.  TEST INFRASTRUCTURE ONLY.

Notation: x [T, width] is the residual stream of one sequence, t / i / j are positions from 0.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Callable, Dict, List, Optional

import torch

Weights = Dict[str, torch.Tensor]


# ---- mechanisms ----------------------------------------------------------------------------------------------
def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def tanh_norm(x: torch.Tensor, alpha: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """Element by element: no mean, no variance."""
    return torch.tanh(alpha * x) * w + b


def frequencies(rot: dict) -> torch.Tensor:
    """Angle per position of every pair.  With scaling: pairs that turn often within the original context keep their frequency,
    pairs that turn rarely are slowed down by the factor, a ramp over the pair's number lies between."""
    dims, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if sc:
        def pair_of(turns):                         # the (real) pair number that turns so many times in the original context
            return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(pair_of(sc["fast"])), 0), min(math.ceil(pair_of(sc["slow"])), dims - 1)
        for i in range(dims // 2):
            ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / sc["factor"] * ramp + f[i] * (1 - ramp)
    return torch.tensor(f, dtype=torch.float64)


def magnitude(rot: dict) -> float:
    """Multiplier of cos and sin."""
    return 0.1 * math.log(rot["scaling"]["factor"]) + 1.0 if rot.get("scaling") else 1.0


def turn(u: torch.Tensor, v: torch.Tensor, rot: dict, i: int):
    """Pair i of a head at every position.  u, v [T, heads]."""
    a = torch.arange(u.shape[0], dtype=u.dtype)[:, None] * frequencies(rot)[i].to(u.dtype)
    c, s = torch.cos(a) * magnitude(rot), torch.sin(a) * magnitude(rot)
    return u * c - v * s, v * c + u * s


def rotate_half(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, D]: channels i and i + dims / 2 are pair i; channels >= dims pass."""
    out, dims = x.clone(), rot["dims"]
    for i in range(dims // 2):
        out[:, :, i], out[:, :, i + dims // 2] = turn(x[:, :, i], x[:, :, i + dims // 2], rot, i)
    return out


def rotate_pairs(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """The same with the neighbours 2 i and 2 i + 1 as pair i."""
    out = x.clone()
    for i in range(rot["dims"] // 2):
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = turn(x[:, :, 2 * i], x[:, :, 2 * i + 1], rot, i)
    return out


def attention(q, k, v, scale: float) -> torch.Tensor:
    """Causal.  q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            out[i, h] = torch.softmax((k[:i + 1, g] @ q[i, h]) * scale, 0) @ v[:i + 1, g]
    return out


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def decayed_sum(q, k, v, decay) -> torch.Tensor:
    """S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  q, k [T, H, D], v [T, H, Dv] -> [T, H, Dv]."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=q.dtype)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.relu(z) ** 2


def clamped_glu(g: torch.Tensor, u: torch.Tensor, limit: float) -> torch.Tensor:
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def expert(h, gate, up, down, limit):
    return down @ clamped_glu(gate @ h, up @ h, limit)


def route(z: torch.Tensor, top: int):
    """One token's router logits -> (chosen experts, their weights)."""
    s = torch.sigmoid(z)
    chosen = sorted(range(z.shape[0]), key=lambda e: (-float(s[e]), e))[:top]
    return chosen, s[chosen]


def expert_mlp(h, W, p, mlp):
    """The weight scales what an expert reads; one more expert reads every token and its output is gated."""
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, w = route(W[p + "router"] @ h[t], mlp["router"]["top"])
        for e, s in zip(chosen, w):
            out[t] += expert(s * h[t], W[f"{p}e{e}.gate"], W[f"{p}e{e}.up"], W[f"{p}e{e}.down"], mlp["expert"]["limit"])
        if mlp.get("shared"):
            y = expert(h[t], W[p + "shared.gate"], W[p + "shared.up"], W[p + "shared.down"], mlp["shared"]["limit"])
            out[t] += torch.sigmoid(W[p + "shared.sg"][0] @ h[t]) * y
    return out


def dense_mlp(h, W, p, mlp):
    return relu_squared(h @ W[p + "up"].T) @ W[p + "down"].T


# ---- layers --------------------------------------------------------------------------------------------------
def left_mixer(h, W, p, m):
    T, H, G, D, Dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = (rotate_half((h @ W[p + n].T).view(T, -1, D), m["rot"]) for n in ("q", "k"))
    return attention(q, k, (h @ W[p + "v"].T).view(T, G, Dv), m["scale"]).reshape(T, H * Dv) @ W[p + "o"].T


def right_mixer(h, W, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v = (silu(h @ W[p + n].T).view(T, H, -1) for n in ("q", "k", "v"))
    o = decayed_sum(q, k, v, m["decay"]).reshape(T, -1)
    return (rms(o, eps) * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel_mixer(h, W, p, m, eps):
    return m["left_scale"] * left_mixer(h, W, p + "left.", m["left"]) + m["right_scale"] * right_mixer(h, W, p + "right.", m["right"], eps)


def latent_mixer(h, W, p, m, eps):
    T, H, D, R, Dv, L = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = ((rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, D + R)
    down = h @ W[p + "dkv"].T
    c = rms(down[:, :L], eps) * W[p + "dkv.norm"]
    k = torch.cat([(c @ W[p + "uk"].T).view(T, H, D), rotate_pairs(down[:, None, L:], m["rot"]).expand(T, H, R)], -1)
    q = torch.cat([q[..., :D], rotate_pairs(q[..., D:], m["rot"])], -1)
    o = attention(q, k, (c @ W[p + "uv"].T).view(T, H, Dv), m["scale"])
    return (o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]).reshape(T, H * Dv) @ W[p + "o"].T


MIXERS: Dict[str, Callable] = {"parallel": parallel_mixer, "latent_attention": latent_mixer}
MLPS: Dict[str, Callable] = {"dense": dense_mlp, "moe": expert_mlp}


def output(x, W, config):
    z = tanh_norm(x, W["final.norm.alpha"], W["final.norm"], W["final.norm.b"]) @ W["embed"].T * config["logit_scale"]
    return config["logit_softcap"] * torch.tanh(z / config["logit_softcap"])


@dataclass
class Run:
    logits: torch.Tensor                        # [T, vocab]
    layers: List[torch.Tensor] = field(default_factory=list)   # residual stream after every layer


def forward(config: dict, weights: Weights, tokens, dtype: Optional[torch.dtype] = torch.float64) -> Run:
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = W["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    out = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."

        def norm(x, name):
            return tanh_norm(x, W[p + name + ".alpha"], W[p + name], W[p + name + ".b"])
        x = x + m * MIXERS[layer["type"]](norm(x, "norm1"), W, p + "mix.", layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + m * MLPS[layer["mlp"]["kind"]](norm(x, "norm2"), W, p + "mlp.", layer["mlp"])
        out.append(x)
    return Run(output(x, W, config), out)
