"""Plain CPU statement of the Viladra decoder: one function per mechanism, whole score rows for attention, one token at a time for
the recurrences, the short convolutions and the routed feed-forward.  No caches, no batches, no chunks; float64 by default so that a
comparison measures the product's rounding only.  TEST INFRASTRUCTURE ONLY.

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


def shifted_sum(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal convolution of every channel: the last column of w [width, taps] weighs the token itself, the one before it the token
    before, and so on; nothing stands ahead of the first token."""
    out = torch.zeros_like(h)
    taps = w.shape[1]
    for t in range(h.shape[0]):
        for back in range(min(taps, t + 1)):
            out[t] += w[:, taps - 1 - back] * h[t - back]
    return out


def mixed_input(h: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return h + shifted_sum(h, w)


def depth_average(a: torch.Tensor, results: List[torch.Tensor]) -> torch.Tensor:
    """results: the embedding and every layer's result so far; a: one number for each."""
    assert a.shape[0] == len(results)
    return sum(c * r for c, r in zip(a, results))


def rotate_half(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, D]: channels i and i + dims / 2 turn by t * base^(-2 i / dims); channels >= dims pass."""
    out, dims = x.clone(), rot["dims"]
    for i in range(dims // 2):
        a = torch.arange(x.shape[0], dtype=x.dtype)[:, None] * rot["base"] ** (-2.0 * i / dims)
        u, v = x[:, :, i], x[:, :, i + dims // 2]
        out[:, :, i], out[:, :, i + dims // 2] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return out


def decayed_sum(q, k, v, decay) -> torch.Tensor:
    """S_t = decay_h S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  q, k [T, H, D], v [T, H, Dv] -> [T, H, Dv]."""
    return gated_sum(q, k, v, torch.as_tensor(decay, dtype=q.dtype)[None, :, None].expand(q.shape))


def gated_sum(q, k, v, alpha) -> torch.Tensor:
    """The same with a decay per token, head and key channel: S_t = diag(alpha_t) S_{t-1} + k_t v_t^T.  alpha [T, H, D]."""
    T, H, D = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        S = torch.zeros(D, v.shape[-1], dtype=q.dtype)
        for t in range(T):
            S = alpha[t, h][:, None] * S + torch.outer(k[t, h], v[t, h])
            out[t, h] = S.T @ q[t, h]
    return out


def channel_decay(z: torch.Tensor, tau: float) -> torch.Tensor:
    return torch.sigmoid(z) ** (1.0 / tau)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def sigmoid_attention(q, k, v, scale: float, shift: torch.Tensor, window: int) -> torch.Tensor:
    """Weights sigmoid(scale q . k + shift_h), not normalised; i sees j with 0 <= i - j < window (0: every j <= i).  q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for i in range(T):
            first = max(0, i - window + 1) if window else 0
            out[i, h] = torch.sigmoid((k[first:i + 1, g] @ q[i, h]) * scale + shift[h]) @ v[first:i + 1, g]
    return out


def relu_squared(z: torch.Tensor) -> torch.Tensor:
    return torch.relu(z) ** 2


def expert(h, up, down):
    return down @ relu_squared(up @ h)


def route(z: torch.Tensor, top: int, scale: float):
    """One token's router logits -> (chosen experts, their weights)."""
    s = torch.softmax(z, -1)
    chosen = sorted(range(z.shape[0]), key=lambda e: (-float(s[e]), e))[:top]
    return chosen, s[chosen] * scale


def expert_mlp(h, W, p, mlp):
    out = torch.zeros_like(h)
    r = mlp["router"]
    for t in range(h.shape[0]):
        chosen, w = route(W[p + "router"] @ h[t], r["top"], r["scale"])
        for e, s in zip(chosen, w):
            out[t] += s * expert(h[t], W[f"{p}e{e}.up"], W[f"{p}e{e}.down"])
        if mlp.get("shared"):
            out[t] += expert(h[t], W[p + "shared.up"], W[p + "shared.down"])
    return out


# ---- layers --------------------------------------------------------------------------------------------------
def heads_of(h, w, n):
    return (h @ w.T).view(h.shape[0], n, -1)


def retention_mixer(h, W, p, m, eps):
    H = m["heads"]
    q, k = (rotate_half(heads_of(h, W[p + n], H), m["rot"]) for n in "qk")
    o = decayed_sum(q, k * m["dim"] ** -0.5, heads_of(h, W[p + "v"], H), m["decay"])
    return (rms(o, eps).reshape(h.shape[0], -1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def gla_mixer(h, W, p, m, eps):
    H = m["heads"]
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    o = gated_sum(heads_of(h, W[p + "q"], H) * m["dim"] ** -0.5, heads_of(h, W[p + "k"], H), heads_of(h, W[p + "v"], H),
                  channel_decay(z, m["tau"]).view(h.shape[0], H, -1))
    return ((rms(o, eps) * W[p + "norm"]).reshape(h.shape[0], -1) * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def attention_mixer(h, W, p, m, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (h @ W[p + n].T + W[p + n + ".b"] for n in "qkv")
    q, k = rms(q, eps) * W[p + "q.norm"], rms(k, eps) * W[p + "k.norm"]        # over all heads at once
    o = sigmoid_attention(q.view(T, H, -1), k.view(T, G, -1), v.view(T, G, -1), m["scale"], W[p + "pb"], (m.get("mask") or {}).get("size", 0))
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ W[p + "o"].T + W[p + "o.b"]


MIXERS: Dict[str, Callable] = {"retention": retention_mixer, "attention": attention_mixer, "gla": gla_mixer}


def output(x, W, config):
    z = (rms(x, config["norm"]["eps"]) * W["final.norm"]) @ W["embed"].T
    return config["logit_softcap"] * torch.tanh(z / config["logit_softcap"])


@dataclass
class Run:
    logits: torch.Tensor                        # [T, vocab]
    layers: List[torch.Tensor] = field(default_factory=list)   # residual stream after every layer


def forward(config: dict, weights: Weights, tokens, dtype: Optional[torch.dtype] = torch.float64) -> Run:
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = W["embed"][torch.as_tensor(list(tokens), dtype=torch.long)] * config["embedding"]["scale"]
    results, out = [x], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + rms(MIXERS[layer["type"]](mixed_input(x, W[p + "canon1"]), W, p + "mix.", layer["mixer"], eps), eps) * W[p + "norm1"]
        if layer["mlp"] is not None:
            x = x + rms(expert_mlp(mixed_input(x, W[p + "canon2"]), W, p + "mlp.", layer["mlp"]), eps) * W[p + "norm2"]
        results.append(x)
        x = depth_average(W[p + "dwa"], results)
        out.append(x)
    return Run(output(x, W, config), out)
