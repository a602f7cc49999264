"""Plain CPU statement of the Folizen decoder: one function per mechanism, token by token where a recurrence is
involved, whole score rows where attention is.  No caches, no batches, no blocking; float64 by default so that a
comparison measures the product's rounding only.  TEST INFRASTRUCTURE ONLY.

Notation: x [T, width] is the residual stream of one sequence, t / i / j are positions from 0.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import torch

Weights = Dict[str, torch.Tensor]


# ---- mechanisms ----------------------------------------------------------------------------------------------
def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    """v / sqrt(mean(v^2) + eps) over the last axis."""
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """c0 rms(z) + c1 rms(z^2) + c2 rms(z^3) + c3, powers element-wise, rms over the row."""
    return coef[0] * rms(z, eps) + coef[1] * rms(z ** 2, eps) + coef[2] * rms(z ** 3, eps) + coef[3]


def distance_slope(h: int, n_heads: int) -> float:
    return 2.0 ** (-8.0 * (h + 1) / n_heads)


def window_attention(q, k, v, temp, *, kv_heads: int, scale: float, window: Optional[int]) -> torch.Tensor:
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv].  Position i sees j with 0 <= i - j < window;
    logit = (q_i . k_j) * scale * temp[h] - slope_h * (i - j)."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // kv_heads)
        slope = distance_slope(h, H)
        for i in range(T):
            lo = 0 if window is None else max(0, i - window + 1)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale * temp[h]
            s = s - slope * torch.arange(i - lo, -1, -1, dtype=q.dtype)
            out[i, h] = torch.softmax(s, 0) @ v[lo:i + 1, g]
    return out


def general_delta(r, k, v, w, a, state: Optional[torch.Tensor] = None):
    """One head.  r, k, w, a [T, D] and v [T, D]; w the per-channel decay, a the removal rate.
    S_t = diag(w_t) S_{t-1} - (a_t u_t)(u_t^T S_{t-1}) + k_t v_t^T with u_t = k_t / sqrt(|k_t|^2 + 1e-6); o_t = S_t^T r_t.
    Returns (o [T, D], final S)."""
    T, D = r.shape
    S = torch.zeros(D, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    o = torch.zeros(T, v.shape[-1], dtype=r.dtype)
    for t in range(T):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        S = w[t][:, None] * S - torch.outer(a[t] * u, u @ S) + torch.outer(k[t], v[t])
        o[t] = S.T @ r[t]
    return o, S


def delta_decay(h, w1, w2, w0):
    """exp(-e^{-1/2} sigmoid(W2 tanh(W1 h) + w0)), per head and key channel."""
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w1.T) @ w2.T + w0))


# ---- layers --------------------------------------------------------------------------------------------------
def attention_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms((h @ W[p + "q"].T).view(T, H, D), eps) * W[p + "q.norm"]
    k = rms((h @ W[p + "k"].T).view(T, G, D), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).view(T, G, Dv)
    window = m["mask"]["size"] if m.get("mask") else None
    o = window_attention(q, k, v, W[p + "temp"], kv_heads=G, scale=m["scale"], window=window)
    return o.reshape(T, H * Dv) @ W[p + "o"].T


def delta_mixer(h, W, p, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    r, k, v = (h @ W[p + n].T for n in "rkv")
    w = delta_decay(h, W[p + "w1"], W[p + "w2"], W[p + "w0"])
    a = torch.sigmoid(h @ W[p + "a"].T + W[p + "a.b"])
    o = torch.empty(T, H * D, dtype=h.dtype)
    for i in range(H):
        c = slice(i * D, (i + 1) * D)
        o[:, c] = rms(general_delta(r[:, c], k[:, c], v[:, c], w[:, c], a[:, c])[0], eps)
    return (o * W[p + "norm"] * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def dense_mlp(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def token_side(x, tokens, W, p, layer, dim, eps):
    e = W["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ W[p + "side.gate"].T) * e) @ W[p + "side.proj"].T
    return x + rms(y, eps) * W[p + "side.norm"]


MIXERS = {"attention": attention_mixer, "general_delta": delta_mixer}


@dataclass
class Run:
    logits: torch.Tensor                        # [T, vocab]
    layers: List[torch.Tensor] = field(default_factory=list)   # residual stream after every layer


def forward(config: dict, weights: Weights, tokens, dtype=torch.float64) -> Run:
    W = {k: v.to(dtype) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    ids = torch.as_tensor(list(tokens), dtype=torch.long)
    x = W["embed"][ids]
    out = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + rms(MIXERS[layer["type"]](x, W, p + "mix.", layer["mixer"], eps), eps) * W[p + "norm1"]
        if layer["mlp"] is not None:
            x = x + rms(dense_mlp(x, W, p + "mlp.", eps), eps) * W[p + "norm2"]
        if config.get("token_side"):
            x = token_side(x, ids, W, p, i, config["token_side"]["dim"], eps)
        out.append(x)
    return Run((rms(x, eps) * W["final.norm"]) @ W["head"].T, out)
