"""Small seeded Temuvik models for the tests: configuration, weights, and models in which one key or one router margin stands
out.  Engine, steps and error measure are those of folizen_util."""
from __future__ import annotations

import torch

from folizen_util import LIMIT, engine, error, run_portions, step, taps, tokens  # noqa: F401


def experts(n=8, top=2, ff=48, groups=(2, 1)):
    router = {"experts": n, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def attention(heads=4, kv_heads=2, dim=32, vdim=24, scale=0.2, size=40, keep=5, rot=16, base=1e4, mlp=None):
    mask = None if size is None else {"size": size, "keep_first": keep}
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": mask,
                                                       "rot": {"base": base, "dims": rot}}}


def latent(heads=3, dim=24, rot=8, vdim=40, q_rank=56, kv_rank=48, scale=0.2, size=30, base=3e4, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                              "scale": scale, "mask": None if size is None else {"size": size},
                                                              "rot": {"base": base, "dims": rot}}}


def config(layers, width=96, vocab=150, eps=1e-5, scale=3.0, loop=None):
    out = {"architecture": "Temuvik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}, "layers": layers}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


MIXED = [attention(mlp=experts(top=3, groups=(4, 2))), latent(mlp=experts(n=6, ff=40, groups=(3, 2))),
         latent(heads=5, dim=32, rot=16, vdim=32, q_rank=40, kv_rank=72, size=70, mlp=None),
         attention(heads=3, kv_heads=3, dim=40, vdim=40, size=64, keep=70, rot=40, mlp=experts(n=5, top=1, ff=72, groups=None))]
MIXED_LOOP = (1, 3, 2)


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,), p + "mix.o": (W, H * Dv)})
        if l["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                out.update({p + f"mix.{n}": (rows, W), p + f"mix.{n}.b": (rows,)})
        else:
            R, q, L = m["rot_dim"], m["q_rank"], m["kv_rank"]
            out.update({p + "mix.dq": (q, W), p + "mix.dq.norm": (q,), p + "mix.uq": (H * (D + R), q), p + "mix.dkv": (L + R, W), p + "mix.dkv.norm": (L,),
                        p + "mix.uk": (H * D, L), p + "mix.uv": (H * Dv, L), p + "mix.sink": (H,), p + "mix.g": (H * Dv, W)})
        if l["mlp"]:
            ff, E = l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.router": (E, W)})
            for e in range(E):
                out.update({p + f"mlp.e{e}.gate": (ff, W), p + f"mlp.e{e}.up": (ff, W), p + f"mlp.e{e}.down": (W, ff)})
    return out


def weights(cfg, seed=0, margins=True):
    """margins: the routers read channels that only the embedding writes, with well separated values, so that rounding never
    decides between two experts; every layer shuffles them its own way."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2", "norm1b", "norm2b"):
            t = 1.0 + 0.3 * t
        elif last == "b":
            t = 0.5 * t
        elif last == "router":
            t = 2.0 * t / shape[1] ** 0.5
        elif len(shape) == 2 and name != "embed":
            t = t / shape[1] ** 0.5
        out[name] = t
    routers = [n for n in out if n.endswith("router")]
    if margins and routers:
        n = max(out[r].shape[0] for r in routers)
        V = cfg["vocab"]
        code = torch.linspace(-2, 2, n)
        out["embed"][:, -n:] = torch.stack([code[torch.randperm(n, generator=g)] for _ in range(V)])
        for name, t in out.items():
            if name.endswith(("norm1b", "norm2b")):
                t[-n:] = 0
            elif name.endswith("norm2"):
                t[-n:] = 1
        for r in routers:
            E = out[r].shape[0]
            out[r] = torch.zeros_like(out[r])
            place = torch.randperm(n, generator=g)[:E]
            out[r][torch.arange(E), cfg["width"] - n + place] = 8.0 / n
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def spotlight(layer, width=128, vocab=100, scores=14.0):
    """A one-layer model in which token 1 (query) attends almost only to token 0 (key), wherever that stands; for latent
    attention the sinks come next."""
    cfg = config([layer], width=width, vocab=vocab, scale=1.0)
    w = {k: v.float() for k, v in weights(cfg, seed=11).items()}
    basis, _ = torch.linalg.qr(torch.randn(width, width, generator=torch.Generator().manual_seed(4)))
    w["embed"][:vocab] = basis[:vocab] * width ** 0.5
    key, query = basis[0], basis[1]
    w["l0.norm1"][:] = 1
    m = layer["mixer"]

    def aim(name, direction, rows):
        """W[name] forgets the direction, then answers to it in the given rows only."""
        t = w["l0.mix." + name]
        t -= torch.outer(t @ direction, direction)
        t[rows] += 3.0 * direction
    if layer["type"] == "attention":
        D = m["dim"]
        for name, n, d in (("q", m["heads"], query), ("k", m["kv_heads"], key)):
            w[f"l0.mix.{name}.b"][:] = 0
            aim(name, d, torch.arange(n) * D + D - 1)                  # the last channel is not rotated
        m["scale"] = scores / D
    else:
        for name, d in (("dq", query), ("dkv", key)):
            aim(name, d, torch.tensor([0]))
            w[f"l0.mix.{name}.norm"][:] = 1
        D, R = m["dim"], m["rot_dim"]
        for name, step in (("uq", D + R), ("uk", D)):
            t = w["l0.mix." + name]
            t[:, 0] = 0
            t[torch.arange(m["heads"]) * step, 0] = 1.0
        m["scale"] = scores / (m["q_rank"] * m["kv_rank"]) ** 0.5
        w["l0.mix.sink"][:] = torch.linspace(5, 9, m["heads"])
    return cfg, {k: v.to(torch.bfloat16) for k, v in w.items()}
