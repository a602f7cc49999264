"""Small seeded Vekolix models for the tests: configuration, weights, and models in which one key or one router margin stands
out.  Engine, steps and error measure are those of folizen_util."""
from __future__ import annotations

import torch

from folizen_util import LIMIT, engine, error, run_portions, step, taps, tokens  # noqa: F401


def dense(ff=88):
    return {"kind": "dense", "ff": ff}


def experts(n=8, top=2, ff=48, limit=0.9, shared=(40, 1.4)):
    out = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": n, "top": top}}
    if shared is not None:
        out["shared"] = {"ff": shared[0], "limit": shared[1]}
    return out


def yarn(factor=4.0, original=64, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def rotation(dims, base, scaling):
    return {"base": base, "dims": dims} if scaling is None else {"base": base, "dims": dims, "scaling": scaling}


def parallel(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.25, rot=16, base=500.0, scaling=yarn(), lin_heads=3, lin_dim=20, lin_vdim=28, decay=None, scales=(0.8, 1.3),
             mlp=None):
    if decay is None:
        decay = [0.5, 0.93, 0.995, 0.999, 0.8, 1.0][:lin_heads] + [0.97] * max(0, lin_heads - 6)
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation(rot, base, scaling)}, "left_scale": scales[0],
        "right": {"heads": lin_heads, "dim": lin_dim, "vdim": lin_vdim, "decay": decay}, "right_scale": scales[1]}}


def latent(heads=3, dim=24, rot=8, vdim=40, q_rank=56, kv_rank=48, scale=0.2, base=3e4, mlp=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                              "scale": scale, "rot": {"base": base, "dims": rot}}}


def config(layers, width=96, vocab=150, eps=1e-5, mult=0.6, logit_scale=0.7, softcap=12.0):
    return {"architecture": "Vekolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit_scale,
            "logit_softcap": softcap, "layers": layers}


MIXED = [parallel(mlp=dense()), latent(mlp=experts(top=3)), latent(heads=5, dim=32, rot=16, vdim=32, q_rank=40, kv_rank=72),
         parallel(heads=3, kv_heads=3, dim=40, vdim=72, rot=40, scaling=None, lin_heads=5, lin_dim=36, lin_vdim=16, scales=(1.1, 0.7),
                  mlp=experts(n=5, top=1, ff=72, limit=1.5, shared=(104, 0.6)))]


def shapes(cfg):
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, W)}

    def norm(name):
        out.update({name: (W,), name + ".b": (W,), name + ".alpha": ()})
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        norm(p + "norm1")
        if l["type"] == "parallel":
            a, b = m["left"], m["right"]
            out.update({p + "mix.left." + n: (r, W) for n, r in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"]))})
            out[p + "mix.left.o"] = (W, a["heads"] * a["vdim"])
            qk, v = b["heads"] * b["dim"], b["heads"] * b["vdim"]
            out.update({p + "mix.right." + n: (r, W) for n, r in (("q", qk), ("k", qk), ("v", v), ("g", v))})
            out.update({p + "mix.right.o": (W, v), p + "mix.right.norm": (v,)})
        else:
            H, D, R, Dv, q, L = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["q_rank"], m["kv_rank"]
            out.update({p + "mix.dq": (q, W), p + "mix.dq.norm": (q,), p + "mix.uq": (H * (D + R), q), p + "mix.dkv": (L + R, W), p + "mix.dkv.norm": (L,),
                        p + "mix.uk": (H * D, L), p + "mix.uv": (H * Dv, L), p + "mix.g": (H, W), p + "mix.o": (W, H * Dv)})
        if not l["mlp"]:
            continue
        norm(p + "norm2")
        if l["mlp"]["kind"] == "dense":
            ff = l["mlp"]["ff"]
            out.update({p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
            continue
        units = [(f"e{e}", l["mlp"]["expert"]["ff"]) for e in range(l["mlp"]["router"]["experts"])]
        out[p + "mlp.router"] = (l["mlp"]["router"]["experts"], W)
        if l["mlp"].get("shared"):
            units.append(("shared", l["mlp"]["shared"]["ff"]))
            out[p + "mlp.shared.sg"] = (1, W)
        for n, ff in units:
            out.update({f"{p}mlp.{n}.gate": (ff, W), f"{p}mlp.{n}.up": (ff, W), f"{p}mlp.{n}.down": (W, ff)})
    norm("final.norm")
    return out


def weights(cfg, seed=0, margins=True):
    """margins: the routers read channels that only the embedding writes, with well separated values, so that rounding never
    decides between two experts; every token shuffles them its own way."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last == "alpha":
            t = 0.7 + 0.1 * t
        elif last in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.3 * t
        elif last == "b":
            t = 0.2 * t
        elif last == "router":
            t = 4.0 * t / shape[1] ** 0.5
        elif len(shape) == 2 and name != "embed":
            t = (3.0 if last in ("gate", "up", "sg", "g") else 1.7) * t / shape[1] ** 0.5
        out[name] = t
    routers = [n for n in out if n.endswith("router")]
    if margins and routers:
        n = max(out[r].shape[0] for r in routers)
        code = torch.linspace(-1.5, 1.5, n) if n > 1 else torch.zeros(1)
        out["embed"][:, -n:] = torch.stack([code[torch.randperm(n, generator=g)] for _ in range(cfg["vocab"])])
        for name, t in out.items():
            if name.endswith((".o", "down")):
                t[-n:] = 0
            elif name.endswith("norm2"):
                t[-n:] = 1
            elif name.endswith("norm2.b"):
                t[-n:] = 0
        for r in routers:
            E = out[r].shape[0]
            out[r] = torch.zeros_like(out[r])
            out[r][torch.arange(E), cfg["width"] - n + torch.randperm(n, generator=g)[:E]] = 2.5
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def spotlight(layer, width=128, vocab=100, scores=14.0):
    """A one-layer model in which token 1 (query) attends almost only to token 0 (key), wherever that stands: channel 0 is
    written by the key's embedding alone, channel 1 by the query's."""
    cfg = config([layer], width=width, vocab=vocab, mult=1.0, logit_scale=0.5, softcap=30.0)
    w = {k: v.float() for k, v in weights(cfg, seed=11).items()}
    w["embed"][:, :2] = 0
    w["embed"][0, 0] = w["embed"][1, 1] = 3.0
    w["l0.norm1"][:2], w["l0.norm1.b"][:2] = 1, 0
    for name, t in w.items():
        if name.endswith((".o", "down")):
            t[:2] = 0
    m = layer["mixer"]

    def aim(name, channel, rows, gain):
        """W[name] answers to the channel in the given rows only."""
        t = w["l0.mix." + name]
        t[:, channel] = 0
        t[rows, channel] = gain
    if layer["type"] == "parallel":
        m = m["left"]
        D = m["dim"]
        assert m["rot"]["dims"] < D                                    # the last channel is not rotated
        for name, n, ch in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
            aim("left." + name, ch, torch.arange(n) * D + D - 1, 8.0)
            w["l0.mix.left." + name] *= 0.5
        m["scale"] = scores / 16.0
        w["l0.mix.left.v"] *= 2
    else:
        for name, ch in (("dq", 1), ("dkv", 0)):
            aim(name, ch, torch.tensor([0]), 40.0)
            w[f"l0.mix.{name}.norm"][:] = 1
        D, R = m["dim"], m["rot_dim"]
        for name, per in (("uq", D + R), ("uk", D)):
            t = w["l0.mix." + name]
            t[:, 0] = 0
            t[torch.arange(m["heads"]) * per, 0] = 1.0
        m["scale"] = scores / (m["q_rank"] * m["kv_rank"]) ** 0.5
    return cfg, {k: v.to(torch.bfloat16) for k, v in w.items()}
