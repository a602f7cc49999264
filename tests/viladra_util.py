"""Small seeded Viladra models for the tests: configuration, weights, and models in which one key, one window edge or one router
margin stands out.  Engine, steps and error measure are those of folizen_util."""
from __future__ import annotations

import numpy as np
import torch

from folizen_util import LIMIT, engine, error, run_portions, step, taps, tokens  # noqa: F401


def row_errors(got, ref):
    """folizen_util.error, row by row."""
    d = np.asarray(got, dtype=np.float64) - ref
    d -= d.mean(-1, keepdims=True)
    scale = np.sqrt(((ref - ref.mean(-1, keepdims=True)) ** 2).mean())
    return np.sqrt((d ** 2).mean(-1)) / scale


def experts(n=8, top=2, ff=48, scale=1.5, shared=40):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top, "scale": scale}}
    if shared is not None:
        out["shared"] = {"ff": shared}
    return out


def retention(heads=3, dim=20, vdim=28, rot=16, base=500.0, decay=None, mlp=None):
    if decay is None:
        decay = [0.93, 0.995, 0.5, 0.999, 0.8, 1.0][:heads] + [0.97] * max(0, heads - 6)
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay, "rot": {"base": base, "dims": rot}}}


def gla(heads=3, dim=24, vdim=36, tau=8.0, mlp=None):
    return {"type": "gla", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}}


def attention(heads=4, kv_heads=2, dim=24, vdim=40, scale=0.3, size=70, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        m["mask"] = {"size": size}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def config(layers, width=96, vocab=150, eps=1e-5, taps=4, embed=1.3, softcap=12.0):
    return {"architecture": "Viladra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps}, "embedding": {"scale": embed},
            "logit_softcap": softcap, "layers": layers}


MIXED = [gla(mlp=experts(top=3)), retention(mlp=experts(n=5, top=1, ff=72, scale=2.5, shared=104)), attention(),
         attention(heads=6, kv_heads=2, dim=32, vdim=24, size=33, mlp=experts(shared=None)), retention(heads=2, dim=36, vdim=72, rot=36), gla(heads=2, dim=40, vdim=16, tau=3.0)]

RANK = 12


def shapes(cfg, rank=RANK):
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "canon1": (W, taps), p + "dwa": (i + 2,), p + "mix.o": (W, H * Dv)})
        if l["type"] == "attention":
            G = m["kv_heads"]
            for n, r in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                out.update({p + "mix." + n: (r, W), p + "mix." + n + ".b": (r,)})
            out.update({p + "mix.q.norm": (H * D,), p + "mix.k.norm": (G * D,), p + "mix.pb": (H,), p + "mix.g": (H, W), p + "mix.o.b": (W,)})
        else:
            out.update({p + "mix." + n: (r, W) for n, r in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv))})
            if l["type"] == "gla":
                out.update({p + "mix.norm": (Dv,), p + "mix.a1": (rank, W), p + "mix.a2": (H * D, rank), p + "mix.a2.b": (H * D,)})
        if not l["mlp"]:
            continue
        out.update({p + "norm2": (W,), p + "canon2": (W, taps), p + "mlp.router": (l["mlp"]["router"]["experts"], W)})
        units = [(f"e{e}", l["mlp"]["expert"]["ff"]) for e in range(l["mlp"]["router"]["experts"])]
        if l["mlp"].get("shared"):
            units.append(("shared", l["mlp"]["shared"]["ff"]))
        for n, ff in units:
            out.update({f"{p}mlp.{n}.up": (ff, W), f"{p}mlp.{n}.down": (W, ff)})
    return out


def weights(cfg, seed=0, margins=True, rank=RANK):
    """margins: the routers read channels that only the embedding writes, with well separated values, so that rounding never
    decides between two experts; every token shuffles them its own way."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg, rank).items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            t = 1.0 + 0.3 * t
        elif last in ("canon1", "canon2"):
            t = 0.5 * t
        elif last == "dwa":
            t = 0.25 * t
            t[-1] += 0.9
        elif name.endswith("a2.b"):
            t = 2.5 + t
        elif last == "pb":
            t = -2.0 + 0.5 * t
        elif last == "b":
            t = 0.2 * t
        elif last == "router":
            t = 4.0 * t / shape[1] ** 0.5
        elif len(shape) == 2 and name != "embed":
            t = (3.0 if last in ("up", "g") else 1.7) * t / shape[1] ** 0.5
        out[name] = t
    routers = [n for n in out if n.endswith("router")]
    if margins and routers:
        n = max(out[r].shape[0] for r in routers)
        code = torch.linspace(-1.5, 1.5, n) if n > 1 else torch.zeros(1)
        out["embed"][:, -n:] = torch.stack([code[torch.randperm(n, generator=g)] for _ in range(cfg["vocab"])])
        for name, t in out.items():
            if name.endswith((".norm1", ".norm2")):                    # the sublayers leave these channels alone
                t[-n:] = 0
            elif name.endswith(("canon1", "canon2")):                  # and a token sees no other's
                t[-n:] = 0
        for r in routers:
            E = out[r].shape[0]
            out[r] = torch.zeros_like(out[r])
            out[r][torch.arange(E), cfg["width"] - n + torch.randperm(n, generator=g)[:E]] = 2.5 / cfg["embedding"]["scale"]
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def isolate(w, keep):
    """Silences the sublayers other than `keep` ("mix" or "mlp") through their norms."""
    other = {"mix": ".norm2", "mlp": ".norm1", "none": (".norm1", ".norm2")}[keep]
    return {k: torch.zeros_like(v) if k.endswith(other) else v for k, v in w.items()}


def spotlight(layer, width=128, vocab=100, score=9.0):
    """A one-layer attention model in which token 1 (query) gives weight almost only to token 0 (key), wherever that stands: channel 0 is
    written by the key's embedding alone, channel 1 by the query's.  Norms over all heads are fed by the biases of the other channels."""
    cfg = config([layer], width=width, vocab=vocab, embed=1.0, softcap=30.0)
    w = {k: v.float() for k, v in weights(cfg, seed=11).items()}
    m = layer["mixer"]
    D = m["dim"]
    w["embed"][:, :2] = 0
    w["embed"][0, 0] = w["embed"][1, 1] = 3.0
    w["l0.canon1"][:] = 0                                              # the neighbours see nothing of it
    w["l0.norm1"][:2] = 0
    for name, n, ch in (("q", m["heads"], 1), ("k", m["kv_heads"], 0)):
        t, b, c = w["l0.mix." + name], w[f"l0.mix.{name}.b"], w[f"l0.mix.{name}.norm"]
        t *= 0.05
        t[:, :2] = 0
        first = torch.arange(n) * D
        t[first, ch] = 4.0
        b[:] = 0
        b[first + D - 1] = 1.0                                         # keeps the root mean square away from zero
        c[:] = 1
        c[first + D - 1] = 0
    w["l0.mix.pb"][:] = -7.0
    rms = (D / (144.0 + 1.0)) ** 0.5 * 12.0                             # what the aimed channel becomes
    m["scale"] = (7.0 + score) / rms ** 2
    w["l0.mix.v"] *= 2
    w["l0.dwa"] = torch.tensor([0.2, 1.0])
    return cfg, {k: v.to(torch.bfloat16) for k, v in w.items()}
