"""Small seeded Folizen models for the tests: configuration, weights, checkpoint, engine, and the CPU statement beside it."""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np
import torch

import cabi
from oracle import folizen


def attention(heads=3, kv_heads=1, dim=32, vdim=32, scale=0.2, size=40, ff=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if size is not None:
        mixer["mask"] = {"size": size}
    return {"type": "attention", "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def delta(heads=2, dim=32, ff=None):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=96, vocab=150, side=16, eps=1e-5):
    out = {"architecture": "Folizen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}
    if side:
        out["token_side"] = {"dim": side}
    return out


MIXED = [attention(ff=112), delta(), attention(heads=4, kv_heads=2, dim=24, vdim=40, size=70, ff=80), delta(heads=3, dim=48, ff=72)]


def shapes(cfg, rank=8):
    W, V, side = cfg["width"], cfg["vocab"], (cfg.get("token_side") or {}).get("dim", 0)
    out = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    if side:
        out["side.embed"] = (V, side * len(cfg["layers"]))
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = (W,)
        if l["type"] == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            out.update({p + "mix.q": (H * D, W), p + "mix.k": (G * D, W), p + "mix.v": (G * Dv, W), p + "mix.q.norm": (D,),
                        p + "mix.k.norm": (D,), p + "mix.temp": (H,), p + "mix.o": (W, H * Dv)})
        else:
            HD = m["heads"] * m["dim"]
            for n in "rkvga":
                out[p + "mix." + n] = (HD, W)
            out.update({p + "mix.a.b": (HD,), p + "mix.w1": (rank, W), p + "mix.w2": (HD, rank), p + "mix.w0": (HD,),
                        p + "mix.norm": (HD,), p + "mix.o": (W, HD)})
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff), p + "mlp.act": (4,)})
        if side:
            out.update({p + "side.gate": (side, W), p + "side.proj": (W, side), p + "side.norm": (W,)})
    return out


def weights(cfg, seed=0, rank=8):
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in shapes(cfg, rank).items():
        t = torch.randn(shape, generator=g)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2") or last == "temp":
            t = 1.0 + 0.3 * t
        elif name in ("embed", "side.embed"):
            pass
        elif len(shape) == 2:
            t = t / shape[1] ** 0.5
        elif last == "act":
            t = torch.tensor([0.7, -0.4, 0.5, 0.2]) + 0.1 * t
        out[name] = t.to(torch.bfloat16)
    return out


def tokens(cfg, n, seed=1):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def engine(tmp_path, cfg, w, dtype="fp32", *, pool=1024, live=4, requests=(), max_new=16, graph=True, name="", temperature=0.0, seed=0, stop=()):
    import edge_fm
    from safetensors.torch import save_file
    d = os.path.join(str(tmp_path), "model")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(d, "model.safetensors"))
    ec = {"prefill_model_path": d, "runtime": {"device": "cuda", "compute_dtype": dtype, "use_cuda_graph": graph},
          "kvcache": {"dtype": dtype, "attention_type": "gqa", "requests": list(requests), "pool_tokens": pool, "max_live_requests": live},
          "sampling": {"temperature": temperature, "top_p": 1.0, "top_k": 1, "seed": seed, "max_new_tokens": max_new, "stop_token_ids": list(stop)}}
    if name:
        ec["model_name"] = name
    path = os.path.join(str(tmp_path), f"engine_{dtype}.json")
    with open(path, "w") as f:
        json.dump(ec, f)
    return edge_fm.EdgeFM(path)


def step(eng, entries):
    """entries: (id, tokens, want) -> fp32 [wanted, vocab]."""
    rows = eng.step(entries)
    return np.stack([np.frombuffer(r, dtype=np.float32) for r in rows]) if rows else np.zeros((0, eng.vocab_size()), np.float32)


def run_portions(eng, rid, toks, cuts):
    """The whole sequence in portions of the given sizes (the last size repeats); logits of every position."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        out.append(step(eng, [(rid, toks[at:at + n], list(range(n)))]))
        at, k = at + n, k + 1
    eng.finish(rid)
    return np.concatenate(out)


def error(got, ref):
    """Worst row error: root mean square over the vocabulary after removing the mean, relative to the reference's spread."""
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    d = got - ref
    d -= d.mean(-1, keepdims=True)
    scale = np.sqrt(((ref - ref.mean(-1, keepdims=True)) ** 2).mean())
    return float((np.sqrt((d ** 2).mean(-1)) / scale).max())


def taps(eng, n_layers, rows, width, fn):
    """Residual stream after every layer of what fn() runs: [layers, rows, width]."""
    L, h = cabi.lib(), cabi.P(eng.backend_handle())
    assert L.efm_b200_decoder_set_taps(h, rows) == 0
    fn()
    out = np.zeros((n_layers, rows, width), np.float32)
    assert L.efm_b200_decoder_read_taps(h, out.ctypes.data_as(C.POINTER(C.c_float))) == 0
    assert L.efm_b200_decoder_set_taps(h, 0) == 0
    return out


LIMIT = {"fp32": 5e-5, "bf16": 1e-1}      # worst row; a mistake of one position shows as 0.3 and more
