"""CPU: host side of the Folizen decoder (configuration reader, registry, page and state bookkeeping, step scheduler, trace
runner's command line) and the plain statement's own consistency."""
import importlib.util
import json
import os
import subprocess
import sys

import pytest
import torch

import folizen_util as fu
from folizen_util import attention, config, delta
from oracle import folizen

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
PKG = os.path.join(ROOT, "edge-fm-x_b200")


def load_build():
    spec = importlib.util.spec_from_file_location("efm_build", os.path.join(PKG, "build.py"))
    m = importlib.util.module_from_spec(spec)
    spec.loader.exec_module(m)
    return m


# ---- scheduler -----------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def driver(built, tmp_path_factory):
    build = load_build()
    exe = str(tmp_path_factory.mktemp("ss") / "step_scheduler_check")
    cmd = ["g++", "-O1", "-std=c++17", os.path.join(ROOT, "tests", "cpp", "step_scheduler_check.cpp"), "-o", exe,
           "-I", os.path.join(PKG, "src", "engine"), "-I", os.path.join(PKG, "include"), "-I", os.path.join(ROOT, "include"),
           "-I", build.dlpack_include(), "-L", os.path.join(PKG, "lib"), "-ledge_fm", "-lefm_b200", "-Wl,-rpath," + os.path.join(PKG, "lib"),
           "-Wl,-rpath,/usr/local/cuda/lib64"]
    subprocess.run(cmd, check=True, capture_output=True, text=True)
    return exe


@pytest.mark.parametrize("pages,states,live,seed", [(11, 4, 4, 1), (40, 4, 4, 2), (6, 2, 2, 3), (30, 0, 3, 4)])
def test_pages_and_states(driver, pages, states, live, seed):
    r = subprocess.run([driver, str(pages), str(states), str(live), str(seed), "600"], capture_output=True, text=True)
    assert r.stdout.strip() == "ok", r.stdout


# ---- configuration -------------------------------------------------------------------------------------------------------
def open_engine(tmp_path, cfg, w=None, **kw):
    return fu.engine(tmp_path, cfg, w if w is not None else fu.weights(cfg), **kw)


BAD = {
    "unknown type": (lambda c: c["layers"][0].__setitem__("type", "convolution"), "unknown type"),
    "no heads": (lambda c: c["layers"][1]["mixer"].pop("heads"), "heads"),
    "bad mlp": (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "routed"), "unknown kind"),
    "no width": (lambda c: c.pop("width"), "width"),
    "negative window": (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", -3), "size"),
    "no layers": (lambda c: c.__setitem__("layers", []), "layers"),
}


@pytest.mark.parametrize("name", sorted(BAD))
def test_configuration_errors(built, tmp_path, name):
    cfg = config([attention(ff=32), delta()])
    w = fu.weights(cfg)
    change, match = BAD[name]
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    with pytest.raises(ValueError, match=match):
        open_engine(tmp_path, cfg, w)


def test_registry(built, tmp_path):
    cfg = config([attention()])
    w = fu.weights(cfg)
    with pytest.raises(ValueError, match="model_name.*folizen"):
        open_engine(tmp_path, cfg, w, name="Llama")
    with pytest.raises(ValueError, match="model_name"):
        open_engine(tmp_path, dict(cfg, architecture="SomethingElse"), w)
    with pytest.raises(ValueError, match="compute_dtype"):
        open_engine(tmp_path, cfg, w, dtype="fp16")
    with pytest.raises(ValueError, match="neither requests nor pool_tokens"):
        open_engine(tmp_path, cfg, w, pool=0)


def test_trace_run_command_line(built, tmp_path):
    build = load_build()
    exe = build.build_trace_run()
    r = subprocess.run([exe, "--model", str(tmp_path)], capture_output=True, text=True)
    assert r.returncode == 2 and "usage" in r.stderr
    r = subprocess.run([exe, "--model", str(tmp_path), "--out", str(tmp_path), "--max-tokens", "64", "--dtype", "int8"], capture_output=True, text=True)
    assert r.returncode == 2
    r = subprocess.run([exe, "--model", str(tmp_path), "--out", str(tmp_path), "--max-tokens", "64"], capture_output=True, text=True)
    assert r.returncode == 1 and "config.json" in r.stderr
    wrapper = os.path.join(ROOT, "bin", "trace_run")
    assert os.access(wrapper, os.X_OK)
    assert subprocess.run([sys.executable, wrapper, "--nonsense"], capture_output=True).returncode == 2


# ---- the plain statement ---------------------------------------------------------------------------------------------------
def test_statement_is_consistent():
    """Each mechanism against a second formulation, and causality: a later token never changes an earlier logit."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(30, n, 8, generator=g, dtype=torch.float64) for n in (4, 2, 2))
    temp = torch.tensor([1.0, -0.5, 2.0, 0.3], dtype=torch.float64)
    out = folizen.window_attention(q, k, v, temp, kv_heads=2, scale=0.7, window=5)
    i, j = torch.arange(30)[:, None], torch.arange(30)[None, :]
    for h in range(4):
        s = (q[:, h] @ k[:, h // 2].T) * 0.7 * temp[h] - 2.0 ** (-8 * (h + 1) / 4) * (i - j)
        s[(j > i) | (i - j >= 5)] = -torch.inf
        assert torch.allclose(torch.softmax(s, -1) @ v[:, h // 2], out[:, h])
    r, kk, vv = (torch.randn(20, 6, generator=g, dtype=torch.float64) for _ in range(3))
    w, a = (torch.rand(20, 6, generator=g, dtype=torch.float64) for _ in range(2))
    o, S = folizen.general_delta(r, kk, vv, w, a)
    o1, S1 = folizen.general_delta(r[:7], kk[:7], vv[:7], w[:7], a[:7])
    o2, S2 = folizen.general_delta(r[7:], kk[7:], vv[7:], w[7:], a[7:], S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)
    # one step as a matrix: S = (diag(w) - (a u) u^T) S + k v^T
    u = kk / torch.sqrt((kk * kk).sum(-1, keepdim=True) + 1e-6)
    M = torch.zeros(6, 6, dtype=torch.float64)
    for t in range(20):
        M = (torch.diag(w[t]) - torch.outer(a[t] * u[t], u[t])) @ M + torch.outer(kk[t], vv[t])
    assert torch.allclose(M, S)
    cfg = config(fu.MIXED)
    W = fu.weights(cfg)
    toks = fu.tokens(cfg, 80)
    full, short = folizen.forward(cfg, W, toks).logits, folizen.forward(cfg, W, toks[:50]).logits
    assert torch.allclose(full[:50], short)
    changed = folizen.forward(cfg, W, toks[:79] + [(toks[79] + 1) % cfg["vocab"]]).logits
    assert torch.equal(changed[:79], full[:79])


def test_every_mechanism_shows_in_the_test_models():
    """Mistakes planted in the statement move the logits by more than the limits the GPU tests allow (1e-1 in bf16, 5e-5 in fp32)."""
    cfg = config(fu.MIXED)
    W = fu.weights(cfg, seed=7)
    toks = fu.tokens(cfg, 120)
    ref = folizen.forward(cfg, W, toks).logits.numpy()

    def moved(fn, original, name):
        setattr(folizen, name, fn)
        try:
            return fu.error(folizen.forward(cfg, W, toks).logits.numpy(), ref)
        finally:
            setattr(folizen, name, original)
    keep = folizen.distance_slope
    assert moved(lambda h, n: 0.0, keep, "distance_slope") > 0.15
    assert moved(lambda h, n: keep(h + 1, n), keep, "distance_slope") > 0.15
    keep_poly = folizen.poly_norm
    assert moved(lambda z, c, e: keep_poly(z, c * torch.tensor([1, 1, 1, 0]), e), keep_poly, "poly_norm") > 0.15
    assert moved(lambda z, c, e: keep_poly(z, c[[1, 0, 2, 3]], e), keep_poly, "poly_norm") > 0.15
    keep_delta = folizen.general_delta
    assert moved(lambda r, k, v, w, a, s=None: keep_delta(r, k, v, w, a * 0, s), keep_delta, "general_delta") > 0.15
    assert moved(lambda r, k, v, w, a, s=None: keep_delta(r, k, v, w * 0 + 1, a, s), keep_delta, "general_delta") > 0.15
    keep_side = folizen.token_side
    assert moved(lambda x, t, W, p, l, d, e: keep_side(x, t, W, p, 0, d, e), keep_side, "token_side") > 0.15
    for size in (39, 41):
        c2 = json.loads(json.dumps(cfg))
        c2["layers"][0]["mixer"]["mask"]["size"] = size
        assert fu.error(folizen.forward(c2, W, toks).logits.numpy(), ref) > 0
