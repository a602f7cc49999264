"""CPU: host side of the Temuvik decoder (configuration reader, registry) and the plain statement's own consistency."""
import json

import pytest
import torch

import temuvik_util as tu
from oracle import temuvik
from temuvik_util import attention, config, experts, latent


BAD = {
    "unknown type": (lambda c: c["layers"][0].__setitem__("type", "convolution"), "unknown type"),
    "no heads": (lambda c: c["layers"][1]["mixer"].pop("heads"), "heads"),
    "no latent width": (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    "rotated part": (lambda c: c["layers"][1]["mixer"].__setitem__("rot_dim", 6), "rot_dim"),
    "no rotation": (lambda c: c["layers"][0]["mixer"].pop("rot"), "rot"),
    "odd rotation": (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 7), "even number"),
    "rotation too wide": (lambda c: c["layers"][0]["mixer"]["rot"].__setitem__("dims", 34), "rotated channels"),
    "bad mlp": (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "unknown kind"),
    "no router": (lambda c: c["layers"][0]["mlp"].pop("router"), "router"),
    "groups": (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("groups", {"count": 3, "keep": 1}), "equal groups"),
    "too many choices": (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 5), "at least expert_top"),
    "no width": (lambda c: c.pop("width"), "width"),
    "no embedding scale": (lambda c: c.pop("embedding"), "embedding"),
    "negative window": (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", -3), "size"),
    "negative keep": (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("keep_first", -1), "keep_first"),
    "no layers": (lambda c: c.__setitem__("layers", []), "layers"),
    "loop": (lambda c: c.__setitem__("loop", {"start": 1, "stop": 3, "times": 2}), "loop"),
    "kv heads": (lambda c: c["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple of kv_heads"),
}


@pytest.mark.parametrize("name", sorted(BAD))
def test_configuration_errors(built, tmp_path, name):
    cfg = config([attention(mlp=experts()), latent()])
    w = tu.weights(cfg)
    change, match = BAD[name]
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    with pytest.raises(ValueError, match=match):
        tu.engine(tmp_path, cfg, w)


def test_registry(built, tmp_path):
    cfg = config([attention()])
    w = tu.weights(cfg)
    with pytest.raises(ValueError, match="model_name.*temuvik"):
        tu.engine(tmp_path, cfg, w, name="Llama")
    with pytest.raises(ValueError, match="neither requests nor pool_tokens"):
        tu.engine(tmp_path, cfg, w, name="Temuvik", pool=0)


# ---- the plain statement -----------------------------------------------------------------------------------------------
def test_statement_is_consistent():
    """Each mechanism against a second formulation, and causality: a later token never changes an earlier logit."""
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(30, n, 8, generator=g, dtype=torch.float64) for n in (4, 2, 2))
    sink = torch.tensor([1.0, -0.5, 2.0, 30.0], dtype=torch.float64)
    out = temuvik.attention(q, k, v, scale=0.7, size=5, keep=3, sink=sink)
    i, j = torch.arange(30)[:, None], torch.arange(30)[None, :]
    for h in range(4):
        s = (q[:, h] @ k[:, h // 2].T) * 0.7
        s[(j > i) | ((i - j >= 5) & (j >= 3))] = -torch.inf
        p = torch.softmax(torch.cat([s, sink[h].expand(30, 1)], 1), -1)[:, :30]
        assert torch.allclose(p @ v[:, h // 2], out[:, h])
    # rotations as complex numbers; a score depends on the distance only
    x = torch.randn(20, 2, 12, generator=g, dtype=torch.float64)
    a = torch.arange(20, dtype=torch.float64)[:, None] * 50.0 ** (-torch.arange(4, dtype=torch.float64) / 4)
    z = torch.polar(torch.ones_like(a), a)[:, None, :]
    half = torch.complex(x[..., :4], x[..., 4:8]) * z
    assert torch.allclose(temuvik.rotate_half(x, 50.0, 8), torch.cat([half.real, half.imag, x[..., 8:]], -1))
    pairs = torch.view_as_complex(x[..., :8].reshape(20, 2, 4, 2).contiguous()) * z
    assert torch.allclose(temuvik.rotate_pairs(x, 50.0, 8), torch.cat([torch.view_as_real(pairs).reshape(20, 2, 8), x[..., 8:]], -1))
    same = torch.randn(1, 1, 12, generator=g, dtype=torch.float64).expand(20, 1, 12)
    r = temuvik.rotate_pairs(same, 50.0, 12)[:, 0]
    assert torch.allclose((r @ r.T).diagonal(3), (r @ r.T)[0, 3].expand(17))
    # the router: the best group's best experts, weights as they are
    logits = torch.tensor([1.0, 5.0, 4.9, 4.8, 0.0, 4.95], dtype=torch.float64)
    s = torch.softmax(logits, 0)
    assert temuvik.route(logits, 2, 3, 1)[0] == [1, 0] and temuvik.route(logits, 2, 1, 1)[0] == [1, 5]
    assert temuvik.route(logits, 3, 3, 2)[0] == [1, 5, 0]
    assert torch.equal(temuvik.route(logits, 2, 3, 1)[1], s[[1, 0]])
    assert temuvik.layer_order({"layers": [0] * 5, "loop": {"start": 1, "stop": 3, "times": 3}}) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    cfg = config(tu.MIXED, loop=tu.MIXED_LOOP)
    W = tu.weights(cfg)
    toks = tu.tokens(cfg, 80)
    full, short = temuvik.forward(cfg, W, toks).logits, temuvik.forward(cfg, W, toks[:50]).logits
    assert torch.allclose(full[:50], short)
    changed = temuvik.forward(cfg, W, toks[:79] + [(toks[79] + 1) % cfg["vocab"]]).logits
    assert torch.allclose(changed[:79], full[:79], atol=1e-12)


def test_latent_attention_in_the_latent_space():
    """Scores and sums over the latents themselves, queries and results carried through the up-projections: the same numbers."""
    layer = latent(heads=3, dim=10, rot=4, vdim=6, q_rank=12, kv_rank=14, size=9)
    cfg = config([layer], width=20, vocab=30)
    W = {k: v.double() for k, v in tu.weights(cfg, seed=1).items()}
    m, p, eps = layer["mixer"], "l0.mix.", 1e-5
    h = torch.randn(25, 20, generator=torch.Generator().manual_seed(2), dtype=torch.float64)
    down = h @ W[p + "dkv"].T
    c = temuvik.rms(down[:, :14], eps) * W[p + "dkv.norm"]
    r = temuvik.rotate_pairs(down[:, None, 14:], m["rot"]["base"], 4)[:, 0]
    q = ((temuvik.rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T).view(25, 3, 14)
    qr = temuvik.rotate_pairs(q[..., 10:], m["rot"]["base"], 4)
    out = torch.zeros(25, 3, 6, dtype=torch.float64)
    for hd in range(3):
        qa = q[:, hd, :10] @ W[p + "uk"].view(3, 10, 14)[hd]
        for i in range(25):
            lo = max(0, i - 8)
            s = (c[lo:i + 1] @ qa[i] + r[lo:i + 1] @ qr[i, hd]) * m["scale"]
            e, sink = torch.exp(s), torch.exp(W[p + "sink"][hd])
            out[i, hd] = W[p + "uv"].view(3, 6, 14)[hd] @ (e @ c[lo:i + 1]) / (e.sum() + sink)
    want = (out.reshape(25, 18) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T
    assert torch.allclose(temuvik.latent_mixer(h, W, p, m, eps), want)


def test_every_mechanism_shows_in_the_test_models(monkeypatch):
    """Mistakes planted in the statement move the logits by more than the limits the GPU tests allow (1e-1 in bf16, 5e-5 in fp32)."""
    cfg = config(tu.MIXED, loop=tu.MIXED_LOOP)
    W = tu.weights(cfg, seed=7)
    toks = tu.tokens(cfg, 120)
    ref = temuvik.forward(cfg, W, toks).logits.numpy()

    def moved(name, fn):
        with monkeypatch.context() as mp:
            mp.setattr(temuvik, name, fn)
            return tu.error(temuvik.forward(cfg, W, toks).logits.numpy(), ref)
    half, pairs, att, route, expert, order = (getattr(temuvik, n) for n in ("rotate_half", "rotate_pairs", "attention", "route", "expert", "layer_order"))
    assert moved("rotate_half", lambda x, b, d: pairs(x, b, d)) > 0.15
    assert moved("rotate_pairs", lambda x, b, d: half(x, b, d)) > 0.15
    assert moved("rotate_pairs", lambda x, b, d: x) > 0.15
    assert moved("attention", lambda q, k, v, sink=None, **kw: att(q, k, v, **kw)) > 0.15                      # no sink
    assert moved("attention", lambda q, k, v, sink=None, **kw: att(q, k, v, sink=None if sink is None else sink * kw["scale"], **kw)) > 0.05
    assert moved("attention", lambda q, k, v, keep=0, **kw: att(q, k, v, **kw)) > 0.1                          # first tokens lost
    assert moved("route", lambda z, t, g, n: route(z, t, 1, 1)) > 0.15                                         # no groups
    assert moved("route", lambda z, t, g, n: (lambda c, w: (c, w / w.sum()))(*route(z, t, g, n))) > 0          # renormalised weights
    assert moved("route", lambda z, t, g, n: (lambda c, w: (c[::-1], w))(*route(z, t, g, n))) > 0.15
    assert moved("expert", lambda h, g, u, d: expert(h, u, g, d)) > 0.15
    assert moved("layer_order", lambda c: list(range(len(c["layers"])))) > 0.15
    for change in (lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("size", 41), lambda c: c["layers"][0]["mixer"]["mask"].__setitem__("keep_first", 4),
                   lambda c: c["layers"][2]["mixer"]["mask"].__setitem__("size", 69), lambda c: c["embedding"].__setitem__("scale", 1.0)):
        c2 = json.loads(json.dumps(cfg))
        change(c2)
        assert tu.error(temuvik.forward(c2, W, toks).logits.numpy(), ref) > 1e-3
