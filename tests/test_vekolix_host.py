"""CPU: host side of the Vekolix decoder (configuration reader, registry) and the plain statement's own consistency."""
import json
import math

import pytest
import torch

import vekolix_util as vu
from oracle import vekolix
from vekolix_util import config, dense, experts, latent, parallel, yarn


def left(c):
    return c["layers"][0]["mixer"]["left"]


def right(c):
    return c["layers"][0]["mixer"]["right"]


BAD = {
    "unknown type": (lambda c: c["layers"][0].__setitem__("type", "attention"), "unknown type"),
    "no left half": (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    "no heads": (lambda c: right(c).pop("heads"), "heads"),
    "no latent width": (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), "kv_rank"),
    "rotated part": (lambda c: c["layers"][1]["mixer"].__setitem__("rot_dim", 6), "rot_dim"),
    "no rotation": (lambda c: left(c).pop("rot"), "rot"),
    "odd rotation": (lambda c: left(c)["rot"].__setitem__("dims", 7), "even number"),
    "rotation too wide": (lambda c: left(c)["rot"].__setitem__("dims", 26), "rotated channels"),
    "scaling": (lambda c: left(c)["rot"]["scaling"].__setitem__("factor", 0.0), "factor"),
    "scaling without a context": (lambda c: left(c)["rot"]["scaling"].pop("original"), "original"),
    "decays": (lambda c: right(c)["decay"].pop(), "decay"),
    "growing state": (lambda c: right(c)["decay"].__setitem__(0, 1.01), "decays"),
    "no scale": (lambda c: c["layers"][0]["mixer"].pop("right_scale"), "right_scale"),
    "wide head": (lambda c: right(c).__setitem__("vdim", 257), "above 256"),
    "kv heads": (lambda c: left(c).__setitem__("kv_heads", 3), "multiple of kv_heads"),
    "bad mlp": (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "gated"), "unknown kind"),
    "no router": (lambda c: c["layers"][0]["mlp"].pop("router"), "router"),
    "no limit": (lambda c: c["layers"][0]["mlp"]["shared"].pop("limit"), "limit"),
    "too many choices": (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 9), "at least expert_top"),
    "no multiplier": (lambda c: c.pop("residual_mult"), "residual_mult"),
    "negative cap": (lambda c: c.__setitem__("logit_softcap", -1.0), "logit_softcap"),
    "no layers": (lambda c: c.__setitem__("layers", []), "layers"),
}


@pytest.mark.parametrize("name", sorted(BAD))
def test_configuration_errors(built, tmp_path, name):
    cfg = config([parallel(mlp=experts()), latent(mlp=dense())])
    w = vu.weights(cfg)
    change, match = BAD[name]
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    with pytest.raises(ValueError, match=match):
        vu.engine(tmp_path, cfg, w)


def test_registry(built, tmp_path):
    cfg = config([latent()])
    w = vu.weights(cfg)
    with pytest.raises(ValueError, match="model_name.*vekolix"):
        vu.engine(tmp_path, cfg, w, name="Llama")
    with pytest.raises(ValueError, match="neither requests nor pool_tokens"):
        vu.engine(tmp_path, cfg, w, name="Vekolix", pool=0)


# ---- the plain statement -----------------------------------------------------------------------------------------------
def test_statement_is_consistent():
    """Each mechanism against a second formulation, and causality: a later token never changes an earlier logit."""
    g = torch.Generator().manual_seed(0)

    def rand(*s):
        return torch.randn(*s, generator=g, dtype=torch.float64)
    q, k, v = rand(30, 4, 8), rand(30, 2, 8), rand(30, 2, 6)
    out = vekolix.attention(q, k, v, 0.7)
    i, j = torch.arange(30)[:, None], torch.arange(30)[None, :]
    for h in range(4):
        s = ((q[:, h] @ k[:, h // 2].T) * 0.7).masked_fill(j > i, -torch.inf)
        assert torch.allclose(torch.softmax(s, -1) @ v[:, h // 2], out[:, h])
    # the recurrence as a masked product
    decay = [0.9, 1.0, 0.3, 0.0]
    v4 = rand(30, 4, 6)
    o = vekolix.decayed_sum(q, q.flip(0), v4, decay)
    for h in range(4):
        d = torch.tensor(decay[h], dtype=torch.float64) ** (i - j).clamp(min=0) * (j <= i)
        assert torch.allclose(((q[:, h] @ q.flip(0)[:, h].T) * d) @ v4[:, h], o[:, h])
    # rotations as complex numbers, scaled ones included
    x = rand(20, 2, 12)
    for rot in ({"base": 50.0, "dims": 8}, {"base": 50.0, "dims": 8, "scaling": yarn(factor=6.0, original=40, fast=4.0, slow=0.5)}):
        a = torch.arange(20, dtype=torch.float64)[:, None] * vekolix.frequencies(rot)
        z = torch.polar(torch.full_like(a, vekolix.magnitude(rot)), a)[:, None, :]
        half = torch.complex(x[..., :4], x[..., 4:8]) * z
        assert torch.allclose(vekolix.rotate_half(x, rot), torch.cat([half.real, half.imag, x[..., 8:]], -1))
        pairs = torch.view_as_complex(x[..., :8].reshape(20, 2, 4, 2).contiguous()) * z
        assert torch.allclose(vekolix.rotate_pairs(x, rot), torch.cat([torch.view_as_real(pairs).reshape(20, 2, 8), x[..., 8:]], -1))
    # scaled frequencies: fast pairs as they are, slow ones divided, the rest between
    rot = {"base": 1e4, "dims": 64, "scaling": yarn(factor=10.0, original=1000, fast=20.0, slow=1.0)}
    f, plain = vekolix.frequencies(rot), vekolix.frequencies({"base": 1e4, "dims": 64})
    turns = plain * 1000 / (2 * math.pi)
    ratio = f / plain
    assert torch.allclose(ratio[turns > 30], torch.ones(1, dtype=torch.float64)) and torch.allclose(ratio[turns < 0.7], torch.full((1,), 0.1, dtype=torch.float64))
    assert (ratio.diff() <= 1e-12).all() and ((ratio > 0.11) & (ratio < 0.99)).sum() > 5
    # the router, and an expert whose input carries the weight
    assert vekolix.route(torch.tensor([0.1, 2.0, -1.0, 1.9]), 2)[0] == [1, 3]
    assert torch.allclose(vekolix.route(torch.tensor([0.1, 2.0]), 2)[1], torch.sigmoid(torch.tensor([2.0, 0.1])))
    lim = vekolix.clamped_glu(torch.tensor([-9.0, 9.0, 0.5]), torch.tensor([9.0, -9.0, 0.5]), 1.0)
    s = torch.sigmoid(1.702 * torch.tensor([-9.0, 1.0, 0.5]))
    assert torch.allclose(lim, torch.tensor([-9.0, 1.0, 0.5]) * s * torch.tensor([2.0, 0.0, 1.5]))
    cfg = config(vu.MIXED)
    W = vu.weights(cfg)
    toks = vu.tokens(cfg, 80)
    full, short = vekolix.forward(cfg, W, toks).logits, vekolix.forward(cfg, W, toks[:50]).logits
    assert torch.allclose(full[:50], short)
    changed = vekolix.forward(cfg, W, toks[:79] + [(toks[79] + 1) % cfg["vocab"]]).logits
    assert torch.allclose(changed[:79], full[:79], atol=1e-12)


def test_every_mechanism_shows_in_the_test_models(monkeypatch):
    """Mistakes planted in the statement move the logits by more than the limits the GPU tests allow (1e-1 in bf16, 5e-5 in fp32)."""
    cfg = config(vu.MIXED)
    W = vu.weights(cfg, seed=7)
    toks = vu.tokens(cfg, 120)
    ref = vekolix.forward(cfg, W, toks).logits.numpy()

    def moved(name, fn):
        with monkeypatch.context() as mp:
            mp.setattr(vekolix, name, fn)
            return vu.error(vekolix.forward(cfg, W, toks).logits.numpy(), ref)
    half, pairs, mag, freq, sums, glu, expert, route, att = (getattr(vekolix, n) for n in (
        "rotate_half", "rotate_pairs", "magnitude", "frequencies", "decayed_sum", "clamped_glu", "expert", "route", "attention"))
    unscaled = {"base": 500.0, "dims": 16}
    assert moved("rotate_half", pairs) > 0.15
    assert moved("rotate_pairs", half) > 0.1
    assert moved("rotate_pairs", lambda x, r: x) > 0.1
    assert moved("magnitude", lambda r: 1.0) > 0.05
    assert moved("frequencies", lambda r: freq(unscaled) if r.get("scaling") else freq(r)) > 0.15
    assert moved("decayed_sum", lambda q, k, v, d: sums(q, k, v, [x * 0.98 for x in d])) > 0.05
    assert moved("decayed_sum", lambda q, k, v, d: sums(q, k, v, d) - (q * k).sum(-1, keepdim=True) * v) > 0.15        # without the token itself
    assert moved("decayed_sum", lambda q, k, v, d: torch.cat([sums(q[a:a + 64], k[a:a + 64], v[a:a + 64], d) for a in (0, 64)])) > 0.15      # a state lost
    assert moved("silu", lambda z: z) > 0.15
    assert moved("relu_squared", torch.relu) > 0.15
    assert moved("clamped_glu", lambda g, u, lim: glu(g, u, 1e9)) > 0.15
    assert moved("clamped_glu", lambda g, u, lim: glu(g, u - 1, lim)) > 0.15
    assert moved("expert", lambda h, a, b, c, lim: expert(h, b, a, c, lim)) > 0.15
    assert moved("route", lambda z, t: (lambda c, w: (c, torch.ones_like(w)))(*route(z, t))) > 0.1                     # weights lost
    assert moved("route", lambda z, t: (lambda c, w: (c, w / w.sum()))(*route(z, t))) > 0.1                            # renormalised
    assert moved("attention", lambda q, k, v, s: att(q, k, v, s * 1.5)) > 0.15
    assert moved("tanh_norm", lambda x, a, w, b: torch.tanh(a * x) * w) > 0.15
    assert moved("tanh_norm", lambda x, a, w, b: torch.tanh(x) * w + b) > 0.15
    for change in (lambda c: c.__setitem__("residual_mult", 0.5), lambda c: c["layers"][0]["mixer"].__setitem__("left_scale", 1.0),
                   lambda c: c["layers"][3]["mixer"].__setitem__("right_scale", 1.0), lambda c: c.__setitem__("logit_softcap", 30.0),
                   lambda c: c["layers"][1]["mlp"]["shared"].__setitem__("limit", 0.9), lambda c: c["layers"][1]["mlp"].__setitem__("shared", None)):
        c2 = json.loads(json.dumps(cfg))
        change(c2)
        assert vu.error(vekolix.forward(c2, W, toks).logits.numpy(), ref) > 1e-2
