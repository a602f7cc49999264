"""CPU: host side of the Viladra decoder (configuration reader, registry) and the plain statement's own consistency."""
import json

import pytest
import torch

import viladra_util as vu
from oracle import viladra
from viladra_util import attention, config, experts, gla, retention


def mixer(c, i=0):
    return c["layers"][i]["mixer"]


BAD = {
    "unknown type": (lambda c: c["layers"][0].__setitem__("type", "linear"), "unknown type"),
    "no heads": (lambda c: mixer(c).pop("heads"), "heads"),
    "no value size": (lambda c: mixer(c, 1).pop("vdim"), "vdim"),
    "no rotation": (lambda c: mixer(c).pop("rot"), "rot"),
    "odd rotation": (lambda c: mixer(c)["rot"].__setitem__("dims", 7), "even number"),
    "rotation too wide": (lambda c: mixer(c)["rot"].__setitem__("dims", 22), "rotated channels"),
    "decays": (lambda c: mixer(c)["decay"].pop(), "decay"),
    "growing state": (lambda c: mixer(c)["decay"].__setitem__(0, 1.01), "decays"),
    "no tau": (lambda c: mixer(c, 1).pop("tau"), "tau"),
    "bad tau": (lambda c: mixer(c, 1).__setitem__("tau", 0), "tau"),
    "wide head": (lambda c: mixer(c, 1).__setitem__("vdim", 257), "above 256"),
    "no scale": (lambda c: mixer(c, 2).pop("scale"), "scale"),
    "kv heads": (lambda c: mixer(c, 2).__setitem__("kv_heads", 3), "multiple of kv_heads"),
    "empty window": (lambda c: mixer(c, 2)["mask"].__setitem__("size", 0), "mask.size"),
    "bad mlp": (lambda c: c["layers"][0]["mlp"].__setitem__("kind", "dense"), "unknown kind"),
    "no router": (lambda c: c["layers"][0]["mlp"].pop("router"), "router"),
    "no router scale": (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "scale"),
    "too many choices": (lambda c: c["layers"][0]["mlp"]["router"].__setitem__("top", 9), "expert_top"),
    "no taps": (lambda c: c["canon"].pop("taps"), "taps"),
    "too many taps": (lambda c: c["canon"].__setitem__("taps", 17), "conv_taps"),
    "no embedding scale": (lambda c: c.pop("embedding"), "embedding"),
    "no cap": (lambda c: c.pop("logit_softcap"), "logit_softcap"),
    "no eps": (lambda c: c.pop("norm"), "norm"),
    "no layers": (lambda c: c.__setitem__("layers", []), "layers"),
}


@pytest.mark.parametrize("name", sorted(BAD))
def test_configuration_errors(built, tmp_path, name):
    cfg = config([retention(mlp=experts()), gla(), attention()])
    w = vu.weights(cfg)
    change, match = BAD[name]
    cfg = json.loads(json.dumps(cfg))
    change(cfg)
    with pytest.raises(ValueError, match=match):
        vu.engine(tmp_path, cfg, w)


def test_registry(built, tmp_path):
    cfg = config([gla()])
    w = vu.weights(cfg)
    with pytest.raises(ValueError, match="model_name.*viladra"):
        vu.engine(tmp_path, cfg, w, name="Llama")
    with pytest.raises(ValueError, match="neither requests nor pool_tokens"):
        vu.engine(tmp_path, cfg, w, name="Viladra", pool=0)


# ---- the plain statement -----------------------------------------------------------------------------------------------
def test_statement_is_consistent():
    """Each mechanism against a second formulation, and causality: a later token never changes an earlier logit."""
    g = torch.Generator().manual_seed(0)

    def rand(*s):
        return torch.randn(*s, generator=g, dtype=torch.float64)
    i, j = torch.arange(30)[:, None], torch.arange(30)[None, :]
    # attention as masked products
    q, k, v, shift = rand(30, 4, 8), rand(30, 2, 8), rand(30, 2, 6), rand(4)
    for window in (0, 1, 7):
        out = viladra.sigmoid_attention(q, k, v, 0.7, shift, window)
        seen = (j <= i) & ((i - j < window) if window else torch.tensor(True))
        for h in range(4):
            s = torch.sigmoid((q[:, h] @ k[:, h // 2].T) * 0.7 + shift[h]) * seen
            assert torch.allclose(s @ v[:, h // 2], out[:, h])
    # the recurrences as masked products: constant decays, and decays per channel
    decay, k4, v4 = [0.9, 1.0, 0.3, 0.0], rand(30, 4, 8), rand(30, 4, 6)
    o = viladra.decayed_sum(q, k4, v4, decay)
    alpha = viladra.channel_decay(rand(30, 4, 8), 3.0)
    z = rand(5)
    assert torch.allclose(viladra.channel_decay(z, 2.0) ** 2, torch.sigmoid(z))
    o2 = viladra.gated_sum(q, k4, v4, alpha)
    sums = torch.cumsum(torch.log(alpha), 0)
    for h in range(4):
        d = torch.tensor(decay[h], dtype=torch.float64) ** (i - j).clamp(min=0) * (j <= i)
        assert torch.allclose(((q[:, h] @ k4[:, h].T) * d) @ v4[:, h], o[:, h])
        e = torch.exp((sums[:, None, h] - sums[None, :, h]).masked_fill((j > i)[..., None], -torch.inf))
        assert torch.allclose(torch.einsum("td,sd,tsd->ts", q[:, h], k4[:, h], e) @ v4[:, h], o2[:, h])
    # the rotation as complex numbers
    x, rot = rand(20, 2, 12), {"base": 50.0, "dims": 8}
    a = torch.arange(20, dtype=torch.float64)[:, None] * 50.0 ** (-torch.arange(4, dtype=torch.float64) / 4)
    half = torch.complex(x[..., :4], x[..., 4:8]) * torch.polar(torch.ones_like(a), a)[:, None, :]
    assert torch.allclose(viladra.rotate_half(x, rot), torch.cat([half.real, half.imag, x[..., 8:]], -1))
    # the convolution as torch's
    h, w = rand(20, 5), rand(5, 3)
    conv = torch.nn.functional.conv1d(torch.nn.functional.pad(h.T[None], (2, 0)), w[:, None, :], groups=5)[0].T
    assert torch.allclose(viladra.shifted_sum(h, w), conv)
    assert torch.allclose(viladra.depth_average(torch.tensor([2.0, -1.0], dtype=torch.float64), [h, conv]), 2 * h - conv)
    # the router
    assert viladra.route(torch.tensor([0.1, 2.0, -1.0, 1.9]), 2, 1.0)[0] == [1, 3]
    assert torch.allclose(viladra.route(torch.tensor([0.1, 2.0]), 1, 3.0)[1], 3 * torch.softmax(torch.tensor([0.1, 2.0]), 0)[1:])
    assert torch.allclose(viladra.relu_squared(torch.tensor([-2.0, 3.0])), torch.tensor([0.0, 9.0]))
    cfg = config(vu.MIXED)
    W = vu.weights(cfg)
    toks = vu.tokens(cfg, 80)
    full, short = viladra.forward(cfg, W, toks).logits, viladra.forward(cfg, W, toks[:50]).logits
    assert torch.allclose(full[:50], short)
    changed = viladra.forward(cfg, W, toks[:79] + [(toks[79] + 1) % cfg["vocab"]]).logits
    assert torch.allclose(changed[:79], full[:79], atol=1e-12)


def test_every_mechanism_shows_in_the_test_models(monkeypatch):
    """Mistakes planted in the statement move the logits by more than the limits the GPU tests allow (1e-1 in bf16, 5e-5 in fp32)."""
    cfg = config(vu.MIXED)
    W = vu.weights(cfg, seed=7)
    toks = vu.tokens(cfg, 120)
    ref = viladra.forward(cfg, W, toks).logits.numpy()

    def moved(name, fn):
        with monkeypatch.context() as mp:
            mp.setattr(viladra, name, fn)
            return vu.error(viladra.forward(cfg, W, toks).logits.numpy(), ref)
    conv, avg, half, sums, gated, decay, att, expert, route = (getattr(viladra, n) for n in (
        "shifted_sum", "depth_average", "rotate_half", "decayed_sum", "gated_sum", "channel_decay", "sigmoid_attention", "expert", "route"))
    assert moved("shifted_sum", lambda h, w: conv(h, w.flip(1))) > 0.15
    assert moved("shifted_sum", lambda h, w: conv(h, torch.cat([torch.zeros_like(w[:, :1]), w[:, 1:]], 1))) > 0.15       # the oldest token lost
    assert moved("shifted_sum", lambda h, w: torch.cat([conv(h[:64], w), conv(h[64:], w)])) > 0.15                       # the state lost
    assert moved("mixed_input", lambda h, w: conv(h, w)) > 0.15
    assert moved("depth_average", lambda a, r: avg(a[1:], r[1:])) > 0.15
    assert moved("depth_average", lambda a, r: avg(a[:-1], r[:-1]) + r[-1]) > 0.1
    assert moved("rotate_half", lambda x, r: x) > 0.15
    assert moved("rotate_half", lambda x, r: half(x, {**r, "base": r["base"] * 1.2})) > 0.05
    assert moved("decayed_sum", lambda q, k, v, d: sums(q, k, v, [x * 0.97 for x in d])) > 0.1
    assert moved("decayed_sum", lambda q, k, v, d: sums(q, k, v, d) - (q * k).sum(-1, keepdim=True) * v) > 0.15          # without the token itself
    assert moved("decayed_sum", lambda q, k, v, d: torch.cat([sums(q[:64], k[:64], v[:64], d), sums(q[64:], k[64:], v[64:], d)])) > 0.15
    assert moved("gated_sum", lambda q, k, v, a: gated(q, k, v, torch.cat([a[1:], a[:1]]))) > 0.15                       # the next token's decay
    assert moved("gated_sum", lambda q, k, v, a: gated(q, k, v, a.mean(-1, keepdim=True).expand(a.shape))) > 0.1         # one decay for all channels
    assert moved("channel_decay", lambda z, tau: decay(z, 1.0)) > 0.15
    assert moved("silu", torch.sigmoid) > 0.15
    assert moved("sigmoid_attention", lambda q, k, v, s, b, w: att(q, k, v, s, b, w + 1)) > 0.02
    assert moved("sigmoid_attention", lambda q, k, v, s, b, w: att(q, k, v, s, 0 * b, w)) > 0.15
    assert moved("sigmoid_attention", lambda q, k, v, s, b, w: att(q, k, v, 1.0, b, w)) > 0.15
    assert moved("relu_squared", torch.relu) > 0.15
    assert moved("route", lambda z, t, s: route(z, t, 1.0)) > 0.1
    assert moved("route", lambda z, t, s: (lambda c, w: (c, w / w.sum()))(*route(z, t, s))) > 0.1                        # renormalised
    assert moved("expert", lambda h, u, d: 0 * expert(h, u, d)) > 0.15
    for change in (lambda c: c["embedding"].__setitem__("scale", 1.0), lambda c: c.__setitem__("logit_softcap", 30.0), lambda c: c["norm"].__setitem__("eps", 0.1),
                   lambda c: c["layers"][1]["mlp"].__setitem__("shared", None), lambda c: c["layers"][3]["mixer"].pop("mask")):
        c2 = json.loads(json.dumps(cfg))
        change(c2)
        assert vu.error(viladra.forward(c2, W, toks).logits.numpy(), ref) > 1e-2
    for name in ("l2.mix.g", "l2.mix.o.b", "l3.mix.q.b", "l3.mix.v.b", "l0.mix.g", "l0.mix.a2.b", "l5.mix.norm", "l1.mlp.shared.up"):
        w2 = {**W, name: torch.zeros_like(W[name])}
        assert vu.error(viladra.forward(cfg, w2, toks).logits.numpy(), ref) > 0.02, name


def test_spotlight_models_show_one_key():
    """Replacing the one key that stands out changes what the query reads; a window one token shorter does, too."""
    cfg, w = vu.spotlight(attention(size=50))
    toks = (2 + torch.randint(0, 90, (120,), generator=torch.Generator().manual_seed(0))).tolist()
    toks[119] = 1

    def last(place, size=50):
        t = list(toks)
        if place is not None:
            t[place] = 0
        c = json.loads(json.dumps(cfg))
        c["layers"][0]["mixer"]["mask"]["size"] = size
        return viladra.forward(c, w, t).logits[-1:].numpy()
    blind = last(None)
    assert vu.error(last(70), blind) > 0.2                             # the first token inside
    assert vu.error(last(69), blind) < 1e-2                            # the last one outside
    assert vu.error(last(70, 49), last(70)) > 0.2 and vu.error(last(69, 51), last(69)) > 0.2
