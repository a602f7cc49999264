"""GPU: the Folizen decoder against its plain CPU statement: every mechanism alone, odd sizes, portions, batches, reused
pages and state slots, window edges, far keys, long decoding, and generation through the engine's own entry points."""
import ctypes as C

import numpy as np
import pytest
import torch

import folizen_util as fu
from folizen_util import attention, config, delta
from oracle import folizen

pytestmark = pytest.mark.gpu


def reference(cfg, w, toks):
    return folizen.forward(cfg, w, toks)


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
def isolate(w, keep):
    """Silences sublayers by zeroing their output projections (rms(0) = 0): only `keep` moves the residual stream."""
    out = dict(w)
    for k, v in w.items():
        if (k.endswith("mix.o") and keep != "mixer") or (k.endswith("mlp.down") and keep != "mlp") or (k.endswith("side.proj") and keep != "side"):
            out[k] = torch.zeros_like(v)
    return out


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("what,layer", [("mixer", attention(ff=48)), ("mixer", delta(ff=48)), ("mlp", attention(ff=200)), ("mlp", delta(ff=36)),
                                        ("side", attention()), ("side", delta())])
def test_mechanism_alone(built, tmp_path, dtype, what, layer):
    cfg = config([layer, layer])
    w = isolate(fu.weights(cfg, seed=3), what)
    toks = fu.tokens(cfg, 90)
    eng = fu.engine(tmp_path, cfg, w, dtype)
    ref = reference(cfg, w, toks)
    got = fu.taps(eng, 2, 90, cfg["width"], lambda: fu.step(eng, [("w", toks, [])]))
    eng.finish("w")
    for i in range(2):
        r = ref.layers[i].numpy()
        err = np.abs(got[i] - r).max() / np.abs(r).max()
        assert err < (2e-5 if dtype == "fp32" else 2e-2), (i, err)
    # the same layer one token at a time: the last token's stream
    fu.step(eng, [("d", toks[:89], [])])
    got = fu.taps(eng, 2, 1, cfg["width"], lambda: fu.step(eng, [("d", toks[89:], [0])]))
    for i in range(2):
        r = ref.layers[i][89:].numpy()
        assert np.abs(got[i] - r).max() / np.abs(r).max() < (2e-5 if dtype == "fp32" else 2e-2)
    eng.finish("d")


# ---- sizes -----------------------------------------------------------------------------------------------------------
SIZES = {
    "single": (config([attention(heads=1, kv_heads=1, dim=8, vdim=8, size=1, ff=8), delta(heads=1, dim=8)], width=16, vocab=32, side=8), 1),
    "odd": (config([attention(heads=5, kv_heads=5, dim=20, vdim=12, size=33, ff=50), delta(heads=3, dim=20, ff=30)], width=76, vocab=131, side=10,
                   eps=1e-3), 9),
    "wide_group": (config([attention(heads=12, kv_heads=1, dim=64, vdim=96, size=100, ff=256), delta(heads=1, dim=96)], width=192, vocab=301, side=24), 24),
    "no_window": (config([attention(heads=4, kv_heads=4, dim=48, vdim=128, size=None), delta(heads=4, dim=64)], width=128, vocab=96, side=40), 40),
    "large_heads": (config([attention(heads=2, kv_heads=1, dim=160, vdim=72, size=64, ff=96), delta(heads=1, dim=160), delta(heads=1, dim=256)],
                           width=160, vocab=90, side=12), 33),
    "no_side": (config([delta(heads=2, dim=128, ff=64), attention(heads=6, kv_heads=3, dim=128, vdim=64, size=129)], width=256, vocab=80, side=0), 16),
    "value_256": (config([attention(heads=3, kv_heads=1, dim=256, vdim=256, size=65), attention(heads=2, kv_heads=2, dim=192, vdim=192, size=20)],
                         width=64, vocab=70, side=8), 8),
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(built, tmp_path, name, dtype):
    cfg, rank = SIZES[name]
    w = fu.weights(cfg, seed=5, rank=rank)
    toks = fu.tokens(cfg, 150)
    ref = reference(cfg, w, toks).logits.numpy()
    eng = fu.engine(tmp_path, cfg, w, dtype)
    assert fu.error(fu.run_portions(eng, "w", toks, [150]), ref) < fu.LIMIT[dtype]
    assert fu.error(fu.run_portions(eng, "d", toks, [130, 1]), ref) < fu.LIMIT[dtype]


# ---- schedules -------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=["fp32", "bf16"])
def mixed(request, tmp_path_factory, built):
    cfg = config(fu.MIXED)
    w = fu.weights(cfg, seed=7)
    seqs = {k: fu.tokens(cfg, n, seed=20 + i) for i, (k, n) in enumerate((("a", 260), ("b", 131), ("c", 64), ("d", 1), ("e", 200)))}
    refs = {k: reference(cfg, w, t).logits.numpy() for k, t in seqs.items()}
    eng = fu.engine(tmp_path_factory.mktemp("mixed"), cfg, w, request.param, pool=704)
    return cfg, w, eng, seqs, refs, fu.LIMIT[request.param]


@pytest.mark.parametrize("cuts", [[260], [1], [2], [3, 2], [64], [63, 1, 65, 2], [17, 2, 40, 5], [128, 15, 16, 2]])
def test_portions(mixed, cuts):
    _, _, eng, seqs, refs, limit = mixed
    assert fu.error(fu.run_portions(eng, "p", seqs["a"], cuts), refs["a"]) < limit


def test_batches_of_unequal_requests_and_reuse(mixed):
    """Portions beside decoded tokens, four live at a time, requests that pause, pages and slots that are used again."""
    _, _, eng, seqs, refs, limit = mixed
    rng = np.random.default_rng(3)
    pending = [(f"{k}{r}", k) for r in range(3) for k in "abcde"]
    live, worst = {}, 0.0
    while pending or live:
        while pending and len(live) < 4 and sum((len(seqs[k]) + 63) // 64 for k, _ in live.values()) + (len(seqs[pending[0][1]]) + 63) // 64 <= 11:
            rid, k = pending.pop(0)
            live[rid] = (k, 0)
        entries, spans = [], []
        for rid, (k, at) in live.items():
            if len(live) > 1 and rng.random() < 0.2:
                continue                                             # left out of this step
            n = min(int(rng.choice([1, 1, 2, 3, 16, 40, 90])), len(seqs[k]) - at)
            entries.append((rid, seqs[k][at:at + n], list(range(n))))
            spans.append((rid, k, at, n))
        if not entries:
            continue
        got, row = fu.step(eng, entries), 0
        for rid, k, at, n in spans:
            worst = max(worst, fu.error(got[row:row + n], refs[k][at:at + n]))
            row += n
            if at + n == len(seqs[k]):
                eng.finish(rid)
                del live[rid]
            else:
                live[rid] = (k, at + n)
    assert worst < 1.5 * limit, worst


def test_steps_longer_than_one_pass(built, tmp_path):
    cfg = config([attention(size=50), delta()], vocab=64)
    w = fu.weights(cfg, seed=2)
    toks = fu.tokens(cfg, 2300)
    eng = fu.engine(tmp_path, cfg, w, "bf16", pool=4096)
    whole = fu.step(eng, [("s", toks[:60], [59]), ("w", toks, [10, 2047, 2048, 2299])])
    eng.finish("w")
    parts = fu.run_portions(eng, "p", toks, [1000])
    assert fu.error(whole[1:], parts[[10, 2047, 2048, 2299]]) < 2e-2
    assert fu.error(whole[:1], parts[[59]]) < 2e-2


# ---- far keys, window edges --------------------------------------------------------------------------------------------
def spotlight(size, heads=4, kv_heads=2, dim=64, vdim=32, scale=0.75):
    """A one-layer model in which token 1 (query) attends almost only to token 0 (key), wherever that stands."""
    cfg = config([attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, size=size)], width=128, vocab=100, side=8)
    w = {k: v.float() for k, v in fu.weights(cfg, seed=11).items()}
    q, _ = torch.linalg.qr(torch.randn(128, 128, generator=torch.Generator().manual_seed(4)))
    w["embed"][:100] = q[:100] * 128 ** 0.5
    key, query = q[0], q[1]
    for name, n, d in (("q", heads, query), ("k", kv_heads, key)):
        m = w[f"l0.mix.{name}"]
        m -= torch.outer(m @ d, d)                                    # forget the direction, then give it channel 0 alone
        m.view(n, dim, 128)[:, 0] += 3.0 * d
    w["l0.mix.q.norm"][:] = 1
    w["l0.mix.k.norm"][:] = 1
    w["l0.mix.temp"][:] = 1
    return cfg, {k: v.to(torch.bfloat16) for k, v in w.items()}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("size", [64, 65, 90, 128, 200])
def test_window_edge(built, tmp_path, size, dtype):
    cfg, w = spotlight(size)
    wrong = {}
    for delta_size in (-1, 1):
        c2, _ = spotlight(size + delta_size)
        wrong[delta_size] = c2
    eng = fu.engine(tmp_path, cfg, w, dtype)
    n = size + 140
    rng = np.random.default_rng(size)
    shown = 0
    for place in (0, 63, 64, 100):                                   # where the key stands: page borders among them
        for dist in (size - 2, size - 1, size, size + 1):
            toks = (2 + rng.integers(0, 97, n)).tolist()
            toks[place] = 0
            i = place + dist
            toks[i] = 1
            toks = toks[:i + 1]
            ref = reference(cfg, w, toks).logits[-1:].numpy()
            other = reference(wrong[-1 if dist == size - 1 else 1], w, toks).logits[-1:].numpy()
            shows = fu.error(other, ref)
            if dist in (size - 1, size):
                shown += shows > 0.3
            prompt = fu.step(eng, [("p", toks, [i])])
            eng.finish("p")
            fu.step(eng, [("d", toks[:-1], [])])
            decoded = fu.step(eng, [("d", toks[-1:], [0])])
            eng.finish("d")
            fu.step(eng, [("c", toks[:-2], []), ("o", toks[:7], [])])
            batched = fu.step(eng, [("o", toks[7:20], []), ("c", toks[-2:], [1])])
            eng.finish("c")
            eng.finish("o")
            for got in (prompt, decoded, batched):
                assert fu.error(got, ref) < fu.LIMIT[dtype], (place, dist)
    assert shown >= 4                                                # a window one off would have shown


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_far_key_without_window(built, tmp_path, dtype):
    cfg, w = spotlight(None, heads=8, scale=1.5)                     # the last heads' slopes are small: they see far
    eng = fu.engine(tmp_path, cfg, w, dtype)
    rng = np.random.default_rng(1)
    for place in (0, 63, 64, 200):
        toks = (2 + rng.integers(0, 97, 400)).tolist()
        toks[place] = 0
        toks[399] = 1
        ref = reference(cfg, w, toks).logits[-1:].numpy()
        blind = list(toks)
        blind[place] = 5
        assert fu.error(reference(cfg, w, blind).logits[-1:].numpy(), ref) > 0.2
        for cuts in ([400], [399, 1], [350, 2]):
            assert fu.error(fu.run_portions(eng, "r", toks, cuts)[-1:], ref) < fu.LIMIT[dtype], (place, cuts)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_first_tokens(mixed, dtype):
    _, _, eng, seqs, refs, limit = mixed
    for n in (1, 2, 3, 5):
        got = fu.run_portions(eng, "f", seqs["b"][:n], [1] if dtype == "fp32" else [2])
        assert fu.error(got, refs["b"][:n]) < limit
    got = fu.step(eng, [("x", seqs["a"][:1], [0]), ("y", seqs["b"][:1], [0]), ("z", seqs["d"], [0])])
    for i, k in enumerate("abd"):
        assert fu.error(got[i:i + 1], refs[k][:1]) < limit
    for r in "xyz":
        eng.finish(r)


def test_recurrent_state_matters_and_is_zero_for_a_new_request(mixed):
    """A slot that held another sequence starts from nothing."""
    _, _, eng, seqs, refs, limit = mixed
    for _ in range(2):
        for k in ("a", "c", "d", "b"):
            assert fu.error(fu.run_portions(eng, "n" + k, seqs[k], [1 if len(seqs[k]) < 100 else 77]), refs[k]) < limit


# ---- generation --------------------------------------------------------------------------------------------------------
def greedy_check(cfg, w, prompt, out, limit):
    """Every generated id is the plain statement's arg-max, or within the rounding of it."""
    logits = reference(cfg, w, prompt + out[:-1]).logits.numpy()[len(prompt) - 1:]
    spread = logits.std()
    for t, row in zip(out, logits):
        assert row.max() - row[t] <= 4 * limit * spread, (t, int(row.argmax()))


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_generate(built, tmp_path, dtype):
    import edge_fm
    cfg = config(fu.MIXED)
    w = fu.weights(cfg, seed=9)
    prefix = fu.tokens(cfg, 70, seed=31)
    reqs = [{"request_id": 0, "max_tokens": 400}, {"request_id": 7, "max_tokens": 256, "prefix_token_ids": prefix}]
    eng = fu.engine(tmp_path, cfg, w, dtype, requests=reqs, max_new=120, name="Folizen")
    prompts = [fu.tokens(cfg, n, seed=40 + n) for n in (1, 2, 30, 150)]
    outs = []
    for p in prompts + prompts:                                       # again: captured prefill, used slot
        outs.append(eng.generate(edge_fm.Request(0, p)).token_ids())
        assert len(outs[-1]) == 120
    for p, o in zip(prompts, outs):
        greedy_check(cfg, w, p, list(o), fu.LIMIT[dtype])
    assert [list(o) for o in outs[:4]] == [list(o) for o in outs[4:]]
    for tail in ([3], [4, 5], fu.tokens(cfg, 40, seed=2), [3]):        # behind a fixed prefix, whose state is kept
        out = list(eng.generate(edge_fm.Request(7, prefix + tail)).token_ids())
        greedy_check(cfg, w, prefix + tail, out, fu.LIMIT[dtype])
    # many at once: the same ids as one at a time
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(100 + i, p) for i, p in enumerate(prompts + prompts[::-1])])]
    for p, o in zip(prompts + prompts[::-1], batch):
        assert len(o) == 120
        greedy_check(cfg, w, p, o, fu.LIMIT[dtype])
    if dtype == "fp32":
        assert batch[:4] == [list(o) for o in outs[:4]]


def test_generate_without_graph_and_stages(built, tmp_path):
    import edge_fm
    cfg = config(fu.MIXED)
    w = fu.weights(cfg, seed=9)
    reqs = [{"request_id": 0, "max_tokens": 200}]
    prompt = fu.tokens(cfg, 33)
    a = fu.engine(tmp_path, cfg, w, "fp32", requests=reqs, max_new=20, graph=False)
    out = list(a.generate(edge_fm.Request(0, prompt)).token_ids())
    greedy_check(cfg, w, prompt, out, fu.LIMIT["fp32"])
    ids = torch.tensor(prompt, dtype=torch.int32)
    t = edge_fm.Tensor(ids.data_ptr(), [33], edge_fm.DType.Int32, edge_fm.Device.CPU, 0)
    got = [a.prefill(0, {"token_ids": t})]
    for _ in range(4):
        got.append(a.decode(0, {}))
    first = [C.c_int32.from_address(g["next_token"].data_ptr()).value for g in got]
    assert first == out[:5]


def test_sampled_generation_is_the_same_alone_and_in_a_batch(built, tmp_path):
    import edge_fm
    cfg = config(fu.MIXED)
    w = fu.weights(cfg, seed=9)
    eng = fu.engine(tmp_path, cfg, w, "fp32", requests=[{"request_id": 0, "max_tokens": 200}], max_new=24, temperature=0.8, seed=5)
    prompts = [fu.tokens(cfg, n, seed=n) for n in (20, 45, 3)]
    alone = [list(eng.generate(edge_fm.Request(0, p)).token_ids()) for p in prompts]
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(i, p) for i, p in enumerate(prompts)])]
    assert alone == batch
    assert len({tuple(o) for o in alone}) == 3


def test_pool_limits_are_errors(mixed):
    _, _, eng, seqs, refs, limit = mixed
    toks = (seqs["a"] + seqs["a"] + seqs["a"])[:700]
    fu.step(eng, [("a", toks, [])])
    with pytest.raises(ValueError, match="room"):
        fu.step(eng, [("b", seqs["b"], [])])
    with pytest.raises(ValueError, match="twice"):
        fu.step(eng, [("a", [1], []), ("a", [2], [])])
    with pytest.raises(ValueError):
        fu.step(eng, [("a", [10 ** 6], [])])
    eng.finish("a")
    with pytest.raises(ValueError, match="not live"):
        eng.finish("a")
    assert fu.error(fu.run_portions(eng, "b", seqs["b"], [50]), refs["b"]) < limit
