"""GPU: the Temuvik decoder against its plain CPU statement: every mechanism alone, odd sizes, portions, batches, reused pages
and slots, window and kept-token edges, sinks, far keys, loops, long decoding, and generation through the engine's own entry
points."""
import ctypes as C
import json

import numpy as np
import pytest
import torch

import temuvik_util as tu
from oracle import temuvik
from temuvik_util import attention, config, experts, latent

pytestmark = pytest.mark.gpu


def reference(cfg, w, toks):
    return temuvik.forward(cfg, w, toks)


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
def isolate(w, keep):
    """Silences the other sublayers by zeroing their output projections (rms(0) = 0): only `keep` moves the residual stream."""
    out = dict(w)
    for k, v in w.items():
        if (k.endswith("mix.o") and keep != "mixer") or (k.endswith("down") and keep != "mlp"):
            out[k] = torch.zeros_like(v)
    return out


ALONE = {"attention": ("mixer", attention(mlp=None)), "latent": ("mixer", latent(mlp=None)),
         "experts": ("mlp", attention(mlp=experts(n=16, top=3, ff=40, groups=(4, 2)))),
         "one_group": ("mlp", latent(mlp=experts(n=5, top=2, ff=130, groups=None))), "one_expert": ("mlp", latent(mlp=experts(n=1, top=1, ff=64, groups=(1, 1)))),
         "every_expert": ("mlp", attention(mlp=experts(n=4, top=4, ff=8, groups=(4, 4))))}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(built, tmp_path, name, dtype):
    what, layer = ALONE[name]
    cfg = config([layer, layer])
    w = isolate(tu.weights(cfg, seed=3, margins=dtype == "bf16"), what)
    toks = tu.tokens(cfg, 90)
    eng = tu.engine(tmp_path, cfg, w, dtype)
    ref = reference(cfg, w, toks)
    limit = 2e-5 if dtype == "fp32" else 2e-2
    got = tu.taps(eng, 2, 90, cfg["width"], lambda: tu.step(eng, [("w", toks, [])]))
    eng.finish("w")
    for i in range(2):
        r = ref.layers[i].numpy()
        assert np.abs(got[i] - r).max() / np.abs(r).max() < limit, i
    tu.step(eng, [("d", toks[:89], [])])                              # the same layer one token at a time: the last token's stream
    got = tu.taps(eng, 2, 1, cfg["width"], lambda: tu.step(eng, [("d", toks[89:], [0])]))
    for i in range(2):
        r = ref.layers[i].numpy()
        assert np.abs(got[i] - r[89:]).max() / np.abs(r).max() < limit
    eng.finish("d")


# ---- sizes -----------------------------------------------------------------------------------------------------------
SIZES = {
    "tiny": config([attention(heads=1, kv_heads=1, dim=8, vdim=8, size=1, keep=1, rot=8, mlp=experts(n=2, top=1, ff=8, groups=(2, 1))),
                    latent(heads=1, dim=8, rot=2, vdim=8, q_rank=8, kv_rank=8, size=1)], width=16, vocab=32),
    "odd": config([latent(heads=3, dim=20, rot=6, vdim=12, q_rank=30, kv_rank=36, size=33, mlp=experts(n=9, top=3, ff=50, groups=(3, 2))),
                   attention(heads=5, kv_heads=1, dim=20, vdim=12, size=25, keep=3, rot=6, mlp=experts(n=7, top=2, ff=20, groups=None))],
                  width=76, vocab=131, eps=1e-3, scale=0.7),
    "wide_group": config([attention(heads=12, kv_heads=1, dim=64, vdim=96, size=100, keep=0, rot=32), latent(heads=12, dim=64, rot=32, vdim=96, size=100)],
                         width=192, vocab=301),
    "no_window": config([attention(heads=4, kv_heads=4, dim=48, vdim=128, size=None, rot=48, mlp=experts()), latent(heads=4, dim=128, vdim=128, rot=64, size=None)],
                        width=128, vocab=96),
    "large_latent": config([latent(heads=6, dim=128, rot=64, vdim=128, q_rank=192, kv_rank=512, size=90, mlp=experts(n=4, top=2, ff=64, groups=None))],
                           width=160, vocab=90),
    "beyond_tensor_cores": config([latent(heads=2, dim=160, rot=72, vdim=144, q_rank=64, kv_rank=640, size=50), latent(heads=2, dim=16, rot=80, vdim=16, size=77),
                                   attention(heads=2, kv_heads=1, dim=256, vdim=200, size=65, keep=9, rot=200)], width=64, vocab=70),
    "many_heads": config([latent(heads=34, dim=16, rot=16, vdim=16, q_rank=24, kv_rank=264, size=200)], width=104, vocab=60),
    "many_experts": config([attention(mlp=experts(n=96, top=8, ff=24, groups=(12, 4)))], width=256, vocab=60),
    "loop_all": config([attention(mlp=experts()), latent()], loop=(0, 2, 3)),
    "loop_last": config([latent(size=12), attention(), latent(mlp=experts())], loop=(2, 3, 2)),
    "loop_once": config([latent(), attention()], loop=(0, 1, 1)),
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(built, tmp_path, name, dtype):
    cfg = SIZES[name]
    w = tu.weights(cfg, seed=5, margins=dtype == "bf16")
    toks = tu.tokens(cfg, 150)
    ref = reference(cfg, w, toks).logits.numpy()
    eng = tu.engine(tmp_path, cfg, w, dtype)
    assert tu.error(tu.run_portions(eng, "w", toks, [150]), ref) < tu.LIMIT[dtype]
    assert tu.error(tu.run_portions(eng, "d", toks, [130, 1]), ref) < tu.LIMIT[dtype]
    assert tu.error(tu.run_portions(eng, "s", toks, [100, 20, 3, 14]), ref) < tu.LIMIT[dtype]


# ---- schedules -------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=["fp32", "bf16"])
def mixed(request, tmp_path_factory, built):
    cfg = config(tu.MIXED, loop=tu.MIXED_LOOP)
    w = tu.weights(cfg, seed=7)
    seqs = {k: tu.tokens(cfg, n, seed=20 + i) for i, (k, n) in enumerate((("a", 260), ("b", 131), ("c", 64), ("d", 1), ("e", 200)))}
    refs = {k: reference(cfg, w, t).logits.numpy() for k, t in seqs.items()}
    eng = tu.engine(tmp_path_factory.mktemp("mixed"), cfg, w, request.param, pool=704)
    return cfg, w, eng, seqs, refs, tu.LIMIT[request.param]


@pytest.mark.parametrize("cuts", [[260], [1], [2], [3, 2], [64], [63, 1, 65, 2], [17, 2, 40, 5], [128, 15, 16, 2]])
def test_portions(mixed, cuts):
    _, _, eng, seqs, refs, limit = mixed
    assert tu.error(tu.run_portions(eng, "p", seqs["a"], cuts), refs["a"]) < limit


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
        got, row = tu.step(eng, entries), 0
        for rid, k, at, n in spans:
            worst = max(worst, tu.error(got[row:row + n], refs[k][at:at + n]))
            row += n
            if at + n == len(seqs[k]):
                eng.finish(rid)
                del live[rid]
            else:
                live[rid] = (k, at + n)
    assert worst < 1.5 * limit, worst


def test_a_batch_is_each_request_alone(mixed):
    """The same portions alone and beside others: equal to rounding, whatever the neighbours are."""
    _, _, eng, seqs, refs, limit = mixed
    alone = {k: tu.run_portions(eng, "s", seqs[k][:60], [40, 4, 16]) for k in "abe"}
    rows = {k: [] for k in "abe"}
    for lo, hi in ((0, 40), (40, 44), (44, 60)):
        got = tu.step(eng, [(k, seqs[k][lo:hi], list(range(hi - lo))) for k in "abe"] + [("x%d" % lo, seqs["c"][:1 + lo], [])])
        for i, k in enumerate("abe"):
            rows[k].append(got[i * (hi - lo):(i + 1) * (hi - lo)])
        eng.finish("x%d" % lo)
    for k in "abe":
        eng.finish(k)
        assert tu.error(np.concatenate(rows[k]), alone[k]) < (1e-5 if limit < 1e-3 else 2e-2)


def test_steps_longer_than_one_pass(built, tmp_path):
    cfg = config([attention(size=50), latent(size=40, mlp=experts())], vocab=64, loop=(0, 2, 2))
    w = tu.weights(cfg, seed=2)
    toks = tu.tokens(cfg, 2300)
    eng = tu.engine(tmp_path, cfg, w, "bf16", pool=4096)
    whole = tu.step(eng, [("s", toks[:60], [59]), ("w", toks, [10, 2047, 2048, 2299])])
    eng.finish("w")
    parts = tu.run_portions(eng, "p", toks, [1000])
    assert tu.error(whole[1:], parts[[10, 2047, 2048, 2299]]) < 2e-2
    assert tu.error(whole[:1], parts[[59]]) < 2e-2


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_first_tokens(mixed, dtype):
    _, _, eng, seqs, refs, limit = mixed
    for n in (1, 2, 3, 5):
        got = tu.run_portions(eng, "f", seqs["b"][:n], [1] if dtype == "fp32" else [2])
        assert tu.error(got, refs["b"][:n]) < limit
    got = tu.step(eng, [("x", seqs["a"][:1], [0]), ("y", seqs["b"][:1], [0]), ("z", seqs["d"], [0])])
    for i, k in enumerate("abd"):
        assert tu.error(got[i:i + 1], refs[k][:1]) < limit
    for r in "xyz":
        eng.finish(r)


# ---- far keys, window and kept-token edges, sinks ---------------------------------------------------------------------------
def ways(eng, toks):
    """Logits of the last token by a whole prompt, decoded alone, and as the end of a portion in a batch."""
    i = len(toks) - 1
    yield tu.step(eng, [("p", toks, [i])])
    eng.finish("p")
    tu.step(eng, [("d", toks[:-1], [])])
    yield tu.step(eng, [("d", toks[-1:], [0])])
    eng.finish("d")
    if len(toks) > 3:
        tu.step(eng, [("c", toks[:-2], []), ("o", toks[:7], [])])
        yield tu.step(eng, [("o", toks[7:20], []), ("c", toks[-2:], [1])])
        eng.finish("c")
        eng.finish("o")
    if len(toks) > 21:
        tu.step(eng, [("e", toks[:-20], [])])
        yield tu.step(eng, [("e", toks[-20:], [19])])
        eng.finish("e")


def scene(n, place, i, seed, vocab=100):
    """Random tokens with the key (0) at `place` and the query (1) at i, the last one."""
    toks = (2 + np.random.default_rng(seed).integers(0, vocab - 3, n)).tolist()
    toks[place] = 0
    toks[i] = 1
    return toks[:i + 1]


LAYERS = {"attention": lambda size, keep: attention(heads=4, kv_heads=2, dim=64, vdim=32, rot=32, size=size, keep=keep),
          "latent": lambda size, keep: latent(heads=4, dim=48, rot=16, vdim=32, q_rank=64, kv_rank=80, size=size)}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("size", [64, 65, 90, 130])
@pytest.mark.parametrize("kind", sorted(LAYERS))
def test_window_edge(built, tmp_path, kind, size, dtype):
    cfg, w = tu.spotlight(LAYERS[kind](size, 0))
    wrong = {d: tu.spotlight(LAYERS[kind](size + d, 0))[0] for d in (-1, 1)}
    eng = tu.engine(tmp_path, cfg, w, dtype)
    shown = 0
    for place in (0, 63, 64, 100):                                   # where the key stands: page borders among them
        for dist in (size - 2, size - 1, size, size + 1):
            toks = scene(size + 140, place, place + dist, size)
            ref = reference(cfg, w, toks).logits[-1:].numpy()
            other = reference(wrong[-1 if dist == size - 1 else 1], w, toks).logits[-1:].numpy()
            shown += dist in (size - 1, size) and tu.error(other, ref) > 0.3
            for k, got in enumerate(ways(eng, toks)):
                assert tu.error(got, ref) < tu.LIMIT[dtype], (place, dist, k)
    assert shown >= 6                                                # a window one off would have shown


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("keep,size", [(1, 50), (20, 64), (64, 33), (65, 100), (130, 40)])
def test_kept_first_tokens(built, tmp_path, keep, size, dtype):
    cfg, w = tu.spotlight(LAYERS["attention"](size, keep))
    wrong = {d: tu.spotlight(LAYERS["attention"](size, keep + d))[0] for d in (-1, 1)}
    eng = tu.engine(tmp_path, cfg, w, dtype)
    shown = 0
    for place in {0, max(0, keep - 2), keep - 1, keep, keep + 1}:
        for i in (place + size - 1, place + size, keep + size + 70, 250):
            if i <= place:
                continue
            toks = scene(260, place, i, keep)
            ref = reference(cfg, w, toks).logits[-1:].numpy()
            if i == 250 and place in (keep - 1, keep):
                other = reference(wrong[-1 if place == keep - 1 else 1], w, toks).logits[-1:].numpy()
                shown += tu.error(other, ref) > 0.3
            for k, got in enumerate(ways(eng, toks)):
                assert tu.error(got, ref) < tu.LIMIT[dtype], (place, i, k)
    assert shown == 2


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_sink(built, tmp_path, dtype):
    """Sinks above, near and far below the scores, and negative ones: with nothing to attend to they take the weight."""
    cfg, w = tu.spotlight(LAYERS["latent"](60, 0))
    w["l0.mix.sink"] = torch.tensor([20.0, 12.0, -3.0, -60.0]).to(torch.bfloat16)
    eng = tu.engine(tmp_path, cfg, w, dtype)
    none = dict(w, **{"l0.mix.sink": torch.full((4,), -1e4).to(torch.bfloat16)})
    for place, i in ((3, 50), (3, 80), (0, 1), (0, 59), (0, 60)):
        toks = scene(100, place, i, 9)
        ref = reference(cfg, w, toks).logits[-1:].numpy()
        assert tu.error(reference(cfg, none, toks).logits[-1:].numpy(), ref) > 0.2
        for k, got in enumerate(ways(eng, toks)):
            assert tu.error(got, ref) < tu.LIMIT[dtype], (place, i, k)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("kind", sorted(LAYERS))
def test_far_key_without_window(built, tmp_path, kind, dtype):
    cfg, w = tu.spotlight(LAYERS[kind](None, 0))
    eng = tu.engine(tmp_path, cfg, w, dtype)
    for place in (0, 63, 64, 200):
        toks = scene(400, place, 399, 1)
        ref = reference(cfg, w, toks).logits[-1:].numpy()
        blind = list(toks)
        blind[place] = 5
        assert tu.error(reference(cfg, w, blind).logits[-1:].numpy(), ref) > 0.2
        for k, got in enumerate(ways(eng, toks)):
            assert tu.error(got, ref) < tu.LIMIT[dtype], (place, k)


def test_every_pass_of_a_loop_has_its_own_cache(built, tmp_path):
    """A later pass sees the keys of its own pass: the same layers with one shared cache would give other logits."""
    cfg = config([attention(mlp=experts()), latent()], loop=(0, 2, 3))
    w = tu.weights(cfg, seed=4)
    toks = tu.tokens(cfg, 80)
    ref = reference(cfg, w, toks)
    once = reference(json.loads(json.dumps(dict(cfg, loop=None))), w, toks)
    assert len(ref.layers) == 6 and tu.error(once.logits.numpy(), ref.logits.numpy()) > 0.3
    eng = tu.engine(tmp_path, cfg, w, "fp32")
    assert tu.error(tu.run_portions(eng, "a", toks, [50, 1, 7]), ref.logits.numpy()) < tu.LIMIT["fp32"]
    got = tu.taps(eng, 6, 80, cfg["width"], lambda: tu.step(eng, [("t", toks, [])]))
    for i in range(6):
        assert np.abs(got[i] - ref.layers[i].numpy()).max() / np.abs(ref.layers[i].numpy()).max() < 2e-5


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
    cfg = config(tu.MIXED, loop=tu.MIXED_LOOP)
    w = tu.weights(cfg, seed=9)
    prefix = tu.tokens(cfg, 70, seed=31)
    reqs = [{"request_id": 0, "max_tokens": 400}, {"request_id": 7, "max_tokens": 256, "prefix_token_ids": prefix}]
    eng = tu.engine(tmp_path, cfg, w, dtype, requests=reqs, max_new=120, name="Temuvik")
    prompts = [tu.tokens(cfg, n, seed=40 + n) for n in (1, 2, 30, 150)]
    outs = [list(eng.generate(edge_fm.Request(0, p)).token_ids()) for p in prompts + prompts]      # again: captured prefill, used slot
    for p, o in zip(prompts, outs):
        assert len(o) == 120
        greedy_check(cfg, w, p, o, tu.LIMIT[dtype])
    assert outs[:4] == outs[4:]
    for tail in ([3], [4, 5], tu.tokens(cfg, 40, seed=2), [3]):        # behind a fixed prefix
        greedy_check(cfg, w, prefix + tail, list(eng.generate(edge_fm.Request(7, prefix + tail)).token_ids()), tu.LIMIT[dtype])
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(100 + i, p) for i, p in enumerate(prompts + prompts[::-1])])]
    for p, o in zip(prompts, batch):
        assert len(o) == 120
        greedy_check(cfg, w, p, o, tu.LIMIT[dtype])
    if dtype == "fp32":
        assert batch == outs[:4] + outs[:4][::-1]


def test_generate_without_graph_and_stages(built, tmp_path):
    import edge_fm
    cfg = config(tu.MIXED, loop=tu.MIXED_LOOP)
    w = tu.weights(cfg, seed=9)
    prompt = tu.tokens(cfg, 33)
    a = tu.engine(tmp_path, cfg, w, "fp32", requests=[{"request_id": 0, "max_tokens": 200}], max_new=20, graph=False)
    out = list(a.generate(edge_fm.Request(0, prompt)).token_ids())
    greedy_check(cfg, w, prompt, out, tu.LIMIT["fp32"])
    ids = torch.tensor(prompt, dtype=torch.int32)
    t = edge_fm.Tensor(ids.data_ptr(), [33], edge_fm.DType.Int32, edge_fm.Device.CPU, 0)
    got = [a.prefill(0, {"token_ids": t})]
    for _ in range(4):
        got.append(a.decode(0, {}))
    assert [C.c_int32.from_address(g["next_token"].data_ptr()).value for g in got] == out[:5]


def test_sampled_generation_is_the_same_alone_and_in_a_batch(built, tmp_path):
    import edge_fm
    cfg = config(tu.MIXED, loop=tu.MIXED_LOOP)
    w = tu.weights(cfg, seed=9)
    eng = tu.engine(tmp_path, cfg, w, "fp32", requests=[{"request_id": 0, "max_tokens": 200}], max_new=24, temperature=0.8, seed=5)
    prompts = [tu.tokens(cfg, n, seed=n) for n in (20, 45, 3)]
    alone = [list(eng.generate(edge_fm.Request(0, p)).token_ids()) for p in prompts]
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(i, p) for i, p in enumerate(prompts)])]
    assert alone == batch
    assert len({tuple(o) for o in alone}) == 3


def test_pool_limits_are_errors(mixed):
    _, _, eng, seqs, refs, limit = mixed
    toks = (seqs["a"] + seqs["a"] + seqs["a"])[:700]
    tu.step(eng, [("a", toks, [])])
    with pytest.raises(ValueError, match="room"):
        tu.step(eng, [("b", seqs["b"], [])])
    eng.finish("a")
    assert tu.error(tu.run_portions(eng, "b", seqs["b"], [50]), refs["b"]) < limit
