"""GPU: the Viladra decoder against its plain CPU statement: every mechanism alone, odd sizes, portions, batches, reused pages and
slots, window and chunk edges, long memories and strong decays of the recurrences, far keys, long decoding, and generation through the
engine's own entry points."""
import ctypes as C

import numpy as np
import pytest
import torch

import viladra_util as vu
from oracle import viladra
from viladra_util import attention, config, experts, gla, retention

pytestmark = pytest.mark.gpu


def reference(cfg, w, toks):
    return viladra.forward(cfg, w, toks)


def agrees(got, ref, dtype, fp32=vu.LIMIT["fp32"]):
    """fp32: every row.  bf16: all rows but a few whose retention output is nearly zero before its norm divides by its size."""
    e = vu.row_errors(got, ref)
    return e.max() < fp32 if dtype == "fp32" else np.quantile(e, 0.95) < vu.LIMIT["bf16"] and np.median(e) < 0.3 * vu.LIMIT["bf16"]


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
ALONE = {"retention": ("mix", retention()), "retention_part_rotated": ("mix", retention(dim=40, rot=8, vdim=64)), "gla": ("mix", gla()), "attention": ("mix", attention()),
         "attention_everywhere": ("mix", attention(size=None)), "convolution_and_depth": ("none", gla()), "experts": ("mlp", gla(mlp=experts(n=16, top=3, ff=40))),
         "one_expert": ("mlp", gla(mlp=experts(n=1, top=1, ff=64, shared=8))), "every_expert": ("mlp", gla(mlp=experts(n=4, top=4, ff=130, shared=200, scale=0.7))),
         "no_shared": ("mlp", gla(mlp=experts(n=6, top=2, shared=None))), "odd_widths": ("mlp", gla(mlp=experts(n=6, top=2, ff=33, shared=21)))}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(built, tmp_path, name, dtype):
    what, layer = ALONE[name]
    cfg = config([layer, layer])
    w = vu.isolate(vu.weights(cfg, seed=3, margins=dtype == "bf16"), what)
    toks = vu.tokens(cfg, 150)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    ref = reference(cfg, w, toks)
    limit = 2e-5 if dtype == "fp32" else 4e-2
    got = vu.taps(eng, 2, 150, cfg["width"], lambda: vu.step(eng, [("w", toks, [])]))
    eng.finish("w")
    for i in range(2):
        r = ref.layers[i].numpy()
        assert np.abs(got[i] - r).max() / np.abs(r).max() < limit, i
    vu.step(eng, [("d", toks[:149], [])])                             # the same layer one token at a time: the last token's stream
    got = vu.taps(eng, 2, 1, cfg["width"], lambda: vu.step(eng, [("d", toks[149:], [0])]))
    for i in range(2):
        r = ref.layers[i].numpy()
        assert np.abs(got[i] - r[149:]).max() / np.abs(r).max() < limit
    eng.finish("d")


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("cap", [3.0, 100.0])
def test_output_alone(built, tmp_path, cap, dtype):
    """Final norm, tied head without the embedding's scale, cap of the logits (one that nearly every logit reaches, too)."""
    cfg = config([gla()], softcap=cap, vocab=83, embed=0.4)
    w = vu.isolate(vu.weights(cfg, seed=6), "none")
    toks = vu.tokens(cfg, 40)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    ref = reference(cfg, w, toks).logits.numpy()
    assert np.abs(ref).max() > 0.99 * cap or cap > 10
    assert vu.error(vu.run_portions(eng, "w", toks, [38, 1]), ref) < (1e-5 if dtype == "fp32" else 2e-2)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("taps", [1, 2, 3, 5, 16])
def test_convolution_taps(built, tmp_path, taps, dtype):
    """Filters from the token alone to sixteen tokens, cut so that a portion is shorter than the filter, and slots used again."""
    cfg = config([retention(mlp=experts()), attention()], taps=taps)
    w = vu.weights(cfg, seed=4)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    for seed, cuts in enumerate(([120], [1], [2], [3, 5, 1, 1, 2, 16, 17, 30], [15, 16, 33])):
        toks = vu.tokens(cfg, 120, seed=60 + seed)
        assert vu.error(vu.run_portions(eng, "c", toks, cuts), reference(cfg, w, toks).logits.numpy()) < vu.LIMIT[dtype], cuts


# ---- sizes -----------------------------------------------------------------------------------------------------------
SIZES = {
    "tiny": config([retention(heads=1, dim=4, vdim=4, rot=2, mlp=experts(n=2, top=1, ff=8, shared=8)), gla(heads=1, dim=4, vdim=4),
                    attention(heads=1, kv_heads=1, dim=8, vdim=8, size=1, mlp=experts(n=1, top=1, ff=2, shared=2))], width=16, vocab=32, taps=2, eps=0.1),
    "odd": config([retention(heads=5, dim=18, vdim=12, rot=6, mlp=experts(n=9, top=3, ff=50, shared=70)), attention(heads=6, kv_heads=3, dim=20, vdim=12, size=23),
                   gla(heads=3, dim=7, vdim=9, tau=1.0, mlp=experts(n=7, top=7, ff=19, shared=None))], width=76, vocab=131, eps=0.1, taps=3),
    "unaligned_rows": config([attention(heads=3, kv_heads=3, dim=9, vdim=5), retention(heads=5, dim=14, vdim=3, rot=14), gla(heads=5, dim=13, vdim=3)], width=50, vocab=77),
    "wide_group": config([attention(heads=12, kv_heads=1, dim=64, vdim=96, size=100), gla(heads=2, dim=64, vdim=128), retention(heads=2, dim=64, vdim=128, rot=32)],
                         width=192, vocab=301),
    "wide_heads": config([retention(heads=2, dim=128, vdim=160, rot=128), gla(heads=2, dim=128, vdim=192), attention(heads=4, kv_heads=2, dim=96, vdim=192)], width=128, vocab=96),
    "widest": config([retention(heads=2, dim=256, vdim=256, rot=256), gla(heads=2, dim=256, vdim=256), attention(heads=2, kv_heads=1, dim=256, vdim=256)], width=96, vocab=64),
    "narrow_values": config([gla(heads=1, dim=200, vdim=24), retention(heads=1, dim=112, vdim=8, rot=64), attention(heads=2, kv_heads=2, dim=128, vdim=16)], width=96, vocab=64),
    "many_heads": config([retention(heads=21, dim=8, vdim=8, rot=8), gla(heads=20, dim=8, vdim=8), attention(heads=20, kv_heads=20, dim=16, vdim=16)], width=104, vocab=60, eps=0.1),
    "many_experts": config([gla(mlp=experts(n=96, top=8, ff=24, shared=256, scale=4.0))], width=256, vocab=60),
    "one_layer": config([retention()], taps=2),
    "deep": config([gla(heads=2, dim=16, vdim=16) if i % 3 else attention(heads=2, kv_heads=1, dim=16, vdim=16, size=20) for i in range(9)], width=160, vocab=60, taps=3, eps=0.1),
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(built, tmp_path, name, dtype):
    cfg = SIZES[name]
    if name == "deep" and dtype == "bf16":
        cfg = {**cfg, "layers": cfg["layers"][:4]}                    # nine random layers amplify 8 bits of mantissa too much
    rank = {"odd": 1, "wide_heads": 40, "widest": 100}.get(name, vu.RANK)
    w = vu.weights(cfg, seed=5, margins=dtype == "bf16", rank=rank)
    toks = vu.tokens(cfg, 150)
    ref = reference(cfg, w, toks).logits.numpy()
    eng = vu.engine(tmp_path, cfg, w, dtype)
    for cuts in ([150], [130, 1], [100, 20, 3, 14]):
        assert agrees(vu.run_portions(eng, "s", toks, cuts), ref, dtype), cuts


# ---- schedules -------------------------------------------------------------------------------------------------------
@pytest.fixture(scope="module", params=["fp32", "bf16"])
def mixed(request, tmp_path_factory, built):
    cfg = config(vu.MIXED)
    w = vu.weights(cfg, seed=7)
    seqs = {k: vu.tokens(cfg, n, seed=20 + i) for i, (k, n) in enumerate((("a", 260), ("b", 131), ("c", 64), ("d", 1), ("e", 200)))}
    refs = {k: reference(cfg, w, t).logits.numpy() for k, t in seqs.items()}
    eng = vu.engine(tmp_path_factory.mktemp("mixed"), cfg, w, request.param, pool=704)
    return cfg, w, eng, seqs, refs, vu.LIMIT[request.param]


@pytest.mark.parametrize("cuts", [[260], [1], [2], [3, 2], [64], [63, 1, 65, 2], [17, 2, 40, 5], [128, 15, 16, 2]])
def test_portions(mixed, cuts):
    _, _, eng, seqs, refs, limit = mixed
    assert vu.error(vu.run_portions(eng, "p", seqs["a"], cuts), refs["a"]) < limit


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
        got, row = vu.step(eng, entries), 0
        for rid, k, at, n in spans:
            worst = max(worst, vu.error(got[row:row + n], refs[k][at:at + n]))
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
    alone = {k: vu.run_portions(eng, "s", seqs[k][:60], [40, 4, 16]) for k in "abe"}
    rows = {k: [] for k in "abe"}
    for lo, hi in ((0, 40), (40, 44), (44, 60)):
        got = vu.step(eng, [(k, seqs[k][lo:hi], list(range(hi - lo))) for k in "abe"] + [("x%d" % lo, seqs["c"][:1 + lo], [])])
        for i, k in enumerate("abe"):
            rows[k].append(got[i * (hi - lo):(i + 1) * (hi - lo)])
        eng.finish("x%d" % lo)
    for k in "abe":
        eng.finish(k)
        assert vu.error(np.concatenate(rows[k]), alone[k]) < (1e-5 if limit < 1e-3 else 4e-2)


def test_steps_longer_than_one_pass(built, tmp_path):
    cfg = config([gla(), attention(mlp=experts()), retention()], vocab=64)
    w = vu.weights(cfg, seed=2)
    toks = vu.tokens(cfg, 2300)
    eng = vu.engine(tmp_path, cfg, w, "bf16", pool=4096)
    whole = vu.step(eng, [("s", toks[:60], [59]), ("w", toks, [10, 2047, 2048, 2299])])
    eng.finish("w")
    parts = vu.run_portions(eng, "p", toks, [1000])
    assert vu.error(whole[1:], parts[[10, 2047, 2048, 2299]]) < 4e-2
    assert vu.error(whole[:1], parts[[59]]) < 4e-2


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_first_tokens(mixed, dtype):
    _, _, eng, seqs, refs, limit = mixed
    for n in (1, 2, 3, 5):
        got = vu.run_portions(eng, "f", seqs["b"][:n], [1] if dtype == "fp32" else [2])
        assert vu.error(got, refs["b"][:n]) < limit
    got = vu.step(eng, [("x", seqs["a"][:1], [0]), ("y", seqs["b"][:1], [0]), ("z", seqs["d"], [0])])
    for i, k in enumerate("abd"):
        assert vu.error(got[i:i + 1], refs[k][:1]) < limit
    for r in "xyz":
        eng.finish(r)


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
def test_long_decoding(built, tmp_path, dtype):
    """Hundreds of tokens one by one, past several pages and windows."""
    cfg = config(vu.MIXED)
    w = vu.weights(cfg, seed=12)
    toks = vu.tokens(cfg, 420)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    assert vu.error(vu.run_portions(eng, "l", toks, [2, 1]), reference(cfg, w, toks).logits.numpy()) < vu.LIMIT[dtype]


# ---- memory of the recurrences -----------------------------------------------------------------------------------------
CHUNK_CUTS = ([300], [64, 64, 64, 108], [63, 2, 64, 1, 65, 105], [1, 2], [129, 1, 1, 62, 107], [192, 1], [128, 128, 44])


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("decay", [[1.0, 0.9995], [0.0, 1.0], [0.3, 0.98]])
def test_constant_decay_over_chunk_edges(built, tmp_path, decay, dtype):
    """The recurrence cut at and beside the edges of its chunks; with decays near one a state that is lost, kept from another request or
    decayed once too often shows hundreds of tokens later."""
    cfg = config([retention(heads=2, dim=24, vdim=20, decay=decay)], taps=2, eps=0.1)
    w = vu.weights(cfg, seed=4)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    for seed, cuts in enumerate(CHUNK_CUTS):
        toks = vu.tokens(cfg, 300, seed=50 + seed)
        ref = reference(cfg, w, toks).logits.numpy()
        forgot = reference(cfg, w, toks[192:]).logits.numpy()
        assert decay[-1] < 0.99 or vu.error(forgot[-20:], ref[-20:]) > 0.15
        # with decay 0 a token reads q . k of its own alone, which the norm magnifies where it is nearly zero
        assert agrees(vu.run_portions(eng, "r", toks, cuts), ref, dtype, 2e-4 if decay[0] == 0.0 else vu.LIMIT["fp32"]), cuts


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("bias,tau", [(6.0, 16.0), (0.0, 16.0), (-4.0, 8.0), (-2.0, 0.5), (None, 2.0)])
def test_channel_decays_over_chunk_edges(built, tmp_path, bias, tau, dtype):
    """From channels that forget nothing within a prompt to channels that forget everything at once, and (None) both side by side."""
    cfg = config([gla(heads=2, dim=40, vdim=24, tau=tau)], taps=2)
    w = vu.weights(cfg, seed=4)
    b = w["l0.mix.a2.b"]
    b[:] = torch.where(torch.arange(80) % 2 == 0, 9.0, -9.0).to(b) if bias is None else bias
    eng = vu.engine(tmp_path, cfg, w, dtype)
    for seed, cuts in enumerate(CHUNK_CUTS):
        toks = vu.tokens(cfg, 300, seed=50 + seed)
        ref = reference(cfg, w, toks).logits.numpy()
        if bias is None or bias > 5:
            assert vu.error(reference(cfg, w, toks[192:]).logits.numpy()[-20:], ref[-20:]) > 0.15
        assert vu.error(vu.run_portions(eng, "r", toks, cuts), ref) < vu.LIMIT[dtype], cuts


# ---- windows and far keys ------------------------------------------------------------------------------------------------
def ways(eng, toks):
    """Logits of the last token by a whole prompt, decoded alone, and as the end of a portion in a batch."""
    i = len(toks) - 1
    yield vu.step(eng, [("p", toks, [i])])
    eng.finish("p")
    vu.step(eng, [("d", toks[:-1], [])])
    yield vu.step(eng, [("d", toks[-1:], [0])])
    eng.finish("d")
    if len(toks) > 20:
        vu.step(eng, [("c", toks[:-2], []), ("o", toks[:7], [])])
        yield vu.step(eng, [("o", toks[7:20], []), ("c", toks[-2:], [1])])
        eng.finish("c")
        eng.finish("o")
    if len(toks) > 21:
        vu.step(eng, [("e", toks[:-20], [])])
        yield vu.step(eng, [("e", toks[-20:], [19])])
        eng.finish("e")


LAYERS = {"grouped": dict(heads=4, kv_heads=2, dim=64, vdim=96), "narrow": dict(heads=3, kv_heads=3, dim=40, vdim=200), "wide": dict(heads=2, kv_heads=1, dim=144, vdim=64)}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("kind", sorted(LAYERS))
@pytest.mark.parametrize("size", [1, 50, 64, 129, 300, None])
def test_far_key_and_window_edge(built, tmp_path, kind, size, dtype):
    """One key stands out among hundreds: the first one inside the window, the last one outside, rows at page borders."""
    cfg, w = vu.spotlight(attention(size=size, **LAYERS[kind]))
    eng = vu.engine(tmp_path, cfg, w, dtype)
    last = 399
    places = [(0, last), (63, last), (64, 128), (200, last), (398, last), (5, 6)] + ([] if size in (None, 1) else [
        (last - size + 1, last), (last - size, last), (128 - min(size, 129) + 1, 128), (max(0, 256 - size), 256), (max(0, 255 - size + 1), 255)])
    for place, end in places:
        toks = (2 + np.random.default_rng(place).integers(0, cfg["vocab"] - 3, 400)).tolist()[:end + 1]
        blind = list(toks)
        toks[place], toks[end], blind[end] = 0, 1, 1
        if place == end:
            continue
        ref, without = (reference(cfg, w, t).logits[-1:].numpy() for t in (toks, blind))
        inside = size is None or end - place < size
        assert (vu.error(without, ref) > 0.2) == inside, (place, end)
        for k, got in enumerate(ways(eng, toks)):
            assert vu.error(got, ref) < vu.LIMIT[dtype], (place, end, k)


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
    cfg = config(vu.MIXED)
    w = vu.weights(cfg, seed=9)
    prefix = vu.tokens(cfg, 70, seed=31)
    reqs = [{"request_id": 0, "max_tokens": 400}, {"request_id": 7, "max_tokens": 256, "prefix_token_ids": prefix}]
    eng = vu.engine(tmp_path, cfg, w, dtype, requests=reqs, max_new=60, name="Viladra")
    prompts = [vu.tokens(cfg, n, seed=40 + n) for n in (1, 2, 30, 150)]
    outs = [list(eng.generate(edge_fm.Request(0, p)).token_ids()) for p in prompts + prompts]      # again: captured prefill, used slot
    for p, o in zip(prompts, outs):
        assert len(o) == 60
        greedy_check(cfg, w, p, o, vu.LIMIT[dtype])
    assert outs[:4] == outs[4:]
    for tail in ([3], [4, 5], vu.tokens(cfg, 40, seed=2), [3]):        # behind a fixed prefix, whose state is restored
        greedy_check(cfg, w, prefix + tail, list(eng.generate(edge_fm.Request(7, prefix + tail)).token_ids()), vu.LIMIT[dtype])
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(100 + i, p) for i, p in enumerate(prompts + prompts[::-1])])]
    for p, o in zip(prompts, batch):
        assert len(o) == 60
        greedy_check(cfg, w, p, o, vu.LIMIT[dtype])
    if dtype == "fp32":
        assert batch == outs[:4] + outs[:4][::-1]


def test_generate_without_graph_and_stages(built, tmp_path):
    import edge_fm
    cfg = config(vu.MIXED)
    w = vu.weights(cfg, seed=9)
    prompt = vu.tokens(cfg, 33)
    a = vu.engine(tmp_path, cfg, w, "fp32", requests=[{"request_id": 0, "max_tokens": 200}], max_new=20, graph=False)
    out = list(a.generate(edge_fm.Request(0, prompt)).token_ids())
    greedy_check(cfg, w, prompt, out, vu.LIMIT["fp32"])
    ids = torch.tensor(prompt, dtype=torch.int32)
    t = edge_fm.Tensor(ids.data_ptr(), [33], edge_fm.DType.Int32, edge_fm.Device.CPU, 0)
    got = [a.prefill(0, {"token_ids": t})]
    for _ in range(4):
        got.append(a.decode(0, {}))
    assert [C.c_int32.from_address(g["next_token"].data_ptr()).value for g in got] == out[:5]


def test_sampled_generation_is_the_same_alone_and_in_a_batch(built, tmp_path):
    import edge_fm
    cfg = config(vu.MIXED)
    w = vu.weights(cfg, seed=9)
    eng = vu.engine(tmp_path, cfg, w, "fp32", requests=[{"request_id": 0, "max_tokens": 200}], max_new=24, temperature=0.8, seed=5)
    prompts = [vu.tokens(cfg, n, seed=n) for n in (20, 45, 3)]
    alone = [list(eng.generate(edge_fm.Request(0, p)).token_ids()) for p in prompts]
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(i, p) for i, p in enumerate(prompts)])]
    assert alone == batch
    assert len({tuple(o) for o in alone}) == 3


def test_pool_limits_are_errors(mixed):
    _, _, eng, seqs, refs, limit = mixed
    toks = (seqs["a"] + seqs["a"] + seqs["a"])[:700]
    vu.step(eng, [("a", toks, [])])
    with pytest.raises(ValueError, match="room"):
        vu.step(eng, [("b", seqs["b"], [])])
    eng.finish("a")
    assert vu.error(vu.run_portions(eng, "b", seqs["b"], [50]), refs["b"]) < limit
