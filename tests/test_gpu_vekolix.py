"""GPU: the Vekolix decoder against its plain CPU statement: every mechanism alone, odd sizes, portions, batches, reused pages
and slots, chunk edges and long memories of the recurrence, far keys, long decoding, and generation through the engine's own
entry points."""
import ctypes as C

import numpy as np
import pytest
import torch

import vekolix_util as vu
from oracle import vekolix
from vekolix_util import config, dense, experts, latent, parallel, yarn

pytestmark = pytest.mark.gpu


def reference(cfg, w, toks):
    return vekolix.forward(cfg, w, toks)


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
def isolate(w, keep):
    """Zeroes the output projections of everything but `keep` ("left", "right", "mix" or "mlp")."""
    def out(k):
        return k.endswith(".o") or k.endswith(".down")

    def kept(k):
        return ".left." in k if keep == "left" else ".right." in k if keep == "right" else (".mix." in k if keep == "mix" else ".mlp." in k)
    return {k: torch.zeros_like(v) if out(k) and not kept(k) else v for k, v in w.items()}


ALONE = {"left": ("left", parallel()), "left_unscaled": ("left", parallel(scaling=None, rot=24)), "right": ("right", parallel()), "latent": ("mix", latent()),
         "both": ("mix", parallel()), "dense": ("mlp", latent(mlp=dense(72))), "experts": ("mlp", parallel(mlp=experts(n=16, top=3, ff=40))),
         "one_expert": ("mlp", latent(mlp=experts(n=1, top=1, ff=64, shared=(8, 0.5)))), "every_expert": ("mlp", latent(mlp=experts(n=4, top=4, ff=130, shared=(200, 5.0)))),
         "no_shared": ("mlp", latent(mlp=experts(n=6, top=2, shared=None)))}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(built, tmp_path, name, dtype):
    what, layer = ALONE[name]
    cfg = config([layer, layer])
    w = isolate(vu.weights(cfg, seed=3, margins=dtype == "bf16"), what)
    toks = vu.tokens(cfg, 90)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    ref = reference(cfg, w, toks)
    limit = 2e-5 if dtype == "fp32" else 2e-2
    got = vu.taps(eng, 2, 90, cfg["width"], lambda: vu.step(eng, [("w", toks, [])]))
    eng.finish("w")
    for i in range(2):
        r = ref.layers[i].numpy()
        assert np.abs(got[i] - r).max() / np.abs(r).max() < limit, i
    vu.step(eng, [("d", toks[:89], [])])                              # the same layer one token at a time: the last token's stream
    got = vu.taps(eng, 2, 1, cfg["width"], lambda: vu.step(eng, [("d", toks[89:], [0])]))
    for i in range(2):
        r = ref.layers[i].numpy()
        assert np.abs(got[i] - r[89:]).max() / np.abs(r).max() < limit
    eng.finish("d")


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("scale,cap", [(1.0, 5.0), (3.0, 2.0), (0.25, 100.0)])
def test_output_alone(built, tmp_path, scale, cap, dtype):
    """Elementwise norm, tied head, scale and cap of the logits (caps that nearly every logit reaches among them)."""
    cfg = config([latent()], logit_scale=scale, softcap=cap, vocab=83)
    w = isolate(vu.weights(cfg, seed=6), "none of them")
    toks = vu.tokens(cfg, 40)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    ref = reference(cfg, w, toks).logits.numpy()
    assert np.abs(ref).max() > 0.9 * cap or scale < 1
    assert vu.error(vu.run_portions(eng, "w", toks, [38, 1]), ref) < (1e-5 if dtype == "fp32" else 2e-2)


@pytest.mark.parametrize("scaling", [yarn(factor=8.0, original=16, fast=32.0, slow=1.0), yarn(factor=2.5, original=5000, fast=2.0, slow=1.9),
                                     yarn(factor=40.0, original=300, fast=4.0, slow=0.01), yarn(factor=1.0, original=100, fast=3.0, slow=3.0),
                                     yarn(factor=3.0, original=64, fast=0.5, slow=2.0)])
def test_scaled_rotations(built, tmp_path, scaling):
    """Ramps that begin below the first pair, end above the last, have no width or run backwards."""
    layer = parallel(rot=20, base=200.0, scaling=scaling)
    cfg = config([layer])
    w = isolate(vu.weights(cfg, seed=8), "left")
    toks = vu.tokens(cfg, 300)
    eng = vu.engine(tmp_path, cfg, w, "fp32")
    ref = reference(cfg, w, toks).logits.numpy()
    other = reference(config([parallel(rot=20, base=200.0, scaling=None)]), w, toks).logits.numpy()
    assert vu.error(other, ref) > 1e-2 or scaling["factor"] == 1.0
    assert vu.error(vu.run_portions(eng, "w", toks, [270, 1, 29]), ref) < vu.LIMIT["fp32"]


# ---- sizes -----------------------------------------------------------------------------------------------------------
SIZES = {
    "tiny": config([parallel(heads=1, kv_heads=1, dim=8, vdim=8, rot=2, lin_heads=1, lin_dim=4, lin_vdim=4, mlp=experts(n=2, top=1, ff=8, shared=(8, 0.3))),
                    latent(heads=1, dim=8, rot=2, vdim=8, q_rank=8, kv_rank=8, mlp=dense(8))], width=16, vocab=32),
    "odd": config([latent(heads=3, dim=20, rot=6, vdim=12, q_rank=30, kv_rank=36, mlp=experts(n=9, top=3, ff=50, shared=(70, 1.0))),
                   parallel(heads=5, kv_heads=1, dim=20, vdim=12, rot=6, lin_heads=3, lin_dim=7, lin_vdim=9, mlp=dense(90))], width=76, vocab=131, eps=1e-1, mult=0.4),
    "unaligned_rows": config([parallel(heads=3, kv_heads=3, dim=9, vdim=5, rot=4, lin_heads=5, lin_dim=13, lin_vdim=3, mlp=dense(33))], width=50, vocab=77),
    "wide_group": config([parallel(heads=12, kv_heads=1, dim=64, vdim=96, rot=32, lin_heads=2, lin_dim=64, lin_vdim=128), latent(heads=12, dim=64, rot=32, vdim=96)],
                         width=192, vocab=301),
    "wide_values": config([parallel(heads=4, kv_heads=2, dim=96, vdim=192, rot=96, lin_heads=2, lin_dim=96, lin_vdim=160), latent(heads=2, dim=64, vdim=200, rot=64, mlp=dense())],
                          width=128, vocab=96),
    "widest": config([parallel(heads=2, kv_heads=1, dim=256, vdim=256, rot=256, lin_heads=2, lin_dim=256, lin_vdim=256)], width=96, vocab=64),
    "narrow_values": config([parallel(heads=2, kv_heads=2, dim=128, vdim=16, rot=64, lin_heads=1, lin_dim=200, lin_vdim=24)], width=96, vocab=64),
    "large_latent": config([latent(heads=6, dim=128, rot=64, vdim=128, q_rank=192, kv_rank=512, mlp=experts(n=4, top=2, ff=64))], width=160, vocab=90),
    "beyond_tensor_cores": config([latent(heads=2, dim=160, rot=72, vdim=144, q_rank=64, kv_rank=640), latent(heads=2, dim=16, rot=80, vdim=16),
                                   parallel(heads=2, kv_heads=1, dim=200, vdim=200, rot=200, lin_heads=9, lin_dim=16, lin_vdim=8)], width=64, vocab=70),
    "many_heads": config([latent(heads=34, dim=16, rot=16, vdim=16, q_rank=24, kv_rank=264), parallel(heads=20, kv_heads=20, dim=16, vdim=16, lin_heads=21, lin_dim=8, lin_vdim=8)],
                         width=104, vocab=60),
    "many_experts": config([parallel(mlp=experts(n=96, top=8, ff=24, shared=(256, 0.8)))], width=256, vocab=60),
    "no_mlp": config([parallel(), latent(), parallel()], mult=0.25),
}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("name", sorted(SIZES))
def test_sizes(built, tmp_path, name, dtype):
    cfg = SIZES[name]
    w = vu.weights(cfg, seed=5, margins=dtype == "bf16")
    toks = vu.tokens(cfg, 150)
    ref = reference(cfg, w, toks).logits.numpy()
    eng = vu.engine(tmp_path, cfg, w, dtype)
    assert vu.error(vu.run_portions(eng, "w", toks, [150]), ref) < vu.LIMIT[dtype]
    assert vu.error(vu.run_portions(eng, "d", toks, [130, 1]), ref) < vu.LIMIT[dtype]
    assert vu.error(vu.run_portions(eng, "s", toks, [100, 20, 3, 14]), ref) < vu.LIMIT[dtype]


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
        assert vu.error(np.concatenate(rows[k]), alone[k]) < (1e-5 if limit < 1e-3 else 2e-2)


def test_steps_longer_than_one_pass(built, tmp_path):
    cfg = config([parallel(mlp=dense()), latent(mlp=experts())], vocab=64)
    w = vu.weights(cfg, seed=2)
    toks = vu.tokens(cfg, 2300)
    eng = vu.engine(tmp_path, cfg, w, "bf16", pool=4096)
    whole = vu.step(eng, [("s", toks[:60], [59]), ("w", toks, [10, 2047, 2048, 2299])])
    eng.finish("w")
    parts = vu.run_portions(eng, "p", toks, [1000])
    assert vu.error(whole[1:], parts[[10, 2047, 2048, 2299]]) < 2e-2
    assert vu.error(whole[:1], parts[[59]]) < 2e-2


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
    """Hundreds of tokens one by one, past several pages."""
    cfg = config(vu.MIXED)
    w = vu.weights(cfg, seed=12)
    toks = vu.tokens(cfg, 420)
    eng = vu.engine(tmp_path, cfg, w, dtype)
    assert vu.error(vu.run_portions(eng, "l", toks, [2, 1]), reference(cfg, w, toks).logits.numpy()) < vu.LIMIT[dtype]


# ---- memory of the recurrence ------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("decay", [[1.0, 0.9995], [0.0, 1.0], [0.3, 0.98]])
def test_state_over_chunk_edges(built, tmp_path, decay, dtype):
    """The recurrence alone, cut at and beside the edges of its chunks; with decays near one a state that is lost, kept from
    another request or decayed once too often shows hundreds of tokens later."""
    cfg = config([parallel(lin_heads=2, lin_dim=24, lin_vdim=20, decay=decay, scales=(1.0, 2.0))])
    w = isolate(vu.weights(cfg, seed=4), "right")
    eng = vu.engine(tmp_path, cfg, w, dtype)
    for seed, cuts in enumerate(([300], [64, 64, 64, 108], [63, 2, 64, 1, 65, 105], [1, 2], [129, 1, 1, 62, 107], [192, 1])):
        toks = vu.tokens(cfg, 300, seed=50 + seed)
        ref = reference(cfg, w, toks).logits.numpy()
        forgot = reference(cfg, w, toks[192:]).logits.numpy()
        assert decay[-1] < 0.99 or vu.error(forgot[-20:], ref[-20:]) > 0.15
        assert vu.error(vu.run_portions(eng, "r", toks, cuts), ref) < vu.LIMIT[dtype], cuts


# ---- far keys ------------------------------------------------------------------------------------------------------------
def ways(eng, toks):
    """Logits of the last token by a whole prompt, decoded alone, and as the end of a portion in a batch."""
    i = len(toks) - 1
    yield vu.step(eng, [("p", toks, [i])])
    eng.finish("p")
    vu.step(eng, [("d", toks[:-1], [])])
    yield vu.step(eng, [("d", toks[-1:], [0])])
    eng.finish("d")
    if len(toks) > 3:
        vu.step(eng, [("c", toks[:-2], []), ("o", toks[:7], [])])
        yield vu.step(eng, [("o", toks[7:20], []), ("c", toks[-2:], [1])])
        eng.finish("c")
        eng.finish("o")
    if len(toks) > 21:
        vu.step(eng, [("e", toks[:-20], [])])
        yield vu.step(eng, [("e", toks[-20:], [19])])
        eng.finish("e")


LAYERS = {"left": lambda: parallel(heads=4, kv_heads=2, dim=64, vdim=96, rot=32), "left_narrow": lambda: parallel(heads=3, kv_heads=3, dim=40, vdim=200, rot=16, scaling=None),
          "latent": lambda: latent(heads=4, dim=48, rot=16, vdim=32, q_rank=64, kv_rank=80)}


@pytest.mark.parametrize("dtype", ["fp32", "bf16"])
@pytest.mark.parametrize("kind", sorted(LAYERS))
def test_far_key(built, tmp_path, kind, dtype):
    """One key stands out among hundreds, first and last rows of pages among its places."""
    cfg, w = vu.spotlight(LAYERS[kind]())
    if kind != "latent":
        w = isolate(w, "left")
    eng = vu.engine(tmp_path, cfg, w, dtype)
    for place, last in ((0, 399), (63, 399), (64, 399), (200, 399), (127, 128), (5, 64), (300, 301)):
        toks = (2 + np.random.default_rng(place).integers(0, cfg["vocab"] - 3, 400)).tolist()[:last + 1]
        toks[place], toks[last] = 0, 1
        ref = reference(cfg, w, toks).logits[-1:].numpy()
        blind = list(toks)
        blind[place] = 5
        assert vu.error(reference(cfg, w, blind).logits[-1:].numpy(), ref) > 0.2, place
        for k, got in enumerate(ways(eng, toks)):
            assert vu.error(got, ref) < vu.LIMIT[dtype], (place, k)


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
    eng = vu.engine(tmp_path, cfg, w, dtype, requests=reqs, max_new=100, name="Vekolix")
    prompts = [vu.tokens(cfg, n, seed=40 + n) for n in (1, 2, 30, 150)]
    outs = [list(eng.generate(edge_fm.Request(0, p)).token_ids()) for p in prompts + prompts]      # again: captured prefill, used slot
    for p, o in zip(prompts, outs):
        assert len(o) == 100
        greedy_check(cfg, w, p, o, vu.LIMIT[dtype])
    assert outs[:4] == outs[4:]
    for tail in ([3], [4, 5], vu.tokens(cfg, 40, seed=2), [3]):        # behind a fixed prefix, whose state is restored
        greedy_check(cfg, w, prefix + tail, list(eng.generate(edge_fm.Request(7, prefix + tail)).token_ids()), vu.LIMIT[dtype])
    batch = [list(r.token_ids()) for r in eng.generate_batch([edge_fm.Request(100 + i, p) for i, p in enumerate(prompts + prompts[::-1])])]
    for p, o in zip(prompts, batch):
        assert len(o) == 100
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
