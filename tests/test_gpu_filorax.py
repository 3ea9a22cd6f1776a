"""Filorax on the GPU against the plain statement (filorax_plain.py): mechanisms alone, prompts, portions, batches, pages and state
slots that are used again, far keys and window edges, long decoding, generation through the scheduler."""
import json

import numpy as np
import pytest

import filorax_make as S
import filorax_plain as P
from gpu_common import backend, error, greedy_plain, run  # noqa: F401

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")
TOL = {"float32": 3e-5, "bfloat16": 4e-2}  # of the logits' spread


def make(backend, cfg, w, dtype, pool=512, rows=256, seq=None, slots=8):
    from orangu_b200.filorax import FiloraxModel

    return FiloraxModel(backend, cfg, w, dtype=dtype, max_seq_len=seq or pool, max_batch_tokens=rows, kv_pool_tokens=pool, state_slots=slots)


# ---- mechanisms ------------------------------------------------------------------------------------------------------------
ALONE = {
    "window": S.config([S.window()]),
    "window of one": S.config([S.window(heads=1, dim=8, vdim=8, size=1)]),
    "window, all ones": S.config([S.window(heads=1, dim=1, vdim=1, kv_rank=1, size=2)], width=8, groups=8, taps=1),
    "window, values of one": S.config([S.window(heads=5, dim=10, vdim=1, size=23)]),
    "window past the sequence": S.config([S.window(heads=2, dim=33, vdim=17, kv_rank=50, size=400)]),
    "window, many heads": S.config([S.window(heads=37, dim=18, vdim=12, kv_rank=24, size=21)]),
    "window, wide values": S.config([S.window(heads=2, dim=40, vdim=150, size=37)]),
    "window, values beyond the prompt kernels": S.config([S.window(heads=2, dim=16, vdim=264, size=17)]),
    "window, latents beyond the tensor-core kernels": S.config([S.window(heads=2, dim=24, vdim=16, kv_rank=600, size=30)]),
    "window, sizes of a large model": S.config([S.window(heads=8, dim=128, vdim=128, kv_rank=512, size=50)], width=256, groups=2),
    "plain window": S.config([S.window(plain=True)]),
    "plain window, many heads": S.config([S.window(heads=20, dim=24, vdim=30, kv_rank=100, size=50, plain=True)]),
    "causal": S.config([S.causal()]),
    "causal, least sizes": S.config([S.causal(heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1)]),
    "causal, mostly rotated": S.config([S.causal(heads=4, dim=6, rot_dim=70, vdim=36, kv_rank=30, base=50.0)]),
    "causal, sizes of a large model": S.config([S.causal(heads=8, dim=128, rot_dim=64, vdim=128, kv_rank=512)], width=256, groups=1),
    "causal, keys beyond tcgen05": S.config([S.causal(heads=2, dim=200, rot_dim=64, vdim=40, kv_rank=72)]),
    "causal, more heads than a tile": S.config([S.causal(heads=70, dim=16, rot_dim=8, vdim=12, kv_rank=20)]),
    "one norm group": S.config([S.causal()], ff=S.experts(), groups=1),
    "groups of whole warps": S.config([S.window()], ff=S.experts(), width=384, groups=3),
    "groups of odd sizes": S.config([S.causal()], ff=S.experts(), width=110, groups=10),
    "odd width": S.config([S.window()], ff=S.experts(), width=91, groups=7),
    "a group per entry": S.config([S.window()], ff=S.experts(), groups=96, eps=0.3),
    "wide": S.config([S.window(heads=1, dim=8, vdim=8)], width=4160, groups=5),
    "one tap": S.config([S.causal()], ff=S.experts(), taps=1),
    "two taps": S.config([S.causal()], ff=S.experts(), taps=2),
    "three taps, odd width": S.config([S.causal()], ff=S.experts(), taps=3, width=85, groups=5),
    "five taps": S.config([S.causal()], ff=S.experts(), taps=5),
    "sixteen taps": S.config([S.causal()], taps=16, width=60, groups=2),
    "one group of experts": S.config([S.window()], ff=S.experts(7, 2, 30, groups=1, keep=1, scale=0.3)),
    "every expert a group": S.config([S.window()], ff=S.experts(12, 4, 16, groups=12, keep=5)),
    "only the best group": S.config([S.window()], ff=S.experts(12, 3, 16, groups=3, keep=1, shared=40)),
    "one expert of forty, large shared": S.config([S.window()], ff=S.experts(40, 1, 7, groups=8, keep=3, shared=100)),
    "all experts": S.config([S.window()], ff=S.experts(4, 4, 130, groups=2, keep=2, shared=131)),
    "only expert": S.config([S.window()], ff=S.experts(1, 1, 33, groups=1, keep=1, shared=33)),
    "nothing shared": S.config([S.window()], ff=S.experts(8, 2, 40, shared=None)),
    "depth": S.config([S.window(), S.causal(), S.window(plain=True), S.causal(heads=1), S.window(size=2), S.causal(), S.window()], mult=1.3),
    "everything": S.config([S.window(plain=True), S.window(), S.causal(), S.causal(heads=1, dim=30), S.window(size=30, plain=True)],
                           ff=[S.experts(), S.experts(6, 2, 40, groups=2, keep=1), None, S.experts(9, 4, 20, groups=3, keep=2, shared=70), S.experts(5, 2, 16, groups=5, keep=3)]),
    "everything, other widths": S.config([S.causal(heads=6, vdim=22), S.window(heads=2, dim=50, vdim=70, kv_rank=90, size=40), S.causal(heads=2, rot_dim=6)],
                                         ff=[S.experts(6, 4, 90, groups=1, keep=1), None, S.experts(16, 6, 24, scale=3.0)], width=204, groups=17, taps=3, vocab=150, eps=0.03, mult=0.2),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_mechanism(backend, name, dtype):
    cfg = ALONE[name]
    w, toks = S.weights(cfg, 11, gain=1.5), S.tokens(cfg, 75, 12)
    want, hidden = P.forward(cfg, S.values(w), toks)
    m = make(backend, cfg, w, dtype)
    kv = m.new_kv_cache(128)
    got = run(m, kv, toks)
    assert error(m.last_hidden(75), hidden[-1]) < TOL[dtype]
    assert error(got, want) < TOL[dtype]
    # the same tokens one by one, and in portions
    one = m.new_kv_cache(128)
    assert error(run(m, one, toks, range(1, 75)), want) < TOL[dtype]
    cut = m.new_kv_cache(128)
    assert error(run(m, cut, toks, (2, 4, 5, 16, 18, 33, 34, 64, 66)), want) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer(backend, dtype):
    """Models of the first layers: what each layer hands on."""
    full = ALONE["everything"]
    w, toks = S.weights(full, 13), S.tokens(full, 70, 14)
    hidden = P.forward(full, S.values(w), toks)[1]
    for n in range(1, 6):
        m = make(backend, dict(full, layers=full["layers"][:n]), w, dtype)
        run(m, m.new_kv_cache(80), toks)
        assert error(m.last_hidden(70), hidden[n - 1]) < TOL[dtype]
        m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_rows_per_expert(backend, dtype):
    """Enough pairs and rows for the widest tiles of the grouped products, and the logits of the router as a product."""
    cfg = S.config([S.window(heads=1, dim=4, vdim=4)], ff=S.experts(4, 2, 2200, groups=2, keep=1, shared=300), width=64, groups=2)
    w, toks = S.weights(cfg, 15), S.tokens(cfg, 560, 16)
    want, _ = P.forward(cfg, S.values(w), toks)
    m = make(backend, cfg, w, dtype, pool=1024, rows=600)
    assert error(run(m, m.new_kv_cache(600), toks), want) < TOL[dtype]
    m.close()


def test_logits_that_are_no_numbers_choose_some_expert(backend):
    """Weights that overflow make logits that are not numbers: the step still ends, and the model goes on with other weights."""
    cfg = S.config([S.window()], ff=S.experts())
    w, toks = S.weights(cfg, 17), S.tokens(cfg, 90, 18)
    broken = dict(w)
    broken["l0.mix.o"] = np.full_like(w["l0.mix.o"], 0x7f80)  # infinite
    m = make(backend, cfg, broken, "bfloat16")
    kv = m.new_kv_cache(128)
    assert not np.isfinite(np.concatenate([m.forward_rows([kv], [toks[:80]], range(80)), m.forward_rows([kv], [toks[80:83]], range(3)), m.forward_rows([kv], [toks[83:84]], [0])])).any()
    m.close()
    m = make(backend, cfg, w, "bfloat16")
    assert error(run(m, m.new_kv_cache(128), toks), P.forward(cfg, S.values(w), toks)[0]) < TOL["bfloat16"]
    m.close()


def test_cache_and_states_hold_what_the_design_says(backend):
    cfg = S.config([S.window(), S.causal(dim=20, rot_dim=12)], ff=[None, S.experts()], taps=5)
    w, toks = S.weights(cfg, 21), S.tokens(cfg, 90, 22)
    v, eps = S.values(w), cfg["norm"]["eps"]
    inputs = []
    P.forward(cfg, v, toks, inputs)
    m = make(backend, cfg, w, "float32")
    for cuts in ((), (17, 20, 21), (88, 89), (1, 2, 3, 70)):
        kv = m.new_kv_cache(96, paged=True)
        run(m, kv, toks, cuts)
        for layer, x in enumerate(inputs):
            part, mx = P.part(v, f"l{layer}.mix."), cfg["layers"][layer]["mixer"]
            c, kr = P.latent(P.input_conv(x[0], v[f"l{layer}.canon1"]), part, mx, eps)
            got_c, got_r = kv.read(layer, 0, 90)
            assert error(got_c, c) < 1e-5
            if layer:
                assert error(got_r, np.stack([P.rotate(kr[p], p, mx["rot"]["base"]) for p in range(90)])) < 1e-5
            got = kv.read_state(layer)
            assert got.shape == (len(x), 4, 96)
            for g, h in zip(got, x):
                assert error(g, h[-4:]) < 1e-5
        kv.truncate(0)
    m.close()


# ---- batches, pages, slots -----------------------------------------------------------------------------------------------------
MIX = S.config([S.window(size=13), S.causal(), S.window(size=23, heads=5, plain=True), S.causal(heads=2, dim=12)], ff=[S.experts(), S.experts(6, 2, 40, groups=2, keep=1), None, S.experts(5, 1, 72, groups=5)])


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch(backend, dtype):
    """Portions of prompts beside single tokens; every request's logits are those it has alone."""
    w = S.weights(MIX, 31)
    prompts = [S.tokens(MIX, n, 32 + n) for n in (90, 41, 67, 3)]
    want = [P.forward(MIX, S.values(w), p)[0] for p in prompts]
    m = make(backend, MIX, w, dtype, rows=64)  # fewer rows than the largest steps: those run in parts
    kvs = [m.new_kv_cache(96, paged=True) for _ in prompts]
    at, got = [0] * 4, [[] for _ in prompts]
    rng = np.random.default_rng(33)
    sizes = (1, 1, 2, 3, 16, 17, 40)
    while any(at[i] < len(p) for i, p in enumerate(prompts)):
        live = [i for i, p in enumerate(prompts) if at[i] < len(p) and rng.random() < 0.8]
        if not live:
            continue
        n = [min(int(rng.choice(sizes)), len(prompts[i]) - at[i]) for i in live]
        lg = m.forward_rows([kvs[i] for i in live], [prompts[i][at[i]:at[i] + k] for i, k in zip(live, n)], range(sum(n)))
        o = 0
        for i, k in zip(live, n):
            got[i].append(lg[o:o + k])
            at[i] += k
            o += k
    for g, x in zip(got, want):
        assert error(np.concatenate(g), x) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size, vdim", ((1, 18), (37, 40), (90, 130), (128, 21), (400, 18)))
def test_long_portions(backend, size, vdim, dtype):
    """Portions long enough for the prompt kernels, started anywhere, beside short ones and single tokens."""
    cfg = S.config([S.window(size=size, dim=40, vdim=vdim), S.causal(heads=6, dim=72, rot_dim=24, vdim=vdim), S.window(heads=2, size=size + 9, plain=True, vdim=vdim)],
                   ff=[S.experts(), None, S.experts(4, 2, 24, groups=1, keep=1)])
    w = S.weights(cfg, 36, gain=2.0)
    prompts = [S.tokens(cfg, n, 37 + n) for n in (390, 165, 131)]
    want = [P.forward(cfg, S.values(w), p)[0] for p in prompts]
    m = make(backend, cfg, w, dtype, pool=1024, rows=512)
    kvs = [m.new_kv_cache(400, paged=True) for _ in prompts]
    got = [[] for _ in prompts]
    at = [0, 0, 0]
    for sizes in ((3, 70, 64), (65, 1, 0), (1, 64, 66), (64, 30, 1), (257, 0, 0)):
        live = [i for i in range(3) if sizes[i]]
        lg = m.forward_rows([kvs[i] for i in live], [prompts[i][at[i]:at[i] + sizes[i]] for i in live], range(sum(sizes)))
        o = 0
        for i in live:
            got[i].append(lg[o:o + sizes[i]])
            at[i] += sizes[i]
            o += sizes[i]
    assert at == [390, 165, 131]
    for g, x in zip(got, want):
        assert error(np.concatenate(g), x) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_prompts_and_single_tokens_in_one_step(backend, dtype):
    """More spans than a warp looks through at once, more long ones than are expanded at a time, more tokens than a step."""
    cfg = S.config([S.window(size=50), S.causal()], ff=[S.experts(), None])
    w = S.weights(cfg, 46)
    prompts = [S.tokens(cfg, 66 + i if i % 3 == 0 else 1 + i % 7, 47 + i) for i in range(44)]
    m = make(backend, cfg, w, dtype, pool=4096, rows=900, seq=128, slots=44)
    kvs = [m.new_kv_cache(128, paged=True) for _ in prompts]
    ends = np.cumsum([len(p) for p in prompts]) - 1
    lg = m.forward_rows(kvs, prompts, ends)
    nxt = m.forward_batch_decode(kvs, [p[0] for p in prompts], want_logits=True)[1]
    for i in (0, 1, 4, 6, 12, 31, 36, 40, 42, 43):
        want = P.forward(cfg, S.values(w), prompts[i] + prompts[i][:1])[0]
        assert error(np.stack([lg[i], nxt[i]]), want[-2:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("kind", ("window", "causal", "causal, large keys"))
def test_more_pieces_of_prompts_than_processors(backend, kind):
    """One long prompt, then many short ones (every second stream of rows is empty), on many heads: every CTA of the prompt attention
    takes several pieces.  Large keys leave room for one stage of them, and the streams of a piece end at different tiles."""
    layer = {"window": S.window(heads=40, dim=24, vdim=16, size=150), "causal": S.causal(heads=40, dim=24, rot_dim=8, vdim=24),
             "causal, large keys": S.causal(heads=40, dim=128, rot_dim=64, vdim=72)}[kind]
    cfg = S.config([layer], width=64, groups=2)
    w = S.weights(cfg, 48)
    long, short = S.tokens(cfg, 1100, 49), [S.tokens(cfg, 64 + i % 9, 50 + i) for i in range(13)]
    m = make(backend, cfg, w, "bfloat16", pool=4096, rows=2048, seq=2048, slots=16)
    want = P.forward(cfg, S.values(w), long)[0]
    places = list(range(0, 1100, 7))
    assert error(m.forward_rows([m.new_kv_cache(1536, paged=True)], [long], places), want[places]) < TOL["bfloat16"]
    kvs = [m.new_kv_cache(96, paged=True) for _ in short]
    ends = np.cumsum([len(p) for p in short]) - 1
    got = m.forward_rows(kvs, short, ends)
    for g, p in zip(got, short):
        assert error(g[None], P.forward(cfg, S.values(w), p)[0][-1:]) < TOL["bfloat16"]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_single_tokens(backend, dtype):
    """A decode batch wide enough for the tensor-core products, at unequal lengths."""
    w = S.weights(MIX, 41)
    seqs = [S.tokens(MIX, 5 + 3 * i, 42 + i) for i in range(9)]
    m = make(backend, MIX, w, dtype, pool=1024, slots=9)
    kvs = [m.new_kv_cache(64) for _ in seqs]
    m.forward_rows(kvs, [s[:-2] for s in seqs], [])
    first = m.forward_rows(kvs, [[s[-2]] for s in seqs], range(9))
    toks, second = m.forward_batch_decode(kvs, [s[-1] for s in seqs], want_logits=True)
    for i, s in enumerate(seqs):
        want = P.forward(MIX, S.values(w), s)[0]
        assert error(np.stack([first[i], second[i]]), want[-2:]) < TOL[dtype]
        assert toks[i] == np.argmax(second[i])
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_are_used_again(backend, dtype):
    from orangu_b200 import OranguError

    w = S.weights(MIX, 51)
    m = make(backend, MIX, w, dtype, pool=96, slots=2)
    assert m.free_pages == 6 and m.free_slots == 2
    a, b, c = (m.new_kv_cache(96, paged=True) for _ in range(3))
    x, y, z = (S.tokens(MIX, n, 52 + n) for n in (50, 20, 70))
    run(m, a, x)
    run(m, b, y)
    assert m.free_pages == 0 and m.free_slots == 0
    with pytest.raises(OranguError, match="pool exhausted|no free state slot"):
        m.forward_rows([c], [z[:5]], [])
    with pytest.raises(OranguError, match="not rolled back"):
        b.truncate(7)
    a.truncate(0)
    assert m.free_pages == 4 and m.free_slots == 1
    want_z, want_y = P.forward(MIX, S.values(w), z)[0], P.forward(MIX, S.values(w), y + z[:12])[0]
    # the third sequence on the first one's pages and state, beside the second, which goes on
    got_z = [m.forward_rows([c, b], [z[:40], z[:1]], range(41))]
    got_y = [got_z[0][40:]]
    got_z[0] = got_z[0][:40]
    for i in range(1, 12):
        lg = m.forward_rows([b, c], [[z[i]], z[39 + i:40 + i]], range(2))
        got_y.append(lg[:1])
        got_z.append(lg[1:])
    assert error(np.concatenate(got_z), want_z[:51]) < TOL[dtype] and error(np.concatenate(got_y), want_y[20:]) < TOL[dtype]
    for kv in (b, c):
        kv.truncate(0)
    assert m.free_pages == 6 and m.free_slots == 2
    m.close()


@pytest.mark.parametrize("taps", (2, 4, 6))
@pytest.mark.parametrize("first", (1, 2, 3, 5))
def test_short_starts_in_used_slots(backend, first, taps):
    """Sequences whose first portions are shorter than the convolution reaches back, in slots that held others."""
    cfg = S.config([S.window(), S.causal()], ff=[S.experts(), None], taps=taps)
    w = S.weights(cfg, 55)
    m = make(backend, cfg, w, "float32", slots=2)
    a, b = m.new_kv_cache(64, paged=True), m.new_kv_cache(64, paged=True)
    x, y, z = (S.tokens(cfg, n, 56 + n) for n in (30, 12, 17))
    m.forward_rows([a, b], [x, y], [])
    for kv in (a, b):
        kv.truncate(0)
    got = m.forward_rows([a, b], [y[:first], z[:1]], range(first + 1))
    got_a, got_b = [got[:first]], [got[first:]]
    for i in range(8):  # one by one beside portions of two
        more, pair = y[first + i:first + i + 1], z[1 + 2 * i:3 + 2 * i]
        lg = m.forward_rows([b, a], [pair, more], range(3)) if more else m.forward_rows([b], [pair], range(2))
        got_b.append(lg[:2])
        got_a.append(lg[2:])
    got_a = np.concatenate(got_a)
    assert error(got_a, P.forward(cfg, S.values(w), y)[0][:len(got_a)]) < 3e-5
    assert error(np.concatenate(got_b), P.forward(cfg, S.values(w), z)[0]) < 3e-5
    m.close()


def test_copy_of_a_sequence_goes_its_own_way(backend):
    w = S.weights(MIX, 61)
    x, y, z = S.tokens(MIX, 37, 62), S.tokens(MIX, 9, 63), S.tokens(MIX, 9, 64)
    m = make(backend, MIX, w, "float32")
    a, b = m.new_kv_cache(64), m.new_kv_cache(64, paged=True)
    run(m, a, x)
    b.copy_prefix_from(a, 37)
    assert error(run(m, a, y), P.forward(MIX, S.values(w), x + y)[0][37:]) < 3e-5
    assert error(run(m, b, z), P.forward(MIX, S.values(w), x + z)[0][37:]) < 3e-5
    m.close()


# ---- far keys, window edges, first tokens -----------------------------------------------------------------------------------------
def edge_model(layer):
    """One layer in which single keys stand out: large queries, no rotated part in the scores, no other token mixed into an input,
    sinks that do not drown them."""
    cfg = S.config([layer], mult=1.0)
    w = S.weights(cfg, 71, gain=6.0, conv=False)
    m = layer["mixer"]
    if "rot_dim" in m:
        q = w["l0.mix.q"].reshape(m["heads"], m["dim"] + m["rot_dim"], -1).copy()
        q[:, m["dim"]:] = 0
        w["l0.mix.q"] = q.reshape(w["l0.mix.q"].shape)
    if "l0.mix.sink" in w:
        w["l0.mix.sink"] = S.bf16_bits(np.linspace(-1.0, 0.5, m["heads"]))
    return cfg, w


def standing_out(cfg, w):
    """Tokens (query, key, filler): the query's score with the key is far above its score with the filler (first head), so that
    whether the key is seen decides that head's output."""
    v, mx = S.values(w), cfg["layers"][0]["mixer"]
    part, D = P.part(v, "l0.mix."), mx["dim"]
    h = P.grouped_norm(v["embed"], v["l0.norm1"], cfg["norm"]["groups"], cfg["norm"]["eps"])
    h = h + h * v["l0.canon1"][:, -1]
    q = (h @ part["q"].T)[:, :D]
    c, _ = P.latent(h, part, mx, cfg["norm"]["eps"])
    s = q @ (c @ part["uk"].T)[:, :D].T * mx["scale"]
    best = np.unravel_index(np.argmax(s.max(1)[:, None] - s), s.shape)  # query row and its worst key: the filler
    return int(best[0]), int(np.argmax(s[best[0]])), int(best[1])


def check_seen(m, v, cfg, w, wrong, j, i, dtype):
    """A key at j asked for at i, in a prompt, decoded, and at the start of long portions; `wrong`: a window under which the answer
    would be another, or None: without the key it would."""
    qt, kt, filler = standing_out(cfg, w)
    toks = [filler] * (i + 1)
    toks[i] = qt
    without = P.forward(cfg, v, toks)[0]
    toks[j], toks[i] = kt, qt
    want = P.forward(cfg, v, toks)[0]
    layer = cfg["layers"][0]
    other = without if wrong is None else P.forward({**cfg, "layers": [{**layer, "mixer": {**layer["mixer"], "mask": {"size": wrong}}}]}, v, toks)[0]
    assert error(other[i:], want[i:]) > 0.15
    whole, step, two, far = (m.new_kv_cache(1024, paged=True) for _ in range(4))
    assert error(run(m, whole, toks)[i:], want[i:]) < TOL[dtype]
    if i:
        assert error(run(m, step, toks, (i,))[i:], want[i:]) < TOL[dtype]
    assert error(run(m, two, toks, (j, i - 1) if i - 1 > j > 0 else (j,) if j else ())[i:], want[i:]) < TOL[dtype]
    longer = toks + [filler] * 70
    assert error(run(m, far, longer, tuple(c for c in sorted({j, i}) if c))[i:i + 1], want[i:]) < TOL[dtype]
    for kv in (whole, step, two, far):
        kv.truncate(0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("plain", (False, True))
@pytest.mark.parametrize("size", (2, 3, 16, 17, 31, 64, 65))
def test_window_edges(backend, size, plain, dtype):
    """A key just inside and just outside the window, at page borders and elsewhere, from the sequence's first token on.  The plain
    statement with a window one longer or one shorter is far off, so a shifted edge could not pass."""
    cfg, w = edge_model(S.window(heads=2, size=size, plain=plain))
    m, v = make(backend, cfg, w, dtype, pool=4096, rows=1024), S.values(w)
    for j in (0, 1, 5, 15, 16, 31, 47):
        check_seen(m, v, cfg, w, size - 1, j, j + size - 1, dtype)
        check_seen(m, v, cfg, w, size + 1, j, j + size, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_at_the_edge_of_a_long_window(backend, dtype):
    """Hundreds of keys between question and key: decoding shares them among CTAs whose parts are put together afterwards."""
    cfg, w = edge_model(S.window(heads=2, size=460))
    m, v = make(backend, cfg, w, dtype, pool=4096, rows=1024), S.values(w)
    for j in (0, 4, 17):
        check_seen(m, v, cfg, w, 459, j, j + 459, dtype)
        check_seen(m, v, cfg, w, 461, j, j + 460, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("vdim", (20, 140))
def test_far_key_of_a_causal_layer(backend, vdim, dtype):
    """One key up to hundreds of positions away, at the sequence's start and at page borders."""
    cfg, w = edge_model(S.causal(heads=2, vdim=vdim))
    m, v = make(backend, cfg, w, dtype, pool=4096, rows=1024), S.values(w)
    for j, i in ((0, 1), (0, 640), (15, 641), (16, 80), (255, 700)):
        check_seen(m, v, cfg, w, None, j, i, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_far_into_a_sequence(backend, dtype):
    """Scores that live on the rotated part alone, also where it has turned many times."""
    cfg = S.config([S.causal(heads=2, dim=8, rot_dim=32, base=20.0)])
    w, toks = S.weights(cfg, 72, gain=2.0), S.tokens(cfg, 700, 73)
    q = w["l0.mix.q"].reshape(2, 40, -1).copy()
    q[:, :8] = 0
    w["l0.mix.q"] = q.reshape(80, -1)
    want = P.forward(cfg, S.values(w), toks)[0]
    m = make(backend, cfg, w, dtype, pool=1024, rows=1024)
    for cuts in ((), (64, 130, 600), tuple(range(640, 700))):
        kv = m.new_kv_cache(704, paged=True)
        assert error(run(m, kv, toks, cuts), want) < TOL[dtype]
        kv.truncate(0)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", (-30.0, 0.0, 9.0, 60.0, 300.0))
@pytest.mark.parametrize("kind", ("window", "causal", "wide"))
def test_sinks(backend, kind, sink, dtype):
    """Sinks far below, among and far above the scores, in all forms of the attention; the second head has another."""
    cfg = S.config([{"window": S.window(heads=2, size=40, scale=0.5), "causal": S.causal(heads=2, scale=0.5), "wide": S.causal(heads=2, vdim=140, scale=0.5)}[kind]])
    w, toks = S.weights(cfg, 74, gain=2.0), S.tokens(cfg, 140, 75)
    w["l0.mix.sink"] = S.bf16_bits([sink, 0.5])
    want = P.forward(cfg, S.values(w), toks)[0]
    m = make(backend, cfg, w, dtype)
    for cuts in ((), (70,), range(100, 140), (3, 50)):
        kv = m.new_kv_cache(160, paged=True)
        assert error(run(m, kv, toks, cuts), want) < TOL[dtype]
        kv.truncate(0)
    m.close()


# ---- decoding ------------------------------------------------------------------------------------------------------------------------
def test_long_decoding(backend):
    """Hundreds of decoded tokens through captured graphs; the plain statement then judges every choice at once."""
    cfg = MIX
    w = S.weights(cfg, 91)
    for dtype in DTYPES:
        m = make(backend, cfg, w, dtype, pool=1024)
        prompts = [S.tokens(cfg, n, 92 + n) for n in (18, 1)]
        kvs = [m.new_kv_cache(512, paged=True) for _ in prompts]
        first = [m.forward_maybe_sampling(kv, p, 0) for kv, p in zip(kvs, prompts)]
        steps = m.decode_loop(kvs, first, 250)
        single = [m.decode_greedy(kvs[0], int(steps[-1, 0]))]
        for _ in range(20):
            single.append(m.decode_greedy(kvs[0], single[-1]))
        for i, p in enumerate(prompts):
            got = [first[i]] + steps[:, i].tolist() + (single if i == 0 else [])
            lg = P.forward(cfg, S.values(w), p + got[:-1])[0][len(p) - 1:]
            behind = lg.max(-1) - lg[np.arange(len(got)), got]  # a choice may differ only where the two are within rounding
            assert behind.max() < TOL[dtype] * np.sqrt((lg ** 2).mean())
        assert [len(kv) for kv in kvs] == [18 + 250 + 21, 1 + 250]
        m.close()


def test_generation_through_scheduler_and_files(backend, tmp_path):
    """A folder on disk, the registry, the slot pool with more prompts than fit one step, greedy tokens and repeat penalty."""
    from orangu_b200.__main__ import generate
    from orangu_b200.registry import load_model
    from orangu_b200.safetensors import save

    w = S.weights(MIX, 101)
    (tmp_path / "config.json").write_text(json.dumps(MIX))
    save(str(tmp_path / "model.safetensors"), w)
    m = load_model(backend, str(tmp_path), dtype="float32", max_seq_len=128, max_batch_tokens=32, kv_pool_tokens=512, state_slots=5)
    prompts = [S.tokens(MIX, n, 102 + n) for n in (45, 2, 17, 33, 8)]
    got = generate(m, prompts, 12, prefill_batch=10)
    for p, g in zip(prompts, got):
        want, lead = greedy_plain(P, MIX, S.values(w), p, 12)
        assert lead > 1e-5 and g == want  # seeds chosen so that no two tokens tie within rounding
    assert m.free_pages == 32 and m.free_slots == 5
    # repeat penalty: the penalised argmax of the logits without it
    p = prompts[0]
    a = generate(m, [p], 2, repeat_penalty=1.8, repeat_last_n=64)[0]
    lg = P.forward(MIX, S.values(w), p)[0][-1]
    seen = list(set(p))
    lg[seen] = np.where(lg[seen] > 0, lg[seen] / 1.8, lg[seen] * 1.8)
    assert a[0] == int(np.argmax(lg))
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(backend, tmp_path, dtype):
    """Requests that come, pause, end and make room for others; logits files in the order asked for."""
    from orangu_b200 import trace

    w = S.weights(MIX, 111)
    v = S.values(w)
    m = make(backend, MIX, w, dtype, pool=192, rows=192, slots=4)
    t = {k: S.tokens(MIX, n, 112 + n) for k, n in (("a", 40), ("b", 64), ("c", 30), ("d", 5), ("e", 60))}
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": t["a"][:38], "want": [37, 0]}, {"id": "b", "tokens": t["b"][:1], "want": [0]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": t["b"][1:20], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "c", "tokens": t["c"], "want": [29]}, {"id": "a", "tokens": t["a"][38:39], "want": [0]}], "end": ["c"]},
        {"step": 4, "entries": [{"id": "a", "tokens": t["a"][39:], "want": [0]}, {"id": "d", "tokens": t["d"], "want": [1, 4]}], "end": ["a", "d"]},
        {"step": 5, "entries": [{"id": "e", "tokens": t["e"], "want": [59]}, {"id": "b", "tokens": t["b"][20:], "want": [0, 43]}], "end": ["b", "e"]},
    ]
    want = {0: [("a", 37), ("a", 0), ("b", 0)], 2: [("c", 29), ("a", 38)], 4: [("a", 39), ("d", 1), ("d", 4)], 5: [("e", 59), ("b", 20), ("b", 63)]}
    said = []
    trace.replay(m, [json.dumps(s) + "\n" for s in steps], str(tmp_path), 192, said.append)
    assert said == [f"done {n}" for n in (0, 1, 2, 4, 5)] and not (tmp_path / "1.f32").exists()
    for n, places in want.items():
        got = np.fromfile(tmp_path / f"{n}.f32", np.float32).reshape(len(places), -1)
        exp = np.stack([P.forward(MIX, v, t[k][:p + 1])[0][p] for k, p in places])
        assert error(got, exp) < TOL[dtype]
    m.close()


def test_descriptions_the_library_refuses(backend):
    """What a reader could get wrong comes back as an error, before anything is made."""
    from orangu_b200 import OranguError, capi
    from orangu_b200.filorax import FiloraxModel
    from orangu_b200.layered import LayeredModel

    init = LayeredModel.__init__

    def description(change):
        def changed(self, be, desc, blocks):
            change(desc, blocks)
            init(self, be, desc, blocks)

        LayeredModel.__init__ = changed
        try:
            FiloraxModel(backend, MIX, S.weights(MIX, 121), kv_pool_tokens=64, max_seq_len=64, state_slots=2).close()
        finally:
            LayeredModel.__init__ = init

    description(lambda d, b: None)
    empty = capi.MatrixDesc()
    for change, message in (
        (lambda d, b: setattr(d, "norm_groups", 5), "does not divide the width"),
        (lambda d, b: setattr(d, "conv_taps", 17), "taps"),
        (lambda d, b: setattr(d, "final_norm", None), "last norm"),
        (lambda d, b: setattr(b[1], "conv1", None), "convolution of an input"),
        (lambda d, b: setattr(b[1], "conv2", None), "convolution of an input"),
        (lambda d, b: setattr(b[1], "depth", None), "average over depth"),
        (lambda d, b: setattr(b[1], "pre_norm2", None), "norm of the feed-forward"),
        (lambda d, b: setattr(b[0], "post_norm1", b[0].pre_norm1), "plain sums"),
        (lambda d, b: setattr(b[0], "n_expert_group", 3), "groups do not divide"),
        (lambda d, b: setattr(b[0], "n_group_used", 5), "groups do not divide"),
        (lambda d, b: setattr(b[0], "n_group_used", 1), "than its groups hold"),
        (lambda d, b: setattr(b[0], "router_softmax", 3), "unknown scores"),
        (lambda d, b: setattr(b[0].mixer, "w_gate", b[0].mixer.wo), "gate"),
        (lambda d, b: setattr(b[1].mixer, "rot_dims", 18), "rot_dims"),
        (lambda d, b: setattr(b[1].mixer, "w_uk", empty), "w_uk"),
    ):
        with pytest.raises(OranguError, match=message):
            description(change)
