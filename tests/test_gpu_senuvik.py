"""Senuvik on the GPU against the plain statement (senuvik_plain.py): mechanisms alone, prompts, portions, batches, pages and state
slots that are used again, far tokens and window edges, long decoding, generation through the scheduler."""
import json

import numpy as np
import pytest

import senuvik_make as S
import senuvik_plain as P
from gpu_common import backend, error, greedy_plain, run  # noqa: F401

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")
TOL = {"float32": 3e-5, "bfloat16": 4e-2}  # of the logits' spread


def make(backend, cfg, w, dtype, pool=512, rows=256, seq=None, slots=8):
    from orangu_b200.senuvik import SenuvikModel

    return SenuvikModel(backend, cfg, w, dtype=dtype, max_seq_len=seq or pool, max_batch_tokens=rows, kv_pool_tokens=pool, state_slots=slots)


def close(got, want, dtype):
    """Every position within the tolerance; in bfloat16 a norm of little that is left after cancelling may magnify the rounding at a
    few of them."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    e = np.sort(np.sqrt(((got - want) ** 2).mean(-1)) / np.sqrt((want ** 2).mean()))
    return e[-1] < TOL[dtype] if dtype == "float32" else e[-1] < 5 * TOL[dtype] and e[int(0.96 * len(e)) - 1] < TOL[dtype]


# ---- mechanisms ------------------------------------------------------------------------------------------------------------
PLAIN = S.space(heads=1, vdim=4, state=2, groups=1, norm_groups=1, conv=1)  # a mixer that does not matter
ALONE = {
    "window": S.config([S.window()]),
    "window, one head, window of one, nothing kept": S.config([S.window(heads=1, kv_heads=1, dim=8, vdim=8, size=1, keep=0, rot_dims=2, factor=1.0)]),
    "window, window of one, first kept": S.config([S.window(heads=2, kv_heads=1, dim=10, vdim=1, size=1, keep=1, rot_dims=10)]),
    "window, one key head": S.config([S.window(heads=5, kv_heads=1, dim=34, vdim=50, size=23, keep=17, rot_dims=34)]),
    "window, more kept than a page": S.config([S.window(heads=4, kv_heads=4, dim=64, vdim=48, size=9, keep=35, rot_dims=32)]),
    "window past the sequence": S.config([S.window(heads=8, kv_heads=2, dim=64, vdim=128, size=400, keep=4, rot_dims=64)]),
    "window, everything kept": S.config([S.window(size=5, keep=300)]),
    "window, wide values": S.config([S.window(heads=2, kv_heads=1, dim=40, vdim=150, size=37, keep=2, rot_dims=24)]),
    "window, beyond the tensor-core kernels": S.config([S.window(heads=2, kv_heads=1, dim=16, vdim=264, keep=5, rot_dims=16)]),
    "window, many heads on one key head": S.config([S.window(heads=37, kv_heads=1, dim=18, vdim=12, size=21, keep=1, rot_dims=6)]),
    "window, sizes of a large model": S.config([S.window(heads=8, kv_heads=2, dim=128, vdim=128, size=50, keep=4, rot_dims=64)], width=256),
    "shared keys": S.config([S.window(size=9, keep=2), S.window(size=21, keep=5, kv_from=0), S.window(heads=2, kv_heads=1), S.window(size=4, keep=0, kv_from=0),
                             S.window(heads=2, kv_heads=1, size=30, kv_from=2)]),
    "state space": S.config([S.space()]),
    "state space, all ones": S.config([S.space(heads=1, vdim=1, state=1, groups=1, norm_groups=1, conv=1)]),
    "state space, one group, two taps": S.config([S.space(heads=5, vdim=32, state=64, groups=1, norm_groups=1, conv=2)]),
    "state space, parts across heads, three taps": S.config([S.space(heads=9, vdim=8, state=33, groups=9, norm_groups=4, conv=3)]),
    "state space, parts within heads, many taps": S.config([S.space(heads=2, vdim=50, state=128, groups=2, norm_groups=10, conv=16)]),
    "state space, large state": S.config([S.space(heads=4, vdim=65, state=200, groups=2, norm_groups=2, conv=5)]),
    "beside": S.config([S.beside()]),
    "beside, ones": S.config([S.beside(heads=1, kv_heads=1, dim=4, vdim=1, rot_dims=2, factor=1.0, left=1.0, right=1.0, time_heads=1, time_dim=1)]),
    "beside, wide values": S.config([S.beside(heads=2, kv_heads=1, dim=40, vdim=150, rot_dims=24, time_heads=2, time_dim=64)]),
    "beside, beyond the tensor-core kernels": S.config([S.beside(heads=2, kv_heads=2, dim=16, vdim=264, rot_dims=16, time_heads=5, time_dim=33)]),
    "beside, sizes of a large model": S.config([S.beside(heads=8, kv_heads=2, dim=128, vdim=128, rot_dims=128, softcap=30.0, time_heads=2, time_dim=128)], width=256),
    "beside, large state": S.config([S.beside(heads=3, kv_heads=3, dim=80, vdim=72, rot_dims=16, softcap=1.5, time_heads=2, time_dim=160)]),
    "gated gelu": S.config([PLAIN], ff=S.dense(250)),
    "one expert of twelve": S.config([PLAIN], ff=S.experts(12, 1, 44)),
    "three experts of four, small shared": S.config([PLAIN], ff=S.experts(4, 3, 60, shared=7)),
    "five experts of forty, large shared": S.config([PLAIN], ff=S.experts(40, 5, 7, shared=100)),
    "all experts": S.config([PLAIN], ff=S.experts(2, 2, 130, shared=131)),
    "only expert": S.config([PLAIN], ff=S.experts(1, 1, 33, shared=33)),
    "no feed-forward": S.config([S.beside(), S.space()]),
    "everything": S.config([S.window(), S.space(), S.beside(), S.window(size=30, keep=5, kv_from=0), S.beside(heads=1, kv_heads=1), S.space(heads=2, groups=1, norm_groups=3, conv=3)],
                           ff=[S.dense(40), S.experts(5, 3, 20, shared=50), None, S.experts(4, 1, 30, shared=12), S.dense(24), S.experts(9, 2, 16)]),
    "everything, other widths": S.config([S.beside(heads=6, kv_heads=3, left=0.3), S.window(heads=6, kv_heads=3, vdim=22), S.space(heads=4, groups=2, norm_groups=1),
                                          S.window(heads=3, kv_heads=3, vdim=22, kv_from=1)], ff=[S.experts(6, 4, 90), None, S.dense(33), None], width=203, vocab=150, eps=0.03),
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
    assert close(m.last_hidden(75), hidden[-1], dtype)
    assert close(got, want, dtype)
    # the same tokens one by one, and in portions
    one = m.new_kv_cache(128)
    assert close(run(m, one, toks, range(1, 75)), want, dtype)
    cut = m.new_kv_cache(128)
    assert close(run(m, cut, toks, (2, 4, 5, 16, 18, 33, 34, 64, 66)), want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_rows_per_expert(backend, dtype):
    """Enough pairs and rows for the widest tiles of the grouped products, and the logits of the router as a product."""
    cfg = S.config([PLAIN], ff=S.experts(3, 2, 2200, shared=300), width=64)
    w, toks = S.weights(cfg, 15), S.tokens(cfg, 560, 16)
    want, _ = P.forward(cfg, S.values(w), toks)
    m = make(backend, cfg, w, dtype, pool=1024, rows=600)
    assert error(run(m, m.new_kv_cache(600), toks), want) < TOL[dtype]
    m.close()


def test_cache_and_states_hold_what_the_design_says(backend):
    cfg = S.config([S.window(), S.window(size=30, kv_from=0), S.space(), S.beside()])
    w, toks = S.weights(cfg, 21), S.tokens(cfg, 90, 22)
    v, eps = S.values(w), cfg["norm"]["eps"]
    m = make(backend, cfg, w, "float32")
    kv = m.new_kv_cache(96)
    run(m, kv, toks, (17, 20, 21))
    k, val = kv.read(0, 0, 90)
    h = P.norm(v["embed"][toks], v["l0.norm1"], eps)
    want_k, want_v = P.window_keys_values(h, P.part(v, "l0.mix."), cfg["layers"][0]["mixer"], eps)
    assert error(k, want_k.reshape(90, -1)) < 1e-5 and error(val, want_v.reshape(90, -1)) < 1e-5
    again, _ = kv.read(1, 0, 90)
    assert (again == k).all()
    states = []
    P.forward(cfg, v, toks, states)
    for layer, want in zip((2, 3), states):
        got = kv.read_state(layer)
        assert error(got.reshape(want.shape[0], -1), want.reshape(want.shape[0], -1)) < 2e-5
    m.close()


# ---- batches, pages, slots -----------------------------------------------------------------------------------------------------
MIX = S.config([S.window(size=13, keep=5), S.beside(), S.space(), S.window(heads=6, size=23, keep=2, kv_from=0)],
               ff=[S.experts(6, 2, 40, shared=24), S.dense(104), S.experts(5, 1, 72), None])


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
@pytest.mark.parametrize("window, keep", ((1, 3), (37, 20), (50, 140), (90, 0), (400, 6)))
def test_long_portions(backend, window, keep, dtype):
    """Portions long enough for the prompt kernels, started anywhere, beside short ones and single tokens."""
    cfg = S.config([S.window(size=window, keep=keep, dim=40, vdim=18), S.beside(heads=6, kv_heads=1, dim=72, rot_dims=24, time_heads=2, time_dim=72),
                    S.space(heads=4, vdim=40, state=96, groups=2, norm_groups=2, conv=3), S.window(heads=2, size=window + 9, keep=keep // 2, dim=40, vdim=18, kv_from=0)],
                   ff=[S.dense(40), S.experts(4, 2, 24), None, None])
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
    """More spans than a warp looks through at once, some long, more tokens than a step."""
    cfg = S.config([S.window(size=50), S.beside(heads=3, kv_heads=1, dim=32, rot_dims=32), S.space()], ff=[S.experts(8, 2, 16), None, S.dense(20)])
    w = S.weights(cfg, 46)
    prompts = [S.tokens(cfg, 66 + i if i % 4 == 0 else 1 + i % 7, 47 + i) for i in range(44)]
    m = make(backend, cfg, w, dtype, pool=4096, rows=700, seq=128, slots=44)
    kvs = [m.new_kv_cache(128, paged=True) for _ in prompts]
    ends = np.cumsum([len(p) for p in prompts]) - 1
    lg = m.forward_rows(kvs, prompts, ends)
    nxt = m.forward_batch_decode(kvs, [p[0] for p in prompts], want_logits=True)[1]
    for i in (0, 1, 4, 5, 12, 31, 36, 40, 42, 43):
        want = P.forward(cfg, S.values(w), prompts[i] + prompts[i][:1])[0]
        assert error(np.stack([lg[i], nxt[i]]), want[-2:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("kind", ("window", "beside"))
def test_more_pieces_of_prompts_than_processors(backend, kind):
    """One long prompt, then many short ones (every second stream of rows is empty), on sixteen key/value heads: every CTA of the
    prompt attention takes several pieces."""
    layer = S.window(heads=32, kv_heads=16, dim=24, vdim=16, size=150, keep=9) if kind == "window" else S.beside(heads=32, kv_heads=16, dim=24, vdim=40)
    cfg = S.config([layer], width=64)
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


@pytest.mark.parametrize("first", range(1, 7))
def test_short_starts_in_used_slots(backend, first):
    """Sequences whose first portions are shorter than the convolution reaches back, in slots that held others."""
    cfg = S.config([S.space(conv=5), S.beside()])
    w = S.weights(cfg, 55)
    m = make(backend, cfg, w, "float32", slots=2)
    a, b = m.new_kv_cache(64, paged=True), m.new_kv_cache(64, paged=True)
    x, y, z = (S.tokens(cfg, n, 56 + n) for n in (30, 12, 14))
    m.forward_rows([a, b], [x, y], [])
    for kv in (a, b):
        kv.truncate(0)
    got = [m.forward_rows([a, b], [y[:first], z[:1]], range(first + 1))]
    got_a, got_b = [got[0][:first]], [got[0][first:]]
    for i in range(first, 12):
        lg = m.forward_rows([a, b], [y[i:i + 1], z[2 * (i - first) + 1:2 * (i - first) + 3]], range(1 + len(z[2 * (i - first) + 1:2 * (i - first) + 3]))) if 2 * (i - first) + 1 < 14 \
            else m.forward_rows([a], [y[i:i + 1]], range(1))
        got_a.append(lg[:1])
        got_b.append(lg[1:])
    got_b = np.concatenate(got_b)
    assert error(np.concatenate(got_a), P.forward(cfg, S.values(w), y)[0]) < 3e-5
    assert error(got_b, P.forward(cfg, S.values(w), z)[0][:len(got_b)]) < 3e-5
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


# ---- far keys, window edges ------------------------------------------------------------------------------------------------------
def edge_model(window, keep):
    """One layer in which single keys stand out: large query norms, no score in the entries that rotate, sinks that do not drown
    them."""
    cfg = S.config([S.window(heads=2, kv_heads=1, size=window, keep=keep, rot_dims=8)])
    w = S.weights(cfg, 71, gain=6.0)
    q = S.bf16_values(w["l0.mix.q.norm"]).reshape(2, -1)
    q[:, :8] = 0.0
    w["l0.mix.q.norm"], w["l0.mix.sink"] = S.bf16_bits(q.reshape(-1)), S.bf16_bits([-1.0, 0.5])
    return cfg, w


def standing_out(cfg, w):
    """Tokens (query, key, filler): the query's score with the key is far above its score with the filler (first head), so that
    whether the key is seen decides that head's output."""
    v, mx = S.values(w), cfg["layers"][0]["mixer"]
    part, D, eps = P.part(v, "l0.mix."), mx["dim"], cfg["norm"]["eps"]
    h = P.norm(v["embed"], v["l0.norm1"], eps)
    q = P.norm(h @ part["q"].T + part["q.b"], part["q.norm"], eps)[:, :D]
    k = P.norm(h @ part["k"].T + part["k.b"], part["k.norm"], eps)[:, :D]
    s = q @ k.T * mx["scale"]
    best = np.unravel_index(np.argmax(s.max(1)[:, None] - s), s.shape)  # query row and its worst key: the filler
    return int(best[0]), int(np.argmax(s[best[0]])), int(best[1])


def check_seen(m, v, cfg, w, wrong, j, i, dtype):
    """A key at j asked for at i, in a prompt, decoded, and at the start of long portions; `wrong`: a mask under which the answer
    would be another."""
    qt, kt, filler = standing_out(cfg, w)
    toks = [filler] * (i + 1)
    toks[j], toks[i] = kt, qt
    want = P.forward(cfg, v, toks)[0]
    if wrong is not None:
        layer = cfg["layers"][0]
        other = {**cfg, "layers": [{**layer, "mixer": {**layer["mixer"], "mask": wrong}}]}
        assert error(P.forward(other, v, toks)[0][i:], want[i:]) > 0.2
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
@pytest.mark.parametrize("window", (1, 3, 16, 17, 31, 64, 65))
def test_window_edges(backend, window, dtype):
    """A key just inside and just outside the window, at page borders and elsewhere.  The plain statement with a window one longer
    or one shorter is far off, so a shifted edge could not pass."""
    cfg, w = edge_model(window, 0 if window == 17 else 2)
    m, v = make(backend, cfg, w, dtype, pool=4096, rows=1024), S.values(w)
    keep = cfg["layers"][0]["mixer"]["mask"]["keep_first"]
    for j in (keep, 5, 15, 16, 31, 47):
        check_seen(m, v, cfg, w, {"size": window - 1, "keep_first": keep} if window > 1 else None, j, j + window - 1, dtype)
        check_seen(m, v, cfg, w, {"size": window + 1, "keep_first": keep}, j, j + window, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("keep", (1, 3, 15, 16, 17, 40))
def test_edge_of_the_kept_tokens(backend, keep, dtype):
    """The last kept token and the first that is not, asked for from beyond the window: near it, pages away, tiles away."""
    cfg, w = edge_model(12, keep)
    m, v = make(backend, cfg, w, dtype, pool=4096, rows=1024), S.values(w)
    for i in (keep + 12, keep + 13, keep + 40, keep + 150, 300):
        check_seen(m, v, cfg, w, {"size": 12, "keep_first": keep - 1}, keep - 1, i, dtype)
        check_seen(m, v, cfg, w, {"size": 12, "keep_first": keep + 1}, keep, i, dtype)
        check_seen(m, v, cfg, w, {"size": 12, "keep_first": 0}, 0, i, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_at_the_edge_of_a_long_window(backend, dtype):
    """Hundreds of keys between question and key: decoding shares them among the CTAs of a cluster."""
    cfg, w = edge_model(460, 4)
    m, v = make(backend, cfg, w, dtype, pool=4096, rows=1024), S.values(w)
    for j in (4, 17):
        check_seen(m, v, cfg, w, {"size": 459, "keep_first": 4}, j, j + 459, dtype)
        check_seen(m, v, cfg, w, {"size": 461, "keep_first": 4}, j, j + 460, dtype)
    check_seen(m, v, cfg, w, {"size": 460, "keep_first": 3}, 3, 600, dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sink", (-30.0, 0.0, 9.0, 60.0))
def test_sinks(backend, sink, dtype):
    """Sinks far below, among and far above the scores."""
    cfg = S.config([S.window(size=40, keep=2, scale=0.5)])
    w, toks = S.weights(cfg, 74, gain=2.0), S.tokens(cfg, 140, 75)
    w["l0.mix.sink"] = S.bf16_bits([sink, 0.0, sink + 1.0, -sink])
    want = P.forward(cfg, S.values(w), toks)[0]
    m = make(backend, cfg, w, dtype)
    for cuts in ((), (70,), range(100, 140), (3, 50)):
        assert error(run(m, m.new_kv_cache(160), toks, cuts), want) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("softcap", (0.05, 2.0, 50.0, 3000.0))
def test_soft_caps(backend, softcap, dtype):
    """From caps that flatten every score to caps nobody reaches; scores up to hundreds."""
    cfg = S.config([S.beside(softcap=softcap, scale=1.0)])
    w, toks = S.weights(cfg, 76, gain=3.0), S.tokens(cfg, 140, 77)
    want = P.forward(cfg, S.values(w), toks)[0]
    m = make(backend, cfg, w, dtype)
    tol = TOL[dtype] * (3 if dtype == "bfloat16" and softcap > 10 else 1)  # scores this large turn a rounded query into another weight
    for cuts in ((), (70,), range(100, 140)):
        assert error(run(m, m.new_kv_cache(160), toks, cuts), want) < tol
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key_of_a_capped_layer(backend, dtype):
    """One key hundreds of positions away, whose capped score stands out."""
    cfg = S.config([S.beside(heads=2, kv_heads=1, rot_dims=2, softcap=9.0, right=0.1)])
    w = S.weights(cfg, 78, gain=8.0)
    v = S.values(w)
    part, mx = P.part(v, "l0.mix.left."), cfg["layers"][0]["mixer"]["left"]
    h = P.norm(v["embed"], v["l0.norm1"], cfg["norm"]["eps"])
    s = (h @ part["q"].T)[:, 2:24] @ (h @ part["k"].T)[:, 2:24].T * mx["scale"]
    qt, filler = np.unravel_index(np.argmax(s.max(1)[:, None] - s), s.shape)
    kt = int(np.argmax(s[qt]))
    m = make(backend, cfg, w, dtype, pool=4096, rows=1024)
    for j, i in ((0, 640), (15, 641), (255, 700)):
        toks = [int(filler)] * (i + 1)
        without = P.forward(cfg, v, toks[:i] + [int(qt)])[0]
        toks[j], toks[i] = kt, int(qt)
        want = P.forward(cfg, v, toks)[0]
        assert error(without[i:], want[i:]) > 0.2
        for cuts in ((), (i,), (j + 1, i - 1)):
            kv = m.new_kv_cache(1024, paged=True)
            assert error(run(m, kv, toks, cuts)[i:], want[i:]) < TOL[dtype]
            kv.truncate(0)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ("space", "time"))
def test_far_token_through_a_state(backend, kind, dtype):
    """Slow decays: the first token still shows hundreds of tokens later, however the sequence is cut."""
    cfg = S.config([S.space(state=16) if kind == "space" else S.beside(left=0.05, time_dim=24)])
    w = S.weights(cfg, 81)
    if kind == "space":
        w["l0.mix.A_log"], w["l0.mix.dt_bias"] = S.bf16_bits(np.full(6, -9.0)), S.bf16_bits(np.full(6, -1.0))
    else:
        w["l0.mix.right.w0"] = S.bf16_bits(np.full(72, -9.0))
    v = S.values(w)
    toks = [5] + [7] * 400 + S.tokens(cfg, 3, 82)
    want = P.forward(cfg, v, toks)[0]
    assert error(P.forward(cfg, v, [6] + toks[1:])[0][-3:], want[-3:]) > (2e-3 if kind == "space" else 1e-4)
    m = make(backend, cfg, w, dtype)
    for cuts in ((), (1,), (2, 66, 131, 402), tuple(range(350, 404))):
        assert error(run(m, m.new_kv_cache(416), toks, cuts)[-3:], want[-3:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_extreme_decays(backend, dtype):
    """Decays that forget within a token beside ones that never do: nothing overflows, in portions of any kind."""
    cfg = S.config([S.space(heads=4, groups=2, norm_groups=1), S.beside(time_dim=16)])
    w, toks = S.weights(cfg, 84), S.tokens(cfg, 200, 85)
    w["l0.mix.A_log"], w["l0.mix.dt_bias"] = S.bf16_bits([5.0, -12.0, 3.0, 0.0]), S.bf16_bits([4.0, 3.0, -20.0, 30.0])
    w["l1.mix.right.w0"] = S.bf16_bits(np.tile([6.0, -14.0, 0.0, 3.0], 12))
    want = P.forward(cfg, S.values(w), toks)[0]
    m = make(backend, cfg, w, dtype)
    for cuts in ((), (64, 129, 131), range(150, 200)):
        assert error(run(m, m.new_kv_cache(256), toks, cuts), want) < TOL[dtype]
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
    from orangu_b200.layered import LayeredModel
    from orangu_b200.senuvik import SenuvikModel

    init = LayeredModel.__init__

    def description(change):
        def changed(self, be, desc, blocks):
            change(blocks)
            init(self, be, desc, blocks)

        LayeredModel.__init__ = changed
        try:
            SenuvikModel(backend, MIX, S.weights(MIX, 121), kv_pool_tokens=64, max_seq_len=64, state_slots=2).close()
        finally:
            LayeredModel.__init__ = init

    description(lambda b: None)
    empty = capi.MatrixDesc()
    for change, message in (
        (lambda b: setattr(b[0].mixer, "n_map", 2), "one map"),
        (lambda b: setattr(b[0].mixer, "k_norm", None), "norm missing"),
        (lambda b: setattr(b[0].mixer, "wk", empty), "wk"),
        (lambda b: setattr(b[3].mixer, "kv_layer", 4), "earlier layer"),
        (lambda b: setattr(b[3].mixer, "kv_layer", 3), "other ones"),
        (lambda b: setattr(b[3].mixer, "wk", b[0].mixer.wk), "of its own"),
        (lambda b: setattr(b[2].mixer, "n_group", 4), "n_group"),
        (lambda b: setattr(b[2].mixer, "n_norm_group", 5), "n_norm_group"),
        (lambda b: setattr(b[2].mixer, "conv_taps", 17), "taps"),
        (lambda b: setattr(b[2].mixer, "dim", 300), "256"),
        (lambda b: setattr(b[2].mixer, "a_log", None), "vectors missing"),
        (lambda b: setattr(b[1].mixer2, "vdim", 4), "keys' size"),
        (lambda b: setattr(b[1].mixer2, "bonus", None), "vectors missing"),
        (lambda b: setattr(b[1].mixer2, "kind", capi.MIXER_ATTENTION), "two mixers"),
        (lambda b: setattr(b[1].mixer2, "w_decay1", empty), "w_decay1"),
        (lambda b: setattr(b[1], "pre_norm1", None), "normed inputs"),
        (lambda b: setattr(b[1], "pre_norm2", None), "norm of the feed-forward"),
        (lambda b: setattr(b[1], "w_gate", empty), "ff gate"),
        (lambda b: setattr(b[0], "router_softmax", 0), "weighted outputs"),
        (lambda b: setattr(b[0], "w_shared_scale", empty), "shared expert"),
    ):
        with pytest.raises(OranguError, match=message):
            description(change)
