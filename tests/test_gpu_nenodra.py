"""Nenodra on the GPU against the plain statement (nenodra_plain.py): mechanisms alone, prompts, portions, batches, pages that are
used again, far keys and window edges, long decoding, generation through the scheduler."""
import json

import numpy as np
import pytest

import nenodra_make as N
import nenodra_plain as P
from gpu_common import backend, error, greedy_plain, run  # noqa: F401

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")
TOL = {"float32": 3e-5, "bfloat16": 4e-2}  # of the logits' spread


def make(backend, cfg, w, dtype, pool=512, rows=256, seq=None):
    from orangu_b200.nenodra import NenodraModel

    return NenodraModel(backend, cfg, w, dtype=dtype, max_seq_len=seq or pool, max_batch_tokens=rows, kv_pool_tokens=pool)


# ---- mechanisms ------------------------------------------------------------------------------------------------------------
ALONE = {
    "differential": N.config([N.differential()]),
    "differential, one head, window of one": N.config([N.differential(heads=1, kv_heads=1, dim=8, vdim=8, window=1, rot_dims=2)]),
    "differential, one key head": N.config([N.differential(heads=5, kv_heads=1, dim=34, vdim=50, window=23, rot_dims=34)]),
    "differential, window past the sequence": N.config([N.differential(heads=4, kv_heads=4, dim=64, vdim=128, window=400, rot_dims=32)]),
    "differential, wide values": N.config([N.differential(heads=2, kv_heads=1, dim=40, vdim=150, window=37, rot_dims=40)]),
    "differential, widest values": N.config([N.differential(heads=2, kv_heads=2, dim=128, vdim=256, window=29, rot_dims=64)]),
    "differential, odd values": N.config([N.differential(heads=6, kv_heads=2, dim=22, vdim=27, window=33, rot_dims=4)]),
    "differential, beyond the tensor-core kernels": N.config([N.differential(heads=2, kv_heads=1, dim=16, vdim=264, rot_dims=16)]),
    "gated": N.config([N.gated()]),
    "gated, equal heads": N.config([N.gated(heads=3, kv_heads=3, dim=16, window=2, rot_dims=8)]),
    "gated, many heads on one key head": N.config([N.gated(heads=37, kv_heads=1, dim=18, window=21, rot_dims=18)]),
    "gated, sizes of a large model": N.config([N.gated(heads=8, kv_heads=2, dim=128, window=50, rot_dims=128)], width=256),
    "gated, odd": N.config([N.gated(heads=4, kv_heads=2, dim=75, window=19, rot_dims=10)]),
    "gated, wide": N.config([N.gated(heads=2, kv_heads=1, dim=250, window=45, rot_dims=100)]),
    "gated, beyond the tensor-core kernels": N.config([N.gated(heads=2, kv_heads=1, dim=264, window=31)]),
    "squared relu": N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.dense(250)),
    "one expert of twelve": N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.experts(12, 1, 44)),
    "three experts of four": N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.experts(4, 3, 60)),
    "five experts of forty": N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.experts(40, 5, 7)),
    "all experts": N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.experts(2, 2, 130)),
    "only expert": N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.experts(1, 1, 33)),
    "everything": N.config([N.differential(), N.gated(), N.gated(heads=2, kv_heads=1), N.differential(heads=2, window=7)],
                           ff=[N.experts(5, 2, 36), N.dense(72), N.experts(9, 1, 50), None]),
    "everything, other widths": N.config([N.gated(heads=4, kv_heads=1, window=9), N.differential(heads=5, kv_heads=5, window=19, diff=0.8)],
                                         ff=[N.dense(33), N.experts(6, 4, 90)], width=202, vocab=150, eps=0.03, mult=1.0, logit_scale=1.0),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_mechanism(backend, name, dtype):
    cfg = ALONE[name]
    w, toks = N.weights(cfg, 11), N.tokens(cfg, 75, 12)
    want, hidden = P.forward(cfg, N.values(w), toks)
    m = make(backend, cfg, w, dtype)
    kv = m.new_kv_cache(128)
    got = run(m, kv, toks)
    assert error(m.last_hidden(75), hidden[-1]) < TOL[dtype]
    assert error(got, want) < TOL[dtype]
    # the same tokens one by one, and in portions
    one = m.new_kv_cache(128)
    assert error(run(m, one, toks, range(1, 75)), want) < TOL[dtype]
    cut = m.new_kv_cache(128)
    assert error(run(m, cut, toks, (2, 5, 16, 18, 33, 34, 64)), want) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_rows_per_expert(backend, dtype):
    """Enough pairs and rows for the widest tiles of the grouped products, and the logits of the router as a product."""
    cfg = N.config([N.gated(heads=1, kv_heads=1, dim=4, window=1, rot_dims=4)], ff=N.experts(3, 2, 2200), width=64)
    w, toks = N.weights(cfg, 15), N.tokens(cfg, 560, 16)
    want, _ = P.forward(cfg, N.values(w), toks)
    m = make(backend, cfg, w, dtype, pool=1024, rows=600)
    assert error(run(m, m.new_kv_cache(600), toks), want) < TOL[dtype]
    m.close()


def test_cache_holds_what_the_design_says(backend):
    cfg = N.config([N.differential(), N.gated()])
    w, toks = N.weights(cfg, 21), N.tokens(cfg, 30, 22)
    v, eps = N.values(w), cfg["norm"]["eps"]
    m = make(backend, cfg, w, "float32")
    kv = m.new_kv_cache(64)
    run(m, kv, toks, (17,))
    x = v["embed"][toks]
    for layer, maps in ((0, 2), (1, 1)):
        k, val = kv.read(layer, 0, 30)
        part, mx = P.part(v, f"l{layer}.mix."), cfg["layers"][layer]["mixer"]
        kp = x @ part["k"].T + part.get("k.b", 0.0)
        want_k = P.normed_rotated(kp.reshape(30, mx["kv_heads"], maps, mx["dim"]), part["k.norm"], mx, eps)
        assert error(k, want_k.reshape(30, -1)) < 1e-5
        assert error(val, x @ part["v"].T + part["v.b"] if layer == 0 else kp) < 1e-5
        x = P.forward({**cfg, "layers": cfg["layers"][:1]}, v, toks)[1][0]
    m.close()


# ---- batches, pages ------------------------------------------------------------------------------------------------------------
MIX = N.config([N.differential(window=13), N.gated(window=30), N.differential(heads=2, kv_heads=1, window=23)],
               ff=[N.experts(6, 2, 40), N.dense(104), N.experts(5, 1, 72)])


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch(backend, dtype):
    """Portions of prompts beside single tokens; every request's logits are those it has alone."""
    w = N.weights(MIX, 31)
    prompts = [N.tokens(MIX, n, 32 + n) for n in (90, 41, 67, 3)]
    want = [P.forward(MIX, N.values(w), p)[0] for p in prompts]
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
@pytest.mark.parametrize("window", (1, 37, 90, 400))
def test_long_portions(backend, window, dtype):
    """Portions long enough for the attention of prompts, started anywhere, beside short ones and single tokens."""
    cfg = N.config([N.differential(window=window, dim=40, vdim=18), N.gated(window=window, heads=6, kv_heads=1, dim=72, rot_dims=24)], ff=[N.dense(40), N.experts(4, 2, 24)])
    w = N.weights(cfg, 36, gain=2.0)
    prompts = [N.tokens(cfg, n, 37 + n) for n in (230, 165, 131)]
    want = [P.forward(cfg, N.values(w), p)[0] for p in prompts]
    m = make(backend, cfg, w, dtype, pool=1024, rows=512)
    kvs = [m.new_kv_cache(256, paged=True) for _ in prompts]
    got = [[] for _ in prompts]
    at = [0, 0, 0]
    for sizes in ((3, 70, 64), (65, 1, 0), (1, 64, 66), (64, 30, 1), (97, 0, 0)):
        live = [i for i in range(3) if sizes[i]]
        lg = m.forward_rows([kvs[i] for i in live], [prompts[i][at[i]:at[i] + sizes[i]] for i in live], range(sum(sizes)))
        o = 0
        for i in live:
            got[i].append(lg[o:o + sizes[i]])
            at[i] += sizes[i]
            o += sizes[i]
    assert at == [230, 165, 131]
    for g, x in zip(got, want):
        assert error(np.concatenate(g), x) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_prompts_and_single_tokens_in_one_step(backend, dtype):
    """More spans than a warp looks through at once, some long, more tokens than a step."""
    cfg = N.config([N.differential(window=50), N.gated(heads=3, kv_heads=1, dim=32, rot_dims=32, window=20)], ff=[N.experts(8, 2, 16), None])
    w = N.weights(cfg, 46)
    prompts = [N.tokens(cfg, 66 + i if i % 4 == 0 else 1 + i % 7, 47 + i) for i in range(44)]
    m = make(backend, cfg, w, dtype, pool=4096, rows=700, seq=128)
    kvs = [m.new_kv_cache(128, paged=True) for _ in prompts]
    ends = np.cumsum([len(p) for p in prompts]) - 1
    lg = m.forward_rows(kvs, prompts, ends)
    nxt = m.forward_batch_decode(kvs, [p[0] for p in prompts], want_logits=True)[1]
    for i in (0, 1, 4, 5, 12, 31, 36, 40, 42, 43):
        want = P.forward(cfg, N.values(w), prompts[i] + prompts[i][:1])[0]
        assert error(np.stack([lg[i], nxt[i]]), want[-2:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("kind", ("differential", "gated"))
def test_more_pieces_of_prompts_than_processors(backend, kind):
    """One long prompt, then many short ones (with one map every second stream of rows is empty), on sixteen key/value heads: every
    CTA of the prompt attention takes several pieces."""
    layer = N.differential(heads=16, kv_heads=16, dim=16, vdim=24, window=150, rot_dims=16) if kind == "differential" else N.gated(heads=32, kv_heads=16, dim=24, window=150, rot_dims=16)
    cfg = N.config([layer], width=64)
    w = N.weights(cfg, 48)
    long, short = N.tokens(cfg, 1500, 49), [N.tokens(cfg, 64 + i % 9, 50 + i) for i in range(13)]
    m = make(backend, cfg, w, "bfloat16", pool=4096, rows=2048, seq=2048)
    want = P.forward(cfg, N.values(w), long)[0]
    places = list(range(0, 1500, 7)) + [1499]
    assert error(m.forward_rows([m.new_kv_cache(1536, paged=True)], [long], places), want[places]) < TOL["bfloat16"]
    kvs = [m.new_kv_cache(96, paged=True) for _ in short]
    ends = np.cumsum([len(p) for p in short]) - 1
    got = m.forward_rows(kvs, short, ends)
    for g, p in zip(got, short):
        assert error(g[None], P.forward(cfg, N.values(w), p)[0][-1:]) < TOL["bfloat16"]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_single_tokens(backend, dtype):
    """A decode batch wide enough for the tensor-core products, at unequal lengths."""
    w = N.weights(MIX, 41)
    seqs = [N.tokens(MIX, 5 + 3 * i, 42 + i) for i in range(9)]
    m = make(backend, MIX, w, dtype, pool=1024)
    kvs = [m.new_kv_cache(64) for _ in seqs]
    m.forward_rows(kvs, [s[:-2] for s in seqs], [])
    first = m.forward_rows(kvs, [[s[-2]] for s in seqs], range(9))
    toks, second = m.forward_batch_decode(kvs, [s[-1] for s in seqs], want_logits=True)
    for i, s in enumerate(seqs):
        want = P.forward(MIX, N.values(w), s)[0]
        assert error(np.stack([first[i], second[i]]), want[-2:]) < TOL[dtype]
        assert toks[i] == np.argmax(second[i])
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_are_used_again(backend, dtype):
    from orangu_b200 import OranguError

    w = N.weights(MIX, 51)
    m = make(backend, MIX, w, dtype, pool=96)
    assert m.free_pages == 6 and m.free_slots == 0  # nothing recurrent
    a, b, c = (m.new_kv_cache(96, paged=True) for _ in range(3))
    x, y, z = (N.tokens(MIX, n, 52 + n) for n in (50, 20, 70))
    run(m, a, x)
    run(m, b, y)
    assert m.free_pages == 0
    with pytest.raises(OranguError, match="pool exhausted"):
        m.forward_rows([c], [z[:5]], [])
    a.truncate(0)
    assert m.free_pages == 4
    want_z, want_y = P.forward(MIX, N.values(w), z)[0], P.forward(MIX, N.values(w), y + z[:12])[0]
    # the third sequence on the first one's pages, beside the second, which goes on
    got_z = [m.forward_rows([c, b], [z[:40], z[:1]], range(41))]
    got_y = [got_z[0][40:]]
    got_z[0] = got_z[0][:40]
    for i in range(1, 12):
        lg = m.forward_rows([b, c], [[z[i]], z[39 + i:40 + i]], range(2))
        got_y.append(lg[:1])
        got_z.append(lg[1:])
    assert error(np.concatenate(got_z), want_z[:51]) < TOL[dtype] and error(np.concatenate(got_y), want_y[20:]) < TOL[dtype]
    # rolled back to the middle of a page and on with other tokens
    b.truncate(21)
    assert error(run(m, b, x[:3]), P.forward(MIX, N.values(w), y + z[:1] + x[:3])[0][21:]) < TOL[dtype]
    for kv in (b, c):
        kv.truncate(0)
    assert m.free_pages == 6
    m.close()


def test_copy_of_a_prefix_goes_its_own_way(backend):
    w = N.weights(MIX, 61)
    x, y, z = N.tokens(MIX, 37, 62), N.tokens(MIX, 9, 63), N.tokens(MIX, 9, 64)
    m = make(backend, MIX, w, "float32")
    a, b = m.new_kv_cache(64), m.new_kv_cache(64, paged=True)
    run(m, a, x)
    b.copy_prefix_from(a, 20)
    assert error(run(m, a, y), P.forward(MIX, N.values(w), x + y)[0][37:]) < 3e-5
    assert error(run(m, b, z), P.forward(MIX, N.values(w), x[:20] + z)[0][20:]) < 3e-5
    m.close()


# ---- far keys, window edges ------------------------------------------------------------------------------------------------------
def edge_model(kind, window):
    """One layer in which single keys stand out: large query norms, and no score in the entries that rotate."""
    layer = N.differential(heads=2, kv_heads=1, window=window, rot_dims=8, diff=0.2) if kind == "differential" else N.gated(heads=2, kv_heads=1, window=window, rot_dims=8)
    cfg = N.config([layer])
    w = N.weights(cfg, 71, gain=6.0)
    q = N.bf16_values(w["l0.mix.q.norm"])
    q[:8] = 0.0
    w["l0.mix.q.norm"] = N.bf16_bits(q)
    return cfg, w


def standing_out(cfg, w):
    """Tokens (query, key, filler): the query's score with the key is far above its score with the filler (first map of the first
    head), so that whether the key is seen decides that head's output."""
    v, mx = N.values(w), cfg["layers"][0]["mixer"]
    part, D, eps = P.part(v, "l0.mix."), mx["dim"], cfg["norm"]["eps"]
    q = (v["embed"] @ part["q"].T + part.get("q.b", 0.0))[:, :D]
    k = (v["embed"] @ part["k"].T + part.get("k.b", 0.0))[:, :D]
    s = (P.over_rms(q, eps) * part["q.norm"]) @ (P.over_rms(k, eps) * part["k.norm"]).T * mx["scale"]
    best = np.unravel_index(np.argmax(s.max(1)[:, None] - s), s.shape)  # query row and its worst key: the filler
    return int(best[0]), int(np.argmax(s[best[0]])), int(best[1])


def check_edge(backend, kind, window, places, dtype):
    cfg, w = edge_model(kind, window)
    qt, kt, filler = standing_out(cfg, w)
    mx = cfg["layers"][0]["mixer"]
    other = {d: {**cfg, "layers": [{**cfg["layers"][0], "mixer": {**mx, "mask": {"size": window + d}}}]} for d in (-1, 1)}
    v = N.values(w)
    m = make(backend, cfg, w, dtype, pool=4096, rows=1024)
    for j in places:
        for inside in (True, False):
            i = j + window - 1 if inside else j + window
            toks = [filler] * (i + 1)
            toks[j], toks[i] = kt, qt
            want = P.forward(cfg, v, toks)[0]
            if window > 1 or not inside:
                assert error(P.forward(other[-1 if inside else 1], v, toks)[0][i:], want[i:]) > 0.2
            whole, step, two, far = (m.new_kv_cache(1024, paged=True) for _ in range(4))
            assert error(run(m, whole, toks)[i:], want[i:]) < TOL[dtype]
            if i:
                assert error(run(m, step, toks, (i,))[i:], want[i:]) < TOL[dtype]
            assert error(run(m, two, toks, (j, i - 1) if i - 1 > j > 0 else (j,) if j else ())[i:], want[i:]) < TOL[dtype]
            longer = toks + [filler] * 70  # key and question at the start of long portions
            assert error(run(m, far, longer, tuple(c for c in sorted({j, i}) if c))[i:i + 1], want[i:]) < TOL[dtype]
            for kv in (whole, step, two, far):
                kv.truncate(0)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", (1, 3, 16, 17, 31, 64, 65))
@pytest.mark.parametrize("kind", ("differential", "gated"))
def test_window_edges(backend, kind, window, dtype):
    """A key just inside and just outside the window, at page borders and elsewhere, asked for in a prompt and while decoding.
    The plain statement with a window one longer or one shorter is far off, so a shifted edge could not pass."""
    check_edge(backend, kind, window, (0, 5, 15, 16, 31, 47), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ("differential", "gated"))
def test_far_key_at_the_edge_of_a_long_window(backend, kind, dtype):
    """Hundreds of keys between question and key: decoding shares them among the CTAs of a cluster."""
    check_edge(backend, kind, 460, (0, 17), dtype)


# ---- decoding ------------------------------------------------------------------------------------------------------------------------
def test_long_decoding(backend):
    """Hundreds of decoded tokens through captured graphs; the plain statement then judges every choice at once."""
    cfg = {**MIX, "layers": [MIX["layers"][0], {**MIX["layers"][1], "mixer": {**MIX["layers"][1]["mixer"], "mask": {"size": 200}}}, MIX["layers"][2]]}
    w = N.weights(cfg, 91)
    for dtype in DTYPES:
        m = make(backend, cfg, w, dtype, pool=1024)
        prompts = [N.tokens(cfg, n, 92 + n) for n in (18, 1)]
        kvs = [m.new_kv_cache(512, paged=True) for _ in prompts]
        first = [m.forward_maybe_sampling(kv, p, 0) for kv, p in zip(kvs, prompts)]
        steps = m.decode_loop(kvs, first, 250)
        single = [m.decode_greedy(kvs[0], int(steps[-1, 0]))]
        for _ in range(20):
            single.append(m.decode_greedy(kvs[0], single[-1]))
        for i, p in enumerate(prompts):
            got = [first[i]] + steps[:, i].tolist() + (single if i == 0 else [])
            lg = P.forward(cfg, N.values(w), p + got[:-1])[0][len(p) - 1:]
            behind = lg.max(-1) - lg[np.arange(len(got)), got]  # a choice may differ only where the two are within rounding
            assert behind.max() < TOL[dtype] * np.sqrt((lg ** 2).mean())
        assert [len(kv) for kv in kvs] == [18 + 250 + 21, 1 + 250]
        m.close()


def test_generation_through_scheduler_and_files(backend, tmp_path):
    """A folder on disk, the registry, the slot pool with more prompts than fit one step, greedy tokens and repeat penalty."""
    from orangu_b200.__main__ import generate
    from orangu_b200.registry import load_model
    from orangu_b200.safetensors import save

    w = N.weights(MIX, 101)
    (tmp_path / "config.json").write_text(json.dumps(MIX))
    save(str(tmp_path / "model.safetensors"), w)
    m = load_model(backend, str(tmp_path), dtype="float32", max_seq_len=128, max_batch_tokens=32, kv_pool_tokens=512)
    prompts = [N.tokens(MIX, n, 102 + n) for n in (45, 2, 17, 33, 8)]
    got = generate(m, prompts, 12, prefill_batch=10)
    for p, g in zip(prompts, got):
        want, lead = greedy_plain(P, MIX, N.values(w), p, 12)
        assert lead > 1e-5 and g == want  # seeds chosen so that no two tokens tie within rounding
    assert m.free_pages == 32
    # repeat penalty: the penalised argmax of the logits without it
    p = prompts[0]
    a = generate(m, [p], 2, repeat_penalty=1.8, repeat_last_n=64)[0]
    lg = P.forward(MIX, N.values(w), p)[0][-1]
    seen = list(set(p))
    lg[seen] = np.where(lg[seen] > 0, lg[seen] / 1.8, lg[seen] * 1.8)
    assert a[0] == int(np.argmax(lg))
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(backend, tmp_path, dtype):
    """Requests that come, pause, end and make room for others; logits files in the order asked for."""
    from orangu_b200 import trace

    w = N.weights(MIX, 111)
    v = N.values(w)
    m = make(backend, MIX, w, dtype, pool=192, rows=192)
    t = {k: N.tokens(MIX, n, 112 + n) for k, n in (("a", 40), ("b", 64), ("c", 30), ("d", 5), ("e", 60))}
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

    class Made(Exception):
        pass

    def description(change):
        from orangu_b200.nenodra import NenodraModel

        kept = {}

        class Catch(NenodraModel):
            pass

        init = LayeredModel.__init__

        def catch(self, be, desc, blocks):
            change(desc, blocks)
            kept["ok"] = True
            init(self, be, desc, blocks)

        LayeredModel.__init__ = catch
        try:
            Catch(backend, MIX, N.weights(MIX, 121), kv_pool_tokens=64, max_seq_len=64).close()
        finally:
            LayeredModel.__init__ = init
        raise Made

    with pytest.raises(Made):
        description(lambda d, b: None)
    for change, message in (
        (lambda d, b: setattr(b[0].mixer, "n_kv_head", 3), "divide"),
        (lambda d, b: setattr(b[0].mixer, "n_map", 3), "maps"),
        (lambda d, b: setattr(b[1].mixer, "q_norm", None), "norm missing"),
        (lambda d, b: setattr(b[1].mixer, "scale", 0.0), "scale"),
        (lambda d, b: setattr(b[1].mixer, "vdim", 24), "wo|keys|gate"),
        (lambda d, b: setattr(b[1].mixer, "rot_dims", 42), "rot_dims"),
        (lambda d, b: setattr(b[1], "post_norm1", None), "two kinds"),
        (lambda d, b: setattr(b[1], "post_norm2", None), "norm of the feed-forward"),
        (lambda d, b: setattr(b[0], "n_expert_used", 7), "experts"),
        (lambda d, b: setattr(b[1], "ff_kind", capi.FF_CLAMPED_GLU), "unknown feed-forward"),
    ):
        with pytest.raises(OranguError, match=message):
            description(change)
