"""Fenipel on the GPU against the plain statement (fenipel_plain.py): mechanisms alone, prompts, portions, batches, pages and
slots that are used again, far keys and window edges, long decoding, generation through the scheduler."""
import json

import numpy as np
import pytest

import fenipel_make as F
import fenipel_plain as P
from gpu_common import backend, error, greedy_plain, run  # noqa: F401

pytestmark = pytest.mark.gpu
DTYPES = ("float32", "bfloat16")
TOL = {"float32": 3e-5, "bfloat16": 4e-2}  # of the logits' spread


def make(backend, cfg, w, dtype, pool=512, rows=256, slots=4, seq=None):
    from orangu_b200.fenipel import FenipelModel

    return FenipelModel(backend, cfg, w, dtype=dtype, max_seq_len=seq or pool, max_batch_tokens=rows, kv_pool_tokens=pool, state_slots=slots)


# ---- mechanisms ------------------------------------------------------------------------------------------------------------
ALONE = {
    "latent": F.config([F.latent()], ff=None, side=0),
    "latent, one head, window of one": F.config([F.latent(heads=1, window=1, dim=8, rot_dim=2, vdim=8, kv_rank=8)], ff=None, side=0),
    "latent, window past the sequence": F.config([F.latent(window=400, dim=80, rot_dim=32, vdim=64, kv_rank=48)], ff=None, side=0),
    "latent, wide": F.config([F.latent(heads=20, window=37, dim=72, rot_dim=40, vdim=56, kv_rank=328)], ff=None, side=0),
    "latent, sizes of a large model": F.config([F.latent(heads=32, window=50, dim=128, rot_dim=64, vdim=128, kv_rank=512)], width=256, ff=None, side=0),
    "latent, beyond the tensor-core kernel": F.config([F.latent(heads=2, window=21, kv_rank=560)], ff=None, side=0),
    "retention": F.config([F.retention()], ff=None, side=0),
    "retention, everything rotates": F.config([F.retention(heads=2, dim=72, vdim=48, rot_dims=72)], ff=None, side=0),
    "retention, 128": F.config([F.retention(heads=5, dim=112, vdim=72, rot_dims=112)], ff=None, side=0),
    "retention, 256": F.config([F.retention(heads=1, dim=250, vdim=130, rot_dims=12, decay=[0.99])], ff=None, side=0),
    "feed-forward": F.config([F.retention(heads=1, dim=2, vdim=2, rot_dims=2)], ff=250, limit=0.35, side=0),
    "token input": F.config([F.retention(heads=1, dim=2, vdim=2, rot_dims=2)], ff=None, side=30),
    "everything": F.config([F.latent(), F.retention(), F.retention(heads=2), F.latent(heads=4, window=7)], ff=[40, None, 104, 64]),
    "everything, other widths": F.config([F.retention(heads=4), F.latent(heads=5, window=19)], width=200, vocab=150, side=7, ff=[33, 90], eps=0.03),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ALONE)
def test_mechanism(backend, name, dtype):
    cfg = ALONE[name]
    w, toks = F.weights(cfg, 11), F.tokens(cfg, 75, 12)
    want, hidden = P.forward(cfg, F.values(w), toks)
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


def test_cache_and_state_hold_what_the_design_says(backend):
    cfg = F.config([F.latent(), F.retention()], ff=None)
    w, toks = F.weights(cfg, 21), F.tokens(cfg, 30, 22)
    v = F.values(w)
    m = make(backend, cfg, w, "float32")
    kv = m.new_kv_cache(64)
    run(m, kv, toks, (17,))
    c, kr = kv.read(0, 0, 30)
    part, mx = P.part(v, "l0.mix."), cfg["layers"][0]["mixer"]
    h = P.over_rms(v["embed"][toks], cfg["norm"]["eps"]) * v["l0.norm1"]
    dkv = h @ part["dkv"].T
    want_c = P.over_rms(dkv[:, :40], cfg["norm"]["eps"]) * part["dkv.norm"]
    want_r = np.stack([P.rotate(dkv[p, 40:], p, mx["rot"]["base"], 16, True) for p in range(30)])
    assert error(c, want_c) < 1e-5 and error(kr, want_r) < 1e-5
    _, hidden = P.forward({**cfg, "layers": cfg["layers"][:1]}, {**v, "side.embed": v["side.embed"][:, :12]}, toks)
    h1 = P.over_rms(hidden[-1], cfg["norm"]["eps"]) * v["l1.norm1"]
    _, S = P.retention(h1, P.part(v, "l1.mix."), cfg["layers"][1]["mixer"], cfg["norm"]["eps"])
    got = kv.read_state(1)
    assert np.abs(got - S).max() < 2e-5 * np.abs(S).max()
    m.close()


# ---- batches, pages, slots ---------------------------------------------------------------------------------------------------
MIX = F.config([F.latent(window=13), F.retention(), F.latent(heads=4, window=23)], ff=[104, 40, 72])


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_in_one_batch(backend, dtype):
    """Portions of prompts beside single tokens; every request's logits are those it has alone."""
    w = F.weights(MIX, 31)
    prompts = [F.tokens(MIX, n, 32 + n) for n in (90, 41, 67, 3)]
    want = [P.forward(MIX, F.values(w), p)[0] for p in prompts]
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
    """Portions long enough for the per-head attention of prompts, started anywhere, beside short ones and single tokens."""
    cfg = F.config([F.latent(window=window, dim=40, vdim=18), F.retention(), F.latent(heads=2, window=window, dim=16, rot_dim=8, vdim=72, kv_rank=24)], ff=[40, 40, None])
    w = F.weights(cfg, 36, gain=2.0)
    prompts = [F.tokens(cfg, n, 37 + n) for n in (230, 165, 131)]
    want = [P.forward(cfg, F.values(w), p)[0] for p in prompts]
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
def test_many_prompts_in_one_step(backend, dtype):
    """More long portions than one launch of the prompt attention takes, and more tokens than a step."""
    cfg = F.config([F.latent(window=50)], ff=None)
    w = F.weights(cfg, 46)
    prompts = [F.tokens(cfg, 66 + i, 47 + i) for i in range(11)]
    m = make(backend, cfg, w, dtype, pool=2048, rows=700, seq=128)
    kvs = [m.new_kv_cache(128, paged=True) for _ in prompts]
    ends = np.cumsum([len(p) for p in prompts]) - 1
    lg = m.forward_rows(kvs, prompts, ends)
    for g, p in zip(lg, prompts):
        want = P.forward(cfg, F.values(w), p)[0]
        assert error(g[None], want[-1:]) < TOL[dtype]
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_single_tokens(backend, dtype):
    """A decode batch wide enough for the tensor-core products, at unequal lengths."""
    w = F.weights(MIX, 41)
    seqs = [F.tokens(MIX, 5 + 3 * i, 42 + i) for i in range(9)]
    m = make(backend, MIX, w, dtype, pool=1024, slots=9)
    kvs = [m.new_kv_cache(64) for _ in seqs]
    m.forward_rows(kvs, [s[:-2] for s in seqs], [])
    first = m.forward_rows(kvs, [[s[-2]] for s in seqs], range(9))
    toks, second = m.forward_batch_decode(kvs, [s[-1] for s in seqs], want_logits=True)
    for i, s in enumerate(seqs):
        want = P.forward(MIX, F.values(w), s)[0]
        assert error(np.stack([first[i], second[i]]), want[-2:]) < TOL[dtype]
        assert toks[i] == np.argmax(second[i])
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_and_slots_are_used_again(backend, dtype):
    from orangu_b200 import OranguError

    w = F.weights(MIX, 51)
    m = make(backend, MIX, w, dtype, pool=96, slots=2)
    pages, slots = m.free_pages, m.free_slots
    assert (pages, slots) == (6, 2)
    a, b, c = (m.new_kv_cache(96, paged=True) for _ in range(3))
    x, y, z = (F.tokens(MIX, n, 52 + n) for n in (50, 20, 70))
    run(m, a, x)
    run(m, b, y)
    assert (m.free_pages, m.free_slots) == (0, 0)
    with pytest.raises(OranguError, match="pool exhausted"):
        m.forward_rows([c], [z[:5]], [])
    a.truncate(0)
    assert (m.free_pages, m.free_slots) == (4, 1)
    want_z, want_y = P.forward(MIX, F.values(w), z)[0], P.forward(MIX, F.values(w), y + z[:12])[0]
    # the third sequence on the first one's pages and slot, beside the second, which goes on
    got_z = [m.forward_rows([c, b], [z[:40], z[:1]], range(41))]
    got_y = [got_z[0][40:]]
    got_z[0] = got_z[0][:40]
    with pytest.raises(OranguError, match="free state slot"):
        m.forward_rows([a], [x[:2]], [])
    for i in range(1, 12):
        lg = m.forward_rows([b, c], [[z[i]], z[39 + i:40 + i]], range(2))
        got_y.append(lg[:1])
        got_z.append(lg[1:])
    assert error(np.concatenate(got_z), want_z[:51]) < TOL[dtype] and error(np.concatenate(got_y), want_y[20:]) < TOL[dtype]
    with pytest.raises(OranguError, match="rolled back"):
        b.truncate(3)
    for kv in (b, c):
        kv.truncate(0)
    assert (m.free_pages, m.free_slots) == (pages, slots)
    m.close()


def test_copy_of_a_sequence_goes_its_own_way(backend):
    from orangu_b200 import OranguError

    w = F.weights(MIX, 61)
    x, y, z = F.tokens(MIX, 37, 62), F.tokens(MIX, 9, 63), F.tokens(MIX, 9, 64)
    m = make(backend, MIX, w, "float32")
    a, b = m.new_kv_cache(64), m.new_kv_cache(64, paged=True)
    run(m, a, x)
    with pytest.raises(OranguError, match="copied whole"):
        b.copy_prefix_from(a, 20)
    b.copy_prefix_from(a, 37)
    assert error(run(m, a, y), P.forward(MIX, F.values(w), x + y)[0][37:]) < 3e-5
    assert error(run(m, b, z), P.forward(MIX, F.values(w), x + z)[0][37:]) < 3e-5
    m.close()


# ---- far keys, window edges ------------------------------------------------------------------------------------------------------
def standing_out(cfg, w):
    """Tokens (query, key, filler): in the first layer the query's score with the key is far above its score with the filler,
    so that whether the key is seen decides the output.  Rotation is slow (base) and left out here."""
    v, mx = F.values(w), cfg["layers"][0]["mixer"]
    part = P.part(v, "l0.mix.")
    h = P.over_rms(v["embed"], cfg["norm"]["eps"]) * v["l0.norm1"]
    H, D, R, K = mx["heads"], mx["dim"], mx["rot_dim"], mx["kv_rank"]
    q = (h @ part["q"].T).reshape(-1, H, D + R)[:, 0, :D]
    c = P.over_rms((h @ part["dkv"].T)[:, :K], cfg["norm"]["eps"]) * part["dkv.norm"]
    s = q @ (c @ part["uk"].T).reshape(-1, H, D)[:, 0].T * mx["scale"]
    best = np.unravel_index(np.argmax(s.max(1)[:, None] - s), s.shape)  # query row and its worst key: the filler
    qt, filler = int(best[0]), int(best[1])
    return qt, int(np.argmax(s[qt])), filler


EDGE_WINDOWS = (3, 16, 17, 31, 64, 65)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", EDGE_WINDOWS)
def test_window_edges(backend, window, dtype):
    """A key just inside and just outside the window, at page borders and elsewhere, asked for in a prompt and while decoding.
    The plain statement with a window one longer or one shorter is far off, so a shifted edge could not pass."""
    cfg = F.config([F.latent(heads=2, window=window, base=1e9)], ff=None, side=0)
    w = F.weights(cfg, 71, gain=6.0)
    qt, kt, filler = standing_out(cfg, w)
    other = {d: {**cfg, "layers": [{**cfg["layers"][0], "mixer": {**cfg["layers"][0]["mixer"], "mask": {"size": window + d}}}]} for d in (-1, 1)}
    v = F.values(w)
    for j in (5, 15, 16, 31, 47):
        for inside in (True, False):
            i = j + window - 1 if inside else j + window
            toks = [filler] * (i + 1)
            toks[j], toks[i] = kt, qt
            want = P.forward(cfg, v, toks)[0]
            wrong = P.forward(other[-1 if inside else 1], v, toks)[0]
            assert error(wrong[i:], want[i:]) > 0.2
            m = make(backend, cfg, w, dtype, pool=1024)
            whole, step, two, far = (m.new_kv_cache(256, paged=True) for _ in range(4))
            assert error(run(m, whole, toks)[i:], want[i:]) < TOL[dtype]
            assert error(run(m, step, toks, (i,))[i:], want[i:]) < TOL[dtype]
            assert error(run(m, two, toks, (j, i - 1) if i - 1 > j else (j,))[i:], want[i:]) < TOL[dtype]
            longer = toks + [filler] * 70  # key and question at the start of long portions
            assert error(run(m, far, longer, (j, i))[i:i + 1], want[i:]) < TOL[dtype]
            m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_token_through_retention(backend, dtype):
    """The first token's trace in the state, hundreds of tokens later: without it the logits are far off."""
    cfg = F.config([F.retention(heads=2, dim=32, vdim=32, rot_dims=32, base=1e9, decay=[0.9995, 0.9999])], ff=None, side=0)
    w = F.weights(cfg, 81)
    v = F.values(w)
    # token 5 alone has a direction that the keys amplify, token 7 one that the queries turn into the same vector
    r, E = np.random.default_rng(83), cfg["width"]
    d5, d7 = np.linalg.qr(r.normal(size=(E, 2)))[0].T
    e = v["embed"] - np.outer(v["embed"] @ d5, d5) - np.outer(v["embed"] @ d7, d7)
    e[5], e[7] = d5, 0.01 * d7
    u = np.sign(r.normal(size=64))
    w.update({"embed": F.bf16_bits(e), "l0.mix.k": F.bf16_bits(v["l0.mix.k"] + np.outer(u, d5)), "l0.mix.q": F.bf16_bits(v["l0.mix.q"] + np.outer(u, d7))})
    toks = [5] + [8 + t % 60 for t in F.tokens(cfg, 330, 82)] + [7]
    v = F.values(w)
    want = P.forward(cfg, v, toks)[0]
    assert error(P.forward(cfg, v, toks[1:])[0][-1:], want[-1:]) > 0.2
    m = make(backend, cfg, w, dtype, pool=1024, seq=512)
    whole, parts = m.new_kv_cache(400, paged=True), m.new_kv_cache(400, paged=True)
    assert error(run(m, whole, toks)[-1:], want[-1:]) < TOL[dtype]
    assert error(run(m, parts, toks, (1, 3, 100, 260, 329, 331))[-1:], want[-1:]) < TOL[dtype]
    m.close()


# ---- decoding ------------------------------------------------------------------------------------------------------------------------
def test_long_decoding(backend):
    """Hundreds of decoded tokens through captured graphs; the plain statement then judges every choice at once."""
    w = F.weights(MIX, 91)
    for dtype in DTYPES:
        m = make(backend, MIX, w, dtype, pool=1024)
        prompts = [F.tokens(MIX, n, 92 + n) for n in (18, 1)]
        kvs = [m.new_kv_cache(512, paged=True) for _ in prompts]
        first = [m.forward_maybe_sampling(kv, p, 0) for kv, p in zip(kvs, prompts)]
        steps = m.decode_loop(kvs, first, 250)
        single = [m.decode_greedy(kvs[0], int(steps[-1, 0]))]
        for _ in range(20):
            single.append(m.decode_greedy(kvs[0], single[-1]))
        for i, p in enumerate(prompts):
            got = [first[i]] + steps[:, i].tolist() + (single if i == 0 else [])
            lg = P.forward(MIX, F.values(w), p + got[:-1])[0][len(p) - 1:]
            behind = lg.max(-1) - lg[np.arange(len(got)), got]  # a choice may differ only where the two are within rounding
            assert behind.max() < TOL[dtype] * np.sqrt((lg ** 2).mean())
        assert [len(kv) for kv in kvs] == [18 + 250 + 21, 1 + 250]
        m.close()


def test_generation_through_scheduler_and_files(backend, tmp_path):
    """A folder on disk, the registry, the slot pool with more prompts than fit one step, greedy tokens and repeat penalty."""
    from orangu_b200.__main__ import generate
    from orangu_b200.registry import load_model
    from orangu_b200.safetensors import save

    w = F.weights(MIX, 101)
    (tmp_path / "config.json").write_text(json.dumps(MIX))
    save(str(tmp_path / "model.safetensors"), w)
    m = load_model(backend, str(tmp_path), dtype="float32", max_seq_len=128, max_batch_tokens=32, kv_pool_tokens=512, state_slots=5)
    prompts = [F.tokens(MIX, n, 102 + n) for n in (45, 2, 17, 33, 8)]
    got = generate(m, prompts, 12, prefill_batch=10)
    for p, g in zip(prompts, got):
        want, lead = greedy_plain(P, MIX, F.values(w), p, 12)
        assert lead > 1e-4 and g == want  # seeds chosen so that no two tokens tie within rounding
    assert (m.free_pages, m.free_slots) == (32, 5)
    # repeat penalty: the penalised argmax of the logits without it
    p = prompts[0]
    a = generate(m, [p], 2, repeat_penalty=1.8, repeat_last_n=64)[0]
    lg = P.forward(MIX, F.values(w), p)[0][-1]
    seen = list(set(p))
    lg[seen] = np.where(lg[seen] > 0, lg[seen] / 1.8, lg[seen] * 1.8)
    assert a[0] == int(np.argmax(lg))
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay(backend, tmp_path, dtype):
    """Requests that come, pause, end and make room for others; logits files in the order asked for."""
    from orangu_b200 import trace

    w = F.weights(MIX, 111)
    v = F.values(w)
    m = make(backend, MIX, w, dtype, pool=192, rows=192, slots=4)
    t = {k: F.tokens(MIX, n, 112 + n) for k, n in (("a", 40), ("b", 64), ("c", 30), ("d", 5), ("e", 60))}
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
    assert m.free_slots == 4
    m.close()


def test_rows_of_the_llama_graph(backend):
    """forward_rows on a quantized model: the wanted rows are those of single-sequence calls, bit for bit."""
    import orangu_b200
    from orangu_b200 import synth

    cfg = synth.CONFIGS["tiny"]
    m = orangu_b200.LlamaModel(backend, cfg, synth.model_tensors(cfg, seed=3), max_seq_len=64, max_batch_tokens=8, kv_pool_tokens=128)
    toks = np.random.default_rng(4).integers(0, cfg["n_vocab"], 13).tolist()
    a, b, c = (m.new_kv_cache(32) for _ in range(3))
    got = m.forward_rows([a, b], [toks, toks[:3]], [7, 12, 15])
    assert (got[1] == m.forward(c, toks, 0)).all()
    c.truncate(0)
    assert (got[2] == m.forward(c, toks[:3], 0)).all()
    c.truncate(0)
    assert (got[0] == m.forward(c, toks[:8], 0)).all()
    m.close()


def test_what_the_library_refuses(backend):
    from orangu_b200 import OranguError

    w = F.weights(MIX, 121)
    m = make(backend, MIX, w, "float32", pool=64)
    kv = m.new_kv_cache(32)
    for rows in ([3], [1, 1], [1, 0]):
        with pytest.raises(OranguError, match="ascend"):
            m.forward_rows([kv], [[1, 2, 3]], rows)
    with pytest.raises(OranguError, match="vocabulary"):
        m.forward_rows([kv], [[MIX["vocab"]]], [0])
    with pytest.raises(OranguError, match="no recurrent state"):
        kv.read_state(1)
    m.forward_rows([kv], [[1, 2, 3]], [])
    for bad in (lambda: kv.read_state(0), lambda: kv.read(1, 0, 1)):
        with pytest.raises(OranguError):
            bad()
    m.close()
