"""Shared helpers for the GPU parity tests (everything goes through the C ABI)."""
import numpy as np
import pytest

import oracle as O


def bits(a):
    return np.ascontiguousarray(a, np.float32).view(np.uint32)


def assert_bit_equal(got, want, what=""):
    got, want = np.asarray(got, np.float32), np.asarray(want, np.float32)
    assert got.shape == want.shape, (got.shape, want.shape)
    same = bits(got) == bits(want)
    if not same.all():
        bad = np.argwhere(~same)
        i = tuple(bad[0])
        raise AssertionError(f"{what}: {len(bad)} of {same.size} values differ in their bits; first at {i}: got {got[i]!r} want {want[i]!r}")


def rel_err(got, want, magnitude):
    """max |got - want| relative to the term magnitude (sum |w*x|), the reference's own yardstick."""
    return float(np.max(np.abs(np.asarray(got, np.float64) - np.asarray(want, np.float64)) / np.maximum(magnitude, 1e-6)))


# ---- models given as a list of layers
def error(got, want):
    """Worst position: root mean square of the difference over the root mean square of all expected values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all()
    return float(np.sqrt(((got - want) ** 2).mean(-1)).max() / np.sqrt((want ** 2).mean()))


def run(model, kv, toks, cuts=()):
    """Logits at every position, the tokens fed in portions that end at `cuts`."""
    out, at = [], 0
    for end in list(cuts) + [len(toks)]:
        out.append(model.forward_rows([kv], [toks[at:end]], range(end - at)))
        at = end
    return np.concatenate(out)


def greedy_plain(plain, cfg, v, prompt, n):
    """Greedy continuation by a design's plain statement (module) and, per step, how far the best token is ahead of the next."""
    toks, out, lead = list(prompt), [], []
    for _ in range(n):
        lg = plain.forward(cfg, v, toks)[0][-1]
        top = np.sort(lg)[-2:]
        lead.append(top[1] - top[0])
        out.append(int(np.argmax(lg)))
        toks.append(out[-1])
    return out, min(lead)


@pytest.fixture(scope="session")
def backend():
    import orangu_b200

    be = orangu_b200.CudaBackend.init(0)  # raises with the reason: a GPU test never falls back
    yield be
    be.close()
