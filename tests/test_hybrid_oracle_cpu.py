"""No GPU: the plain restatement the GPU tests compare with, checked against direct loops and its own invariances."""
import numpy as np
import pytest

import hybrid_oracle as orc
from hybrid_util import attn, bf16, config, rec, weights

rng = np.random.default_rng(0)


def test_rotation_turns_neighbouring_pairs():
    x = rng.standard_normal((5, 2, 6))
    y = orc.rotate_interleaved(x, [0, 1, 2, 9, 30], 100.0)
    assert np.allclose(y[0], x[0])
    for i in range(3):
        z = (x[..., 2 * i] + 1j * x[..., 2 * i + 1]) * np.exp(1j * np.array([0, 1, 2, 9, 30])[:, None] * 100.0 ** (-2 * i / 6))
        assert np.allclose(y[..., 2 * i], z.real) and np.allclose(y[..., 2 * i + 1], z.imag)
    part = orc.rotate_interleaved(x, [0, 1, 2, 9, 30], 100.0, dims=2)
    assert np.array_equal(part[..., 2:], x[..., 2:])


def test_convolution_and_recurrence_by_loops():
    x, taps, b = rng.standard_normal((7, 3)), rng.standard_normal((3, 4)), rng.standard_normal(3)
    y = orc.causal_conv(x, taps, b)
    for t in range(7):
        want = b + sum(taps[:, 3 - k] * x[t - k] for k in range(4) if t - k >= 0)
        assert np.allclose(y[t], want)
    r, i, u, lam = rng.uniform(0, 1, (6, 3)), rng.uniform(0, 1, (6, 3)), rng.standard_normal((6, 3)), rng.standard_normal(3)
    s = orc.linear_recurrence(r, i, u, lam)
    a = np.exp(-8 * r * np.log1p(np.exp(lam)))
    assert np.allclose(s[0], np.sqrt(1 - a[0] ** 2) * i[0] * u[0])
    assert np.allclose(s[5], sum(np.prod(a[t + 1:6], axis=0) * np.sqrt(1 - a[t] ** 2) * i[t] * u[t] for t in range(6)))


@pytest.mark.parametrize("window", [1, 3, 100])
def test_window_attention_by_loops(window):
    q, k, v = rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 4)), rng.standard_normal((9, 2, 3))
    o = orc.window_attention(q, k, v, 0.7, window)
    for t in range(9):
        lo = max(0, t - window + 1)
        for h in range(2):
            e = np.exp(0.7 * k[lo:t + 1, h] @ q[t, h])
            assert np.allclose(o[t, h], (e / e.sum()) @ v[lo:t + 1, h])


def test_clamped_glu_by_elements():
    w = {"gate": rng.standard_normal((5, 4)), "up": rng.standard_normal((5, 4)), "down": np.eye(5)}
    h = 3 * rng.standard_normal((6, 4))
    y = orc.clamped_glu(h, w, "", 1.25)
    g, u = np.minimum(h @ w["gate"].T, 1.25), np.clip(h @ w["up"].T, -1.25, 1.25)
    assert (h @ w["gate"].T < -1.25).any() and np.allclose(y, g / (1 + np.exp(-1.702 * g)) * (u + 1))


def test_loops_repeat_a_range():
    cfg = config([rec(4, 1, 1)] * 5, 4, 4, loop=(1, 3, 3))
    assert orc.layer_runs(cfg) == [0, 1, 2, 1, 2, 1, 2, 3, 4]
    assert orc.layer_runs(config([rec(4, 1, 1)] * 2, 4, 4)) == [0, 1]


def test_causal_and_blind_behind_the_window():
    cfg = config([attn(2, 6, 4, 5, 9, window=5, ff=12)], 16, 30)
    w = weights(cfg, 3)
    toks = rng.integers(0, 30, 20)
    full, _ = orc.forward(cfg, w, toks)
    assert np.allclose(orc.forward(cfg, w, toks[:13])[0], full[:13])
    other = toks.copy()
    other[7] = (other[7] + 1) % 30
    d = np.abs(orc.forward(cfg, w, other)[0] - full).max(-1)
    assert (d[7:12] > 1e-6).all() and d[:7].max() < 1e-12 and d[12:].max() < 1e-12


def test_bf16_rounding():
    x = np.array([1.0, 1 + 2.0 ** -8, 1 + 3 * 2.0 ** -8, -3.14159], np.float32)
    assert np.array_equal(bf16(x), np.array([1.0, 1.0, 1 + 2.0 ** -6, -3.140625], np.float32))
