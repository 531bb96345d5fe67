"""The plain reference of the layered designs against closed forms and second derivations of the same mathematics: no
GPU, nothing of the product path."""
import numpy as np
import pytest

from layered_helpers import attention, config, distance, gla, mlstm, reference, tensors
from oracle import layers as L

rng = np.random.default_rng(0)


def test_dyt_has_no_statistics():
    x = rng.standard_normal((3, 8))
    y = L.dyt_norm(x, 0.5, np.full(8, 2.0), np.full(8, 0.25))
    assert np.allclose(y, 2 * np.tanh(x / 2) + 0.25)
    assert np.array_equal(y[1], L.dyt_norm(x[1:2], 0.5, np.full(8, 2.0), np.full(8, 0.25))[0])


def test_gelu_and_gates():
    z = np.array([-1e3, -1.0, 0.0, 1.0, 1e3])
    assert np.allclose(L.gelu_tanh(z), [0, -0.15880801, 0, 0.84119199, 1e3])
    assert np.allclose(L.log_sigmoid(z), [-1e3, -1.31326169, -0.69314718, -0.31326169, 0])
    assert np.allclose(L.sigmoid(z), [0, 0.26894142, 0.5, 0.73105858, 1])


def test_rotation_keeps_lengths_and_depends_on_distance_only():
    q, k = rng.standard_normal((2, 1, 1, 8))
    a = [np.sum(L.rotate_interleaved(q, [p], 6, 100.0) * L.rotate_interleaved(k, [p - 5], 6, 100.0)) for p in (5, 50, 500)]
    assert np.allclose(a, a[0])
    r = L.rotate_interleaved(q, [7], 6, 100.0)
    assert np.allclose(np.sum(r ** 2), np.sum(q ** 2)) and np.array_equal(r[..., 6:], q[..., 6:])
    assert np.allclose(r[0, 0, 0] + 1j * r[0, 0, 1], (q[0, 0, 0] + 1j * q[0, 0, 1]) * np.exp(7j))


def test_window_edges():
    T, w = 12, 4
    v = np.eye(T)
    p = L.window_softmax(np.zeros((T, 2)), np.zeros((T, 2)), v, 1.0, w)
    for t in range(T):
        seen = [s for s in range(T) if 0 <= t - s < w]
        assert np.allclose(p[t], np.isin(np.arange(T), seen) / len(seen))
    assert np.allclose(L.window_softmax(np.zeros((T, 2)), np.zeros((T, 2)), v, 1.0, None)[-1], 1 / T)


def test_gla_scan_is_a_decayed_sum():
    T, D, E = 9, 3, 2
    q, k, v, g = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, E)), -rng.random((T, D))
    o, S = L.gla_scan(q, k, v, g, np.zeros((D, E)))
    c = np.cumsum(g, 0)
    for t in range(T):
        want = sum((q[t] * np.exp(c[t] - c[s]) @ k[s]) * v[s] for s in range(t + 1))
        assert np.allclose(o[t], want)
    o1, S1 = L.gla_scan(q[:4], k[:4], v[:4], g[:4], np.zeros((D, E)))
    o2, S2 = L.gla_scan(q[4:], k[4:], v[4:], g[4:], S1)
    assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)


def test_mlstm_maximum_is_only_a_scale_except_for_the_floor():
    T, D, E = 10, 3, 2
    q, k, v = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, E))
    i, f = 2 * rng.standard_normal(T), -rng.random(T)
    o, S, n, m = L.mlstm_scan(q, k, v, i, f, np.zeros((D, E)), np.zeros(D), 0.0)
    c = np.cumsum(f)
    mx = 0.0
    for t in range(T):
        mx = max(f[t] + mx, i[t])
        w = np.array([np.exp(c[t] - c[s] + i[s]) for s in range(t + 1)]) * (k[:t + 1] @ q[t])
        assert np.allclose(o[t], np.exp(-mx) * (w @ v[:t + 1]) / (max(abs(np.exp(-mx) * w.sum()), np.exp(-mx)) + 1e-6))


def test_differential_attention_without_second_map_is_normalised_attention():
    H, D, E, W, T = 2, 4, 6, 8, 7
    h = rng.standard_normal((T, W))
    w = {"q": rng.standard_normal((H * 2 * D, W)), "k": rng.standard_normal((2 * D, W)), "v": rng.standard_normal((E, W)), "o": np.eye(H * E)}
    z = np.zeros(D)
    w.update(lq1=z, lk1=z, lq2=z, lk2=z)      # lambda = diff
    out = L.differential_attention(h, w, H, 1, D, E, 0, 1.0, 0.5, 3, 0.0, 1e-9)
    q = (h @ w["q"].T).reshape(T, H, 2, D)
    k = (h @ w["k"].T).reshape(T, 2, D)
    a = L.window_softmax(q[:, 1, 0], k[:, 0], h @ w["v"].T, 0.5, 3)
    assert np.allclose(out[:, E:], L.unit_rms(a, 1e-9))
    assert np.isclose(L.differential_lambda(*[np.full(2, x) for x in (1.0, 0.5, 0.5, 1.0)], 0.4), 0.4)


@pytest.mark.parametrize("layer", [attention(), gla(), mlstm()], ids=["attention", "gla", "mlstm"])
def test_prefix_of_a_sequence_does_not_see_its_end(layer):
    cfg = config([layer, layer])
    m = reference(cfg, tensors(cfg, 3))
    toks = rng.integers(0, cfg["vocab"], 30)
    assert distance(m.forward(toks)[:17], m.forward(toks[:17])).max() < 1e-12
