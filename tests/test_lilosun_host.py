"""Lilosun without a GPU: its configuration and registry entry, and the plain reference against closed forms and second
derivations of the same mathematics."""
import numpy as np
import pytest

from layered_helpers import YARN, bits, dense, distance, draw, latent, lilosun, mamba2, moe, reference, tensors, write_checkpoint
from oracle import layers as L
from paged_infer_b200 import loader, registry

rng = np.random.default_rng(0)


def test_config_fields_reach_the_layers():
    c = loader.LayeredConfig.from_lilosun(lilosun([latent(5, 10, 6, 7, 21, 9, base=77.0, scale=0.5, mlp=dense(13)), latent(window=None, scaling=None),
                                                   mamba2(6, 8, 12, 3, 4, 5, mlp=moe(10, 2, 33, 1.5, (5, 3), 44, 0.25)), mamba2(mlp=moe(groups=None, shared=None))],
                                                  width=30, vocab=50, eps=1e-4, logit_scale=0.75))
    a, b, s, u = c.layers
    assert (c.width, c.vocab_size, c.norm_eps, c.norm, c.tied, c.logit_scale, c.has_state) == (30, 50, 1e-4, loader.NORM_LAYER, False, 0.75, True)
    assert (a.mixer, a.heads, a.dim, a.rot_dims, a.vdim, a.rank, a.window, a.rot_base, a.scale, a.ff, a.ff_kind) == \
        (loader.MIXER_LATENT, 5, 10, 6, 7, 21, 9, 77.0, 0.5, 13, loader.FF_SILU)
    assert (a.rot_factor, a.rot_original, a.rot_fast, a.rot_slow) == (8.0, 96.0, 20.0, 2.0)
    assert (b.window, b.rot_factor, b.ff) == (None, 1.0, 0)
    assert (s.mixer, s.heads, s.vdim, s.dim, s.groups, s.norm_groups, s.conv) == (loader.MIXER_SSD, 6, 8, 12, 3, 4, 5)
    assert (s.ff_kind, s.experts, s.top, s.ff, s.limit, s.expert_groups, s.keep_groups, s.shared_ff, s.shared_limit) == \
        (loader.FF_EXPERTS, 10, 2, 33, 1.5, 5, 3, 44, 0.25)
    assert (u.expert_groups, u.keep_groups, u.shared_ff) == (1, 1, 0)
    assert not loader.LayeredConfig.from_lilosun(lilosun([latent()])).has_state


def test_unknown_parts_are_refused():
    for change, why in ((lambda l: l.update(type="other"), "unknown mixer"), (lambda l: l.update(mlp={"kind": "other"}), "unknown feed-forward"),
                        (lambda l: l["mixer"]["rot"].update(dims=2), "rotated channels")):
        cfg = lilosun([latent()])
        change(cfg["layers"][0])
        with pytest.raises(ValueError, match=why):
            loader.LayeredConfig.from_lilosun(cfg)


def test_registry_and_checkpoint(tmp_path):
    cfg = lilosun([latent(mlp=moe(experts=6, groups=(2, 1), top=2)), mamba2()])
    t = tensors(cfg, 1)
    folder = write_checkpoint(tmp_path, cfg, t)
    assert registry.family_of(registry.read_config(folder)) == "Lilosun"
    got = loader.read_safetensors(folder + "/model.safetensors")
    assert set(got) == set(t) and all(np.array_equal(got[k], v) for k, v in bits(t).items())


def test_layer_norm():
    x = rng.standard_normal((3, 8)) + 5
    y = L.layer_norm(x, np.full(8, 2.0), 0.0)
    assert np.allclose(y.mean(-1), 0) and np.allclose(y.std(-1), 2)
    assert np.allclose(L.layer_norm(np.full((1, 4), 3.0), np.ones(4), 1e-5), 0)


def test_yarn_ends():
    f, g = L.yarn_frequencies(32, 10000.0, YARN)
    p, one = L.yarn_frequencies(32, 10000.0, None)
    assert one == 1.0 and np.isclose(g, 1 + 0.1 * np.log(8))
    turns = 96 * p / (2 * np.pi)
    assert np.allclose(f[:1], p[:1]) and np.allclose(f[turns < 1], p[turns < 1] / 8)
    assert np.all(np.diff(f) < 0) and np.all(f <= p + 1e-12) and np.all(f >= p / 8 - 1e-12)
    assert np.allclose(L.yarn_frequencies(32, 10000.0, {**YARN, "factor": 1.0})[0], p)


def test_rotation_keeps_lengths_up_to_its_gain():
    q, k = rng.standard_normal((2, 1, 1, 8))
    f, g = L.yarn_frequencies(8, 100.0, YARN)
    a = [np.sum(L.rotate_pairs(q, [p], f, g) * L.rotate_pairs(k, [p - 5], f, g)) for p in (5, 50, 500)]
    assert np.allclose(a, a[0])
    assert np.allclose(np.sum(L.rotate_pairs(q, [7], f, g) ** 2), np.sum(q ** 2) * g * g)


def test_latent_attention_in_latent_space():
    """The same attention with the queries taken into latent space: the cached rows are keys and values of all heads."""
    H, D, R, E, K, W, T, win = 3, 4, 6, 5, 7, 9, 12, 5
    h = rng.standard_normal((T, W))
    w = {n: rng.standard_normal(s) for n, s in (("q", (H * (D + R), W)), ("dkv", (K + R, W)), ("dkv.norm", (K,)), ("uk", (H * D, K)), ("uv", (H * E, K)),
                                                ("g", (H * E, W)), ("o", (W, H * E)))}
    got = L.latent_attention(h, w, H, D, R, E, K, 50.0, YARN, 0.3, win, 1e-5)
    f, g = L.yarn_frequencies(R, 50.0, YARN)
    q = (h @ w["q"].T).reshape(T, H, D + R)
    down = h @ w["dkv"].T
    c = down[:, :K] / np.sqrt((down[:, :K] ** 2).mean(-1, keepdims=True) + 1e-5) * w["dkv.norm"]
    kr = L.rotate_pairs(down[:, None, K:], np.arange(T), f, g)[:, 0]
    qr = L.rotate_pairs(q[:, :, D:], np.arange(T), f, g)
    a = np.zeros((T, H, E))
    for n in range(H):
        rows = np.concatenate([q[:, n, :D] @ w["uk"][n * D:(n + 1) * D], qr[:, n]], -1)
        a[:, n] = L.window_softmax(rows, np.concatenate([c, kr], -1), c, 0.3, win) @ w["uv"][n * E:(n + 1) * E].T
    want = (a.reshape(T, H * E) / (1 + np.exp(-(h @ w["g"].T)))) @ w["o"].T
    assert np.allclose(got, want)


def test_convolution():
    x, w, b = rng.standard_normal((6, 2)), rng.standard_normal((2, 3)), rng.standard_normal(2)
    y = L.causal_conv(x, w, b)
    assert np.allclose(y[0], b + w[:, 2] * x[0])
    assert np.allclose(y[5], b + w[:, 0] * x[3] + w[:, 1] * x[4] + w[:, 2] * x[5])


def test_ssd_scan_is_a_decayed_sum():
    T, N, E = 9, 3, 2
    x, B, C, dt = rng.standard_normal((T, E)), rng.standard_normal((T, N)), rng.standard_normal((T, N)), rng.random(T)
    y, S = L.ssd_scan(x, B, C, dt, 0.3, np.zeros((N, E)))
    F = np.cumsum(-np.exp(0.3) * dt)
    for t in range(T):
        assert np.allclose(y[t], sum((C[t] @ B[s]) * np.exp(F[t] - F[s]) * dt[s] * x[s] for s in range(t + 1)))
    y1, S1 = L.ssd_scan(x[:4], B[:4], C[:4], dt[:4], 0.3, np.zeros((N, E)))
    y2, S2 = L.ssd_scan(x[4:], B[4:], C[4:], dt[4:], 0.3, S1)
    assert np.allclose(np.concatenate([y1, y2]), y) and np.allclose(S2, S)


def test_grouped_norm_and_units():
    x = rng.standard_normal((2, 6))
    y = L.grouped_unit_rms(x, 3, 0.0)
    assert np.allclose((y.reshape(2, 3, 2) ** 2).mean(-1), 1)
    one = np.eye(1)
    assert np.allclose(L.clamped_mlp(np.array([[9.0]]), one, one, one, 2.0), 2 * L.sigmoid(3.404) * 3)
    assert np.allclose(L.clamped_mlp(np.array([[-9.0]]), one, one, one, 2.0), -9 * L.sigmoid(-15.3178) * -1)
    assert np.allclose(L.softplus(np.array([-50.0, 0.0, 50.0])), [0, np.log(2), 50])


def test_routing():
    z = np.array([[2.0, -1.0, 0.5, 0.4, 3.0, -3.0]])
    s = L.sigmoid(z)
    ids, w = L.route(z, np.zeros(6), 2, 1, 1)
    assert sorted(ids[0]) == [0, 4] and np.allclose(np.sort(w), np.sort(s[:, [0, 4]] / s[0, [0, 4]].sum()))
    # groups (0,1) (2,3) (4,5): the pair sums decide, not the best member
    ids, _ = L.route(z, np.zeros(6), 2, 3, 1)
    assert sorted(ids[0]) == [2, 3]
    # a correction moves the choice and not the weights; negative choice scores still beat what is masked
    c = np.array([-5.0, -5, -5, -5, -4, -3])
    ids, w = L.route(z, c, 2, 3, 1)
    assert sorted(ids[0]) == [4, 5] and np.allclose(np.sort(w), np.sort(s[:, [4, 5]] / s[0, [4, 5]].sum()))
    m = L.route_margin(z, np.zeros(6), 2, 3, 1)
    assert np.isclose(m[0], (s[0, 2] + s[0, 3] - max(s[0, 0] + s[0, 1], s[0, 4] + s[0, 5])) / 2)


@pytest.mark.parametrize("layer", [latent(mlp=moe()), mamba2(mlp=dense())], ids=["latent_moe", "mamba2_dense"])
def test_prefix_of_a_sequence_does_not_see_its_end(layer):
    cfg = lilosun([layer, layer])
    t = tensors(cfg, 3)
    m = reference(cfg, t)
    toks = draw(cfg, t, 30, 1)
    assert distance(m.forward(toks)[:17], m.forward(toks[:17])).max() < 1e-12
