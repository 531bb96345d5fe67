"""Noresun without a GPU: its configuration and registry entry, and the plain reference against closed forms and second
derivations of the same mathematics."""
import numpy as np
import pytest

from layered_helpers import BANDS, bits, distance, draw, mingru, noresun, reference, relu2_moe, sigmoid_attention, tensors, write_checkpoint
from oracle import layers as L
from paged_infer_b200 import api, loader, registry

rng = np.random.default_rng(0)


def test_config_fields_reach_the_layers():
    cfg = noresun([sigmoid_attention(6, 3, 10, 7, 9, 4, 77.0, BANDS, 0.5), mingru(33, relu2_moe(10, 2, 31)), sigmoid_attention(4, 3, 10, 7, None, 0, kv_from=0),
                   sigmoid_attention(scaling=None, rot=6)], width=30, vocab=50, eps=1e-4, embed_scale=7.0, alpha=2.5, bigram=(19, 40, 5))
    c = loader.LayeredConfig.from_noresun(cfg)
    a, g, s, p = c.layers
    assert (c.width, c.vocab_size, c.norm_eps, c.norm, c.tied, c.logit_scale, c.has_state) == (30, 50, 1e-4, loader.NORM_SUM, True, 1.0, True)
    assert (c.embed_scale, c.residual_keep, c.sublayer_gate, c.pair_buckets, c.pair_prev, c.pair_cur) == (7.0, 2.5, True, 19, 2, 5)
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, a.ff) == (loader.MIXER_ATTENTION, 6, 3, 10, 7, 9, 0.5, 0)
    assert (a.norm_qk, a.sigmoid_weights, a.kv_from, a.maps) == (True, True, None, 1)
    assert (a.rot_dims, a.rot_base, a.rot_banded, a.rot_factor, a.rot_original, a.rot_fast, a.rot_slow) == (4, 77.0, True, 6.0, 160.0, 5.0, 1.5)
    assert (g.mixer, g.heads, g.vdim) == (loader.MIXER_MINGRU, 1, 33)
    assert (g.ff_kind, g.experts, g.top, g.ff, g.unit, g.score, g.router_bias, g.shared_ff, g.expert_groups) == \
        (loader.FF_EXPERTS, 10, 2, 31, loader.UNIT_RELU2, loader.SCORE_CHOSEN, True, 0, 1)
    assert (s.kv_from, s.window, s.rot_dims) == (0, None, 0) and (p.rot_dims, p.rot_banded, p.rot_factor) == (6, False, 1.0)
    only = [sigmoid_attention(), sigmoid_attention(kv_from=0)]
    assert loader.LayeredConfig.from_noresun(noresun(only)).has_state         # the previous token
    assert not loader.LayeredConfig.from_noresun(noresun(only, bigram=None)).has_state
    lib = api.LayeredModel._config(c, "float32", 8)
    assert [l.kv_from for l in lib.layers[:4]] == [0, 0, 1, 0] and (lib.pair_buckets, lib.pair_prev, lib.residual_keep) == (19, 2, 2.5)


def test_unknown_parts_are_refused():
    for change, why in ((lambda l: l.update(type="gru"), "unknown mixer"), (lambda l: l.update(mlp={"kind": "dense"}), "unknown feed-forward")):
        cfg = noresun([sigmoid_attention()])
        change(cfg["layers"][0])
        with pytest.raises(ValueError, match=why):
            loader.LayeredConfig.from_noresun(cfg)


def test_registry_and_checkpoint(tmp_path):
    cfg = noresun([sigmoid_attention(mlp=relu2_moe(experts=6, top=2)), mingru(), sigmoid_attention(kv_from=0)])
    t = tensors(cfg, 1)
    folder = write_checkpoint(tmp_path, cfg, t)
    assert registry.family_of(registry.read_config(folder)) == "Noresun"
    got = loader.read_safetensors(folder + "/model.safetensors")
    assert set(got) == set(t) and all(np.array_equal(got[k], v) for k, v in bits(t).items())
    assert "l2.mix.k" not in t and "l2.mix.k.norm" not in t and "l2.mix.v" not in t


def test_pair_rows():
    assert L.bigram_rows([4, 9, 2], 11, 5, 3).tolist() == [11, (4 * 5 + 9 * 3) % 11, (9 * 5 + 2 * 3) % 11]
    assert L.bigram_rows([2 ** 31, 2 ** 31], 1000003, 999983, 7)[1] == (2 ** 31 * 999990) % 1000003


def test_banded_frequencies():
    """Short wavelengths stay, long ones are slowed by the factor, and the blend meets both ends."""
    plain = L.banded_frequencies(16, 10000.0, None)
    assert np.allclose(plain, 10000.0 ** (-np.arange(8) / 8))
    f = L.banded_frequencies(16, 10000.0, BANDS)
    turns = BANDS["original"] * plain / (2 * np.pi)
    assert (f[turns > 5] == plain[turns > 5]).all() and np.allclose(f[turns < 1.5], plain[turns < 1.5] / 6)
    mid = (turns <= 5) & (turns >= 1.5)
    assert mid.any() and (f[mid] < plain[mid]).all() and (f[mid] > plain[mid] / 6).all()
    for edge, want in ((5.0, 1.0), (1.5, 1 / 6), (3.25, 0.5 + 0.5 / 6)):       # one pair placed there by the original length
        at = L.banded_frequencies(2, 10000.0, dict(BANDS, original=2 * np.pi * edge))
        assert np.allclose(at, want)


def test_keys_weigh_by_themselves():
    T = 9
    q, k, v = rng.standard_normal((T, 3)), rng.standard_normal((T, 3)), rng.standard_normal((T, 4))
    for window in (1, 4, None):
        o = L.window_sigmoid(q, k, v, 0.7, -0.4, window)
        for t in range(T):
            want = sum(v[s] / (1 + np.exp(-(q[t] @ k[s]) * 0.7 + 0.4)) for s in range(T) if 0 <= t - s < (window or T))
            assert np.allclose(o[t], want)
    zero = np.zeros((T, 3))
    assert np.allclose(L.window_sigmoid(zero, k, np.ones((T, 1)), 1.0, 0.0, 4)[:, 0], np.minimum(np.arange(T) + 1, 4) / 2)   # a sum, no mean


def test_queries_and_keys_are_normalised_over_all_heads():
    W, H, G, D, E = 5, 4, 2, 6, 3
    h = rng.standard_normal((7, W))
    w = {"k": rng.standard_normal((G * D, W)), "k.norm": np.ones(G * D), "v": rng.standard_normal((G * E, W))}
    k, v = L.keys_and_values(h, w, G, D, E, L.banded_frequencies(4, 100.0, BANDS), 0.0)
    assert np.allclose((k ** 2).mean((1, 2)), 1) and not np.allclose((k[:, 0] ** 2).mean(-1), 1)
    assert np.allclose(v.reshape(7, -1), h @ w["v"].T)
    w = {"q": rng.standard_normal((H * D, W)), "q.norm": rng.standard_normal(H * D), "pb": np.zeros(H), "o": np.eye(H * E)}
    a = L.sigmoid_attention(h, w, H, D, [], 1.0, None, 0.0, k, v)
    assert np.allclose(L.sigmoid_attention(h, dict(w, q=3 * w["q"]), H, D, [], 1.0, None, 0.0, k, v), a)
    one = np.repeat([3.0, 1, 1, 1], D)[:, None]                       # one head's rows larger: the other heads' queries shrink
    assert not np.allclose(L.sigmoid_attention(h, dict(w, q=one * w["q"]), H, D, [], 1.0, None, 0.0, k, v)[:, E:], a[:, E:])


def test_min_gru_is_a_weighted_mean_of_its_candidates():
    T, N = 8, 3
    z, c = rng.uniform(0, 1, (T, N)), rng.standard_normal((T, N))
    s, last = L.min_gru_scan(z, c, np.zeros(N))
    for t in range(T):
        assert np.allclose(s[t], sum(z[j] * c[j] * np.prod(1 - z[j + 1:t + 1], axis=0) for j in range(t + 1)))
    s1, mid = L.min_gru_scan(z[:3], c[:3], np.zeros(N))
    s2, end = L.min_gru_scan(z[3:], c[3:], mid)
    assert np.allclose(np.concatenate([s1, s2]), s) and np.allclose(end, last)
    ones = np.ones((T, N))
    assert np.allclose(L.min_gru_scan(ones, c, np.full(N, 9.0))[0], c) and np.allclose(L.min_gru_scan(0 * ones, c, np.full(N, 9.0))[0], 9)


def test_candidates():
    u = np.array([-800.0, -2.0, -1e-9, 0.0, 3.0])
    assert np.allclose(L.positive_candidate(u), [0, 1 / (1 + np.exp(2.0)), 0.5, 0.5, 3.5])


def test_routing():
    z = np.array([[2.0, -1.0, 0.5, 0.4, 1.9, 1.8]])
    ids, w = L.route_chosen(z, 2)
    e = np.exp([2.0, 1.9])
    assert ids.tolist() == [[0, 4]] and np.allclose(w, e / e.sum())
    assert np.allclose(L.route_chosen(z, 1)[1], 1) and np.allclose(L.route_chosen(z, 6)[1].sum(), 1)


def test_experts_square_what_is_positive():
    w = {"router": np.zeros((2, 3)), "router.b": np.array([0.0, np.log(3.0)])}
    for k in range(2):
        w[f"e{k}.up"], w[f"e{k}.down"] = rng.standard_normal((4, 3)), rng.standard_normal((3, 4))
    h = rng.standard_normal((5, 3))
    act = [np.where(h @ w[f"e{k}.up"].T > 0, h @ w[f"e{k}.up"].T, 0) ** 2 @ w[f"e{k}.down"].T for k in range(2)]
    assert np.allclose(L.relu2_moe(h, w, 2), 0.25 * act[0] + 0.75 * act[1]) and np.allclose(L.relu2_moe(h, w, 1), act[1])


def test_norm_of_the_sum_and_the_gate():
    """With a gate that is shut a layer only normalises; the residual stream always leaves a layer at the norm's size."""
    cfg = noresun([mingru(mlp=relu2_moe()), sigmoid_attention()], eps=1e-12)
    t = tensors(cfg, 2)
    for n in list(t):
        if n.endswith((".norm1", ".norm2")):
            t[n][:] = 2.0
    out = []
    reference(cfg, t).forward([5, 6, 7], out)
    assert all(np.allclose((x ** 2).mean(-1), 4) for x in out)
    for n in list(t):
        if ".rg" in n and n.endswith(".b"):
            t[n][:] = -1e4
    out = []
    ref = reference(cfg, t)
    ref.forward([5, 6, 7], out)
    x = ref.embed(np.array([5, 6, 7]))
    assert np.allclose(out[-1], 2 * x / np.sqrt((x ** 2).mean(-1, keepdims=True)))


@pytest.mark.parametrize("layer", [sigmoid_attention(mlp=relu2_moe()), mingru(mlp=relu2_moe())], ids=["attention", "mingru"])
def test_prefix_of_a_sequence_does_not_see_its_end(layer):
    cfg = noresun([layer, layer])
    t = tensors(cfg, 3)
    m = reference(cfg, t)
    toks = draw(cfg, t, 30, 1)
    assert distance(m.forward(toks)[:17], m.forward(toks[:17])).max() < 1e-12


def test_shared_keys_are_the_other_layers():
    """The layer's own queries and window over keys that the other layer's input gave."""
    cfg = noresun([sigmoid_attention(window=5), mingru(), sigmoid_attention(window=11, kv_from=0)])
    t = tensors(cfg, 4)
    toks = list(range(20))
    want = reference(cfg, t).forward(toks)
    for name in ("l0.mix.k", "l0.mix.v", "l0.mix.k.norm", "l2.mix.q", "l2.mix.q.norm", "l2.mix.pb"):
        assert distance(reference(cfg, dict(t, **{name: np.roll(t[name], 1, axis=0)})).forward(toks), want).max() > 1e-3
    own = {**cfg, "layers": cfg["layers"][:2] + [sigmoid_attention(window=11)]}
    t2 = dict(t, **{n.replace("l0", "l2"): t[n] for n in ("l0.mix.k", "l0.mix.v", "l0.mix.k.norm")})
    assert distance(reference(own, t2).forward(toks), want).max() > 1e-2       # the same projections of another input are other keys
