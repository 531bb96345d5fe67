"""Rubuvik without a GPU: its configuration and registry entry, and the plain reference against closed forms and second
derivations of the same mathematics."""
import numpy as np
import pytest

from layered_helpers import biased, bits, dense, distance, draw, lightning, reference, rubuvik, softmax_moe, sunk, tensors, write_checkpoint
from oracle import layers as L
from paged_infer_b200 import api, loader, registry

rng = np.random.default_rng(0)


def test_config_fields_reach_the_layers():
    cfg = rubuvik([biased(6, 3, 10, 7, 9, 0.5, True, (0.25, 33), dense(13)), sunk(4, 4, 8, 12, None, 0.75, False),
                   lightning(2, 5, 6, (0.25, 1.0), softmax_moe(10, 2, 33, (5, 3), 44, 2.25)), lightning(mlp=softmax_moe(groups=None, shared=None))],
                  width=30, vocab=50, eps=1e-4, embed_scale=7.0, mult=0.125, side=3)
    c = loader.LayeredConfig.from_rubuvik(cfg)
    a, b, s, u = c.layers
    assert (c.width, c.vocab_size, c.norm_eps, c.norm, c.tied, c.logit_scale, c.has_state) == (30, 50, 1e-4, loader.NORM_RMS, True, 1.0, True)
    assert (c.embed_scale, c.residual_mult, c.side_dim) == (7.0, 0.125, 3)
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.scale, a.ff, a.ff_kind) == (loader.MIXER_ATTENTION, 6, 3, 10, 7, 9, 0.5, 13, loader.FF_SILU)
    assert (a.distance_bias, a.v_mix, a.q_temp_coef, a.q_temp_every, a.biases, a.unit_qk, a.sink, a.head_gate) == (True, True, 0.25, 33.0, False, False, False, False)
    assert (b.window, b.v_mix, b.q_temp_every, b.distance_bias, b.biases, b.unit_qk, b.sink, b.head_gate, b.ff) == (None, False, 0.0, True, True, True, True, True, 0)
    assert (s.mixer, s.heads, s.dim, s.vdim, s.decay) == (loader.MIXER_LIGHTNING, 2, 5, 6, (0.25, 1.0))
    assert (s.ff_kind, s.experts, s.top, s.ff, s.expert_groups, s.keep_groups, s.shared_ff) == (loader.FF_EXPERTS, 10, 2, 33, 5, 3, 44)
    assert (s.unit, s.score, s.group_best, s.renorm, s.shared_gate, s.route_scale) == (loader.UNIT_SILU, loader.SCORE_SOFTMAX, 1, False, False, 2.25)
    assert (u.expert_groups, u.keep_groups, u.shared_ff) == (1, 1, 0)
    assert not loader.LayeredConfig.from_rubuvik(rubuvik([biased(), sunk()])).has_state
    assert loader.LayeredConfig.from_rubuvik(rubuvik([biased()], side=None)).side_dim == 0
    assert loader.LayeredConfig.from_rubuvik(rubuvik([biased(temp=None)])).layers[0].q_temp_every == 0


def test_the_library_gets_the_decays():
    cfg = loader.LayeredConfig.from_rubuvik(rubuvik([biased(), lightning(2, decay=(0.5, 0.75))]))
    c = api.LayeredModel._config(cfg, "float32", 8)
    assert c.layers[1].decay[:2] == [0.5, 0.75] and not c.layers[0].decay and c.layers[0].window == 30
    cfg.layers[1].heads = 3
    with pytest.raises(ValueError, match="2 decays for 3 heads"):
        api.LayeredModel._config(cfg, "float32", 8)


def test_unknown_parts_are_refused():
    for change, why in ((lambda l: l.update(type="attention_3"), "unknown mixer"), (lambda l: l.update(mlp={"kind": "other"}), "unknown feed-forward")):
        cfg = rubuvik([biased()])
        change(cfg["layers"][0])
        with pytest.raises(ValueError, match=why):
            loader.LayeredConfig.from_rubuvik(cfg)


def test_registry_and_checkpoint(tmp_path):
    cfg = rubuvik([sunk(mlp=softmax_moe(experts=6, groups=(2, 1), top=2)), lightning()])
    t = tensors(cfg, 1)
    folder = write_checkpoint(tmp_path, cfg, t)
    assert registry.family_of(registry.read_config(folder)) == "Rubuvik"
    got = loader.read_safetensors(folder + "/model.safetensors")
    assert set(got) == set(t) and all(np.array_equal(got[k], v) for k, v in bits(t).items())


def test_norm_around_one():
    x = rng.standard_normal((3, 8))
    y = L.rms_around_one(x, np.full(8, 1.0), 0.0)
    assert np.allclose((y * y).mean(-1), 4)
    assert np.allclose(L.rms_around_one(np.zeros((1, 4)), np.zeros(4), 1e-5), 0)


def test_slopes_and_temperature():
    assert np.allclose(L.distance_slopes(8), 0.5 ** np.arange(1, 9))
    s = L.distance_slopes(6)
    assert np.allclose(s[1:] / s[:-1], 2 ** (-8 / 6)) and np.isclose(s[-1], 1 / 256)
    t = L.query_temperature(np.arange(12), 0.5, 4)
    assert np.allclose(t, 1 + 0.5 * np.log([1, 1, 1, 2, 2, 2, 2, 3, 3, 3, 3, 4]))


def test_distance_bias_and_sink_without_scores():
    """With queries of zero only the bias and the sink weigh: a geometric series beside one constant term."""
    T, window, slope = 9, 5, 0.3
    q, k, v = np.zeros((T, 2)), rng.standard_normal((T, 2)), np.eye(T)
    for sink in (None, -40.0, 0.7, 40.0):
        p = L.biased_window_softmax(q, k, v, 1.0, slope, window, sink)
        for t in range(T):
            w = np.array([np.exp(-slope * (t - s)) if 0 <= t - s < window else 0.0 for s in range(T)])
            assert np.allclose(p[t], w / (w.sum() + (0 if sink is None else np.exp(sink))))


def test_bias_alone_orders_the_keys_and_a_shift_of_the_scores_does_not_matter_without_a_sink():
    T = 7
    q, k, v = rng.standard_normal((T, 3)), rng.standard_normal((T, 3)), rng.standard_normal((T, 4))
    far = np.concatenate([k, np.ones((T, 1))], 1), np.concatenate([q, np.full((T, 1), 5.0)], 1)
    a = L.biased_window_softmax(q, k, v, 0.5, 0.1, None)
    assert np.allclose(L.biased_window_softmax(far[1], far[0], v, 0.5, 0.1, None), a)
    assert not np.allclose(L.biased_window_softmax(far[1], far[0], v, 0.5, 0.1, None, 1.0), L.biased_window_softmax(q, k, v, 0.5, 0.1, None, 1.0))
    assert np.allclose(a, L.biased_window_softmax(q, k, v, 0.5, 0.1, T))
    assert np.allclose(L.biased_window_softmax(q, k, v, 0.5, 0.0, 3), L.window_softmax(q, k, v, 0.5, 3))


def test_mixed_values():
    v, f = rng.standard_normal((2, 3, 1, 4))
    assert np.allclose(L.mixed_values(v, f, 0.0), v) and np.allclose(L.mixed_values(v, f, 1.0), f) and np.allclose(L.mixed_values(v, f, 0.25), 0.75 * v + 0.25 * f)


def test_decayed_scan_is_a_decayed_sum():
    T, D, E = 9, 3, 2
    q, k, v = rng.standard_normal((T, D)), rng.standard_normal((T, D)), rng.standard_normal((T, E))
    for a in (0.0, 0.4, 1.0):
        o, S = L.decayed_scan(q, k, v, a, np.zeros((D, E)))
        for t in range(T):
            assert np.allclose(o[t], sum(a ** (t - s) * (q[t] @ k[s]) * v[s] for s in range(t + 1)))
        o1, S1 = L.decayed_scan(q[:4], k[:4], v[:4], a, np.zeros((D, E)))
        o2, S2 = L.decayed_scan(q[4:], k[4:], v[4:], a, S1)
        assert np.allclose(np.concatenate([o1, o2]), o) and np.allclose(S2, S)


def test_lightning_norm_spans_the_heads_and_the_gate_follows():
    H, D, E, W = 2, 3, 4, 5
    w = {n: rng.standard_normal(s) for n, s in (("q", (H * D, W)), ("k", (H * D, W)), ("v", (H * E, W)), ("g", (H * E, W)), ("norm", (H * E,)))}
    w["o"] = np.eye(H * E)
    h = rng.standard_normal((6, W))
    y = L.lightning(h, w, H, D, E, [0.5, 0.9], 0.0) / (w["norm"] / (1 + np.exp(-(h @ w["g"].T))))
    assert np.allclose((y * y).mean(-1), 1) and not np.allclose((y[:, :E] ** 2).mean(-1), 1)


def test_routing():
    z = np.array([[2.0, -1.0, 0.5, 0.4, 1.9, 1.8]])
    s = np.exp(z) / np.exp(z).sum()
    ids, w = L.route_softmax(z, np.zeros(6), 2, 1, 1, 3.0)
    assert ids.tolist() == [[0, 4]] and np.allclose(w, 3 * s[:, [0, 4]])
    # groups (0,1) (2,3) (4,5): the best member decides, not the sum
    assert sorted(L.route_softmax(z, np.zeros(6), 2, 3, 1, 1.0)[0][0]) == [0, 1]
    # a correction moves the choice and not the weights; negative choice scores still beat what is masked
    c = np.array([-5.0, -5, -3, -6, -4, -4])
    ids, w = L.route_softmax(z, c, 2, 3, 1, 1.0)
    assert ids.tolist() == [[2, 3]] and np.allclose(w, s[:, [2, 3]])
    assert np.isclose(L.route_softmax_margin(z, np.zeros(6), 1, 3, 1)[0], min(s[0, 0] - s[0, 4], s[0, 0] - s[0, 1]))


def test_token_side_is_gated_by_the_row_of_the_table():
    x, e = rng.standard_normal((2, 4)), rng.standard_normal((2, 3))
    w = {"gate": rng.standard_normal((3, 4)), "proj": rng.standard_normal((4, 3)), "norm": np.full(4, 2.0)}
    y = L.token_side(x, e, w, 0.0)
    assert np.allclose((y * y).mean(-1), 4)
    assert np.allclose(L.token_side(x, 5 * e, w, 0.0), y) and np.allclose(L.token_side(x, -e, w, 0.0), -y)
    assert np.allclose(L.token_side(x, 0 * e, w, 1e-5), 0)


@pytest.mark.parametrize("layer", [biased(mlp=softmax_moe()), sunk(mlp=dense()), lightning()], ids=["attention_moe", "attention_2_dense", "lightning"])
def test_prefix_of_a_sequence_does_not_see_its_end(layer):
    cfg = rubuvik([layer, layer])
    t = tensors(cfg, 3)
    m = reference(cfg, t)
    toks = draw(cfg, t, 30, 1)
    assert distance(m.forward(toks)[:17], m.forward(toks[:17])).max() < 1e-12


def test_only_the_first_layer_that_mixes_gives_its_values():
    """Its own lambda counts for nothing; the others' do; layers that do not mix neither give nor take."""
    cfg = rubuvik([sunk(v_mix=False, vdim=16), biased(), sunk(), biased()])
    t = tensors(cfg, 4)
    toks = list(range(20))
    want = reference(cfg, t).forward(toks)
    for name, moves in (("l1.mix.vmix", False), ("l2.mix.vmix", True), ("l3.mix.vmix", True)):
        other = dict(t, **{name: t[name] + 0.5})
        assert (distance(reference(cfg, other).forward(toks), want).max() > 1e-3) == moves
    assert "l0.mix.vmix" not in t
