"""Rubuvik on the device against the plain reference: every mechanism alone, prefill against decoding, portions, mixed batches,
blocks and slots used again, window edges, sinks, temperature, value mixing, routing, and generation through the engine.  Both
number formats."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from layered_helpers import (LIMIT, Session, biased, dense, device_model, distance, draw, lightning, reference, rubuvik, softmax_moe, sunk, tensors,
                             write_checkpoint)
from test_gpu_layered import reference_greedy

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("compute", ["float32", "bfloat16"])


@pytest.fixture(scope="module")
def ctx():
    from paged_infer_b200 import api
    return api.Context(0)


# what one layer can be, in sizes that hit the kernels' special cases
ALONE = {
    "attention": biased(),
    "attention_everything": biased(window=None, heads=5, kv_heads=5),
    "attention_window1": biased(window=1, heads=2, kv_heads=1),
    "attention_wide_window": biased(window=1000, scale=0.05, temp=(2.0, 1)),
    "attention_no_temperature": biased(temp=None, v_mix=False),
    "attention_odd": biased(heads=3, kv_heads=3, dim=11, vdim=9, window=19),
    "attention_17_per_group": biased(heads=34, kv_heads=2, dim=16, vdim=16, window=90),
    "attention_one_head": biased(heads=1, kv_heads=1, dim=80, vdim=32, window=65),
    "attention_big_heads": biased(heads=2, kv_heads=1, dim=200, vdim=150, window=50),
    "attention_wide_values": biased(heads=4, kv_heads=2, dim=128, vdim=256, window=77),
    "attention_huge_keys": biased(heads=2, kv_heads=2, dim=300, vdim=20, window=40, scale=0.03),
    "attention_2": sunk(),
    "attention_2_everything": sunk(window=None, heads=7, kv_heads=1),
    "attention_2_window1": sunk(window=1, heads=2, kv_heads=2),
    "attention_2_odd": sunk(heads=9, kv_heads=3, dim=13, vdim=7, window=33),
    "attention_2_one_head": sunk(heads=1, kv_heads=1, dim=80, vdim=32, window=129),
    "attention_2_wide": sunk(heads=8, kv_heads=2, dim=128, vdim=64, window=100),
    "attention_2_huge_keys": sunk(heads=2, kv_heads=1, dim=300, vdim=300, window=70),
    "lightning": lightning(),
    "lightning_one_head": lightning(heads=1, dim=48, vdim=80, decay=(0.99,)),
    "lightning_extremes": lightning(heads=5, dim=16, vdim=16, decay=(0.0, 1e-30, 0.02, 0.99999, 1.0)),
    "lightning_odd": lightning(heads=3, dim=5, vdim=7, decay=(0.3, 0.9, 0.97)),
    "lightning_large": lightning(heads=4, dim=128, vdim=128, decay=(0.6, 0.9, 0.98, 0.999)),
    "lightning_wide_value": lightning(heads=2, dim=40, vdim=200, decay=(0.7, 0.98)),
    "lightning_wide_key": lightning(heads=2, dim=250, vdim=36, decay=(0.7, 0.98)),
    "lightning_state_in_memory": lightning(heads=1, dim=300, vdim=128, decay=(0.95,)),
    "dense": lightning(mlp=dense(50)),
    "dense_odd": biased(heads=2, mlp=dense(13)),
    "moe": lightning(mlp=softmax_moe()),
    "moe_top1": sunk(mlp=softmax_moe(experts=8, top=1, ff=24, groups=(2, 1))),
    "moe_all": lightning(mlp=softmax_moe(experts=4, top=4, ff=33, groups=None)),
    "moe_no_shared": biased(mlp=softmax_moe(experts=10, top=2, ff=48, groups=(5, 3), shared=None)),
    "moe_groups_of_one": sunk(mlp=softmax_moe(experts=6, top=2, ff=20, groups=(6, 4), scale=0.5)),
    "moe_keeps_all_groups": biased(mlp=softmax_moe(experts=6, top=2, ff=20, groups=(2, 2), scale=3.0)),
    "moe_many": lightning(mlp=softmax_moe(experts=70, top=6, ff=17, groups=(7, 3), shared=31)),
}
MIXED = rubuvik([sunk(v_mix=False, vdim=12), biased(mlp=softmax_moe()), lightning(mlp=dense()), sunk(window=44, heads=4, mlp=softmax_moe(experts=10, groups=None, top=2)),
                 lightning(heads=2, dim=16, vdim=48, decay=(0.9, 0.995), mlp=softmax_moe(shared=None)), biased(window=None, heads=2, dim=32, temp=(0.7, 25)),
                 sunk(window=17, heads=8, dim=10, mlp=dense(31))], vocab=500)


@pytest.fixture(scope="module")
def mixed():
    t = tensors(MIXED, 3)
    return t, reference(MIXED, t)


def check_alone(ctx, cfg, t, toks, compute):
    """Residual stream and logits of a model: a prompt in one step, then token by token."""
    layer = []
    want = reference(cfg, t).forward(toks, layer)
    n = len(toks) - 9
    m = device_model(ctx, cfg, t, compute)
    s = Session(m)
    m.trace_layers(True)
    got = s.run([("a", toks[:n])])[0]
    x = m.read_layer(len(layer) - 1, n)
    m.trace_layers(False)
    lim = LIMIT[compute]
    assert distance(x, layer[-1][:n]).max() < lim
    assert distance(got, want[:n]).max() < lim
    for i in range(n, len(toks)):
        assert distance(s.run([("a", [toks[i]])])[0], want[i:i + 1]).max() < 1.5 * lim


@BOTH
@pytest.mark.parametrize("name", sorted(ALONE))
def test_mechanism_alone(ctx, name, compute):
    cfg = rubuvik([ALONE[name]], width=72, vocab=240)
    t = tensors(cfg, 11)
    check_alone(ctx, cfg, t, draw(cfg, t, 150, 5), compute)


@BOTH
@pytest.mark.parametrize("change", [dict(side=None), dict(side=3), dict(side=70, mult=1.0), dict(embed_scale=1.0, mult=0.05), dict(width=75, side=5),
                                    dict(width=1028), dict(width=2052), dict(width=4100), dict(eps=0.3)], ids=str)
def test_sizes_and_constants_around_the_layers(ctx, change, compute):
    """Widths that leave the row kernel's registers, rows of odd length, no table of tokens, constants that are 1."""
    cfg = rubuvik([lightning(mlp=dense(40)), sunk(mlp=None), biased(mlp=softmax_moe(experts=4, top=2, groups=None, ff=24))], **{"vocab": 240, **change})
    t = tensors(cfg, 12)
    check_alone(ctx, cfg, t, draw(cfg, t, 80, 6), compute)


@BOTH
@pytest.mark.parametrize("width,side", [(512, 8), (1024, 384), (2048, 100), (3000, 256)])
def test_token_table_at_every_number_of_rows(ctx, width, side, compute):
    """One launch for few rows, projections and row steps for more, and for matrices that are too large: the same numbers."""
    cfg = rubuvik([sunk(mlp=softmax_moe(experts=6, top=3, groups=None, ff=24)), lightning(mlp=dense(40)), biased()], width=width, vocab=240, side=side)
    t = tensors(cfg, 15)
    toks = draw(cfg, t, 100, 8)
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    at, got = 0, []
    for n in (1, 2, 4, 5, 8, 9, 23, 48):
        got.append(s.run([("a", toks[at:at + n])])[0])
        at += n
    assert at == len(toks) and distance(np.concatenate(got), want).max() < LIMIT[compute]
    seqs = [draw(cfg, t, 9, 50 + i) for i in range(5)]       # five rows of five sequences
    for i in range(9):
        outs = s.run([(f"s{j}", [q[i]]) for j, q in enumerate(seqs)])
    for q, out in zip(seqs, outs):
        assert distance(out, reference(cfg, t).forward(q)[-1:]).max() < 1.5 * LIMIT[compute]


def test_token_table_of_one_channel(ctx):
    """Its normalised contribution is a sign times a vector: in the f32 mode only, where no rounding turns the sign."""
    cfg = rubuvik([lightning(), biased(mlp=dense(20))], width=72, vocab=96, side=1)
    t = tensors(cfg, 13)
    check_alone(ctx, cfg, t, draw(cfg, t, 60, 7), "float32")


@BOTH
def test_decoding_equals_prefill(ctx, mixed, compute):
    t, ref = mixed
    toks = draw(MIXED, t, 100, 8)
    want = ref.forward(toks)
    s = Session(device_model(ctx, MIXED, t, compute), block_size=16)
    whole = s.run([("whole", toks)])[0]
    one = np.concatenate([s.run([("one", [x])])[0] for x in toks])
    assert distance(whole, want).max() < LIMIT[compute]
    assert distance(one, want).max() < LIMIT[compute]


@BOTH
@pytest.mark.parametrize("size", [2, 3, 7, 16, 63, 64, 65, 128, 129])
def test_portions(ctx, mixed, size, compute):
    t, ref = mixed
    toks = draw(MIXED, t, 200 if size > 7 else 70, 9)
    want = ref.forward(toks)
    s = Session(device_model(ctx, MIXED, t, compute), block_size=8)
    got = np.concatenate([s.run([("p", toks[i:i + size])])[0] for i in range(0, len(toks), size)])
    assert distance(got, want).max() < LIMIT[compute]


@BOTH
def test_uneven_batches_and_reuse(ctx, mixed, compute):
    """Portions beside single tokens, requests that pause, end and make room; freed blocks and slots are used at once."""
    t, ref = mixed
    s = Session(device_model(ctx, MIXED, t, compute), blocks=40, slots=3)
    rng = np.random.default_rng(1)
    live, got, done = {}, {}, 0
    for i in range(60):
        while len(live) < 3 and done + len(live) < 9:
            name = f"r{done + len(live)}.{i}"
            live[name] = draw(MIXED, t, int(rng.choice([1, 2, 19, 64, 150])), 100 + i + len(live))
            got[name] = []
        batch = []
        for name in list(live):
            if rng.random() < 0.2:
                continue    # pauses
            n = int(rng.choice([1, 1, 2, 5, 70, 90]))
            at = sum(len(x) for x in got[name])
            if live[name][at:at + n]:
                batch.append((name, live[name][at:at + n]))
        if not batch:
            continue
        for (name, _), out in zip(batch, s.run(batch)):
            got[name].append(out)
        for name in list(live):
            if sum(len(x) for x in got[name]) == len(live[name]):
                assert distance(np.concatenate(got[name]), ref.forward(live[name])).max() < LIMIT[compute], name
                s.close(name)
                del live[name]
                done += 1
    assert done == 9


@BOTH
def test_batch_does_not_change_a_row(ctx, mixed, compute):
    t, _ = mixed
    m = device_model(ctx, MIXED, t, compute)
    toks = {n: draw(MIXED, t, k, 40 + k) for n, k in (("a", 33), ("b", 70), ("c", 5), ("d", 101))}
    alone = {}
    for n in toks:
        s = Session(m, seed=1)
        alone[n] = [s.run([(n, toks[n][:-1])])[0], s.run([(n, toks[n][-1:])])[0]]
    s = Session(m, seed=2)
    first = s.run([(n, toks[n][:-1]) for n in toks])
    last = s.run([(n, toks[n][-1:]) for n in reversed(toks)])
    for i, n in enumerate(toks):
        assert distance(first[i], alone[n][0]).max() < LIMIT[compute] / 2
        assert distance(last[len(toks) - 1 - i], alone[n][1]).max() < LIMIT[compute] / 2


NEEDLE, SEEKER = 1, 2


def needle_model(kind, window):
    """One attention layer in which token SEEKER looks for token NEEDLE through one channel of every head, so that one score stands
    far above all others, whatever the distance takes off it."""
    heads, dim = 4, 12
    cfg = rubuvik([kind(heads, 2, dim, 20, window, 1.0 if kind is biased else 2.5, False)], width=64, vocab=96, embed_scale=1.0)
    t = tensors(cfg, 21)
    e = t["embed"]
    e[:, 40:42] = 0
    e[NEEDLE, 40] = e[SEEKER, 41] = 8.0
    m = "l0.mix."
    for n in ("l0.norm1", "l0.norm1b"):
        t[n][:] = 0.0
    t[m + "q"][:, 40:42] = t[m + "k"][:, 40:42] = 0
    t[m + "v"][:, 40] *= 8                                           # and what it finds there is large
    for name, col in (("q", 41), ("k", 40)):
        for r in range(0, t[m + name].shape[0], dim):
            t[m + name][r] = 0
            t[m + name][r, col] = 4.0 if kind is biased else 16.0    # q and k of unit size: this channel is nearly all of them
            if kind is sunk:
                t[m + name + ".b"][r] = 0.0
    return cfg, t


@BOTH
@pytest.mark.parametrize("kind", [biased, sunk], ids=["attention", "attention_2"])
@pytest.mark.parametrize("window", [1, 2, 16, 17, 47, 64, 65, 130])
def test_window_edge(ctx, kind, window, compute):
    """NEEDLE just inside and just outside the window of SEEKER, at block and tile borders, read in a prompt, in a portion of
    two and when decoded."""
    cfg, t = needle_model(kind, window)
    ref = reference(cfg, t)
    m = device_model(ctx, cfg, t, compute)
    fill = np.random.default_rng(3).integers(3, 96, 400).tolist()
    power = []
    for back in sorted({window - 1, window, window + 1} - {0}):
        for at in (back, back + 15, back + 16, back + 33, back + 63, back + 64):      # NEEDLE at at - back
            toks = fill[:at + 1]
            toks[at - back] = NEEDLE
            toks[at] = SEEKER
            want = ref.forward(toks)[-1:]
            other = list(toks)
            other[at - back] = 50
            power.append((back < window, distance(ref.forward(other)[-1:], want).max()))
            s = Session(m, block_size=16)
            assert distance(s.run([("whole", toks)], False)[0], want).max() < 2 * LIMIT[compute]
            s.run([("decode", toks[:-1])], False)
            assert distance(s.run([("decode", toks[-1:])], False)[0], want).max() < 2 * LIMIT[compute]
            if at > 2:
                s.run([("two", toks[:-2])], False)
                assert distance(s.run([("two", toks[-2:])], False)[0], want).max() < 2 * LIMIT[compute]
    # the test has teeth: inside, the needle matters a lot; outside, not at all
    assert all(p > 0.2 for inside, p in power if inside) and all(p < 1e-9 for inside, p in power if not inside)


@BOTH
@pytest.mark.parametrize("kind", [biased, sunk], ids=["attention", "attention_2"])
def test_far_key_without_a_window(ctx, kind, compute):
    """The first token among hundreds of keys, in a prompt, in portions and decoded far along (keys cut over a cluster)."""
    cfg, t = needle_model(kind, None)
    ref = reference(cfg, t)
    m = device_model(ctx, cfg, t, compute)
    toks = [NEEDLE] + np.random.default_rng(4).integers(3, 96, 700).tolist()
    for i in (1, 63, 64, 300, 517, 690, 699, 700):
        toks[i] = SEEKER
    want = ref.forward(toks)
    assert distance(ref.forward([50] + toks[1:])[-1:], want[-1:]).max() > 0.2
    for bs in (16, 12, 64):
        s = Session(m, block_size=bs)
        got = [s.run([("a", toks[:600])])[0], s.run([("a", toks[600:690])])[0]] + [s.run([("a", [x])])[0] for x in toks[690:]]
        assert distance(np.concatenate(got), want).max() < 2 * LIMIT[compute]


@BOTH
@pytest.mark.parametrize("sink", [-60.0, 0.0, 4.0, 60.0])
def test_sinks_of_every_size(ctx, sink, compute):
    """A sink far below, among and far above the scores (then hardly anything of the values is left), over one and many key tiles."""
    cfg = rubuvik([sunk(window=300, heads=6)], vocab=96)
    t = tensors(cfg, 22)
    t["l0.mix.sink"][:] = sink + np.arange(6)
    ref = reference(cfg, t)
    toks = np.random.default_rng(5).integers(0, 96, 400).tolist()
    want = ref.forward(toks)
    t0 = dict(t, **{"l0.mix.sink": np.full(6, -1e4, np.float32)})
    assert (distance(reference(cfg, t0).forward(toks), want).max() > 0.05) == (sink >= 0)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:380])])[0], s.run([("a", toks[380:383])])[0]] + [s.run([("a", [x])])[0] for x in toks[383:]]
    assert np.isfinite(np.concatenate(got)).all()
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_temperature_steps(ctx, compute):
    """A steep temperature that moves on within portions and between decoded tokens."""
    for every in (1, 5, 64):
        cfg = rubuvik([biased(temp=(3.0, every), scale=0.4, window=None)], vocab=96)
        t = tensors(cfg, 23)
        toks = np.random.default_rng(6).integers(0, 96, 140).tolist()
        want = reference(cfg, t).forward(toks)
        late = {**cfg, "layers": [biased(temp=(3.0, every + 1), scale=0.4, window=None)]}
        assert distance(reference(late, t).forward(toks), want).max() > 1000 * LIMIT["float32"]
        s = Session(device_model(ctx, cfg, t, compute), block_size=16)
        got = [s.run([("a", toks[i:i + 31])])[0] for i in range(0, 124, 31)] + [s.run([("a", [x])])[0] for x in toks[124:]]
        assert distance(np.concatenate(got), want).max() < LIMIT[compute] * (1 if compute == "float32" else 2)


@BOTH
def test_values_of_the_same_token_are_mixed(ctx, compute):
    """lambda = 1: the later layers attend to nothing but the first layer's values, whichever row of the step a token is."""
    cfg = rubuvik([lightning(), biased(), sunk(mlp=dense(20)), sunk(v_mix=False, kv_heads=3), biased(heads=4, window=8)], vocab=96)
    t = tensors(cfg, 24)
    for i in (2, 4):
        t[f"l{i}.mix.vmix"][...] = 1.0
    ref = reference(cfg, t)
    m = device_model(ctx, cfg, t, compute)
    toks = {n: np.random.default_rng(i).integers(0, 96, 90).tolist() for i, n in enumerate("abc")}
    want = {n: ref.forward(v) for n, v in toks.items()}
    s, got = Session(m), {n: [] for n in toks}
    at = dict.fromkeys(toks, 0)
    for sizes in ({"a": 40, "b": 2}, {"b": 60, "c": 1, "a": 1}, {"c": 70, "a": 30}, {"a": 1, "b": 1, "c": 1}, {"b": 27, "c": 18, "a": 18}):
        for (n, k), out in zip(sizes.items(), s.run([(n, toks[n][at[n]:at[n] + k]) for n, k in sizes.items()])):
            got[n].append(out)
            at[n] += k
    for n in toks:
        assert at[n] == 90 and distance(np.concatenate(got[n]), want[n]).max() < LIMIT[compute]


@BOTH
def test_first_token_is_remembered(ctx, compute):
    """Slow decays: the first token still moves the logits hundreds of tokens on, through portions and decoding."""
    cfg = rubuvik([lightning(decay=(1.0, 0.9999, 0.9995, 0.999))], vocab=96)
    t = tensors(cfg, 31)
    t["l0.norm1"][:] = 0.0
    t["embed"][7] = np.abs(t["embed"][7]) * np.sign(t["l0.mix.k"][0] + t["l0.mix.v"][0])
    toks = [7] + np.random.default_rng(5).integers(8, 96, 320).tolist()
    ref = reference(cfg, t)
    want = ref.forward(toks)
    assert distance(ref.forward([8] + toks[1:])[-1:], want[-1:]).max() > 50 * LIMIT["float32"]
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:200])])[0], s.run([("a", toks[200:270])])[0]] + [s.run([("a", [x])])[0] for x in toks[270:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_long_decoding(ctx, mixed, compute):
    t, ref = mixed
    m = device_model(ctx, MIXED, t, compute)
    a, b = draw(MIXED, t, 300, 13), draw(MIXED, t, 300, 14)
    s = Session(m)
    got = [s.run([("a", [x]), ("b", [y])]) for x, y in zip(a, b)]
    for i, toks in enumerate((a, b)):
        assert distance(np.concatenate([g[i] for g in got]), ref.forward(toks)).max() < LIMIT[compute]


def test_wide_model_many_rows(ctx):
    """Sizes that fill the tensor-core tiles, up to several hundred rows; expert tiles of every height."""
    cfg = rubuvik([sunk(heads=8, kv_heads=2, dim=64, vdim=64, window=100, mlp=softmax_moe(experts=16, top=2, ff=136, groups=(4, 2), shared=200)),
                   lightning(heads=4, dim=64, vdim=128, mlp=softmax_moe(experts=5, top=3, ff=300, groups=None, shared=None)),
                   biased(heads=16, kv_heads=2, dim=64, vdim=64, window=200, mlp=dense(1000))], width=520, vocab=1000, side=128)
    t = tensors(cfg, 14)
    toks = draw(cfg, t, 600, 15)
    want = reference(cfg, t).forward(toks)
    m = device_model(ctx, cfg, t, "bfloat16")
    for rows in ((600,), (350, 130, 120), (20, 40, 5, 1, 33, 501)):
        s = Session(m)
        got, at = [], 0
        for n in rows:
            got.append(s.run([("a", toks[at:at + n])])[0])
            at += n
        assert distance(np.concatenate(got), want).max() < LIMIT["bfloat16"]


@BOTH
@pytest.mark.parametrize("shift", [-3.0, 0.0, 3.0])
def test_routing_with_large_corrections(ctx, shift, compute):
    """Choice scores all negative or all far above 1: what is masked counts as minus infinity, and the correction leaves the
    weights alone."""
    cfg = rubuvik([lightning(mlp=softmax_moe(experts=12, top=4, groups=(4, 2), shared=None)), biased(mlp=softmax_moe(experts=9, top=5, groups=(3, 2)))])
    t = tensors(cfg, 51)
    for i in (0, 1):
        t[f"l{i}.mlp.correction"] += np.float32(shift)
    toks = draw(cfg, t, 90, 52)
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:80])])[0]] + [s.run([("a", [x])])[0] for x in toks[80:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@BOTH
def test_groups_compete_by_their_best_expert(ctx, compute):
    """One strong expert beside weak ones against a group of middling ones: the sum of two would choose the other group."""
    cfg = rubuvik([lightning(mlp=softmax_moe(experts=8, top=2, groups=(2, 1), shared=None))])
    t = tensors(cfg, 53)
    t["l0.mlp.correction"][:] = [3.0, -4.0, -4.5, -5.0, 2.0, 1.5, 1.0, 0.5]
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 60).tolist()
    want = reference(cfg, t).forward(toks)
    s = Session(device_model(ctx, cfg, t, compute))
    got = [s.run([("a", toks[:50])])[0]] + [s.run([("a", [x])])[0] for x in toks[50:]]
    assert distance(np.concatenate(got), want).max() < LIMIT[compute]


@pytest.mark.parametrize("layer", [lightning(heads=4, dim=64, vdim=128), lightning(heads=5, dim=24, vdim=20, decay=(0.0, 0.001, 0.5, 0.999, 1.0)),
                                   lightning(heads=3, dim=5, vdim=7, decay=(0.2, 0.9, 0.99)), lightning(heads=2, dim=40, vdim=150, decay=(0.97, 0.9))],
                         ids=lambda l: f"{l['mixer']['dim']}-{l['mixer']['vdim']}")
def test_chunks_equal_token_by_token(ctx, layer):
    """The chunked kernels against the scan on the same projections (both in the bf16 mode): far tighter than bf16 itself."""
    cfg = rubuvik([layer], width=48, vocab=96)
    t = tensors(cfg, 41)
    m = device_model(ctx, cfg, t, "bfloat16")
    toks = np.random.default_rng(42).integers(0, 96, 64 * 3 + 21).tolist()
    outs = []
    for size in (len(toks), 63, 64 + 37):    # all chunks; scan only; both, with the state handed over
        s = Session(m)
        outs.append(np.concatenate([s.run([("a", toks[i:i + size])])[0] for i in range(0, len(toks), size)]))
    assert np.isfinite(outs[0]).all()
    assert distance(outs[0], outs[1]).max() < 6e-3 and distance(outs[2], outs[1]).max() < 6e-3
    want = reference(cfg, t).forward(toks)
    assert distance(outs[0], want).max() < LIMIT["bfloat16"]
    exact = Session(device_model(ctx, cfg, t, "float32")).run([("a", toks)])[0]
    assert distance(exact, want).max() < LIMIT["float32"]


@pytest.mark.parametrize("in_batches", [True, False], ids=["mixed_batches", "prefill_at_admission"])
def test_generation_through_the_engine(ctx, tmp_path, mixed, in_batches):
    """registry -> engine: more requests than state slots, a pool that makes them wait, greedy tokens of every request."""
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    t, ref = mixed
    m = registry.load(ctx, write_checkpoint(tmp_path, MIXED, t), "float32", max_rows=48)
    prompts = [draw(MIXED, t, n, 60 + n) for n in (3, 40, 17, 80, 1, 29, 64)]
    e = Engine(ctx, m, num_blocks=20, block_size=16, prefill_chunk=19, mixed_batches=in_batches, state_slots=3)
    got = e.generate(prompts, 8)
    for p, out in zip(prompts, got):
        want, margin = reference_greedy(ref, p, 8)
        assert margin > 1e-4 and out == want
    assert e.stats()["free_blocks"] == 20 and e.stats()["free_state_slots"] == 3
    assert e.generate([prompts[1]], 4) == [got[1][:4]]


def test_samples_copy_the_state(ctx, tmp_path, mixed):
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    t, ref = mixed
    m = registry.load(ctx, write_checkpoint(tmp_path, MIXED, t), "float32", max_rows=48)
    e = Engine(ctx, m, num_blocks=20, state_slots=4)
    p = draw(MIXED, t, 37, 61)
    e.add_request(5, p, 8, samples=3)
    while e.step():
        pass
    want, _ = reference_greedy(ref, p, 8)
    assert [(i, x) for i, x, _ in e.finished()] == [(5, want)] * 3


def test_prefix_cache_of_a_model_without_state(ctx, tmp_path):
    """Attention alone carries nothing but its cache: a prompt that begins like an earlier one resumes from its blocks."""
    from paged_infer_b200 import registry
    from paged_infer_b200.engine import Engine
    cfg = rubuvik([biased(), sunk(mlp=dense(30)), biased(window=12)], vocab=96)
    t = tensors(cfg, 25)
    ref = reference(cfg, t)
    m = registry.load(ctx, write_checkpoint(tmp_path, cfg, t), "float32", max_rows=64)
    e = Engine(ctx, m, num_blocks=40, block_size=16, prefix_cache=True)
    p = np.random.default_rng(7).integers(0, 96, 53).tolist()
    for prompt in (p, p, p[:40] + [1, 2, 3]):
        want, margin = reference_greedy(ref, prompt, 6)
        assert margin > 1e-4 and e.generate([prompt], 6) == [want]


@BOTH
@pytest.mark.parametrize("n_seqs", [3, 7])
def test_steps_on_the_device_equal_single_steps(ctx, mixed, compute, n_seqs):
    """Greedy steps without returning to the host (one captured graph) choose what single steps choose."""
    t, _ = mixed
    m = device_model(ctx, MIXED, t, compute)
    names = "abcdefg"[:n_seqs]
    prompts = [draw(MIXED, t, n, n) for n in (30, 7, 55, 12, 3, 21, 44)[:n_seqs]]
    s = Session(m, slots=8)
    first = [int(np.argmax(x)) for x in s.run(list(zip(names, prompts)), False)]
    for n in names:   # room for what is to come
        while len(s.seq[n][1]) * s.bs < s.seq[n][0] + 12:
            s.seq[n][1].append(int(s.free.pop(0)))
    out = m.step_multi(first, [s.seq[n][0] for n in names], [s.seq[n][1] for n in names], s.kv, 10, s.state, [s.seq[n][2] for n in names])
    s2 = Session(m, slots=8, seed=3)
    s2.run(list(zip(names, prompts)), False)
    cur, want = first, []
    for _ in range(10):
        cur = [int(np.argmax(x)) for x in s2.run([(n, [c]) for n, c in zip(names, cur)], False)]
        want.append(cur)
    assert out.tolist() == want


def test_replay_and_command_line(tmp_path, mixed):
    """bin/trace_run and the command line as a user calls them."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    t, ref = mixed
    folder = write_checkpoint(tmp_path, MIXED, t)
    a, b = draw(MIXED, t, 70, 1), draw(MIXED, t, 20, 2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:66], "want": [0, 65]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[66:67], "want": []}, {"id": "y", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "y", "tokens": b[19:], "want": [0]}, {"id": "x", "tokens": a[67:], "want": [1, 2]}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": b, "want": [19]}], "end": ["z"]}]
    la, lb = ref.forward(a), ref.forward(b)
    want = {0: la[[0, 65]], 1: lb[[18]], 2: np.stack([lb[19], la[68], la[69]]), 3: lb[[19]]}
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                           input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.split("\n") if x.startswith("done")] == [f"done {i}" for i in range(4)]
        for i, w in want.items():
            assert distance(np.fromfile(out / f"{i}.f32", "<f4").reshape(w.shape), w).max() < LIMIT[dtype]
    r = subprocess.run([sys.executable, "-m", "paged_infer_b200", "generate", "--model", folder, "--dtype", "float32", "--tokens",
                        ",".join(map(str, b)), "--tokens", "5,6", "--max-tokens", "6"], capture_output=True, text=True, cwd=root, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.split() == [",".join(map(str, reference_greedy(ref, p, 6)[0])) for p in (b, [5, 6])]


def test_wrong_configurations_are_errors(ctx):
    from paged_infer_b200.api import PiError
    for layer, why in ((lightning(decay=(0.5, 0.5, 0.5, 1.5)), "decay"), (biased(heads=5, kv_heads=2), "share"), (biased(temp=(1.0, -3)), "grow"),
                       (lightning(mlp=softmax_moe(experts=12, groups=(5, 2))), "groups"), (sunk(mlp=softmax_moe(experts=12, top=5, groups=(3, 1))), "experts per token")):
        cfg = rubuvik([layer])
        with pytest.raises(PiError, match=why):
            device_model(ctx, cfg, tensors(rubuvik([lightning()]), 1), "float32")
    cfg = rubuvik([biased(), biased(vdim=12)])
    with pytest.raises(PiError, match="do not mix"):
        device_model(ctx, cfg, tensors(cfg, 1), "float32")
    cfg = rubuvik([sunk(mlp=softmax_moe())])
    t = tensors(cfg, 4)
    for missing in ("l0.mlp.e11.down", "l0.mix.v.b", "l0.side.norm", "side.embed", "l0.norm2b", "l0.mix.sink"):
        with pytest.raises(PiError, match=f"missing tensor: {missing}"):
            device_model(ctx, cfg, {k: v for k, v in t.items() if k != missing}, "float32")
